"""Rerupel decoder: latent attention without positions, squared-ReLU or mixture-of-experts feed-forwards, a hashed bigram
embedding, and a run of layers that is passed several times.

Everything between two sublayers (add the finished one to the f32 residual with its per-channel scale, sum a token's expert
rows, normalise) is one kernel, `ops.residual_norm`. A sublayer is then
  latent attention   one projection GEMM [q | latent | gate logits], `ops.latent_write` (norm, cache), attention in absorbed or
                     expanded form (`ops.latent`), gated per-head value maps, one output GEMM
  feed-forward       squared-ReLU GEMM and output GEMM; or router GEMM (f32), `ops.moe_experts` and the shared expert's pair
The residual enters each pass of the loop through one product with the embedding output beside it, in f32 out.

A sequence's memory is pages of latents, one set per layer run (every pass of the loop has its own), and its previous token
(`AttnMeta.prev`). In bf16 on CUDA head sizes are padded to multiples of 64 and the latent to 64, 128, 256, 512 or 1024
columns, with zero weights; odd sizes elsewhere are padded when they are loaded."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import reference
from .config import LayerSpec, ModelConfig

GLU_ALPHA, GLU_UP_BIAS = 1.702, 1.0           # y = g sigmoid(1.702 g) (u + 1)
LATENTS = (64, 128, 256, 512, 1024)           # widths of the latent attention kernel


def _up(n: int, m: int = 8) -> int:
    return (n + m - 1) // m * m


def _pad(t: torch.Tensor, rows: int | None = None, cols: int | None = None) -> torch.Tensor:
    r, c = t.shape
    rows, cols = rows or r, cols or c
    if (rows, cols) == (r, c):
        return t
    out = torch.zeros(rows, cols, dtype=t.dtype, device=t.device)
    out[:r, :c] = t
    return out


@dataclass
class SharedExpert:
    w_gu: torch.Tensor
    w_down: torch.Tensor
    glu: ops.Glu


@dataclass
class RerupelLayer:
    spec: LayerSpec
    norm1: torch.Tensor                       # f32
    scale1: torch.Tensor                      # f32: layer scale times the residual multiplier
    w_in: torch.Tensor                        # [q | latent | gate logits]
    latent_norm: torch.Tensor                 # f32 [rank]
    w_qk: torch.Tensor                        # [heads * latent, dim]: key map, transposed per head (absorbed into queries)
    w_kv: torch.Tensor                        # [heads * dim | heads * vdim, latent]: key map, then value map
    wo: torch.Tensor
    norm2: torch.Tensor | None = None
    scale2: torch.Tensor | None = None
    w_up: torch.Tensor | None = None          # dense feed-forward
    w_down: torch.Tensor | None = None
    moe: ops.MoeWeights | None = None
    shared: SharedExpert | None = None


class RerupelModel:
    needs_prev_tokens = True                  # the engine stages the token before each row

    def __init__(self, cfg: ModelConfig, device: torch.device | str = "cpu", dtype: torch.dtype = torch.float32, comm=None):
        if comm is not None and getattr(comm, "world_size", 1) > 1:
            raise ValueError("rerupel runs on one GPU per replica: tensor parallelism is not available for it")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.comm = None
        self.padded = self.device.type == "cuda" and dtype == torch.bfloat16
        self.width = _up(cfg.hidden_size)     # padded columns are zero throughout
        self.runs = cfg.layer_runs()
        for i, s in enumerate(cfg.layers):
            if s.kv_rank > LATENTS[-1]:
                raise ValueError(f"layer {i}: latents of at most {LATENTS[-1]} columns")
            if s.moe is not None and (s.moe.experts > 1024 or s.moe.top > 32):
                raise ValueError(f"layer {i}: at most 1024 experts, of which a token uses at most 32")
        self.layers: list[RerupelLayer] = []
        self.embed = self.bigram = self.loop_in = self.final_norm = None

    # ------------------------------------------------------------------------------------------------
    # weights
    # ------------------------------------------------------------------------------------------------
    def _sizes(self, s: LayerSpec) -> tuple[int, int, int]:
        """(query / key size, value size, latent size) as the kernels see them."""
        if not self.padded:
            return s.dim, s.vdim, s.kv_rank
        return _up(s.dim, 64), _up(s.vdim, 64), next(n for n in LATENTS if n >= s.kv_rank)

    def _put(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=self.dtype).contiguous()

    def _vec(self, t: torch.Tensor, n: int | None = None, factor: float = 1.0) -> torch.Tensor:
        """f32, zero-padded."""
        out = torch.zeros(n or self.width, dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.to(device=self.device, dtype=torch.float32) * factor
        return out

    def global_shapes(self) -> dict[str, tuple]:
        """Checkpoint tensors outside the layers."""
        c = self.cfg
        out = {"embed": (c.vocab_size, c.hidden_size), "final.norm": (c.hidden_size,)}
        if c.bigram is not None:
            out["bigram"] = (c.bigram.buckets + 1, c.hidden_size)
        if c.loop is not None:
            out["loop.in"] = (c.hidden_size, 2 * c.hidden_size)
        return out

    def load_tensor(self, name: str, t: torch.Tensor) -> None:
        want, W = self.global_shapes()[name], self.width
        if tuple(t.shape) != want:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {want}")
        if name == "embed":
            self.embed = self._put(_pad(t, rows=_up(t.shape[0]), cols=W))       # the table is the output matrix as well
        elif name == "bigram":
            self.bigram = self._put(_pad(t, cols=W))
        elif name == "loop.in":
            h = self.cfg.hidden_size
            self.loop_in = self._put(torch.cat([_pad(t[:, :h], W, W), _pad(t[:, h:], W, W)], dim=1))
        else:
            self.final_norm = self._vec(t)

    @staticmethod
    def tensor_shapes(s: LayerSpec, width: int) -> dict[str, tuple]:
        """Checkpoint tensors of one layer and their shapes."""
        H, d, e, R = s.heads, s.dim, s.vdim, s.kv_rank
        out = {"norm1": (width,), "ls1": (width,), "mix.q": (H * d, width), "mix.dkv": (R, width), "mix.dkv.norm": (R,), "mix.uk": (H * d, R),
               "mix.uv": (H * e, R), "mix.g": (H * e, width), "mix.o": (width, H * e)}
        if s.ffn or s.moe is not None:
            out.update(norm2=(width,), ls2=(width,))
        if s.ffn:
            out.update({"mlp.up": (s.ffn, width), "mlp.down": (width, s.ffn)})
        if s.moe is not None:
            out["mlp.router"] = (s.moe.experts, width)
            parts = [(f"mlp.e{j}", s.moe.expert.ffn) for j in range(s.moe.experts)] + ([("mlp.shared", s.moe.shared.ffn)] if s.moe.shared else [])
            for p, f in parts:
                out.update({f"{p}.gate": (f, width), f"{p}.up": (f, width), f"{p}.down": (width, f)})
        return out

    def load_layer(self, idx: int, w: dict[str, torch.Tensor]) -> None:
        """`w`: checkpoint tensors of the layer, named without the layer prefix."""
        s, W, m = self.cfg.layers[idx], self.width, self.cfg.residual_mult
        for name, shape in self.tensor_shapes(s, self.cfg.hidden_size).items():
            if tuple(w[name].shape) != shape:
                raise ValueError(f"layer {idx}: {name} has shape {tuple(w[name].shape)}, expected {shape}")
        H = s.heads
        d, e, R = self._sizes(s)

        def per_head(t, size, pad, cols):
            """[H * size, c] -> [H * pad, cols], every head's rows padded."""
            out = torch.zeros(H, pad, cols, dtype=t.dtype, device=t.device)
            out[:, :size, :t.shape[1]] = t.view(H, size, -1)
            return out.view(H * pad, cols)

        uk = per_head(w["mix.uk"], s.dim, d, R)
        w_in = torch.cat([per_head(w["mix.q"], s.dim, d, W), _pad(w["mix.dkv"], R, W), per_head(w["mix.g"], s.vdim, e, W)])
        wo = per_head(w["mix.o"].t(), s.vdim, e, W).t()
        lw = RerupelLayer(
            spec=s, norm1=self._vec(w["norm1"]), scale1=self._vec(w["ls1"], factor=m), w_in=self._put(_pad(w_in, rows=_up(w_in.shape[0]))),
            latent_norm=self._vec(w["mix.dkv.norm"], s.kv_rank), w_qk=self._put(uk.view(H, d, R).transpose(1, 2).reshape(H * R, d)),
            w_kv=self._put(torch.cat([uk, per_head(w["mix.uv"], s.vdim, e, R)])), wo=self._put(wo))
        if s.ffn or s.moe is not None:
            lw.norm2, lw.scale2 = self._vec(w["norm2"]), self._vec(w["ls2"], factor=m)

        def expert(p, f):
            """(interleaved gate / up rows, down) of one gated feed-forward, its width padded to 16."""
            n = _up(f, 16)
            return reference.interleave_gate_up(_pad(w[f"{p}.gate"], n, W), _pad(w[f"{p}.up"], n, W)), _pad(w[f"{p}.down"], W, n)

        if s.ffn:
            n = _up(s.ffn, 16)
            lw.w_up, lw.w_down = self._put(_pad(w["mlp.up"], n, W)), self._put(_pad(w["mlp.down"], W, n))
        if s.moe is not None:
            E, n = s.moe.experts, _up(s.moe.expert.ffn, 16)
            gu, down = (torch.empty(E, r, c, dtype=self.dtype, device=self.device) for r, c in ((2 * n, W), (W, n)))
            for j in range(E):
                a, b = expert(f"mlp.e{j}", s.moe.expert.ffn)
                gu[j].copy_(a)
                down[j].copy_(b)
            lw.moe = ops.MoeWeights(self._put(_pad(w["mlp.router"], _up(E), W)), gu, down, E, s.moe.top, "sigmoid", False, s.moe.scale,
                                    ops.Glu(s.moe.expert.limit, GLU_ALPHA, GLU_UP_BIAS))
            if s.moe.shared is not None:
                a, b = expert("mlp.shared", s.moe.shared.ffn)
                lw.shared = SharedExpert(self._put(a), self._put(b), ops.Glu(s.moe.shared.limit, GLU_ALPHA, GLU_UP_BIAS))
        assert idx == len(self.layers)
        self.layers.append(lw)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "RerupelModel":
        """Random weights of the architecture: N(0, std) matrices, norms and layer scales of one."""
        cfg = self.cfg
        big = cfg.hidden_size * cfg.vocab_size > (1 << 24)
        dev = self.device if (big and self.device.type == "cuda") else torch.device("cpu")
        g = torch.Generator(device=dev).manual_seed(seed)

        def rnd(name, shape):
            kind = name.rsplit(".", 1)[-1]
            if kind in ("norm", "norm1", "norm2", "ls1", "ls2"):
                return torch.ones(shape, device=dev)
            return (torch.randn(*shape, generator=g, device=dev, dtype=torch.float32) * std).to(self.dtype)

        self.layers.clear()
        for name, shape in self.global_shapes().items():
            self.load_tensor(name, rnd(name, shape))
        for i, spec in enumerate(cfg.layers):
            self.load_layer(i, {n: rnd(n, shape) for n, shape in self.tensor_shapes(spec, cfg.hidden_size).items()})
        return self

    def weight_bytes(self) -> int:
        def tensors(obj):
            for t in vars(obj).values():
                if isinstance(t, torch.Tensor):
                    yield t
                elif isinstance(t, (ops.MoeWeights, SharedExpert)):
                    yield from tensors(t)

        glob = [t for t in (self.embed, self.bigram, self.loop_in, self.final_norm) if t is not None]
        return sum(t.numel() * t.element_size() for lw in self.layers for t in tensors(lw)) + sum(t.numel() * t.element_size() for t in glob)

    # ------------------------------------------------------------------------------------------------
    # caches
    # ------------------------------------------------------------------------------------------------
    def allocate_kv_cache(self, num_pages: int, page_size: int) -> list[torch.Tensor]:
        """Latents [pages, page, latent] of every layer run."""
        from ..utils import guard

        return [guard.zeros((num_pages, page_size, self._sizes(self.cfg.layers[i])[2]), self.dtype, self.device, f"latent cache, layer run {n}")
                for n, (i, _) in enumerate(self.runs)]

    def kv_bytes_per_page(self, page_size: int) -> int:
        esz = torch.empty((), dtype=self.dtype).element_size()
        return sum(self._sizes(self.cfg.layers[i])[2] for i, _ in self.runs) * page_size * esz

    def plan_latent_prefill(self, cu_q, ctx_lens, num_decode: int):
        """Metadata of the expanded attention form for a batch's prompt chunks (None: they run absorbed). All layers take the
        same form, the one that suits the first."""
        if not self.padded or any(self._sizes(s)[:2] != (128, 128) for s in self.cfg.layers):
            return None
        s = max(self.cfg.layers, key=lambda s: s.heads)
        return ops.plan_latent_prefill(cu_q, ctx_lens, num_decode, min(self._sizes(x)[2] for x in self.cfg.layers), s.heads, 128, 128)

    # ------------------------------------------------------------------------------------------------
    # forward
    # ------------------------------------------------------------------------------------------------
    def _attention(self, lw: RerupelLayer, h, positions, slots, meta: ops.AttnMeta, rows, cache) -> torch.Tensor:
        s = lw.spec
        H, (d, e, R) = s.heads, self._sizes(s)
        proj = ops.linear(h, lw.w_in)
        q, g = proj[:, :H * d], proj[:, H * d + R:H * (d + e) + R]
        ops.latent_write(proj[:, H * d:H * d + s.kv_rank], lw.latent_norm, self.cfg.rms_norm_eps, slots, cache)
        o = torch.empty(h.shape[0], H * e, dtype=h.dtype, device=h.device)
        n = h.shape[0] if meta.expand is None else meta.num_decode      # rows that attend in the absorbed form
        if n:
            q_lat = ops.head_linear(q[:n], lw.w_qk, H)
            o_lat = ops.latent_attend(q_lat, cache, meta, rows, H, s.scale, positions)
            ops.head_linear(o_lat, lw.w_kv[H * d:], H, gate=g[:n], out=o[:n])
        if meta.expand is not None:
            ops.latent_prefill(q, cache, lw.w_kv, meta, H, s.scale, g, o)
        return ops.linear(o, lw.wo)

    def _feed_forward(self, lw: RerupelLayer, h: torch.Tensor) -> ops.Finished:
        if lw.moe is None:
            return ops.Finished(lw.scale2, ops.linear(ops.linear_relu2(h, lw.w_up), lw.w_down))
        y = None
        if lw.shared is not None:
            y = ops.linear(ops.linear_swiglu(h, lw.shared.w_gu, glu=lw.shared.glu), lw.shared.w_down)
        return ops.Finished(lw.scale2, y, ops.moe_experts(h, lw.moe))

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, meta: ops.AttnMeta, kv_caches: list[torch.Tensor],
                sample_rows: torch.Tensor | None, greedy: bool = False) -> torch.Tensor:
        """Logits [len(sample_rows), vocab] (every row when sample_rows is None)."""
        cfg, eps, T, W = self.cfg, self.cfg.rms_norm_eps, token_ids.shape[0], self.width
        norm = dict(eps=eps, dtype=self.dtype, mean_width=cfg.hidden_size)
        x = torch.empty(T, W, dtype=torch.float32, device=self.device)
        both = torch.empty(T, 2 * W, dtype=self.dtype, device=self.device) if cfg.loop is not None else None     # [residual | embedding output]
        bg = cfg.bigram
        start = ops.StreamStart(token_ids, self.embed, cfg.embedding_scale, meta.prev, self.bigram, bg.mul_prev if bg else 0, bg.mul_cur if bg else 0,
                                both[:, W:] if both is not None else None)
        rows = ops.token_rows(meta, T, self.device)
        done = None
        for (i, enters), cache in zip(self.runs, kv_caches):
            lw = self.layers[i]
            if enters:
                ops.residual_norm(x, None, done=done, start=start, out=both[:, :W], store=False, **norm)
                x, start, done = ops.linear_f32(both, self.loop_in), None, None
            h = ops.residual_norm(x, lw.norm1, done=done, start=start, **norm)
            start = None
            done = ops.Finished(lw.scale1, self._attention(lw, h, positions, slots, meta, rows, cache))
            if lw.norm2 is not None:
                h = ops.residual_norm(x, lw.norm2, done=done, **norm)
                done = self._feed_forward(lw, h)
        if sample_rows is not None and sample_rows.numel() == 0:
            return torch.empty(0, cfg.vocab_size, dtype=self.dtype, device=self.device)
        h = ops.residual_norm(x, self.final_norm, done=done, start=start, rows=sample_rows, store=False, **norm)
        logits = ops.linear_softcap(h, self.embed, cfg.logit_softcap) if cfg.logit_softcap else ops.linear(h, self.embed)
        return logits[:, :cfg.vocab_size]

    def gemm_shapes(self) -> list[tuple[int, int, int, int]]:
        """(N, K, epilogue, max tokens or 0) of every distinct weight that goes through the bf16 GEMM, for the measured
        configuration tables."""
        if self.dtype != torch.bfloat16:
            return []
        seen: dict = {}

        def add(t, epi, most=0):
            if t is not None:
                seen[(t.shape[0], t.shape[1], epi, most)] = None

        add(self.loop_in, ops.EPI_F32)
        for lw in self.layers:
            for t, epi in ((lw.w_in, ops.EPI_NONE), (lw.wo, ops.EPI_NONE), (lw.w_kv, ops.EPI_NONE), (lw.w_up, ops.EPI_RELU2), (lw.w_down, ops.EPI_NONE)):
                add(t, epi)
            if lw.moe is not None:
                add(lw.moe.router, ops.EPI_F32)
            if lw.shared is not None:
                add(lw.shared.w_gu, ops.EPI_SWIGLU)
                add(lw.shared.w_down, ops.EPI_NONE)
        add(self.embed, ops.EPI_SOFTCAP if self.cfg.logit_softcap else ops.EPI_NONE, 256)
        return list(seen)
