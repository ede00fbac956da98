"""Pilutar decoder: parallel blocks, in which the mixer and the feed-forward of a layer read the same layer-normed input. Mixers
are latent attention with a rotated key part and one output gate per head, or two side by side: windowed grouped-query
attention (biased projections, norms over whole query and key rows, capped scores) and gated linear attention. Feed-forwards
are gated (ReLU), or mixtures of squared-ReLU experts and identity experts, chosen group by group, with a gated shared expert.

Everything between two layers (add all that the finished one produced to the f32 residual, layer-normalise) is one kernel,
`ops.residual_norm`. Since nothing of a layer depends on anything but the normed input, its products are few:
  inputs         one GEMM for all projections of the mixer, one for a dense feed-forward's gated half; router and shared gate
                 together, in f32
  mixers         `ops.norm_qkv` and paged attention, `ops.gated_linear`; or `ops.latent_write` and `ops.latent_attend` /
                 `ops.latent_prefill` with the per-head maps. They write side by side into one matrix ...
  output         ... behind which the dense feed-forward puts its activations, so one GEMM over all those columns is the sum of
                 the output projections. Factors of the mixers' results are applied in their epilogues, in f32.

A sequence's memory is pages (keys and values, or latents with the rotated part) and, where a layer has gated linear
attention, a slot of f32 state. In bf16 on CUDA attention heads are padded to 64, 128 or 256 columns, the query and value
heads of latent attention to multiples of 64, the latent to 64, 128, 256, 512 or 1024 and its rotated part to 64 or 128,
with zero weights; odd sizes elsewhere are padded when they are loaded."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from .. import ops
from ..ops import reference
from .config import LayerSpec, ModelConfig

LATENTS, ROTATED = (64, 128, 256, 512, 1024), (64, 128)      # widths of the latent attention kernel
HEADS = (64, 128, 256)                                       # head sizes of the paged attention kernels
MAX_STATE = 256                                              # key and value sizes of the recurrence


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


def _per_head(t: torch.Tensor, heads: int, rows: int, cols: int) -> torch.Tensor:
    """[heads * size, c] -> [heads * rows, cols], every head's rows padded."""
    out = torch.zeros(heads, rows, cols, dtype=t.dtype, device=t.device)
    out[:, :t.shape[0] // heads, :t.shape[1]] = t.view(heads, -1, t.shape[1])
    return out.view(heads * rows, cols)


@dataclass
class SharedExpert:
    w_up: torch.Tensor
    w_down: torch.Tensor


@dataclass
class PilutarLayer:
    spec: LayerSpec
    norm: torch.Tensor                        # f32
    norm_b: torch.Tensor
    w_in: torch.Tensor                        # the mixer's input projections
    w_out: torch.Tensor                       # [width, mixer columns | feed-forward columns]
    off: dict = field(default_factory=dict)   # columns of w_in's rows by name
    latent_norm: torch.Tensor | None = None   # latent attention: f32 [rank]
    w_qk: torch.Tensor | None = None          # [heads * (latent + rotated), q]: key map, transposed per head, and an identity
    w_kv: torch.Tensor | None = None          # [heads * q | heads * v, latent + rotated]: key map with identity, value map
    qkv: ops.QkvNorm | None = None            # attention beside the recurrence
    w_decay: torch.Tensor | None = None       # recurrence: second factor of the decay map
    linear: ops.GatedLinearParams | None = None
    w_gu: torch.Tensor | None = None          # dense feed-forward, gate / up rows interleaved in blocks of 16
    moe: ops.MoeWeights | None = None         # its router matrix ends with the shared expert's gate
    shared: SharedExpert | None = None


@dataclass
class LayerCache:
    """What one layer keeps between steps: paged keys and values and the recurrence's state, or paged latents."""
    k: torch.Tensor | None = None
    v: torch.Tensor | None = None
    state: torch.Tensor | None = None         # f32 [slots, heads, dim, vdim]
    latent: torch.Tensor | None = None        # [pages, page, latent + rotated]


class PilutarModel:
    def __init__(self, cfg: ModelConfig, device: torch.device | str = "cpu", dtype: torch.dtype = torch.float32, comm=None):
        if comm is not None and getattr(comm, "world_size", 1) > 1:
            raise ValueError("pilutar runs on one GPU per replica: tensor parallelism is not available for it")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.comm = None
        self.padded = self.device.type == "cuda" and dtype == torch.bfloat16
        self.width = _up(cfg.hidden_size)     # padded columns are zero throughout
        for i, s in enumerate(cfg.layers):
            for m in s.parts or [s]:
                if m.mixer == "attention" and max(m.dim, m.vdim) > HEADS[-1]:
                    raise ValueError(f"layer {i}: attention heads of at most {HEADS[-1]} columns")
                if m.mixer == "gated_linear" and max(m.dim, m.vdim) > MAX_STATE:
                    raise ValueError(f"layer {i}: recurrent heads of at most {MAX_STATE} columns")
                if m.mixer == "latent_attention" and (m.kv_rank > LATENTS[-1] or m.rot.dims > ROTATED[-1]):
                    raise ValueError(f"layer {i}: latents of at most {LATENTS[-1]} columns, {ROTATED[-1]} of them rotated")
            if s.moe is not None and (s.moe.experts + s.moe.identity > 1024 or s.moe.top > 32):
                raise ValueError(f"layer {i}: at most 1024 experts, of which a token uses at most 32")
        self.recurrent_state = any(m.mixer == "gated_linear" for m in cfg.mixers())
        self.latent_specs = [s for s in cfg.layers if s.mixer == "latent_attention"]
        self.layers: list[PilutarLayer] = []
        self.embed = self.lm_head = self.final_norm = self.final_norm_b = None
        self._tables: dict[tuple, torch.Tensor] = {}
        self.max_positions = 0
        self.reserve_positions(2048)

    def reserve_positions(self, n: int) -> None:
        """Make the rotary tables cover positions 0 .. n - 1 (the engine calls this with its context limit)."""
        if n <= self.max_positions:
            return
        for m in self.cfg.mixers():
            if m.mixer != "gated_linear":
                self._tables[m.rot.dims, m.rot.base] = reference.rope_table(n, m.rot.dims, m.rot.base).to(self.device)
        self.max_positions = n

    # ------------------------------------------------------------------------------------------------
    # weights
    # ------------------------------------------------------------------------------------------------
    def _head_pad(self, s: LayerSpec) -> int | None:
        """Columns of an attention head in the caches and results; None: keys and values as they are."""
        return next(n for n in HEADS if n >= max(s.dim, s.vdim)) if self.padded else None

    def _latent_sizes(self, s: LayerSpec) -> tuple[int, int, int, int]:
        """(query size, value size, latent size, size of the rotated part) of latent attention as the kernels see them."""
        if not self.padded:
            return s.dim + s.rot.dims, s.vdim, s.kv_rank, s.rot.dims
        return (_up(s.dim + s.rot.dims, 64), _up(s.vdim, 64), next(n for n in LATENTS if n >= s.kv_rank), next(n for n in ROTATED if n >= s.rot.dims))

    def _mixer_cols(self, s: LayerSpec) -> list[int]:
        """Columns of each mixer's result ahead of the output product, each a multiple of 16."""
        if s.parts is None:
            return [_up(s.heads * self._latent_sizes(s)[1], 16)]
        a, b = s.parts
        return [_up(a.heads * (self._head_pad(a) or a.vdim), 16), _up(b.heads * b.vdim, 16)]

    def _put(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=self.dtype).contiguous()

    def _vec(self, t: torch.Tensor, n: int | None = None, factor: float = 1.0) -> torch.Tensor:
        """f32, zero-padded."""
        out = torch.zeros(n or t.numel(), dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.to(device=self.device, dtype=torch.float32) * factor
        return out

    def global_shapes(self) -> dict[str, tuple]:
        """Checkpoint tensors outside the layers."""
        c = self.cfg
        return {"embed": (c.vocab_size, c.hidden_size), "head": (c.vocab_size, c.hidden_size), "final.norm": (c.hidden_size,), "final.norm.b": (c.hidden_size,)}

    def load_tensor(self, name: str, t: torch.Tensor) -> None:
        want = self.global_shapes()[name]
        if tuple(t.shape) != want:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {want}")
        if name == "embed":
            self.embed = self._put(_pad(t, cols=self.width))
        elif name == "head":
            self.lm_head = self._put(_pad(t, rows=_up(t.shape[0]), cols=self.width))
        else:      # the factor of the logits goes into the norm ahead of them, in f32
            setattr(self, "final_norm" if name == "final.norm" else "final_norm_b", self._vec(t, self.width, self.cfg.logit_scale))

    @staticmethod
    def tensor_shapes(s: LayerSpec, width: int) -> dict[str, tuple]:
        """Checkpoint tensors of one layer and their shapes; -1 is a size only the checkpoint tells."""
        out = {"norm1": (width,), "norm1.b": (width,)}
        if s.parts is None:
            H, d, r, e, R = s.heads, s.dim, s.rot.dims, s.vdim, s.kv_rank
            out.update({"mix.q": (H * (d + r), width), "mix.dkv": (R + r, width), "mix.dkv.norm": (R,), "mix.uk": (H * d, R), "mix.uv": (H * e, R),
                        "mix.g": (H, width), "mix.o": (width, H * e)})
        else:
            a, b = s.parts
            for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                out.update({f"mix.left.{n}": (rows, width), f"mix.left.{n}.b": (rows,)})
            nk, nv = b.heads * b.dim, b.heads * b.vdim
            out.update({"mix.left.q.norm": (a.heads * a.dim,), "mix.left.k.norm": (a.kv_heads * a.dim,), "mix.left.o": (width, a.heads * a.vdim),
                        "mix.right.q": (nk, width), "mix.right.k": (nk, width), "mix.right.v": (nv, width), "mix.right.g": (nv, width),
                        "mix.right.o": (width, nv), "mix.right.norm": (b.vdim,), "mix.right.a1": (-1, width), "mix.right.a2": (nk, -1), "mix.right.a2.b": (nk,)})
        if s.ffn:
            out.update({"mlp.gate": (s.ffn, width), "mlp.up": (s.ffn, width), "mlp.down": (width, s.ffn)})
        if s.moe is not None:
            n, sh = s.moe.experts + s.moe.identity, s.moe.shared
            out.update({"mlp.router": (n, width), "mlp.correction": (n,)})
            for p, f in [(f"mlp.e{j}", s.moe.expert.ffn) for j in range(s.moe.experts)] + ([("mlp.shared", sh.ffn)] if sh else []):
                out.update({f"{p}.up": (f, width), f"{p}.down": (width, f)})
            if sh:
                out["mlp.shared.sg"] = (1, width)
        return out

    def load_layer(self, idx: int, w: dict[str, torch.Tensor]) -> None:
        """`w`: checkpoint tensors of the layer, named without the layer prefix."""
        s, W = self.cfg.layers[idx], self.width
        for name, shape in self.tensor_shapes(s, self.cfg.hidden_size).items():
            got = tuple(w[name].shape)
            if len(got) != len(shape) or any(n not in (-1, g) for g, n in zip(got, shape)):
                raise ValueError(f"layer {idx}: {name} has shape {got}, expected {shape}")
        parts, off, outs = [], {}, []          # rows of w_in, where each block of them begins, columns of w_out

        def place(name, t):
            off[name] = sum(p.shape[0] for p in parts)
            parts.append(_pad(t, cols=W))

        def align():                           # the kernels read a block at an 8-column boundary
            n = sum(p.shape[0] for p in parts)
            if n % 8:
                parts.append(torch.zeros(_up(n) - n, W, dtype=parts[0].dtype, device=parts[0].device))

        kw = self._load_latent(s, w, place, align, outs) if s.parts is None else self._load_parallel(s, w, place, align, outs)
        align()
        if s.ffn:
            f = _up(s.ffn, 16)
            kw["w_gu"] = self._put(reference.interleave_gate_up(_pad(w["mlp.gate"], f, W), _pad(w["mlp.up"], f, W)))
            outs.append(_pad(w["mlp.down"], W, f))
        if s.moe is not None:
            kw.update(self._load_experts(s, w))
        assert idx == len(self.layers)
        self.layers.append(PilutarLayer(spec=s, norm=self._vec(w["norm1"], W), norm_b=self._vec(w["norm1.b"], W), w_in=self._put(torch.cat(parts)),
                                        w_out=self._put(torch.cat(outs, dim=1)), off=off, **kw))

    def _load_latent(self, s: LayerSpec, w, place, align, outs) -> dict:
        H, d, r, (dq, e, R, P) = s.heads, s.dim, s.rot.dims, self._latent_sizes(s)
        place("q", _per_head(w["mix.q"], H, dq, self.width))
        align()
        place("c", w["mix.dkv"])
        align()
        place("g", w["mix.g"])
        outs.append(_pad(_per_head(w["mix.o"].t(), H, e, self.width).t(), self.width, self._mixer_cols(s)[0]))
        # a head's key map from [latent | rotated part] to [unrotated | rotated]: the second part passes through
        key = torch.zeros(H, dq, R + P, dtype=w["mix.uk"].dtype, device=w["mix.uk"].device)
        key[:, :d, :s.kv_rank] = w["mix.uk"].view(H, d, s.kv_rank)
        key[:, d:d + r, R:R + r] = torch.eye(r, dtype=key.dtype, device=key.device)
        return dict(latent_norm=self._vec(w["mix.dkv.norm"]), w_qk=self._put(key.transpose(1, 2).reshape(H * (R + P), dq)),
                    w_kv=self._put(torch.cat([key.view(H * dq, R + P), _per_head(w["mix.uv"], H, e, R + P)])))

    def _load_parallel(self, s: LayerSpec, w, place, align, outs) -> dict:
        (a, b), W = s.parts, self.width
        for n in ("q", "k", "v"):
            place(n, w[f"mix.left.{n}"])
        align()
        for n in ("q", "k", "v", "g"):
            place(f"r{n}", w[f"mix.right.{n}"])
        align()
        low = _up(w["mix.right.a1"].shape[0])
        place("low", _pad(w["mix.right.a1"], low))
        ca, cb = self._mixer_cols(s)
        outs += [_pad(_per_head(w["mix.left.o"].t(), a.heads, self._head_pad(a) or a.vdim, W).t(), W, ca), _pad(w["mix.right.o"], W, cb)]
        return dict(qkv=ops.QkvNorm(self._vec(torch.cat([w[f"mix.left.{n}.b"] for n in ("q", "k", "v")])), self._vec(w["mix.left.q.norm"]),
                                    self._vec(w["mix.left.k.norm"])),
                    w_decay=self._put(_pad(w["mix.right.a2"], _up(b.heads * b.dim), low)),
                    linear=ops.GatedLinearParams(self._vec(w["mix.right.a2.b"]), self._vec(w["mix.right.norm"]), b.tau))

    def _load_experts(self, s: LayerSpec, w) -> dict:
        E, n, W = s.moe.experts, _up(s.moe.expert.ffn, 16), self.width
        up, down = (torch.empty(E, r, c, dtype=self.dtype, device=self.device) for r, c in ((n, W), (W, n)))
        for j in range(E):
            up[j].copy_(_pad(w[f"mlp.e{j}.up"], n, W))
            down[j].copy_(_pad(w[f"mlp.e{j}.down"], W, n))
        rows = [w["mlp.router"]] + ([w["mlp.shared.sg"]] if s.moe.shared else [])
        router = _pad(torch.cat(rows), _up(sum(t.shape[0] for t in rows)), W)
        kw = dict(moe=ops.MoeWeights(self._put(router), up, down, E, s.moe.top, "softmax", True, s.moe.scale, None, self._vec(w["mlp.correction"]),
                                     s.moe.groups, s.moe.keep, s.moe.identity))
        if s.moe.shared:
            f = _up(s.moe.shared.ffn, 16)
            kw["shared"] = SharedExpert(self._put(_pad(w["mlp.shared.up"], f, W)), self._put(_pad(w["mlp.shared.down"], W, f)))
        return kw

    def init_random(self, seed: int = 0, std: float = 0.02) -> "PilutarModel":
        """Random weights of the architecture: N(0, std) matrices, norms of one, decays that forget over some hundred tokens."""
        cfg = self.cfg
        big = cfg.hidden_size * cfg.vocab_size > (1 << 24)
        dev = self.device if (big and self.device.type == "cuda") else torch.device("cpu")
        g = torch.Generator(device=dev).manual_seed(seed)

        def rnd(name, shape):
            kind = name.rsplit(".", 1)[-1]
            if kind in ("norm", "norm1"):
                return torch.ones(shape, device=dev)
            if name == "mix.right.a2.b":
                return torch.full(shape, 2.0, device=dev)
            if kind in ("b", "correction"):
                return torch.zeros(shape, device=dev)
            return (torch.randn(*shape, generator=g, device=dev, dtype=torch.float32) * std).to(self.dtype)

        self.layers.clear()
        for name, shape in self.global_shapes().items():
            self.load_tensor(name, rnd(name, shape))
        for i, spec in enumerate(cfg.layers):
            rank = (spec.parts[1].decay_rank if spec.parts else 0) or 16
            self.load_layer(i, {n: rnd(n, tuple(rank if x == -1 else x for x in shape)) for n, shape in self.tensor_shapes(spec, cfg.hidden_size).items()})
        return self

    def weight_bytes(self) -> int:
        def tensors(obj):
            for t in vars(obj).values():
                if isinstance(t, torch.Tensor):
                    yield t
                elif isinstance(t, (ops.MoeWeights, SharedExpert, ops.QkvNorm, ops.GatedLinearParams)):
                    yield from tensors(t)

        glob = (self.embed, self.lm_head, self.final_norm, self.final_norm_b)
        return sum(t.numel() * t.element_size() for lw in self.layers for t in tensors(lw)) + sum(t.numel() * t.element_size() for t in glob)

    # ------------------------------------------------------------------------------------------------
    # caches and state
    # ------------------------------------------------------------------------------------------------
    def _page_cols(self, s: LayerSpec) -> list[int]:
        """Columns a token takes in the layer's paged tensors: latents, or keys and values."""
        if s.parts is None:
            return [sum(self._latent_sizes(s)[2:])]
        a = s.parts[0]
        n = self._head_pad(a)
        return [a.kv_heads * (n or a.dim), a.kv_heads * (n or a.vdim)]

    def allocate_kv_cache(self, num_pages: int, page_size: int, state_slots: int = 0) -> list[LayerCache]:
        from ..utils import guard

        caches = []
        for i, s in enumerate(self.cfg.layers):
            if s.parts is None:
                caches.append(LayerCache(latent=guard.zeros((num_pages, page_size, *self._page_cols(s)), self.dtype, self.device, f"latent cache, layer {i}")))
                continue
            a, b = s.parts
            k, v = (guard.zeros((num_pages, a.kv_heads, page_size, n // a.kv_heads), self.dtype, self.device, f"{x} cache, layer {i}")
                    for x, n in zip("KV", self._page_cols(s)))
            caches.append(LayerCache(k, v, guard.zeros((state_slots, b.heads, b.dim, b.vdim), torch.float32, self.device, f"recurrent state, layer {i}")))
        return caches

    def kv_bytes_per_page(self, page_size: int) -> int:
        esz = torch.empty((), dtype=self.dtype).element_size()
        return sum(n for s in self.cfg.layers for n in self._page_cols(s)) * page_size * esz

    def state_bytes_per_slot(self) -> int:
        return sum(m.heads * m.dim * m.vdim * 4 for m in self.cfg.mixers() if m.mixer == "gated_linear")

    def plan_latent_prefill(self, cu_q, ctx_lens, num_decode: int):
        """Metadata of the expanded attention form for a batch's prompt chunks (None: they run absorbed). All layers take the
        same form."""
        specs = self.latent_specs
        if not specs or not self.padded or any(self._latent_sizes(s)[:2] != (128, 128) for s in specs):
            return None
        windows = [s.window for s in specs]
        return ops.plan_latent_prefill(cu_q, ctx_lens, num_decode, min(self._latent_sizes(s)[2] for s in specs), max(s.heads for s in specs), 128, 128,
                                       0 if 0 in windows else max(windows))

    def _tensor_core_prefill(self, page_size: int) -> bool:
        return self.padded and all(ops.prefill_on_tensor_core(self._head_pad(s), page_size) for s in self.cfg.mixers() if s.mixer == "attention")

    def lists_prefill_work(self, page_size: int) -> bool:
        """Whether prompt chunks want a list of attention work items (eager steps)."""
        return self.recurrent_state and self._tensor_core_prefill(page_size)

    def supports_static_attention(self, page_size: int) -> bool:
        """Whether a step that mixes decode rows and prompt chunks can run with fixed launch shapes (inside a CUDA graph). Latent
        attention cannot: the size of its expansion follows the contexts."""
        return not self.latent_specs and self._tensor_core_prefill(page_size)

    # ------------------------------------------------------------------------------------------------
    # forward
    # ------------------------------------------------------------------------------------------------
    def _latent_attention(self, lw: PilutarLayer, h, positions, slots, meta: ops.AttnMeta, rows, cache: torch.Tensor, out: torch.Tensor) -> None:
        s, off = lw.spec, lw.off
        H, r, (dq, e, R, P) = s.heads, s.rot.dims, self._latent_sizes(s)
        proj = ops.linear(h, lw.w_in)
        q, g, c = proj[:, :H * dq], proj[:, off["g"]:off["g"] + H], off["c"]
        rope = ops.SharedRope(proj[:, c + s.kv_rank:c + s.kv_rank + r], q, H, s.dim, R, self._tables[r, s.rot.base], positions) if r else None
        ops.latent_write(proj[:, c:c + s.kv_rank], lw.latent_norm, self.cfg.rms_norm_eps, slots, cache, rope)
        out = out[:, :H * e]
        n = h.shape[0] if meta.expand is None else meta.num_decode      # rows that attend in the absorbed form
        if n:
            q_lat = ops.head_linear(q[:n], lw.w_qk, H)
            o_lat = ops.latent_attend(q_lat, cache, meta, rows, H, s.scale, positions, R, s.window)
            ops.head_linear(o_lat, lw.w_kv[H * dq:, :R], H, gate=g[:n], out=out[:n])
        if meta.expand is not None:
            ops.latent_prefill(q, cache, lw.w_kv, meta, H, s.scale, g, out, s.window)

    def _parallel(self, lw: PilutarLayer, h, positions, slots, meta: ops.AttnMeta, cache: LayerCache, out_a: torch.Tensor, out_b: torch.Tensor) -> None:
        (a, b), (scale_a, scale_b), off, eps = lw.spec.parts, lw.spec.part_scales, lw.off, self.cfg.rms_norm_eps
        proj = ops.linear(h, lw.w_in)
        z = ops.linear_f32(proj[:, off["low"]:off["low"] + lw.w_decay.shape[1]], lw.w_decay)
        pad = self._head_pad(a)
        q = ops.norm_qkv(proj, lw.qkv, self._tables[a.rot.dims, a.rot.base], positions, slots, cache.k, cache.v, a.heads, a.kv_heads, a.dim, a.vdim,
                         pad or a.dim, eps)
        ops.paged_attention(q, cache.k, cache.v, meta, a.scale, pad or a.dim, out=out_a[:, :a.heads * (pad or a.vdim)], positions=positions,
                            mods=ops.ScoreMods(a.window, a.softcap, scale_a))
        nk, nv = b.heads * b.dim, b.heads * b.vdim
        ops.gated_linear(proj[:, off["rq"]:off["rq"] + 2 * (nk + nv)], z, lw.linear, cache.state, meta.seq, b.heads, b.dim, b.vdim, eps, out_b[:, :nv], scale_b)

    def _layer(self, lw: PilutarLayer, h, positions, slots, meta: ops.AttnMeta, rows, cache: LayerCache) -> ops.Finished:
        s, cols = lw.spec, self._mixer_cols(lw.spec)
        K, used = lw.w_out.shape[1], s.heads * self._latent_sizes(s)[1] if s.parts is None else None
        exact = (used == cols[0]) if s.parts is None else (cols == [s.parts[0].heads * (self._head_pad(s.parts[0]) or s.parts[0].vdim),
                                                                    s.parts[1].heads * s.parts[1].vdim])
        cat = (torch.empty if exact else torch.zeros)(h.shape[0], K, dtype=self.dtype, device=self.device)
        if s.parts is None:
            self._latent_attention(lw, h, positions, slots, meta, rows, cache.latent, cat[:, :cols[0]])
        else:
            self._parallel(lw, h, positions, slots, meta, cache, cat[:, :cols[0]], cat[:, cols[0]:cols[0] + cols[1]])
        if lw.w_gu is not None:
            ops.linear_swiglu(h, lw.w_gu, out=cat[:, sum(cols):], glu=ops.REGLU)
        y = ops.linear(cat, lw.w_out)
        if lw.moe is None:
            return ops.Finished(None, y)
        logits = ops.linear_f32(h, lw.moe.router)
        experts = ops.moe_experts(h, lw.moe, logits)
        if lw.shared is None:
            return ops.Finished(None, y, experts)
        gated = ops.linear(ops.linear_relu2(h, lw.shared.w_up), lw.shared.w_down)
        return ops.Finished(None, y, experts, gated, logits[:, lw.moe.experts + lw.moe.identity])

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, meta: ops.AttnMeta, kv_caches: list[LayerCache],
                sample_rows: torch.Tensor | None, greedy: bool = False) -> torch.Tensor:
        """Logits [len(sample_rows), vocab] (every row when sample_rows is None)."""
        cfg, T, W = self.cfg, token_ids.shape[0], self.width
        norm = dict(eps=cfg.rms_norm_eps, dtype=self.dtype, mean_width=cfg.hidden_size)
        x = torch.empty(T, W, dtype=torch.float32, device=self.device)
        start, done = ops.StreamStart(token_ids, self.embed, cfg.embedding_scale), None
        rows = ops.token_rows(meta, T, self.device) if self.latent_specs else None
        for lw, cache in zip(self.layers, kv_caches):
            h = ops.residual_norm(x, lw.norm, done=done, start=start, bias=lw.norm_b, **norm)
            start, done = None, self._layer(lw, h, positions, slots, meta, rows, cache)
        if sample_rows is not None and sample_rows.numel() == 0:
            return torch.empty(0, cfg.vocab_size, dtype=self.dtype, device=self.device)
        h = ops.residual_norm(x, self.final_norm, done=done, start=start, rows=sample_rows, store=False, bias=self.final_norm_b, **norm)
        return ops.linear(h, self.lm_head)[:, :cfg.vocab_size]

    def gemm_shapes(self) -> list[tuple[int, int, int, int]]:
        """(N, K, epilogue, max tokens or 0) of every distinct weight that goes through the bf16 GEMM, for the measured
        configuration tables."""
        if self.dtype != torch.bfloat16:
            return []
        seen: dict = {}

        def add(t, epi, most=0):
            if t is not None:
                seen[(t.shape[0], t.shape[1], epi, most)] = None

        for lw in self.layers:
            for t, epi in ((lw.w_in, ops.EPI_NONE), (lw.w_out, ops.EPI_NONE), (lw.w_kv, ops.EPI_NONE), (lw.w_decay, ops.EPI_F32), (lw.w_gu, ops.EPI_SWIGLU)):
                add(t, epi)
            if lw.moe is not None:
                add(lw.moe.router, ops.EPI_F32)
            if lw.shared is not None:
                add(lw.shared.w_up, ops.EPI_RELU2)
                add(lw.shared.w_down, ops.EPI_NONE)
        add(self.lm_head, ops.EPI_NONE, 256)
        return list(seen)
