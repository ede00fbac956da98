"""Rekudra decoder: layers of two kinds (attention behind short convolutions, gated delta rule with one decay per key
channel) on a residual of several mixed streams.

Everything between two sublayers (fold the finished one into the streams, read the next one's input, normalise) is one
kernel, `ops.hyper_norm`, on f32 streams. A sublayer is then
  attention      one projection GEMM [q | k | v | gate], `ops.conv_qkv` (convolution, rotation, head norms, cache write),
                 paged attention with the head gate in its epilogue, one output GEMM
  channel_delta  one projection GEMM [q | k | v | low-rank inputs | step sizes], one GEMM for decays and output gates (the two
                 low-rank maps as one block-diagonal matrix), `ops.delta_rule`, one output GEMM
  feed-forward   SwiGLU GEMM, output GEMM
A layer with `kv_from` projects queries only and attends over the named layer's cache.

Two kinds of memory per sequence: pages of keys and values for the attention layers that own some, and one slot of
recurrent state (f32 matrices of the delta rule; the last taps - 1 projected rows of every convolution, in two banks).
Head sizes are padded to what the attention kernels take (64, 128, 256) in bf16 on CUDA; odd sizes elsewhere are padded
with zero weights when they are loaded."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import reference
from .config import LayerSpec, ModelConfig


def _up(n: int, m: int = 8) -> int:
    return (n + m - 1) // m * m


def _pad(t: torch.Tensor, rows: int | None = None, cols: int | None = None) -> torch.Tensor:
    r, c = t.shape[0], t.shape[1]
    rows, cols = rows or r, cols or c
    if (rows, cols) == (r, c):
        return t
    out = torch.zeros(rows, cols, dtype=t.dtype, device=t.device)
    out[:r, :c] = t
    return out


@dataclass
class RekudraLayer:
    spec: LayerSpec
    norm1: torch.Tensor                       # f32, 1 + w
    hc1: ops.HyperMix
    w_in: torch.Tensor                        # stacked input projections
    wo: torch.Tensor
    conv_w: torch.Tensor                      # f32 [taps, channels]
    gate_off: int = 0                         # attention: column of the head-gate logits
    delta: ops.DeltaParams | None = None
    w_dg: torch.Tensor | None = None          # delta rule: block-diagonal [decay | gate] second factors
    low_off: int = 0                          # columns of the low-rank inputs and of the step-size logits
    b_off: int = 0
    norm2: torch.Tensor | None = None
    hc2: ops.HyperMix | None = None
    w_gu: torch.Tensor | None = None          # gate / up rows interleaved in blocks of 16
    w_down: torch.Tensor | None = None


@dataclass
class LayerCache:
    """What one layer keeps between steps: paged keys / values (shared with another layer where `kv_from` says so), the
    banks of its short convolution, the delta rule's matrices."""
    k: torch.Tensor | None = None
    v: torch.Tensor | None = None
    conv: torch.Tensor | None = None          # [2 * slots, taps - 1, channels]
    state: torch.Tensor | None = None         # f32 [slots, heads, dim, vdim]


class RekudraModel:
    recurrent_state = True                    # the engine gives every sequence a state slot

    def __init__(self, cfg: ModelConfig, device: torch.device | str = "cpu", dtype: torch.dtype = torch.float32, comm=None):
        if comm is not None and getattr(comm, "world_size", 1) > 1:
            raise ValueError("rekudra runs on one GPU per replica: tensor parallelism is not available for it")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.comm = None
        self.width = _up(cfg.hidden_size)     # padded columns are zero throughout
        for i, s in enumerate(cfg.layers):
            if s.heads % s.kv_heads or max(s.dim, s.vdim) > 256:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads and head sizes at most 256")
        self.layers: list[RekudraLayer] = []
        self.embed = self.final_norm = self.lm_head = None
        self._tables: dict[tuple, torch.Tensor] = {}
        self.max_positions = 0
        self.reserve_positions(cfg.max_position_embeddings or 2048)

    # ------------------------------------------------------------------------------------------------
    # rotary tables
    # ------------------------------------------------------------------------------------------------
    @staticmethod
    def _rot_key(spec: LayerSpec) -> tuple:
        sc = spec.rot.scaling
        return (spec.rot.dims, spec.rot.base, tuple(sorted(sc.items())) if sc else None)

    def reserve_positions(self, n: int) -> None:
        """Make the rotary tables cover positions 0 .. n - 1 (the engine calls this with its context limit)."""
        if n <= self.max_positions:
            return
        for s in self.cfg.layers:
            if s.mixer != "attention":
                continue
            sc = s.rot.scaling
            scaling = None if not sc else {"rope_type": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"],
                                           "high_freq_factor": sc["high"], "original_max_position_embeddings": sc["original"]}
            self._tables[self._rot_key(s)] = reference.rope_table(n, s.rot.dims, s.rot.base, scaling).to(self.device)
        self.max_positions = n

    # ------------------------------------------------------------------------------------------------
    # weights
    # ------------------------------------------------------------------------------------------------
    def _put(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=self.dtype).contiguous()

    def _f32(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=torch.float32).contiguous()

    def _head_pad(self, spec: LayerSpec) -> tuple[int, int]:
        """(key size, value size) as the caches hold them."""
        if self.device.type == "cuda" and self.dtype == torch.bfloat16:
            n = next(p for p in (64, 128, 256) if p >= max(spec.dim, spec.vdim))
            return n, n
        return spec.dim, spec.vdim

    def _norm(self, w: torch.Tensor) -> torch.Tensor:
        out = torch.zeros(self.width, dtype=torch.float32, device=self.device)
        out[:w.numel()] = 1.0 + w.to(device=self.device, dtype=torch.float32)
        return out

    def load_tensor(self, name: str, t: torch.Tensor) -> None:
        want = {"embed": (self.cfg.vocab_size, self.cfg.hidden_size), "head": (self.cfg.vocab_size, self.cfg.hidden_size),
                "final.norm": (self.cfg.hidden_size,)}[name]
        if tuple(t.shape) != want:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {want}")
        if name == "embed":
            self.embed = self._put(_pad(t, cols=self.width))
        elif name == "head":
            self.lm_head = self._put(_pad(t, rows=_up(t.shape[0]), cols=self.width))
        else:
            self.final_norm = self._norm(t)

    @staticmethod
    def tensor_shapes(spec: LayerSpec, width: int, streams: int) -> dict[str, tuple]:
        """Checkpoint tensors of one layer and their shapes; -1 is a size only the checkpoint tells. With one tap the
        convolution tensors are a factor per channel, and may be missing (`conv_names`)."""
        H, G, d, e, n = spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.conv_taps
        out = {"norm1": (width,)}
        if spec.mixer == "attention":
            mix = {"q": (H * d, width), "g": (H, width)}
            if spec.kv_from is None:
                mix.update(k=(G * d, width), v=(G * e, width))
        else:
            mix = {"q": (G * d, width), "k": (G * d, width), "v": (H * e, width), "b": (H, width), "A_log": (H,), "norm": (e,), "a1": (-1, width),
                   "a2": (H * d, -1), "dt_bias": (H * d,), "g1": (-1, width), "g2": (H * e, -1)}
        if n > 1:
            mix.update({c[4:]: (mix[c[4:5]][0], n) for c in RekudraModel.conv_names(spec)})
        mix["o"] = (width, H * e)
        out.update({f"mix.{k}": v for k, v in mix.items()})
        subs = (1, 2) if spec.ffn else (1,)
        for q in subs:
            out.update({f"hc{q}.in": (streams,), f"hc{q}.out": (streams,), f"hc{q}.mix": (streams, streams)})
        if spec.ffn:
            out.update({"norm2": (width,), "mlp.gate": (spec.ffn, width), "mlp.up": (spec.ffn, width), "mlp.down": (width, spec.ffn)})
        return out

    @staticmethod
    def conv_names(spec: LayerSpec) -> list[str]:
        return [f"mix.{x}.conv" for x in ("q", "k", "v") if x == "q" or spec.kv_from is None]

    def load_layer(self, idx: int, w: dict[str, torch.Tensor]) -> None:
        """`w`: checkpoint tensors of the layer, named without the layer prefix."""
        spec, W = self.cfg.layers[idx], self.width
        for name, shape in self.tensor_shapes(spec, self.cfg.hidden_size, self.cfg.residual_streams).items():
            got = tuple(w[name].shape)
            if len(got) != len(shape) or any(s not in (-1, g) for g, s in zip(got, shape)):
                raise ValueError(f"layer {idx}: {name} has shape {got}, expected {shape}")

        def wide(name, rows=None):
            return _pad(w[name], rows=rows, cols=W)

        def hyper(q):
            return ops.HyperMix(self._f32(w[f"hc{q}.in"]), self._f32(w[f"hc{q}.out"]), self._f32(w[f"hc{q}.mix"]))

        qkv = [n for n in ("q", "k", "v") if f"mix.{n}" in w]
        channels = sum(w[f"mix.{n}"].shape[0] for n in qkv)
        conv = torch.cat([w[f"mix.{n}.conv"] if f"mix.{n}.conv" in w else torch.ones(w[f"mix.{n}"].shape[0], 1) for n in qkv]).t()
        H, d, e = spec.heads, spec.dim, spec.vdim
        parts = [wide(f"mix.{n}") for n in qkv]
        kw: dict = {}
        if spec.mixer == "attention":
            pad_v = self._head_pad(spec)[1]
            wo = torch.zeros(W, H, pad_v, dtype=w["mix.o"].dtype, device=w["mix.o"].device)
            wo[:self.cfg.hidden_size, :, :e] = w["mix.o"].view(-1, H, e)
            wo = wo.view(W, H * pad_v)
            parts.append(wide("mix.g"))
            kw["gate_off"] = channels
        else:
            ra, rg = w["mix.a1"].shape[0], w["mix.g1"].shape[0]
            ra8, rg8 = _up(ra), _up(rg)
            parts[-1] = _pad(parts[-1], rows=parts[-1].shape[0] + _up(channels) - channels)     # the GEMM reads the inputs at an 8-column boundary
            parts += [wide("mix.a1", ra8), wide("mix.g1", rg8), wide("mix.b")]
            dg = torch.zeros(_up(H * (d + e)), ra8 + rg8, dtype=w["mix.a2"].dtype, device=w["mix.a2"].device)
            dg[:H * d, :ra] = w["mix.a2"]
            dg[H * d:H * (d + e), ra8:ra8 + rg] = w["mix.g2"]
            wo = _pad(w["mix.o"], rows=W, cols=_up(H * e))
            kw.update(w_dg=self._put(dg), low_off=_up(channels), b_off=_up(channels) + ra8 + rg8,
                      delta=ops.DeltaParams(self._f32(conv), -torch.exp(self._f32(w["mix.A_log"])), self._f32(w["mix.dt_bias"]), self._f32(w["mix.norm"])))
        w_in = torch.cat(parts)
        if spec.ffn:
            f = _up(spec.ffn, 16)
            kw.update(norm2=self._norm(w["norm2"]), hc2=hyper(2), w_gu=self._put(reference.interleave_gate_up(wide("mlp.gate", f), wide("mlp.up", f))),
                      w_down=self._put(_pad(w["mlp.down"], rows=W, cols=f)))
        assert idx == len(self.layers)
        self.layers.append(RekudraLayer(spec=spec, norm1=self._norm(w["norm1"]), hc1=hyper(1), w_in=self._put(_pad(w_in, rows=_up(w_in.shape[0]))),
                                        wo=self._put(wo), conv_w=self._f32(conv), **kw))

    def init_random(self, seed: int = 0, std: float = 0.02) -> "RekudraModel":
        """Random weights of the architecture: N(0, std) matrices, streams that start as copies of a plain residual."""
        cfg = self.cfg
        big = cfg.hidden_size * cfg.vocab_size > (1 << 27)
        dev = self.device if (big and self.device.type == "cuda") else torch.device("cpu")
        g = torch.Generator(device=dev).manual_seed(seed)

        def rnd(*shape, s=std):
            return torch.randn(*shape, generator=g, device=dev, dtype=torch.float32) * s

        S = cfg.residual_streams
        self.layers.clear()
        self.load_tensor("embed", rnd(cfg.vocab_size, cfg.hidden_size))
        for i, spec in enumerate(cfg.layers):
            w = {}
            for name, shape in self.tensor_shapes(spec, cfg.hidden_size, S).items():
                rank = {"mix.a1": spec.decay_rank, "mix.a2": spec.decay_rank, "mix.g1": spec.gate_rank, "mix.g2": spec.gate_rank}.get(name, 0)
                shape = tuple((rank or spec.dim) if x == -1 else x for x in shape)
                kind = name.rsplit(".", 1)[-1]
                if name.startswith("hc"):
                    w[name] = {"in": torch.full(shape, 1.0 / S), "out": torch.ones(shape), "mix": torch.eye(S)}[kind].to(dev)
                elif kind == "conv":
                    w[name] = rnd(*shape, s=shape[1] ** -0.5)
                elif name in ("norm1", "norm2", "mix.A_log"):
                    w[name] = torch.zeros(shape, device=dev)
                elif name == "mix.norm":
                    w[name] = torch.ones(shape, device=dev)
                elif name == "mix.dt_bias":
                    w[name] = rnd(*shape, s=1.0) - 3.0
                else:
                    w[name] = rnd(*shape)
            self.load_layer(i, w)
        self.load_tensor("final.norm", torch.zeros(cfg.hidden_size))
        self.load_tensor("head", rnd(cfg.vocab_size, cfg.hidden_size))
        return self

    def weight_bytes(self) -> int:
        n = 0
        for lw in self.layers:
            for t in list(vars(lw).values()) + [x for p in (lw.hc1, lw.hc2, lw.delta) if p is not None for x in vars(p).values()]:
                if isinstance(t, torch.Tensor):
                    n += t.numel() * t.element_size()
        return n + sum(t.numel() * t.element_size() for t in (self.embed, self.final_norm, self.lm_head))

    # ------------------------------------------------------------------------------------------------
    # caches and state
    # ------------------------------------------------------------------------------------------------
    def _channels(self, s: LayerSpec) -> int:
        if s.mixer == "channel_delta":
            return 2 * s.kv_heads * s.dim + s.heads * s.vdim
        return s.heads * s.dim + (0 if s.kv_from is not None else s.kv_heads * (s.dim + s.vdim))

    def allocate_kv_cache(self, num_pages: int, page_size: int, state_slots: int) -> list[LayerCache]:
        from ..utils import guard

        caches: list[LayerCache] = []
        for i, s in enumerate(self.cfg.layers):
            c = LayerCache()
            if s.conv_taps > 1:
                c.conv = guard.zeros((2 * state_slots, s.conv_taps - 1, self._channels(s)), self.dtype, self.device, f"convolution banks, layer {i}")
            if s.mixer == "channel_delta":
                c.state = guard.zeros((state_slots, s.heads, s.dim, s.vdim), torch.float32, self.device, f"delta-rule state, layer {i}")
            elif s.kv_from is not None:
                c.k, c.v = caches[s.kv_from].k, caches[s.kv_from].v
            else:
                dk, dv = self._head_pad(s)
                c.k = guard.zeros((num_pages, s.kv_heads, page_size, dk), self.dtype, self.device, f"K cache, layer {i}")
                c.v = guard.zeros((num_pages, s.kv_heads, page_size, dv), self.dtype, self.device, f"V cache, layer {i}")
            caches.append(c)
        return caches

    def kv_bytes_per_page(self, page_size: int) -> int:
        esz = torch.empty((), dtype=self.dtype).element_size()
        return sum(s.kv_heads * page_size * sum(self._head_pad(s)) * esz for s in self.cfg.layers if s.mixer == "attention" and s.kv_from is None)

    def state_bytes_per_slot(self) -> int:
        esz = torch.empty((), dtype=self.dtype).element_size()
        n = 0
        for s in self.cfg.layers:
            n += 2 * (s.conv_taps - 1) * self._channels(s) * esz
            if s.mixer == "channel_delta":
                n += s.heads * s.dim * s.vdim * 4
        return n

    # ------------------------------------------------------------------------------------------------
    # forward
    # ------------------------------------------------------------------------------------------------
    def _attention(self, lw: RekudraLayer, h, positions, slots, meta: ops.AttnMeta, cache: LayerCache) -> torch.Tensor:
        s = lw.spec
        proj = ops.linear(h, lw.w_in)
        own = s.kv_from is None
        pad_dim = self._head_pad(s)[0]
        q = ops.conv_qkv(proj, lw.conv_w, cache.conv, self._tables[self._rot_key(s)], positions, meta.seq, slots if own else None,
                         cache.k if own else None, cache.v if own else None, s.heads, s.kv_heads if own else 0, s.dim, s.vdim, pad_dim,
                         self.cfg.rms_norm_eps)
        o = ops.paged_attention(q, cache.k, cache.v, meta, s.scale, pad_dim, gate=proj[:, lw.gate_off:lw.gate_off + s.heads], positions=positions)
        return ops.linear(o, lw.wo)

    def _channel_delta(self, lw: RekudraLayer, h, meta: ops.AttnMeta, cache: LayerCache) -> torch.Tensor:
        s = lw.spec
        proj = ops.linear(h, lw.w_in)
        dg = ops.linear(proj[:, lw.low_off:lw.b_off], lw.w_dg)
        nk = s.heads * s.dim
        o = ops.delta_rule(proj, dg[:, :nk], dg[:, nk:nk + s.heads * s.vdim], lw.delta, cache.conv, cache.state, meta.seq, lw.b_off, s.heads, s.kv_heads, s.dim, s.vdim, lw.wo.shape[1],
                           self.cfg.rms_norm_eps)
        return ops.linear(o, lw.wo)

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, meta: ops.AttnMeta, kv_caches: list[LayerCache],
                sample_rows: torch.Tensor | None, greedy: bool = False) -> torch.Tensor:
        """Logits [len(sample_rows), vocab] (every row when sample_rows is None)."""
        cfg, eps, W0 = self.cfg, self.cfg.rms_norm_eps, self.cfg.hidden_size
        x = torch.empty(token_ids.shape[0], cfg.residual_streams, self.width, dtype=torch.float32, device=self.device)
        start = dict(ids=token_ids, embed=self.embed, embed_scale=cfg.embedding_scale)     # the first read creates the streams
        done, y = None, None
        for lw, cache in zip(self.layers, kv_caches):
            h = ops.hyper_norm(x, lw.norm1, eps, self.dtype, lw.hc1, done, y, mean_width=W0, **start)
            start = {}
            y = self._attention(lw, h, positions, slots, meta, cache) if lw.spec.mixer == "attention" else self._channel_delta(lw, h, meta, cache)
            done = lw.hc1
            if lw.w_gu is not None:
                h = ops.hyper_norm(x, lw.norm2, eps, self.dtype, lw.hc2, done, y, mean_width=W0)
                y = ops.linear(ops.linear_swiglu(h, lw.w_gu), lw.w_down)
                done = lw.hc2
        if sample_rows is not None and sample_rows.numel() == 0:
            return torch.empty(0, cfg.vocab_size, dtype=self.dtype, device=self.device)
        h = ops.hyper_norm(x, self.final_norm, eps, self.dtype, None, done, y, rows=sample_rows, store=False, mean_width=W0, **start)
        return ops.linear(h, self.lm_head)[:, :cfg.vocab_size]

    def supports_static_attention(self, page_size: int) -> bool:
        """Whether a step that mixes decode rows and prompt chunks can run with fixed launch shapes (inside a CUDA graph):
        every attention layer needs the prefill kernel that takes a device-side work list."""
        return (self.device.type == "cuda" and self.dtype == torch.bfloat16
                and all(ops.prefill_on_tensor_core(self._head_pad(s)[0], page_size) for s in self.cfg.layers if s.mixer == "attention"))

    def gemm_shapes(self) -> list[tuple[int, int, int, int]]:
        """(N, K, epilogue, max tokens or 0) of every distinct weight that goes through the bf16 GEMM, for the measured
        configuration tables."""
        if self.dtype != torch.bfloat16:
            return []
        seen: dict = {}
        for lw in self.layers:
            for t, epi in ((lw.w_in, ops.EPI_NONE), (lw.wo, ops.EPI_NONE), (lw.w_dg, ops.EPI_NONE), (lw.w_gu, ops.EPI_SWIGLU), (lw.w_down, ops.EPI_NONE)):
                if t is not None:
                    seen[(t.shape[0], t.shape[1], epi, 0)] = None
        seen[(self.lm_head.shape[0], self.lm_head.shape[1], ops.EPI_NONE, 256)] = None
        return list(seen)
