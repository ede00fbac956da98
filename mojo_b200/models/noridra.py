"""Noridra decoder: a residual that is normalised after the sum, group by group of its columns, with a short convolution over time
on everything a sublayer reads. Mixers are the gated delta rule with one decay per head, attention inside chunks (values that are
the keys as projected, norms per head, capped scores with a bias by distance and a sink, an output gate by element) and the
selective scan; feed-forwards are mixtures of experts whose weights multiply what the experts read. Positions are learned vectors.

Everything between two sublayers (scale and add the finished one, normalise, convolve) is one kernel, `ops.post_norm`, on an f32
stream that goes from one buffer to another. A sublayer is then
  delta      one projection GEMM [q | k | v | step sizes | decays | gates], `ops.delta_rule`, one output GEMM
  attention  one projection GEMM [q | k | gates], `ops.head_norm_qkv` (norms, cache write), paged attention, one output GEMM
  mamba1     one projection GEMM [x | z], `ops.conv_silu`, one GEMM [step sizes | B | C], one for the step sizes in f32,
             `ops.selective_scan`, one output GEMM
  experts    router in f32, `ops.moe_experts`; their rows are summed by the next `post_norm`

A sequence's memory is pages of keys and values for the attention layers and one slot of state: f32 matrices of the recurrences,
the last rows ahead of every convolution in two banks (those of the residual in f32). In bf16 on CUDA attention heads are padded to
64, 128 or 256 columns; odd sizes elsewhere are padded with zero weights when they are loaded."""
from __future__ import annotations

import math
from dataclasses import dataclass, field

import torch

from .. import ops
from ..ops import reference
from ..ops.mixers import SCAN_STATES
from .config import LayerSpec, ModelConfig

HEADS = (64, 128, 256)                                       # head sizes of the paged attention kernels
MAX_HEAD, MAX_TAPS = 256, 16                                 # of the recurrence; of the convolution on the residual


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


def _per_head(t: torch.Tensor, heads: int, rows: int) -> torch.Tensor:
    """[heads * size, c] -> [heads * rows, c], every head's rows padded."""
    out = torch.zeros(heads, rows, t.shape[1], dtype=t.dtype, device=t.device)
    out[:, :t.shape[0] // heads] = t.view(heads, -1, t.shape[1])
    return out.view(heads * rows, t.shape[1])


@dataclass
class NoridraLayer:
    spec: LayerSpec
    norm1: torch.Tensor                       # f32, as the next three
    scale1: torch.Tensor
    canon1: torch.Tensor                      # [taps, width]
    w_in: torch.Tensor                        # the mixer's input projections
    w_out: torch.Tensor
    off: dict = field(default_factory=dict)   # rows of w_in by name
    delta: ops.DeltaParams | None = None
    q_norm: torch.Tensor | None = None        # attention
    k_norm: torch.Tensor | None = None
    mods: ops.ScoreMods | None = None
    distance: torch.Tensor | None = None
    conv_w: torch.Tensor | None = None        # selective scan: f32 [taps, channels], bias
    conv_b: torch.Tensor | None = None
    w_x: torch.Tensor | None = None           # step sizes | B | C
    w_dt: torch.Tensor | None = None
    scan: ops.ScanParams | None = None
    norm2: torch.Tensor | None = None         # experts
    scale2: torch.Tensor | None = None
    canon2: torch.Tensor | None = None
    moe: ops.MoeWeights | None = None


@dataclass
class LayerCache:
    """What one layer keeps between steps."""
    k: torch.Tensor | None = None             # paged keys and values
    v: torch.Tensor | None = None
    state: torch.Tensor | None = None         # f32 [slots, heads, dim, vdim] or [slots, channels, states]
    conv: torch.Tensor | None = None          # [2 * slots, taps - 1, channels], the mixer's convolution
    in1: torch.Tensor | None = None           # f32 [2 * slots, taps - 1, width], the residual ahead of the mixer ...
    in2: torch.Tensor | None = None           # ... and of the experts


class NoridraModel:
    recurrent_state = True                    # the engine gives every sequence a state slot

    def __init__(self, cfg: ModelConfig, device: torch.device | str = "cpu", dtype: torch.dtype = torch.float32, comm=None):
        if comm is not None and getattr(comm, "world_size", 1) > 1:
            raise ValueError("noridra runs on one GPU per replica: tensor parallelism is not available for it")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.comm = None
        self.padded = self.device.type == "cuda" and dtype == torch.bfloat16
        self.width = _up(cfg.hidden_size)     # padded columns are zero throughout
        self.norm = ops.GroupNorm(cfg.norm_groups, cfg.rms_norm_eps, cfg.hidden_size)
        if not 1 <= cfg.input_taps <= MAX_TAPS:
            raise ValueError(f"convolutions on the residual of at most {MAX_TAPS} taps")
        for i, s in enumerate(cfg.layers):
            if s.mixer == "attention" and s.dim > HEADS[-1]:
                raise ValueError(f"layer {i}: attention heads of at most {HEADS[-1]} columns")
            if s.mixer == "delta" and max(s.dim, s.vdim) > MAX_HEAD:
                raise ValueError(f"layer {i}: recurrent heads of at most {MAX_HEAD} columns")
            if s.mixer == "mamba1" and s.state > SCAN_STATES[-1]:
                raise ValueError(f"layer {i}: channels of at most {SCAN_STATES[-1]} states")
            if s.moe is not None and (s.moe.experts > 1024 or s.moe.top > 32):
                raise ValueError(f"layer {i}: at most 1024 experts, of which a token uses at most 32")
        self.layers: list[NoridraLayer] = []
        self.embed = self.pos = self.lm_head = self.final_norm = None

    # ------------------------------------------------------------------------------------------------
    # weights
    # ------------------------------------------------------------------------------------------------
    def _head_pad(self, s: LayerSpec) -> int:
        """Columns of an attention head in the caches and results."""
        return next(n for n in HEADS if n >= s.dim) if self.padded else s.dim

    @staticmethod
    def _scan_sizes(s: LayerSpec) -> tuple[int, int]:
        """(channels, states) of a selective scan as the kernels see them."""
        return _up(s.inner), next(n for n in SCAN_STATES if n >= s.state)

    def _put(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=self.dtype).contiguous()

    def _vec(self, t: torch.Tensor, n: int | None = None) -> torch.Tensor:
        """f32, zero-padded."""
        out = torch.zeros(n or t.numel(), dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.to(device=self.device, dtype=torch.float32)
        return out

    def _taps(self, t: torch.Tensor, channels: int) -> torch.Tensor:
        """A convolution's weights [channels, taps] as f32 [taps, channels]."""
        return _pad(t.to(device=self.device, dtype=torch.float32), rows=channels).t().contiguous()

    def global_shapes(self) -> dict[str, tuple]:
        """Checkpoint tensors outside the layers."""
        c = self.cfg
        return {"embed": (c.vocab_size, c.hidden_size), "pos": (c.max_position_embeddings, c.hidden_size), "head": (c.vocab_size, c.hidden_size),
                "final.norm": (c.hidden_size,)}

    def load_tensor(self, name: str, t: torch.Tensor) -> None:
        want = self.global_shapes()[name]
        if tuple(t.shape) != want:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {want}")
        if name == "final.norm":
            self.final_norm = self._vec(t, self.width)
        elif name == "head":
            self.lm_head = self._put(_pad(t, rows=_up(t.shape[0]), cols=self.width))
        else:
            setattr(self, name, self._put(_pad(t, cols=self.width)))

    def tensor_shapes(self, s: LayerSpec, width: int) -> dict[str, tuple]:
        """Checkpoint tensors of one layer and their shapes."""
        H, G, d, e, taps, I = s.heads, s.kv_heads, s.dim, s.vdim, s.conv_taps, s.inner
        if s.mixer == "delta":
            mix = {"q": (G * d, width), "k": (G * d, width), "v": (H * e, width), "b": (H, width), "A_log": (H,), "norm": (e,), "a": (H, width), "dt_bias": (H,),
                   "g": (H * e, width), "o": (width, H * e), "q.conv": (G * d, taps), "k.conv": (G * d, taps), "v.conv": (H * e, taps)}
        elif s.mixer == "attention":
            mix = {"q": (H * d, width), "k": (G * d, width), "q.norm": (d,), "k.norm": (d,), "r1": (H,), "r2": (H,), "g": (H * d, width), "o": (width, H * d)}
        else:
            mix = {"in": (2 * I, width), "conv": (I, taps), "conv.b": (I,), "x": (s.dt_rank + 2 * s.state, I), "dt": (I, s.dt_rank), "dt.b": (I,),
                   "A_log": (I, s.state), "D": (I,), "o": (width, I)}
        out = {f"mix.{n}": shape for n, shape in mix.items()}
        for i in (1, 2) if s.moe is not None else (1,):
            out.update({f"norm{i}": (width,), f"ls{i}": (width,), f"canon{i}": (width, self.cfg.input_taps)})
        if s.moe is not None:
            f = s.moe.expert.ffn
            out["mlp.router"] = (s.moe.experts, width)
            for j in range(s.moe.experts):
                out.update({f"mlp.e{j}.gate": (f, width), f"mlp.e{j}.up": (f, width), f"mlp.e{j}.down": (width, f)})
        return out

    def load_layer(self, idx: int, w: dict[str, torch.Tensor]) -> None:
        """`w`: checkpoint tensors of the layer, named without the layer prefix."""
        s, W = self.cfg.layers[idx], self.width
        for name, shape in self.tensor_shapes(s, self.cfg.hidden_size).items():
            if tuple(w[name].shape) != shape:
                raise ValueError(f"layer {idx}: {name} has shape {tuple(w[name].shape)}, expected {shape}")
        load = {"delta": self._load_delta, "attention": self._load_attention, "mamba1": self._load_scan}[s.mixer]
        kw = load(s, w)
        if s.moe is not None:
            kw.update(norm2=self._vec(w["norm2"], W), scale2=self._vec(w["ls2"], W), canon2=self._taps(w["canon2"], W), moe=self._load_experts(s, w))
        assert idx == len(self.layers)
        self.layers.append(NoridraLayer(spec=s, norm1=self._vec(w["norm1"], W), scale1=self._vec(w["ls1"], W), canon1=self._taps(w["canon1"], W), **kw))

    def _stack(self, parts: list[tuple[str, torch.Tensor]]) -> tuple[torch.Tensor, dict]:
        """Projections under one another, each from a multiple of eight rows on, and where they begin."""
        off, rows = {}, []
        for name, t in parts:
            off[name] = sum(r.shape[0] for r in rows)
            rows.append(_pad(t, rows=_up(t.shape[0]), cols=self.width))
        return self._put(torch.cat(rows)), off

    def _load_delta(self, s: LayerSpec, w) -> dict:
        qkv = torch.cat([w[f"mix.{n}"] for n in "qkv"])
        w_in, off = self._stack([("qkv", qkv), ("b", w["mix.b"]), ("a", w["mix.a"]), ("g", w["mix.g"])])
        conv = torch.cat([w[f"mix.{n}.conv"] for n in "qkv"])
        p = ops.DeltaParams(self._taps(conv, conv.shape[0]), -torch.exp(self._vec(w["mix.A_log"])), self._vec(w["mix.dt_bias"]), self._vec(w["mix.norm"]), True)
        return dict(w_in=w_in, off=off, delta=p, w_out=self._put(_pad(w["mix.o"], self.width, _up(s.heads * s.vdim))))

    def _load_attention(self, s: LayerSpec, w) -> dict:
        n = self._head_pad(s)
        w_in, off = self._stack([("qk", torch.cat([w["mix.q"], w["mix.k"]])), ("g", _per_head(w["mix.g"], s.heads, n))])
        distance = torch.stack([self._vec(w["mix.r1"]), self._vec(w["mix.r2"])]).contiguous()
        return dict(w_in=w_in, off=off, q_norm=self._vec(w["mix.q.norm"]), k_norm=self._vec(w["mix.k.norm"]), distance=distance,
                    mods=ops.ScoreMods(softcap=s.softcap, chunk=s.chunk, sink=True, distance=distance),
                    w_out=self._put(_pad(_per_head(w["mix.o"].t(), s.heads, n).t(), self.width, _up(s.heads * n))))

    def _load_scan(self, s: LayerSpec, w) -> dict:
        (C, n), I, r = self._scan_sizes(s), s.inner, _up(s.dt_rank)
        w_in, off = self._stack([("x", w["mix.in"][:I]), ("z", w["mix.in"][I:])])
        x = w["mix.x"]
        w_x = torch.cat([_pad(x[:s.dt_rank], r, C), _pad(x[s.dt_rank:s.dt_rank + s.state], n, C), _pad(x[s.dt_rank + s.state:], n, C)])
        rate = _pad(-torch.exp(w["mix.A_log"].to(device=self.device, dtype=torch.float32)) * math.log2(math.e), C, n).contiguous()
        return dict(w_in=w_in, off=off, conv_w=self._taps(w["mix.conv"], C), conv_b=self._vec(w["mix.conv.b"], C), w_x=self._put(_pad(w_x, rows=_up(r + 2 * n))),
                    w_dt=self._put(_pad(w["mix.dt"], C, r)), scan=ops.ScanParams(rate, self._vec(w["mix.dt.b"], C), self._vec(w["mix.D"], C)),
                    w_out=self._put(_pad(w["mix.o"], self.width, C)))

    def _load_experts(self, s: LayerSpec, w) -> ops.MoeWeights:
        E, n, W = s.moe.experts, _up(s.moe.expert.ffn, 16), self.width
        gu, down = (torch.empty(E, r, c, dtype=self.dtype, device=self.device) for r, c in ((2 * n, W), (W, n)))
        for j in range(E):
            gu[j].copy_(reference.interleave_gate_up(_pad(w[f"mlp.e{j}.gate"], n, W), _pad(w[f"mlp.e{j}.up"], n, W)))
            down[j].copy_(_pad(w[f"mlp.e{j}.down"], W, n))
        return ops.MoeWeights(self._put(_pad(w["mlp.router"], _up(E), W)), gu, down, E, s.moe.top, "sigmoid", on_input=True)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "NoridraModel":
        """Random weights of the architecture: N(0, std) matrices, norms and scales of one, decays that forget over some hundred
        tokens."""
        cfg = self.cfg
        big = cfg.hidden_size * cfg.vocab_size > (1 << 24)
        dev = self.device if (big and self.device.type == "cuda") else torch.device("cpu")
        g = torch.Generator(device=dev).manual_seed(seed)

        def rnd(name, shape):
            kind = name.rsplit(".", 1)[-1]
            if kind.startswith(("norm", "ls")) or kind == "D":
                return torch.ones(shape, device=dev)
            if kind == "A_log":
                return torch.arange(1, shape[1] + 1, device=dev).float().log().expand(shape) if len(shape) == 2 else torch.zeros(shape, device=dev)
            if name in ("mix.dt_bias", "mix.dt.b"):
                return torch.full(shape, -4.0, device=dev)
            if kind in ("r1", "r2"):
                return torch.full(shape, 0.5, device=dev)
            if kind == "b" and len(shape) == 1:
                return torch.zeros(shape, device=dev)
            s = shape[1] ** -0.5 if kind == "conv" else 0.1 if kind.startswith("canon") else std
            return (torch.randn(*shape, generator=g, device=dev, dtype=torch.float32) * s).to(self.dtype)

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
                elif isinstance(t, (ops.MoeWeights, ops.DeltaParams, ops.ScanParams)):
                    yield from tensors(t)

        glob = (self.embed, self.pos, self.lm_head, self.final_norm)
        return sum(t.numel() * t.element_size() for lw in self.layers for t in tensors(lw)) + sum(t.numel() * t.element_size() for t in glob)

    # ------------------------------------------------------------------------------------------------
    # caches and state
    # ------------------------------------------------------------------------------------------------
    def _state_shape(self, s: LayerSpec) -> tuple | None:
        """Recurrent state of a sequence, f32."""
        return {"delta": (s.heads, s.dim, s.vdim), "mamba1": self._scan_sizes(s) if s.mixer == "mamba1" else None}.get(s.mixer)

    def _channels(self, s: LayerSpec) -> int:
        """Channels of the mixer's convolution."""
        return {"delta": 2 * s.kv_heads * s.dim + s.heads * s.vdim, "mamba1": _up(s.inner)}.get(s.mixer, 0)

    def allocate_kv_cache(self, num_pages: int, page_size: int, state_slots: int) -> list[LayerCache]:
        from ..utils import guard

        caches, past = [], self.cfg.input_taps - 1
        for i, s in enumerate(self.cfg.layers):
            c = LayerCache()
            if s.mixer == "attention":
                shape = (num_pages, s.kv_heads, page_size, self._head_pad(s))
                c.k, c.v = (guard.zeros(shape, self.dtype, self.device, f"{x} cache, layer {i}") for x in "KV")
            else:
                c.state = guard.zeros((state_slots, *self._state_shape(s)), torch.float32, self.device, f"recurrent state, layer {i}")
                if s.conv_taps > 1:
                    c.conv = guard.zeros((2 * state_slots, s.conv_taps - 1, self._channels(s)), self.dtype, self.device, f"convolution banks, layer {i}")
            if past:
                c.in1 = guard.zeros((2 * state_slots, past, self.width), torch.float32, self.device, f"residual banks, layer {i}")
                if s.moe is not None:
                    c.in2 = guard.zeros((2 * state_slots, past, self.width), torch.float32, self.device, f"residual banks, layer {i}")
            caches.append(c)
        return caches

    def kv_bytes_per_page(self, page_size: int) -> int:
        esz = torch.empty((), dtype=self.dtype).element_size()
        return sum(2 * s.kv_heads * self._head_pad(s) for s in self.cfg.layers if s.mixer == "attention") * page_size * esz

    def state_bytes_per_slot(self) -> int:
        esz, n = torch.empty((), dtype=self.dtype).element_size(), 0
        for s in self.cfg.layers:
            n += 2 * (self.cfg.input_taps - 1) * self.width * 4 * (2 if s.moe is not None else 1)
            if s.mixer != "attention":
                n += math.prod(self._state_shape(s)) * 4 + 2 * (s.conv_taps - 1) * self._channels(s) * esz
        return n

    def supports_static_attention(self, page_size: int) -> bool:
        """Whether a step that mixes decode rows and prompt chunks can run with fixed launch shapes (inside a CUDA graph):
        every attention layer needs the prefill kernel that takes a device-side work list."""
        return self.padded and all(ops.prefill_on_tensor_core(self._head_pad(s), page_size) for s in self.cfg.layers if s.mixer == "attention")

    # ------------------------------------------------------------------------------------------------
    # forward
    # ------------------------------------------------------------------------------------------------
    def _delta(self, lw: NoridraLayer, h, positions, slots, meta: ops.AttnMeta, cache: LayerCache) -> torch.Tensor:
        s, off = lw.spec, lw.off
        proj = ops.linear(h, lw.w_in)
        return ops.delta_rule(proj, proj[:, off["a"]:off["a"] + s.heads], proj[:, off["g"]:off["g"] + s.heads * s.vdim], lw.delta, cache.conv, cache.state, meta.seq,
                              off["b"], s.heads, s.kv_heads, s.dim, s.vdim, lw.w_out.shape[1], self.cfg.rms_norm_eps)

    def _attention(self, lw: NoridraLayer, h, positions, slots, meta: ops.AttnMeta, cache: LayerCache) -> torch.Tensor:
        s, g, n = lw.spec, lw.off["g"], self._head_pad(lw.spec)
        proj, cols = ops.linear(h, lw.w_in), s.heads * n
        q = ops.head_norm_qkv(proj, lw.q_norm, lw.k_norm, slots, cache.k, cache.v, s.heads, s.kv_heads, s.dim, s.heads * s.dim, n, self.cfg.rms_norm_eps)
        K = lw.w_out.shape[1]
        out = (torch.empty if K == cols else torch.zeros)(h.shape[0], K, dtype=self.dtype, device=self.device)
        ops.paged_attention(q, cache.k, cache.v, meta, s.scale, n, out=out[:, :cols], gate=proj[:, g:g + cols], positions=positions, mods=lw.mods)
        return out

    def _scan(self, lw: NoridraLayer, h, positions, slots, meta: ops.AttnMeta, cache: LayerCache) -> torch.Tensor:
        (C, n), r, z = self._scan_sizes(lw.spec), lw.w_dt.shape[1], lw.off["z"]
        proj = ops.linear(h, lw.w_in)
        u = ops.conv_silu(proj, lw.conv_w, lw.conv_b, cache.conv, meta.seq)
        f = ops.linear(u, lw.w_x)
        return ops.selective_scan(ops.linear_f32(f[:, :r], lw.w_dt), u, proj[:, z:z + C], f[:, r:r + n], f[:, r + n:r + 2 * n], lw.scan, cache.state, meta.seq)

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, meta: ops.AttnMeta, kv_caches: list[LayerCache],
                sample_rows: torch.Tensor | None, greedy: bool = False) -> torch.Tensor:
        """Logits [len(sample_rows), vocab] (every row when sample_rows is None)."""
        cfg = self.cfg
        mixers = {"delta": self._delta, "attention": self._attention, "mamba1": self._scan}
        step = dict(norm=self.norm, dtype=self.dtype, seq=meta.seq)
        sums = dict(start=ops.StreamStart(token_ids, self.embed, pos_table=self.pos, positions=positions))      # what the next norm takes
        x = None
        for lw, cache in zip(self.layers, kv_caches):
            h, x = ops.post_norm(x, conv=ops.InputConv(lw.canon1, cache.in1), **sums, **step)
            y = mixers[lw.spec.mixer](lw, h, positions, slots, meta, cache)
            sums = dict(done=ops.Finished(lw.scale1, ops.linear(y, lw.w_out)), weight=lw.norm1, alpha=cfg.residual_alpha)
            if lw.moe is not None:
                h, x = ops.post_norm(x, conv=ops.InputConv(lw.canon2, cache.in2), **sums, **step)
                sums = dict(done=ops.Finished(lw.scale2, None, ops.moe_experts(h, lw.moe)), weight=lw.norm2, alpha=cfg.residual_alpha)
        if sample_rows is not None and sample_rows.numel() == 0:
            return torch.empty(0, cfg.vocab_size, dtype=self.dtype, device=self.device)
        if sample_rows is None:
            sample_rows = self._all_rows(token_ids.shape[0])
        h, _ = ops.post_norm(x, then=self.final_norm, rows=sample_rows, **sums, **step)
        return ops.linear(h, self.lm_head)[:, :cfg.vocab_size]

    def _all_rows(self, n: int) -> torch.Tensor:
        return torch.arange(n, dtype=torch.int64, device=self.device)

    def gemm_shapes(self) -> list[tuple[int, int, int, int]]:
        """(N, K, epilogue, max tokens or 0) of every distinct weight that goes through the bf16 GEMM, for the measured
        configuration tables."""
        if self.dtype != torch.bfloat16:
            return []
        seen: dict = {}
        for lw in self.layers:
            for t, epi in ((lw.w_in, ops.EPI_NONE), (lw.w_out, ops.EPI_NONE), (lw.w_x, ops.EPI_NONE), (lw.w_dt, ops.EPI_F32),
                           (lw.moe.router if lw.moe is not None else None, ops.EPI_F32)):
                if t is not None:
                    seen[(t.shape[0], t.shape[1], epi, 0)] = None
        seen[(self.lm_head.shape[0], self.lm_head.shape[1], ops.EPI_NONE, 256)] = None
        return list(seen)
