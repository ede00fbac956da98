"""Sequence mixing beyond plain attention: residuals in 32 bits (hyper-connections, that is several mixed streams, or one
stream with a scale per channel, normalised before a sublayer or after the sum), short causal convolutions or norms in front of
attention, the gated delta rule, gated linear attention and the selective scan. CUDA tensors (bf16, or f32 for the exact mode) go to the
sm_100a kernels, CPU tensors to `ops.reference`, as in the rest of `ops`."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import _ext
from . import _state, reference


class SeqRows:
    """Where a step's sequences lie in its flat token rows, and which recurrent-state banks they use.

      row_seq    int32 [T]     sequence of each row (-1: padding)
      seq_rows   int32 [S, 2]  first row and one past the last row (equal: unused entry)
      seq_state  int32 [S, 2]  bank to read (-1: no history), bank to write (-1: unused entry); bank = 2 * slot + parity
    The first `n_decode` entries have one row each; entries [first, first + n_prefill) have any number of rows."""

    __slots__ = ("row_seq", "seq_rows", "seq_state", "n_decode", "first", "n_prefill")

    def __init__(self, row_seq, seq_rows, seq_state, n_decode, first, n_prefill):
        self.row_seq, self.seq_rows, self.seq_state = row_seq, seq_rows, seq_state
        self.n_decode, self.first, self.n_prefill = int(n_decode), int(first), int(n_prefill)


@dataclass
class HyperMix:
    """Mixing coefficients of one sublayer, f32: what it reads from the streams, what it adds to them, stream to stream."""
    w_in: torch.Tensor
    w_out: torch.Tensor
    mix: torch.Tensor


def hyper_norm(x: torch.Tensor, weight: torch.Tensor, eps: float, dtype: torch.dtype, read: HyperMix | None, done: HyperMix | None = None,
               y: torch.Tensor | None = None, ids: torch.Tensor | None = None, embed: torch.Tensor | None = None, embed_scale: float = 1.0,
               rows: torch.Tensor | None = None, store: bool = True, mean_width: int | None = None) -> torch.Tensor:
    """Everything between two sublayers in one launch: fold the finished sublayer's output `y` (coefficients `done`) into
    the streams x [T, streams, width] (f32, in place), read the next sublayer's input (`read`; None: the plain sum) and
    RMS-normalise it with `weight` (f32). `ids`: x starts from the embedding instead. `rows`: only these rows, x untouched."""
    from . import _count

    T, S, W = x.shape
    if not x.is_cuda:
        if ids is not None:
            x.copy_((embed.float()[ids.long()] * embed_scale).unsqueeze(1).expand(T, S, W))
        pick = slice(None) if rows is None else rows.long()
        h, new = reference.hyper_norm(x[pick], weight, eps, read.w_in if read else None, y[pick] if y is not None else None,
                                      done.mix if done else None, done.w_out if done else None, mean_width)
        if store:
            x.copy_(new)
        return h.to(dtype)
    h = torch.empty(T if rows is None else rows.numel(), W, dtype=dtype, device=x.device)
    _ext.require().hyper_norm(x, y, done.mix if done else None, done.w_out if done else None, read.w_in if read else None, weight, h, ids, embed,
                              embed_scale, rows, store, eps, mean_width or W, _state.get(x.device).status)
    _count()
    return h


@dataclass
class StreamStart:
    """How a residual stream begins: embed[id] * scale, plus (where `bigram` is given, [buckets + 1, width]) the row
    (previous id * mul_prev + id * mul_cur) mod buckets of a second table, its last row for a sequence's first token.
    `x0` receives a copy of the result."""
    ids: torch.Tensor
    embed: torch.Tensor
    scale: float = 1.0
    prev: torch.Tensor | None = None          # int32 [T], -1: none
    bigram: torch.Tensor | None = None
    mul_prev: int = 0
    mul_cur: int = 0
    x0: torch.Tensor | None = None
    pos_table: torch.Tensor | None = None     # [max_pos, width]: a learned vector per position (`post_norm` only; scale is 1 there)
    positions: torch.Tensor | None = None     # int32 [T]


@dataclass
class Finished:
    """Sublayers' results on their way into the residual, any of: rows `y`, the weighted rows of every token's experts
    (`ops.ExpertRows`), rows `gated` times sigmoid(gate) with one f32 logit per row. `scale` f32 [width] is applied to their sum
    (None: one)."""
    scale: torch.Tensor | None
    y: torch.Tensor | None = None
    experts: object | None = None
    gated: torch.Tensor | None = None
    gate: torch.Tensor | None = None          # f32 [T], may be a column of a matrix


def residual_norm(x: torch.Tensor, weight: torch.Tensor | None, eps: float, dtype: torch.dtype, done: Finished | None = None,
                  start: StreamStart | None = None, out: torch.Tensor | None = None, rows: torch.Tensor | None = None, store: bool = True,
                  mean_width: int | None = None, bias: torch.Tensor | None = None) -> torch.Tensor:
    """Everything between two sublayers in one launch: add the finished one to the stream x [T, width] (f32, in place) and
    RMS-normalise the sum with `weight` (f32; None: return x itself, rounded), or layer-normalise it where there is a `bias`
    (f32). `start`: x begins from the embedding.
    `rows`: only these rows, compact. `out`: where the result goes (rows may be strided)."""
    from . import _count

    T, W = x.shape
    ex = done.experts if done is not None else None
    y = done.y if done is not None else None
    if not x.is_cuda:
        if start is not None:
            e = start.embed.float()[start.ids.long()] * start.scale
            if start.bigram is not None:
                n, prev = start.bigram.shape[0] - 1, start.prev.long()
                e = e + start.bigram.float()[torch.where(prev < 0, n, (prev * start.mul_prev + start.ids.long() * start.mul_cur) % n)]
            x.copy_(e)
            if start.x0 is not None:
                start.x0.copy_(e)
        pick = slice(None) if rows is None else rows.long()
        add = None
        if done is not None:
            add = torch.zeros(T, W) if y is None else y.float()
            if ex is not None:
                add = add + ex.total()
            if done.gated is not None:
                add = add + torch.sigmoid(done.gate.float()).unsqueeze(-1) * done.gated.float()
            add = add[pick]
        h, new = reference.residual_norm(x[pick], weight, eps, add, done.scale if done is not None else None, mean_width, bias)
        if store:
            x.copy_(new)
        return h.to(dtype) if out is None else out.copy_(h)
    if out is None:
        out = torch.empty(T if rows is None else rows.numel(), W, dtype=dtype, device=x.device)
    s = start
    _ext.require().residual_norm(x, y, ex.rows if ex else None, ex.slot if ex else None, ex.weights if ex else None, done.scale if done else None, weight, out,
                                 s.ids if s else None, s.embed if s else None, s.scale if s else 1.0, s.prev if s and s.bigram is not None else None,
                                 s.bigram if s else None, s.mul_prev if s else 0, s.mul_cur if s else 0, s.x0 if s else None, rows, store, eps,
                                 mean_width or W, _state.get(x.device).status, bias, ex.own if ex else None, done.gated if done else None,
                                 done.gate if done else None)
    _count()
    return out


@dataclass
class GroupNorm:
    """RMS norm of each of `groups` equal runs of the first `width` columns by itself. Weights f32, padded like the rows."""
    groups: int
    eps: float
    width: int


@dataclass
class InputConv:
    """Short causal convolution over time that is added to what a sublayer reads: w f32 [taps, width], `state` f32 [banks, taps - 1,
    width]."""
    w: torch.Tensor
    state: torch.Tensor | None


def post_norm(x: torch.Tensor | None, norm: GroupNorm, dtype: torch.dtype, seq: SeqRows, done: Finished | None = None, weight: torch.Tensor | None = None,
              alpha: float = 1.0, start: StreamStart | None = None, conv: InputConv | None = None, then: torch.Tensor | None = None,
              rows: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor | None]:
    """Everything between two sublayers of a residual that is normalised after the sum, in one launch: x' = norm(alpha x + done) with
    `weight` (None: not normalised), h = x' + conv(x') in `dtype`. Returns (h, x'). `start`: the embedding takes the place of the sum.
    `rows`: only these rows, normalised once more with `then`; no convolution and no x'. Rows of no sequence read as zero."""
    from . import _count

    T, W = (start.ids.shape[0], start.embed.shape[1]) if start is not None else x.shape
    ex, dev = done.experts if done is not None else None, (x if x is not None else start.embed).device
    banks = conv.state.shape[0] if conv is not None and conv.state is not None else 1 << 30
    if dev.type == "cpu":
        if start is not None:
            v = start.embed.float()[start.ids.long()] * start.scale
            if start.pos_table is not None:
                v = v + start.pos_table.float()[start.positions.long()]
        else:
            v = alpha * x
        if done is not None:
            add = torch.zeros(T, W) if done.y is None else done.y.float()
            if ex is not None:
                add = add + ex.total()
            v = v + (add if done.scale is None else done.scale * add)
        if rows is not None:
            v = v[rows.long()]

        def normed(z, w):
            return torch.cat([reference.group_rms(z[:, :norm.width], norm.groups, norm.eps) * w[:norm.width], z[:, norm.width:]], dim=1)

        if weight is not None:
            v = normed(v, weight)
        if then is not None:
            v = normed(v, then)
        if rows is not None:
            return v.to(dtype), None
        used = (seq.row_seq >= 0) & (seq.seq_state[seq.row_seq.clamp_min(0).long(), 1] >= 0)
        v = torch.where(used.unsqueeze(-1), v, 0.0)
        h = v if conv is None else v + reference.short_conv(v, conv.w, conv.state, seq.seq_rows, seq.seq_state)
        return h.to(dtype), v
    make = torch.empty if norm.width == W else torch.zeros
    h = make(T if rows is None else rows.numel(), W, dtype=dtype, device=dev)
    out = make(T, W, dtype=torch.float32, device=dev) if rows is None else None
    s = start
    _ext.require().post_norm(x if s is None else None, out, done.y if done else None, ex.rows if ex else None, ex.slot if ex else None, ex.weights if ex else None,
                             done.scale if done else None, alpha, weight, then, conv.w if conv else None, conv.state if conv else None, h, s.ids if s else None,
                             s.embed if s else None, s.pos_table if s else None, s.positions if s else None, rows, seq.row_seq, seq.seq_rows, seq.seq_state, banks,
                             norm.groups, norm.width, norm.eps, _state.get(dev).status)
    _count()
    return h, out


def conv_qkv(proj: torch.Tensor, conv_w: torch.Tensor, conv_state: torch.Tensor | None, cos_sin: torch.Tensor, positions: torch.Tensor, seq: SeqRows,
             slots: torch.Tensor | None, k_cache: torch.Tensor | None, v_cache: torch.Tensor | None, heads: int, kv_heads: int, dim: int, vdim: int,
             pad_dim: int, eps: float) -> torch.Tensor:
    """Short convolution over the q | k | v channels of `proj`, rotary embedding and RMS norm of every q and k head, k and v
    into the paged cache. kv_heads == 0: queries only. Returns q [T, heads * pad_dim] (zeros past `dim`)."""
    from . import _count

    T = proj.shape[0]
    if not proj.is_cuda:
        u = reference.short_conv(proj, conv_w, conv_state, seq.seq_rows, seq.seq_state)

        def head_norm(z):
            z = reference.apply_rope(z, positions, cos_sin) if cos_sin.shape[1] else z
            return z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps)

        q = head_norm(u[:, :heads * dim].reshape(T, heads, dim))
        if kv_heads:
            kv = (heads + kv_heads) * dim
            k, v = head_norm(u[:, heads * dim:kv].reshape(T, kv_heads, dim)), u[:, kv:].reshape(T, kv_heads, vdim)
            reference.write_kv(k_cache, v_cache, k, v, slots)
        return q.reshape(T, heads * dim).to(proj.dtype)
    q = torch.empty(T, heads * pad_dim, dtype=proj.dtype, device=proj.device)
    banks = conv_state.shape[0] if conv_state is not None else 1 << 30
    _ext.require().conv_qkv(proj, conv_w, conv_state, cos_sin, positions, seq.row_seq, seq.seq_rows, seq.seq_state, banks, q, slots, k_cache,
                            v_cache, heads, kv_heads, dim, vdim, eps, _state.get(proj.device).status)
    _count()
    return q


@dataclass
class QkvNorm:
    """f32 parameters in front of attention: biases of the q | k | v columns, weights of the norms over a whole q and k row."""
    bias: torch.Tensor
    q_norm: torch.Tensor
    k_norm: torch.Tensor


def norm_qkv(proj: torch.Tensor, p: QkvNorm, cos_sin: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor,
             v_cache: torch.Tensor, heads: int, kv_heads: int, dim: int, vdim: int, pad_dim: int, eps: float) -> torch.Tensor:
    """Biases on the q | k | v columns of `proj`, one RMS norm over all of a row's q columns and one over its k columns, rotary
    embedding (halves pair up) of the first columns of every head, k and v into the paged cache. Returns q [T, heads * pad_dim]
    (zeros past `dim`)."""
    from . import _count

    T, nq, nk = proj.shape[0], heads * dim, kv_heads * dim
    if not proj.is_cuda:
        u = proj[:, :nq + nk + kv_heads * vdim].float() + p.bias

        def whole(z, w, n):
            z = (z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps) * w).reshape(T, n, dim)
            return reference.apply_rope(z, positions, cos_sin) if cos_sin.shape[1] else z

        reference.write_kv(k_cache, v_cache, whole(u[:, nq:nq + nk], p.k_norm, kv_heads), u[:, nq + nk:].reshape(T, kv_heads, vdim), slots)
        return whole(u[:, :nq], p.q_norm, heads).reshape(T, nq).to(proj.dtype)
    q = torch.empty(T, heads * pad_dim, dtype=proj.dtype, device=proj.device)
    _ext.require().norm_qkv(proj, p.bias, p.q_norm, p.k_norm, cos_sin, positions, slots, k_cache, v_cache, q, heads, kv_heads, dim, vdim, eps,
                            _state.get(proj.device).status)
    _count()
    return q


def head_norm_qkv(proj: torch.Tensor, q_norm: torch.Tensor, k_norm: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                  heads: int, kv_heads: int, vdim: int, v_off: int, pad_dim: int, eps: float) -> torch.Tensor:
    """RMS norm of every query and key head (weights f32 [dim], the same for all heads), k and the values into the paged cache. proj:
    q | k from column 0, the values from column `v_off` (heads * dim: the keys as projected). Returns q [T, heads * pad_dim] (zeros
    past `dim`)."""
    from . import _count

    T, dim = proj.shape[0], q_norm.numel()
    if not proj.is_cuda:
        def head(z, n, w):
            z = z.float().reshape(T, n, dim)
            return z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps) * w

        nq, nk = heads * dim, kv_heads * dim
        reference.write_kv(k_cache, v_cache, head(proj[:, nq:nq + nk], kv_heads, k_norm), proj[:, v_off:v_off + kv_heads * vdim].reshape(T, kv_heads, vdim), slots)
        return head(proj[:, :nq], heads, q_norm).reshape(T, nq).to(proj.dtype)
    q = torch.empty(T, heads * pad_dim, dtype=proj.dtype, device=proj.device)
    _ext.require().head_norm_qkv(proj, q_norm, k_norm, slots, k_cache, v_cache, q, heads, kv_heads, vdim, v_off, eps, _state.get(proj.device).status)
    _count()
    return q


def conv_silu(proj: torch.Tensor, conv_w: torch.Tensor, bias: torch.Tensor | None, conv_state: torch.Tensor | None, seq: SeqRows) -> torch.Tensor:
    """silu of a short causal convolution over time (conv_w f32 [taps, channels], `bias` f32) of the first columns of proj. Returns
    [T, channels]."""
    from . import _count

    T, (taps, channels) = proj.shape[0], conv_w.shape
    if not proj.is_cuda:
        u = reference.short_conv(proj, conv_w, conv_state, seq.seq_rows, seq.seq_state)
        return reference.silu(u if bias is None else u + bias).to(proj.dtype)
    out = torch.empty(T, channels, dtype=proj.dtype, device=proj.device)
    banks = conv_state.shape[0] if conv_state is not None else 1 << 30
    _ext.require().conv_silu(proj, conv_w, bias, conv_state, out, seq.row_seq, seq.seq_rows, seq.seq_state, banks, _state.get(proj.device).status)
    _count()
    return out


SCAN_STATES = (4, 8, 16, 32, 64, 128, 256)      # states of a channel that the kernels take


@dataclass
class ScanParams:
    """f32 parameters of a selective scan: rate [channels, states] = -exp(A_log) log2(e), bias of the step sizes and direct factor
    [channels]. On CUDA channels are a multiple of 8 and states one of SCAN_STATES, padded with zeros."""
    rate: torch.Tensor
    dt_bias: torch.Tensor
    d: torch.Tensor


def selective_scan(dt: torch.Tensor, u: torch.Tensor, z: torch.Tensor, b: torch.Tensor, c: torch.Tensor, p: ScanParams, state: torch.Tensor,
                   seq: SeqRows) -> torch.Tensor:
    """Selective scan over a step's sequences: per channel and state S <- exp(dt A) S + dt u B, y = S C + D u, times silu(z).
    dt f32 [T, channels] (logits of the step sizes without their bias), u and z [T, channels], b and c [T, states]; `state` f32 [slots,
    channels, states], updated in place. Returns [T, channels]."""
    from . import _count

    if not u.is_cuda:
        step, uf, out = torch.nn.functional.softplus(dt + p.dt_bias), u.float(), torch.zeros_like(u)
        for (lo, hi), (rd, wr) in zip(seq.seq_rows.tolist(), seq.seq_state.tolist()):
            if wr < 0 or hi <= lo:
                continue
            S = state[wr // 2]
            if rd < 0:
                S.zero_()
            y = reference.selective_scan(step[lo:hi], p.rate, uf[lo:hi], b[lo:hi].float(), c[lo:hi].float(), S) + p.d * uf[lo:hi]
            out[lo:hi] = (y * reference.silu(z[lo:hi].float())).to(out.dtype)
        return out
    out = torch.empty(u.shape, dtype=u.dtype, device=u.device)
    _ext.require().selective_scan(dt, u, z, b, c, p.rate, p.dt_bias, p.d, state, out, seq.row_seq, seq.seq_rows, seq.seq_state, seq.n_decode, seq.first,
                                  seq.n_prefill, _state.get(u.device).status)
    _count((1 if seq.n_decode else 0) + (1 if seq.n_prefill else 0))
    return out


@dataclass
class GatedLinearParams:
    """f32 parameters of gated linear attention: bias of the decay logits [heads * dim], output norm [vdim]; decays are
    sigmoid(z)^(1 / tau)."""
    decay_bias: torch.Tensor
    norm_w: torch.Tensor
    tau: float


def gated_linear(proj: torch.Tensor, z: torch.Tensor, p: GatedLinearParams, state: torch.Tensor, seq: SeqRows, heads: int, dim: int, vdim: int, eps: float,
                 out: torch.Tensor, out_scale: float = 1.0) -> torch.Tensor:
    """Gated linear attention over a step's sequences: S <- diag(a) S + k v^T, o = S^T q dim^-0.5, o normalised per head, times
    silu(gate) and `out_scale`. proj [T, q | k | v | gate], z f32 [T, heads * dim] (decay logits without their bias), `state` f32
    [slots, heads, dim, vdim], updated in place. Writes and returns out [T, heads * vdim] (rows may be strided)."""
    from . import _count

    T, nk, nv = proj.shape[0], heads * dim, heads * vdim
    if not proj.is_cuda:
        q, k = proj[:, :nk].float().reshape(T, heads, dim) * dim ** -0.5, proj[:, nk:2 * nk].float().reshape(T, heads, dim)
        v, g = proj[:, 2 * nk:2 * nk + nv].float().reshape(T, heads, vdim), proj[:, 2 * nk + nv:2 * (nk + nv)].float()
        a = torch.exp(torch.nn.functional.logsigmoid(z[:, :nk].float() + p.decay_bias) / p.tau).reshape(T, heads, dim)
        out.zero_()
        for (b, e), (rd, wr) in zip(seq.seq_rows.tolist(), seq.seq_state.tolist()):
            if wr < 0 or e <= b:
                continue
            S = state[wr // 2]
            if rd < 0:
                S.zero_()
            o = reference.gated_linear(q[b:e], k[b:e], v[b:e], a[b:e], S)
            o = (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * p.norm_w).reshape(e - b, nv)
            out[b:e] = (o * reference.silu(g[b:e]) * out_scale).to(out.dtype)
        return out
    C, st = _ext.require(), _state.get(proj.device)
    scratch = torch.empty(C.gated_linear_scratch_floats(heads, dim, vdim, T, seq.seq_rows.shape[0], seq.n_prefill) if seq.n_prefill else 0, dtype=torch.float32, device=proj.device)
    C.gated_linear(proj, z, p.decay_bias, p.norm_w, p.tau, state, seq.row_seq, seq.seq_rows, seq.seq_state, out, scratch, heads, dim, vdim, eps, out_scale,
                   seq.n_decode, seq.first, seq.n_prefill, st.status)
    _count((1 if seq.n_decode else 0) + (C.gated_linear_prefill_launches(heads, vdim, T, seq.n_prefill) if seq.n_prefill else 0))
    return out


@dataclass
class DeltaParams:
    """f32 parameters of a gated delta-rule layer: convolution taps [taps, channels], -exp(A_log) [heads], dt_bias
    [heads * dim] (one decay per key channel) or [heads] (one per head), output norm [vdim]. `gate_silu`: the output gate is silu
    instead of the sigmoid."""
    conv_w: torch.Tensor
    neg_rate: torch.Tensor
    dt_bias: torch.Tensor
    norm_w: torch.Tensor
    gate_silu: bool = False


def delta_rule(proj: torch.Tensor, decay: torch.Tensor, gate: torch.Tensor, p: DeltaParams, conv_state: torch.Tensor | None, state: torch.Tensor, seq: SeqRows, b_off: int,
               heads: int, kv_heads: int, dim: int, vdim: int, out_cols: int, eps: float) -> torch.Tensor:
    """Gated delta rule over a step's sequences, with everything around it: short convolution + silu and unit norms on
    q | k | v of `proj`, step sizes from the logits at column `b_off`, decays from the inputs `decay` [T, heads * dim] or [T, heads], output
    norm and gate (logits `gate` [T, heads * vdim]). `state` f32 [slots, heads, dim, vdim] and `conv_state` are updated in place. Returns [T, out_cols]."""
    from . import _count

    T = proj.shape[0]
    if not proj.is_cuda:
        u = reference.silu(reference.short_conv(proj, p.conv_w, conv_state, seq.seq_rows, seq.seq_state))
        ck, per = kv_heads * dim, heads // kv_heads

        def unit(z):
            z = z.reshape(T, kv_heads, dim)
            return (z * torch.rsqrt(z.pow(2).sum(-1, keepdim=True) + 1e-6)).repeat_interleave(per, dim=1)

        q, k, v = unit(u[:, :ck]) * dim ** -0.5, unit(u[:, ck:2 * ck]), u[:, 2 * ck:].reshape(T, heads, vdim)
        z = torch.nn.functional.softplus(decay[:, :p.dt_bias.numel()].float() + p.dt_bias).reshape(T, heads, -1)
        g = torch.exp(p.neg_rate[None, :, None] * z).expand(T, heads, dim)
        beta = torch.sigmoid(proj[:, b_off:b_off + heads].float())
        out = torch.zeros(T, out_cols, dtype=proj.dtype)
        for (b, e), (rd, wr) in zip(seq.seq_rows.tolist(), seq.seq_state.tolist()):
            if wr < 0 or e <= b:
                continue
            S = state[wr // 2]
            if rd < 0:
                S.zero_()
            o = reference.delta_rule(q[b:e], k[b:e], v[b:e], g[b:e], beta[b:e], S)
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * p.norm_w
            f = gate[b:e, :heads * vdim].float()
            o = o * (reference.silu(f) if p.gate_silu else torch.sigmoid(f)).reshape(e - b, heads, vdim)
            out[b:e, :heads * vdim] = o.reshape(e - b, -1).to(out.dtype)
        return out
    C = _ext.require()
    st = _state.get(proj.device)
    make = torch.empty if out_cols == heads * vdim else torch.zeros
    out = make(T, out_cols, dtype=proj.dtype, device=proj.device)

    scratch = torch.empty(C.delta_scratch_floats(heads, dim, vdim, T, seq.seq_rows.shape[0]), dtype=torch.float32, device=proj.device)
    raw = torch.empty(T, heads * vdim, dtype=torch.float32, device=proj.device) if seq.n_prefill else None
    C.delta_rule(proj, decay, gate, p.gate_silu, p.conv_w, conv_state, p.neg_rate, p.dt_bias, p.norm_w, state, seq.row_seq, seq.seq_rows, seq.seq_state, out, scratch, raw,
                 b_off, heads, kv_heads, dim, vdim, eps, seq.n_decode, seq.first, seq.n_prefill, st.status)
    _count(1 + (1 if seq.n_decode else 0) + (2 if seq.n_prefill else 0))
    return out
