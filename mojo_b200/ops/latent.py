"""Latent attention: one vector per token is cached, and every head's key and value are linear maps of it. Where positions are
rotary, the vector has a second part, the rotated key part that all heads share; the map of a key then holds an identity for
it, so that both forms below treat the two parts alike. Attention runs in one of two equal forms:

  absorbed   the key map is applied to the query and the value map to the result, so a token's heads attend over the cached
             vectors themselves: decode rows, short portions, and every row where the expanded form has no kernel
  expanded   the latents of a prompt's whole context become keys and values by one matrix product, and the tensor-core
             prefill kernel attends over those: fewer operations per (query, key) pair once a portion is long

CUDA tensors (bf16, or f32 for the exact mode) go to the sm_100a kernels, CPU tensors to `ops.reference`."""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np
import torch

from .. import _ext
from . import _state, reference

EXPAND_PAGE = 128                  # tokens in a page of expanded keys and values
EXPAND_BYTES = 2 << 30             # most scratch the expanded form may take
ABSORBED_RATE, PREFILL_RATE, GEMM_RATE = 90.0, 400.0, 900.0      # TFLOP/s of the kernels the two forms run on


@dataclass
class SharedRope:
    """Rotary positions of latent attention, neighbouring columns in pairs. k [T, rot] is the key part that the heads share; it
    goes to the cache columns from `column`. q [T, heads * q_dim] is rotated in place, columns [q_off, q_off + rot) of each
    head. table f32 [positions, rot]: cosines, then sines."""
    k: torch.Tensor
    q: torch.Tensor
    heads: int
    q_off: int
    column: int
    table: torch.Tensor
    positions: torch.Tensor


def latent_write(c: torch.Tensor, weight: torch.Tensor, eps: float, slots: torch.Tensor, cache: torch.Tensor, rope: SharedRope | None = None) -> None:
    """RMS-normalise c [T, rank] (rows may be strided) with `weight` (f32) into cache [pages, page, >= rank] at `slots`; slots
    below 0 are skipped. With `rope` also the shared key part, rotated; the queries rotate in the same launch. Columns that
    hold neither become zero."""
    from . import _count

    if not c.is_cuda:
        x = c.float()
        y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight
        keep = slots >= 0
        flat = cache.view(-1, cache.shape[2])
        flat[slots[keep].long(), :c.shape[1]] = y[keep].to(cache.dtype)
        if rope is not None:
            T, rot = rope.k.shape
            k = reference.apply_rope(rope.k.unsqueeze(1), rope.positions, rope.table, True).squeeze(1)
            flat[slots[keep].long(), rope.column:rope.column + rot] = k[keep].to(cache.dtype)
            part = rope.q.unflatten(1, (rope.heads, -1))[..., rope.q_off:rope.q_off + rot]
            part.copy_(reference.apply_rope(part, rope.positions, rope.table, True))
        return
    C, st = _ext.require(), _state.get(c.device)
    if rope is None:
        C.latent_write(c, weight, eps, slots, cache, st.status)
    else:
        C.latent_write(c, weight, eps, slots, cache, st.status, rope.k, rope.q, rope.heads, rope.q_off, rope.column, rope.table, rope.positions)
    _count()


def head_linear(x: torch.Tensor, w: torch.Tensor, heads: int, gate: torch.Tensor | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """One matrix per head: x [T, heads * K], w [heads * N, K] -> [T, heads * N], times sigmoid(gate): element by element, or
    head by head where the gate has `heads` columns."""
    from . import _count

    T = x.shape[0]
    if out is None:
        out = torch.empty(T, w.shape[0], dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        y = torch.einsum("thk,hnk->thn", x.reshape(T, heads, -1).float(), w.reshape(heads, -1, w.shape[1]).float()).reshape(T, -1)
        if gate is not None:
            y = y * torch.sigmoid(gate.float()).repeat_interleave(y.shape[1] // gate.shape[1], dim=1)
        return out.copy_(y)
    if T == 0:
        return out
    C = _ext.require()
    if x.dtype == torch.float32:
        C.gemm_f32(x, w, out, heads, 0, 0.0, gate)
    else:
        C.head_gemm(x, w, out, heads, gate, _state.get(x.device).status)
    _count()
    return out


def token_rows(meta, tokens: int, device) -> tuple[torch.Tensor, torch.Tensor | None]:
    """(cache positions each row sees, the sequence of each row; None: row i belongs to sequence i) of a batch. One small
    launch per step, shared by all layers."""
    from . import _count

    if device.type != "cuda" or meta.num_decode == meta.num_seqs:
        return meta.ctx_lens, None
    ctx, seq = (torch.empty(tokens, dtype=torch.int32, device=device) for _ in range(2))
    _ext.require().token_rows(meta.cu_q, meta.ctx_lens, ctx, seq)
    _count()
    return ctx, seq


def latent_attend(q: torch.Tensor, cache: torch.Tensor, meta, rows, heads: int, scale: float, positions: torch.Tensor,
                  latent: int | None = None, window: int = 0) -> torch.Tensor:
    """Absorbed form: q [R, heads * columns] (the first R rows of the batch) over the cached vectors; returns what is attended of
    their first `latent` columns (None: all), [R, heads * latent]. `rows` from `token_rows`; `window`: a row sees that many
    positions, its own included (0: all). f32 tensors also need `positions`."""
    from . import _count

    R, D = q.shape[0], cache.shape[2]
    L = latent or D
    if not q.is_cuda:
        qh = q.view(R, heads, D)
        o = reference.mla_attend(qh[..., :L], qh[..., L:], cache, meta.cu_q, meta.ctx_lens, meta.block_tables, scale, window)
        return o.reshape(R, -1).to(q.dtype)
    out = torch.empty(R, heads * L, dtype=q.dtype, device=q.device)
    if R == 0:
        return out
    C, st = _ext.require(), _state.get(q.device)
    row_ctx, row_seq = rows
    if q.dtype == torch.float32:
        if row_seq is None:
            row_seq = torch.arange(R, dtype=torch.int32, device=q.device)
        kv = cache.unsqueeze(1)
        C.attn_f32(q, kv, kv[..., :L], out, row_seq, positions, meta.block_tables, scale, None, st.status, window)
        _count()
        return out
    ctas, splits = R * ((heads + 15) // 16), 1
    max_ctx = min(meta.max_ctx, window) if window else meta.max_ctx
    if ctas < 148 and max_ctx > 256:
        splits = max(1, min((148 + ctas - 1) // ctas, max_ctx // 128, 16))
        splits = max(1, min(splits, _state.ATTN_WORKSPACE_BYTES // (R * heads * (L + 2) * 4)))
    C.latent_attend(q, cache, out, row_ctx, meta.block_tables, row_seq, st.attn_ws, heads, splits, scale, st.status, L, window)
    _count(2 if splits > 1 else 1)
    return out


def plan_latent_prefill(cu_q, ctx_lens, num_decode: int, latent: int, heads: int, dim: int, vdim: int, window: int = 0):
    """Whether the prefill sequences of a batch (host arrays) attend in the expanded form: where that is faster by the kernels'
    rates and its scratch stays small. Returns (pages int32 [n, 2] = (prefill sequence, block of 128 positions), tables int32
    [sequences, blocks]) or None. Blocks that lie outside every row's window are left out; their table entries mean nothing."""
    cu, ctx = np.asarray(cu_q[num_decode:], dtype=np.int64), np.asarray(ctx_lens[num_decode:], dtype=np.int64)
    q_len = cu[1:] - cu[:-1]
    skip = np.maximum(ctx - q_len - window + 1, 0) // EXPAND_PAGE if window else np.zeros_like(ctx)
    blocks = (ctx + EXPAND_PAGE - 1) // EXPAND_PAGE - skip
    n = int(blocks.sum())
    # operations per head, over rates: the prefill kernel works on tiles of 128 query rows
    seen = np.minimum(ctx, window) if window else ctx
    absorbed = float((q_len * seen).sum()) * 4 * latent / ABSORBED_RATE
    tiles = float(((q_len + 127) // 128 * 128 * (np.minimum(ctx, window + EXPAND_PAGE) if window else ctx)).sum())
    expanded = tiles * 2 * (dim + vdim) / PREFILL_RATE + n * EXPAND_PAGE * 2 * latent * (dim + vdim) / GEMM_RATE
    if n == 0 or expanded >= absorbed:
        return None
    if n * EXPAND_PAGE * heads * (dim + vdim) * 2 > EXPAND_BYTES:
        return None
    first = np.cumsum(blocks) - blocks
    seq = np.repeat(np.arange(len(blocks)), blocks)
    pages = np.stack([seq, np.arange(n) - first[seq] + skip[seq]], axis=1).astype(np.int32)
    tables = np.clip((first - skip)[:, None] + np.arange(int((blocks + skip).max()))[None], 0, n - 1).astype(np.int32)
    return pages, tables


def latent_prefill(q: torch.Tensor, cache: torch.Tensor, w_kv: torch.Tensor, meta, heads: int, scale: float, gate: torch.Tensor | None,
                   out: torch.Tensor, window: int = 0) -> None:
    """Expanded form for the prefill sequences of a batch (bf16, heads of 128, `meta.expand` from `plan_latent_prefill`):
    q [T, heads * 128], w_kv [2 * heads * 128, columns of the cache] (all keys, then all values). Writes the rows of those
    sequences in `out` [T, heads * 128], times sigmoid(gate), one per element or one per head."""
    from . import _count, linear

    C, st = _ext.require(), _state.get(q.device)
    pages, tables = meta.expand
    nd = meta.num_decode
    n, W = pages.shape[0], heads * 128
    lat = torch.empty(n * EXPAND_PAGE, cache.shape[2], dtype=q.dtype, device=q.device)
    C.latent_gather(cache, pages, meta.ctx_lens[nd:], meta.block_tables[nd:], lat, st.status)
    kv = linear(lat, w_kv)
    k, v = (kv[:, i * W:(i + 1) * W].view(n, EXPAND_PAGE, heads, 128).permute(0, 2, 1, 3) for i in (0, 1))
    C.attn_prefill_tc(q, k, v, out, meta.cu_q[nd:], meta.ctx_lens[nd:], tables, meta.max_q_len, scale, st.status, meta.work, None, meta.n_items, gate,
                      window)
    _count(2)
