"""Mixture of experts with all experts on one GPU: router, permutation of the token rows, grouped products over a packed list
of tiles. Nothing is read back to the host, so a layer can be captured in a CUDA graph. The weighted sum of the experts'
rows is left to the kernel that adds them to the residual (`ops.residual_norm`). `parallel.ep` spreads experts over ranks."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import _ext
from . import _state, reference
from .activation import SWIGLU, Glu

SCORING = {"softmax": 0, "sigmoid": 1}


@dataclass
class MoeWeights:
    """router [>= experts + identity, width] (rows past those are not looked at here), w_gu [experts, 2 ffn, width] (gate and up
    rows interleaved in blocks of 16; with `glu` None, squared-ReLU experts, [experts, ffn, width]), w_down [experts, width,
    ffn]. A token uses the `top` experts of the largest scores, with their scores (over their sum if `norm_top`) times `scale`
    as weights. `correction` f32 [experts + identity] is added to the scores for the choice alone; the choice is among the
    `keep` of `groups` groups of neighbours with the largest scores in them. The last `identity` experts return their input.
    `on_input`: a weight multiplies what its expert reads, not what it returns."""
    router: torch.Tensor
    w_gu: torch.Tensor
    w_down: torch.Tensor
    experts: int
    top: int
    scoring: str = "softmax"
    norm_top: bool = False
    scale: float = 1.0
    glu: Glu | None = SWIGLU
    correction: torch.Tensor | None = None
    groups: int = 1
    keep: int = 1
    identity: int = 0
    on_input: bool = False


@dataclass
class ExpertRows:
    """Results of a token's experts: rows[slot[t, j]] times weights[t, j], summed over j. A slot of -1 stands for the token's own
    input row, `own[t]`."""
    rows: torch.Tensor
    slot: torch.Tensor                  # int32 [T, top]
    weights: torch.Tensor | None        # f32 [T, top]; None: one
    own: torch.Tensor | None = None

    def total(self) -> torch.Tensor:
        """The weighted sums, f32 [T, width], by plain tensor operations."""
        e = self.rows.float()[self.slot.clamp_min(0).long()]
        if self.own is not None:
            e = torch.where((self.slot < 0).unsqueeze(-1), self.own.float().unsqueeze(1), e)
        return e.sum(1) if self.weights is None else torch.einsum("tk,tkw->tw", self.weights, e)


def tile_rows(rows_per_expert: float) -> int:
    """Token rows of one tile of the grouped product: the narrowest that usually holds an expert's rows."""
    return next((n for n in (16, 32, 64, 128) if rows_per_expert * 1.25 <= n), 256)


def moe_experts(h: torch.Tensor, p: MoeWeights, logits: torch.Tensor | None = None) -> ExpertRows:
    """Run every row of h [T, width] through its experts. `logits`: the router's, f32, where the caller has them already."""
    from . import EPI_NONE, EPI_RELU2, EPI_SWIGLU, _count, linear_f32

    T, W = h.shape
    if logits is None:
        logits = linear_f32(h, p.router)
    own = h if p.identity else None
    n_out = p.experts + p.identity
    if not h.is_cuda:
        weights, ids = reference.moe_route(logits[:, :n_out], p.top, p.norm_top, p.scale, p.scoring == "sigmoid", p.correction, p.groups, p.keep)
        rows = torch.zeros(T, p.top, W, dtype=h.dtype)
        for e in range(p.experts):
            tok, j = torch.where(ids == e)
            if tok.numel():
                x = (h[tok].float() * weights[tok, j].unsqueeze(-1)).to(h.dtype) if p.on_input else h[tok]
                if p.glu is None:
                    act = reference.linear(x, p.w_gu[e]).clamp_min(0.0).square()
                else:
                    act = reference.linear_swiglu_interleaved(x, p.w_gu[e], act=p.glu)
                rows[tok, j] = reference.linear(act.to(h.dtype), p.w_down[e]).to(h.dtype)
        slot = torch.where(ids < p.experts, torch.arange(T * p.top).view(T, p.top), -1).int()
        return ExpertRows(rows.view(T * p.top, W), slot, None if p.on_input else weights.float(), own)
    C, st = _ext.require(), _state.get(h.device)
    dev, R, f32 = h.device, T * p.top, h.dtype == torch.float32
    bn = 64 if f32 else tile_rows(R / n_out)
    weights = torch.empty(T, p.top, dtype=torch.float32, device=dev)
    ids, place, slot = (torch.empty(T, p.top, dtype=torch.int32, device=dev) for _ in range(3))
    counts = st.moe_counts
    C.moe_route(logits, weights, ids, place, counts, p.experts, SCORING[p.scoring], p.norm_top, p.scale, p.correction, p.groups, p.keep, p.identity)
    xs = torch.empty(R, W, dtype=h.dtype, device=dev)
    tiles, n_tiles = torch.empty(p.experts + R // bn, 4, dtype=torch.int32, device=dev), torch.empty(1, dtype=torch.int32, device=dev)
    C.moe_gather(h, ids, place, counts, slot, xs, tiles, n_tiles, p.experts, bn, st.status, weights if p.on_input else None)
    f = p.w_down.shape[2]
    act, y = torch.empty(R, f, dtype=h.dtype, device=dev), torch.empty(R, W, dtype=h.dtype, device=dev)
    launches = 4
    if p.glu is None:
        C.moe_tiles_gemm(xs, p.w_gu, tiles, n_tiles, act, EPI_RELU2, bn, None, st.status)
    elif f32:
        gu = torch.empty(R, 2 * f, dtype=h.dtype, device=dev)
        C.moe_tiles_gemm(xs, p.w_gu, tiles, n_tiles, gu, EPI_NONE, bn, None, st.status)
        C.glu_f32(gu, act, *p.glu)
        launches = 5
    else:
        C.moe_tiles_gemm(xs, p.w_gu, tiles, n_tiles, act, EPI_SWIGLU, bn, (*p.glu, 0.0), st.status)
    C.moe_tiles_gemm(act, p.w_down, tiles, n_tiles, y, EPI_NONE, bn, None, st.status)
    _count(launches)
    return ExpertRows(y, slot, None if p.on_input else weights, own)
