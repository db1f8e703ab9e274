"""Mixture of experts over plain rows: bf16 (or fp32) expert matrices stacked for the grouped linear, a router and an optional
shared expert (gated or not) that read the same input in one fp32-output linear.  Experts are gated units or plain ones (`act`); router
outputs behind the last expert are identity experts, which cost nothing: the row kernel that sums a token's experts adds its input.  The router's weight multiplies an expert's input or its
output; since the projections around the activation are linear it is applied in the activation kernel either way.

Up to 16 rows: one launch routes and lists the experts in use, every listed expert reads all rows.  More rows: selection, counting
sort into tiles, row scatter (`csrc/kernels/moe_prefill.cu`, `moe_rows.cu`).  Both are shapes fixed by the row count alone, so passes
can be captured."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import core as ops
from ..ops import mixers as mx
from ..quant.formats import QuantLinear


@dataclass
class RowExperts:
    """Packed weights of one block."""
    experts: int                         # experts with matrices
    top: int
    ff: int                              # packed width of a routed expert (a multiple of 8)
    limit: float
    w_first: QuantLinear                 # [router rows | shared gate row | shared gate and up rows] over the input, fp32 results
    w_gu: torch.Tensor                   # [experts * 2 ff, Hp] (plain experts: [experts * ff, Hp])
    w_down: torch.Tensor                 # [experts * Hp, ff]
    hidden: int
    sg_col: int = 0                      # columns of w_first's result
    shared_col: int = 0
    shared_ff: int = 0                   # 0: no shared expert
    shared_limit: float = 0.0
    shared_down: Optional[QuantLinear] = None
    alpha: float = 1.702                 # activation: min(g, limit) sigmoid(alpha min(g, limit)) (clamp(u, +-limit) + shift)
    shift: float = 1.0
    score: str = "sigmoid"               # the router's weights (ops.mixers.SCORES)
    weigh_out: bool = False              # they multiply the experts' outputs instead of their inputs
    router_b: Optional[torch.Tensor] = None   # fp32 [outputs]: added to the logits
    correction: Optional[torch.Tensor] = None  # fp32 [outputs]: added to the scores for the choice alone
    norm_topk: bool = False              # weights divided by their sum
    identity: int = 0                    # router outputs whose expert is the input itself
    act: str = ""                        # plain experts: activation between up and down (ops.mixers.ACTS); "": gated units
    shared_gated: bool = True

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    @property
    def up_cols(self) -> int:
        return self.ff * (1 if self.act else 2)

    @property
    def nbytes(self) -> int:
        w = [self.w_gu, self.w_down]
        return sum(t.numel() * t.element_size() for t in w) + self.w_first.nbytes + (self.shared_down.nbytes if self.shared_ff else 0)

    def tile_rows(self, rows: int, f32: bool) -> int:
        """Rows of a tile: about the experts' average share, as the linears take them."""
        if rows <= mx.SMALL_TOKENS:
            return 16
        share = rows * self.top / self.outputs
        return next((bn for bn in (16, 32, 64) if share <= bn), 64 if f32 else 128)

    def max_tiles(self, rows: int, bn: int) -> int:
        pairs = rows * self.top
        return min(self.experts, pairs) + (0 if rows <= mx.SMALL_TOKENS else pairs // bn)


class RowExpertsScratch:
    """Buffers for passes of up to `rows` rows, shared by the blocks of one runner."""

    def __init__(self, blocks, rows: int, dtype: torch.dtype, device):
        f32 = dtype == torch.float32
        # every size grows with the row count while the tile stays the same: the largest count of every tile decides
        counts = lambda b: {min(rows, n) for n in (mx.SMALL_TOKENS, rows, *(bn * b.outputs // b.top for bn in (16, 32, 64)))}
        need = lambda f: max([f(b, n) for b in blocks for n in counts(b)] + [1])
        tiles = lambda b, n: b.max_tiles(n, b.tile_rows(n, f32))
        tr = lambda b, n: tiles(b, n) * b.tile_rows(n, f32)
        e = lambda n, dt: torch.empty(n, dtype=dt, device=device)
        self.first = e(need(lambda b, n: n * b.w_first.n), torch.float32)
        self.ids, self.wts = e(need(lambda b, n: n * b.top), torch.int32), e(need(lambda b, n: n * b.top), torch.float32)
        self.pair_row, self.tiles, self.n_tiles = e(need(lambda b, n: n * b.top), torch.int32), e(need(tiles), torch.int32), e(1, torch.int32)
        self.row_w = torch.zeros(need(tr), dtype=torch.float32, device=device)
        self.xs = e(need(lambda b, n: tr(b, n) * b.hidden), dtype)
        self.h = e(need(lambda b, n: tr(b, n) * b.up_cols), dtype)
        self.act = e(need(lambda b, n: tr(b, n) * b.ff), dtype)
        self.shared_act = e(need(lambda b, n: n * b.shared_ff), dtype)
        self.y = e(need(lambda b, n: tr(b, n) * b.hidden), dtype)
        self.shared = e(need(lambda b, n: n * b.hidden if b.shared_ff else 0), dtype)


def run_experts(b: RowExperts, s: RowExpertsScratch, x: torch.Tensor) -> mx.MoeDelta:
    """x [rows, hidden] -> the block's result as the rows ``stream_norm`` sums."""
    rows, f32 = x.shape[0], x.dtype == torch.float32
    view = lambda buf, *shape: buf[:torch.Size(shape).numel()].view(*shape)
    first = view(s.first, rows, b.w_first.n)
    ops.linear(x, b.w_first, out=first) if f32 else ops.gemm_tc(x, b.w_first, out32=first)
    bn = b.tile_rows(rows, f32)
    nt = b.max_tiles(rows, bn)
    tiles, pair_row, row_w = s.tiles[:nt], s.pair_row[:rows * b.top], s.row_w[:nt * bn]
    wts = view(s.wts, rows, b.top)
    if rows <= mx.SMALL_TOKENS:
        mx.moe_route_small(first, b.experts, b.top, pair_row, tiles, row_w, b.score, b.router_b, b.correction, b.norm_topk, b.identity,
                           wts if b.identity else None)
        xs = x
    else:
        ids = view(s.ids, rows, b.top)
        mx.moe_select(first, b.outputs, b.top, ids, wts, b.score, b.norm_topk, bias=b.router_b, correction=b.correction)
        ops.moe_segment_sort(ids, bn, nt, 0, b.experts, pair_row, tiles, s.n_tiles)
        xs = view(s.xs, nt * bn, b.hidden)
        mx.moe_scatter_rows(x, pair_row, wts, xs, row_w, b.top)
    h = mx.grouped_linear(xs, b.w_gu, b.up_cols, tiles, bn, view(s.h, nt * bn, b.up_cols), shared_rows=xs is x)
    act = view(s.act, nt * bn, b.ff)
    if b.act:
        mx.act_rows(h, act, b.act, row_w, tiles, bn)
    else:
        mx.clamped_glu(h, act, b.limit, b.alpha, row_w, tiles, bn, b.shift, b.weigh_out)
    y = mx.grouped_linear(act, b.w_down, b.hidden, tiles, bn, view(s.y, nt * bn, b.hidden))
    own = dict(self_rows=x, wts=wts) if b.identity else {}
    if not b.shared_ff:
        return mx.MoeDelta(y, pair_row, b.top, **own)
    act = view(s.shared_act, rows, b.shared_ff)
    if b.act:
        mx.act_rows(first[:, b.shared_col:], act, b.act)
    else:
        mx.clamped_glu(first[:, b.shared_col:], act, b.shared_limit, b.alpha, shift=b.shift)
    return mx.MoeDelta(y, pair_row, b.top, ops.linear(act, b.shared_down, out=view(s.shared, rows, b.hidden)),
                       first[:, b.sg_col:] if b.shared_gated else None, **own)
