"""Attention of ``WindowHeads`` layers over the shared page pool, as the runners of several families have it: decode passes in one fused launch
per layer, prompt passes prepared row by row and then attended on the tensor cores (long runs) or row by row with splits (short runs,
fp32).  A subclass calls ``_init_attention`` behind ``_init_pool`` and ``_attend`` once per layer."""
from __future__ import annotations

from typing import List, Optional

import torch

from ..ops import mixers as mx
from .rows import RowRunner, RowRuns

SINGLE_RUN = 8                  # runs of a mixed pass up to this length attend row by row, longer ones on the prompt kernel


class WindowRowRunner(RowRunner):
    def _init_attention(self, heads: List[mx.WindowHeads], max_rows: int, slots: int, page: int, dtype: torch.dtype, device) -> None:
        e = lambda n, dt: torch.empty(max(n, 1), dtype=dt, device=device)
        big = lambda vals: max(list(vals) + [1])
        self.tc_prefill = True
        self.max_span = self.kv.max_blocks * page
        self.max_splits = 32
        self.parts = slots * self.max_splits
        # partial results of single rows; with two maps the outputs of all rows
        cap = lambda g: max(self.parts, max_rows) if g.maps == 2 else self.parts
        self.scratch = (e(big(cap(g) * g.hq * 2 for g in heads), torch.float32), e(big(cap(g) * g.hq * g.DV for g in heads), torch.float32))
        self.conv = e(big(max_rows * g.channels for g in heads if g.taps), dtype)                # convolved prompt rows
        self.turn = e(big(max_rows * g.DV for g in heads if g.vfreq is not None), torch.float32)  # angles of rotated values

    def _plan(self, runs: RowRuns):
        """(single rows, (first rows, lengths, lengths on the host) of the longer runs, rows of the longer runs) on the device; None for
        an empty part, and for a list that would name every row."""
        short, long, start = runs.split(SINGLE_RUN)
        lens = [runs.lens[r] for r in long]
        if not short:
            return None, (runs.start, None, lens), None
        rows = [start[r] + k for r in long for k in range(runs.lens[r])]
        dev = torch.tensor(short + [start[r] for r in long] + lens + rows, dtype=torch.int32).to(self.dev)
        n, k = len(short), len(long)
        return dev[:n], ((dev[n:n + k], dev[n + k:n + 2 * k], lens) if long else None), dev[n + 2 * k:]

    def _attend_rows(self, g, norms, diff, proj, mixed, positions, row_req, cache, splits: int, fused: bool, row_list=None, ring=None) -> None:
        mx.window_attn(g, proj, *norms, cache, self.kv.block_table, row_req, positions, mixed, fused=fused, splits=splits, scratch=self.scratch,
                       row_list=row_list, ring=ring)
        if diff is not None:
            gated, off, lam, factor = diff
            mx.diff_combine(g, self.scratch, gated, off, mixed, lam, factor, splits, row_list)

    def _attend(self, g: mx.WindowHeads, norms, cache, proj, mixed, positions, row_req, runs: Optional[RowRuns], plan, diff=None, ring=None) -> None:
        """proj rows -> mixed [rows, heads * DV].  norms: (query, key) norm weights; plan: `_plan` of the pass; diff: (rows that hold the
        gate, its column, lambda, factor) of differential attention; ring: the convolution's history."""
        bt, rows = self.kv.block_table, proj.shape[0]
        if runs is None:
            return self._attend_rows(g, norms, diff, proj, mixed, positions, row_req, cache, g.splits(rows, self.max_span, self.max_splits), True, ring=ring)
        if g.taps:
            after = self.conv[:rows * g.channels].view(rows, g.channels)
            proj, g = mx.short_conv(proj[:, g.q_off:], g.stacked_bias, g.conv_w, ring, row_req, positions, runs, after), g.after_conv
        tc = self.tc_prefill and mx.window_prefill_usable(g, proj, cache.page)
        turn = self.turn[:rows * g.DV] if tc and g.vfreq is not None else None
        mx.qk_norm_append(g, proj, *norms, cache, bt, row_req, positions, turn)
        if not tc:
            return self._attend_rows(g, norms, diff, proj, mixed, positions, row_req, cache, 1, False)
        short, long, long_rows = plan
        if long is not None:
            raw = self.scratch[1] if g.maps == 2 else None
            mx.window_prefill(g, proj, cache, bt, row_req, positions, runs, mixed, raw=raw, some=long, turn=turn)
            if diff is not None:
                gated, off, lam, factor = diff
                mx.diff_combine(g, raw, gated, off, mixed, lam, factor, row_list=long_rows, finished=True)
        if short is not None:
            n = short.numel()
            splits = min(g.splits(n, self.max_span, self.max_splits), max(1, self.parts // n))
            self._attend_rows(g, norms, diff, proj, mixed, positions, row_req, cache, splits, False, short)
