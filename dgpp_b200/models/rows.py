"""Prefill / decode plumbing shared by the smaller family runners: chunked prefill of one request, batched decode with
one CUDA graph per batch width (static id / position / request tensors; recurrent state saved around warm-up and
capture so that only replays move the model), paged KV reservation, full-attention rows on the tensor-core kernels.
A subclass provides `forward(tokens, positions, row_req, chunk_slot, all_logits, pos0)` and, if it keeps state besides
the KV cache, `_state_tensors()` and `_reset_state(slot)`.  A subclass whose layers take runs of consecutive tokens of
several requests in one pass sets `mixed_runs` and provides `forward_runs`; `step` then carries prompt portions and
single decoded tokens of any requests together.
(reference counterparts: src/engine/graph_engine.hpp capture / replay, src/engine/paged_blocks.hpp.)
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List, Optional

import torch

from ..ops import core as ops


@dataclass
class RowRuns:
    """The rows of one pass as runs of consecutive tokens, one run per request."""
    start: torch.Tensor          # int32 [runs + 1] first row of every run
    row_run0: torch.Tensor       # int32 [rows] first row of the row's run
    lens: List[int]              # tokens per run
    slots: List[int]
    pos0: List[int]              # position of every run's first token

    def split(self, limit: int):
        """(rows of the runs of up to `limit` tokens, indices of the longer runs, first row of every run and behind the last)."""
        start = [0]
        for n in self.lens:
            start.append(start[-1] + n)
        return ([start[r] + k for r, n in enumerate(self.lens) if n <= limit for k in range(n)],
                [r for r, n in enumerate(self.lens) if n > limit], start)


class RowRunner:
    mixed_runs = False           # True: `forward_runs` exists and `step` may be used
    pooled = False               # True: `kv` is the pool that admission has to ask (its blocks are this runner's memory)

    def _init_pool(self, slots: int, device, kv_shapes, kv_dtype, page: int, max_seq_len: int, max_rows: int,
                   pool_tokens: int = 0) -> None:
        """Rows over one shared pool of `pool_tokens` cache positions (default: every slot at full length); kv_shapes lists
        (kv heads, key width, value width[, value heads]) per attention layer."""
        from ..engine.kv_cache import PagedKV

        self._init_rows(slots, device, max_rows=max_rows)
        per = (max_seq_len + page - 1) // page
        blocks = (pool_tokens + page - 1) // page if pool_tokens else slots * per
        self.kv = PagedKV(len(kv_shapes), 0, 0, max(blocks, 1), slots, max(min(per, blocks), 1), page, False, device,
                          shapes=kv_shapes, dtype=kv_dtype)
        self.pooled = True

    def _init_rows(self, slots: int, device, kv_layers: int = 0, kv_heads: int = 0, q_heads: int = 0, head_dim: int = 0,
                   page: int = 64, max_seq_len: int = 0, max_rows: int = 0) -> None:
        from ..engine.kv_cache import PagedKV

        self.dev, self.slots, self.max_rows = device, slots, max_rows
        self.lengths = [0] * slots
        self.use_graphs, self._graphs, self._static = True, {}, {}
        self.pdl_graphs = True      # programmatic-dependent-launch edges between this library's kernels in captured passes
        self.kv = None
        if kv_layers:
            blocks_per = (max_seq_len + page - 1) // page + 1
            self.kv = PagedKV(kv_layers, kv_heads, head_dim, slots * blocks_per + 2, slots, blocks_per, page, True, device)
            self.att_q, self.att_kv, self.att_d = q_heads, kv_heads, head_dim
            self.att_scale = 1.0 / math.sqrt(head_dim)
            self.tc_attn = (torch.device(device).type == "cuda" and head_dim in (128, 256)
                            and q_heads // kv_heads in (1, 2, 4, 8))
            if self.tc_attn:
                r, sp = min(max_rows, 32), 32
                self.att_scratch = (torch.empty(r * q_heads * sp * 2, dtype=torch.float32, device=device),
                                    torch.empty(r * q_heads * sp * head_dim, dtype=torch.float32, device=device))

    # ---- hooks
    def _state_tensors(self):
        return []

    def _reset_state(self, slot: int) -> None:
        pass

    def forward(self, tokens, positions, row_req, chunk_slot=None, all_logits=True, pos0=None, extra=None):
        raise NotImplementedError

    def _extra_rows(self, slots: List[int], tokens: List[int], prefill_slot: Optional[int] = None) -> List[List[int]]:
        """Further int32 rows a pass needs per token (they ride in the same static tensor as ids / positions / requests and
        reach `forward` as `extra`).  prefill_slot given: `tokens` are consecutive tokens of that request."""
        return []

    def _note_tokens(self, slot: int, tokens: List[int]) -> None:
        """Called after `tokens` were appended to request `slot`."""

    # ---- full attention over the paged FP8 cache
    def _attention_rows(self, cache_layer: int, qkv: torch.Tensor, positions, row_req, inv_freq, chunk_slot, pos0,
                        out: torch.Tensor) -> torch.Tensor:
        """qkv [rows, (hq + 2 hkv) d] bf16: rotary embedding, K/V append (FP8), causal attention of every row up to its
        own position -> out [rows, hq d].  Prefill chunks and up to 32 decode rows run on the tcgen05 kernels."""
        hq, hkv, d = self.att_q, self.att_kv, self.att_d
        rows = qkv.shape[0]
        cache = self.kv.layers[cache_layer]
        ops.rope_kv_write(qkv, positions, row_req, self.kv.block_table, inv_freq, cache, hq, hkv, d)
        if self.tc_attn and chunk_slot is not None and pos0 is not None:
            ops.attn_prefill_tc(qkv, qkv.stride(0), cache, self.kv.block_table[chunk_slot], pos0, hq, hkv, d,
                                self.att_scale, out=out, rows=rows)
        elif self.tc_attn and rows <= 32:
            splits = max(1, min(32, -(-160 // (hkv * rows))))
            ops.attn_decode_tc(qkv, qkv.stride(0), cache, self.kv.block_table, row_req, positions, hq, hkv, d,
                               self.att_scale, splits=splits, scratch=self.att_scratch, out=out)
        else:
            ops.attn_decode(qkv, qkv.stride(0), cache, self.kv.block_table, row_req, positions, hq, hkv, d,
                            self.att_scale, out=out)
        return out

    # ---- requests
    def reset(self, slot: int) -> None:
        if self.kv is not None:
            self.kv.release(slot)
        self.lengths[slot] = 0
        self._reset_state(slot)

    def forward_runs(self, tokens, positions, row_req, runs: RowRuns, logit_rows: torch.Tensor):
        """One pass over runs of several requests -> fp32 logits of the rows named by logit_rows (int64)."""
        raise NotImplementedError

    @torch.no_grad()
    def step(self, entries) -> torch.Tensor:
        """One mixed pass: entries = [(slot, tokens, want)], the next tokens of each (distinct) request and the places among
        them whose logits are wanted.  Every request advances by its tokens; returns fp32 logits [wanted, V] in the order
        of the entries and of their `want`.  Passes beyond `max_rows` rows are cut (the state carries over)."""
        assert self.mixed_runs and entries and len({s for s, _, _ in entries}) == len(entries)
        for slot, tokens, _ in entries:
            assert len(tokens) >= 1
            if not self.kv.reserve(slot, self.lengths[slot] + len(tokens)):
                raise RuntimeError("KV pool exhausted")
        if all(len(t) == 1 for _, t, _ in entries):
            logits = self.decode([s for s, _, _ in entries], [t[0] for _, t, _ in entries])
            rows = [i for i, (_, _, want) in enumerate(entries) for _ in want]
            return logits if rows == list(range(len(entries))) else logits[torch.tensor(rows, dtype=torch.long, device=self.dev)]
        parts, order = [], {}                       # logits per pass; (entry, place) -> row of their concatenation
        done, found = [0] * len(entries), 0
        while any(d < len(t) for d, (_, t, _) in zip(done, entries)):
            room, piece = self.max_rows, []
            for i, (slot, tokens, _) in enumerate(entries):
                n = min(len(tokens) - done[i], room)
                if n > 0:
                    piece.append((i, slot, tokens[done[i]:done[i] + n]))
                    room -= n
            toks, pos, req, run0, start, rows = [], [], [], [], [0], []
            for i, slot, part in piece:
                p0 = self.lengths[slot]
                wanted = set(entries[i][2])
                for k in range(len(part)):
                    if done[i] + k in wanted:
                        order[(i, done[i] + k)] = found
                        found += 1
                        rows.append(start[-1] + k)
                toks += part
                pos += range(p0, p0 + len(part))
                req += [slot] * len(part)
                run0 += [start[-1]] * len(part)
                start.append(start[-1] + len(part))
            n = len(toks)
            flat = torch.tensor(toks + pos + req + run0 + start, dtype=torch.int32).to(self.dev)
            runs = RowRuns(flat[4 * n:], flat[3 * n:4 * n], [len(p) for _, _, p in piece], [s for _, s, _ in piece],
                           [self.lengths[s] for _, s, _ in piece])
            out = self.forward_runs(flat[:n], flat[n:2 * n], flat[2 * n:3 * n], runs,
                                    torch.tensor(rows, dtype=torch.long, device=self.dev))
            if rows:
                parts.append(out)
            for i, slot, part in piece:
                self.lengths[slot] += len(part)
                done[i] += len(part)
                self._note_tokens(slot, part)
        idx = [order[(i, k)] for i, (_, _, want) in enumerate(entries) for k in want]
        if not idx:
            return torch.empty(0, 0, dtype=torch.float32, device=self.dev)
        logits = parts[0] if len(parts) == 1 else torch.cat(parts)
        return logits if idx == list(range(logits.shape[0])) else logits[torch.tensor(idx, dtype=torch.long, device=self.dev)]

    @torch.no_grad()
    def prefill(self, slot: int, tokens: List[int], chunk: int = 64) -> torch.Tensor:
        """Appends `tokens` to request `slot`; returns the logits of the last token [1, V]."""
        if self.mixed_runs:
            return self.step([(slot, list(tokens), [len(tokens) - 1])])
        start = self.lengths[slot]
        if self.kv is not None:
            assert self.kv.reserve(slot, start + len(tokens)), "KV pool exhausted"
        out = None
        for o in range(0, len(tokens), chunk):
            part = tokens[o:o + chunk]
            t = torch.tensor(part, dtype=torch.int32, device=self.dev)
            pos = torch.arange(start + o, start + o + len(part), dtype=torch.int32, device=self.dev)
            req = torch.full((len(part),), slot, dtype=torch.int32, device=self.dev)
            ex = self._extra_rows([slot], part, prefill_slot=slot)
            ex = torch.tensor(ex, dtype=torch.int32, device=self.dev) if ex else None
            out = self.forward(t, pos, req, chunk_slot=slot, all_logits=False, pos0=start + o, extra=ex)
            self._note_tokens(slot, part)
        self.lengths[slot] = start + len(tokens)
        return out

    @torch.no_grad()
    def decode(self, slots: List[int], tokens: List[int]) -> torch.Tensor:
        """One token for every listed request -> fp32 logits [len(slots), V]."""
        b = len(slots)
        positions = [self.lengths[s] for s in slots]
        if self.kv is not None:
            for s in slots:
                assert self.kv.reserve(s, self.lengths[s] + 1), "KV pool exhausted"
        host = torch.tensor([tokens, positions, slots] + self._extra_rows(slots, tokens), dtype=torch.int32)
        rest = lambda t: t[3:] if t.shape[0] > 3 else None
        if not (self.use_graphs and torch.device(self.dev).type == "cuda"):
            d = host.to(self.dev)
            out = self.forward(d[0], d[1], d[2], extra=rest(d))
        else:
            st = self._static.get(b)
            if st is None:
                st = self._static[b] = torch.zeros(host.shape[0], b, dtype=torch.int32, device=self.dev)
            st.copy_(host, non_blocking=True)
            g = self._graphs.get(b)
            if g is None:
                saved = [t.clone() for t in self._state_tensors()]
                side = torch.cuda.Stream()
                side.wait_stream(torch.cuda.current_stream())
                with torch.cuda.stream(side):
                    self.forward(st[0], st[1], st[2], extra=rest(st))
                torch.cuda.current_stream().wait_stream(side)
                torch.cuda.synchronize()
                from ..engine.graph import capture_with_pdl
                graph, out, _ = capture_with_pdl(lambda: self.forward(st[0], st[1], st[2], extra=rest(st)), self.pdl_graphs)
                for t, s0 in zip(self._state_tensors(), saved):
                    t.copy_(s0)
                g = self._graphs[b] = (graph, out)
            graph, out = g
            graph.replay()
        for s, t in zip(slots, tokens):
            self.lengths[s] += 1
            self._note_tokens(s, [t])
        return out
