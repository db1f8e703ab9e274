"""Vevapel at the sizes of a real model's layers, beside the closest families at equal size (random weights, one GPU).

    python bench.py --family vevapel [--sizes 2048,4096] [--steps K] [--warmup W]

Kernels: every state, attention, expert and row operator of the family, decode (64 requests, experts also 8) and prefill (2048
tokens of one request), next to the like operator of the family closest to it: the gated delta rule of `models/gdn.py`
(convolution + recurrence + gated norm); for full causal attention and for differential attention the grouped attention of
`models/sitirax.py` over the same 16-bit cache with the same keys per row (per-head norms there); the bf16 experts of
`models/potivik.py`; the norms of that family.  Inputs rotate over more than the 126 MB L2.  `roofline_ms` is the larger of algorithmic
bytes / measured copy bandwidth and FLOPs / measured bf16 throughput (fp32 work on the CUDA cores: FLOPs / 2 x 128 x SMs x clock);
`frac` = roofline_ms / measured.

Models: 8 layer runs of width W (delta, differential and full attention in turn, 64 experts of width / 2, 8 per token), without a loop
and as 6 layers of which two run twice, against the latent + state-space family with equal bf16 experts and the delta-rule + gated
attention family with NVFP4 experts: decode tokens/s at 1, 8 and 64 requests and prefill tokens/s of one 4096-token prompt
(2048-token passes).  A decode step includes the runner's host work and the read-back of its tokens.
"""
from __future__ import annotations

import json
from typing import List

import torch

from .configs import _time_decode, _time_prefill
from .micro import peaks
from .sitirax import _roof, _row

BF = torch.bfloat16


def _state_rows(dev, batch: int, rows: int, heads: int = 32, hk: int = 16, dim: int = 128, copies: int = 3) -> List[dict]:
    from ..models.rows import RowRuns
    from ..ops import core as ops, mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    out, taps, nq, nv = [], 4, hk * dim, heads * dim
    C = 2 * nq + nv
    s = mx.StateHeads(heads, hk, dim, dim, 0, C, 1e-5, rnd(taps, C), rnd(heads) - 2, rnd(heads) - 2, norm_w=rnd(dim), a_off=C + heads, gate_off=C + 2 * heads)
    st = [s.new_state(batch, dev) for _ in range(copies)]
    conv = [torch.zeros(batch, taps - 1, C, device=dev) for _ in range(copies)]
    cw, nw, big = rnd(C, taps).to(BF), rnd(dim).to(BF), max(rows, batch)
    prep = torch.empty(max(s.prep_floats(big, 1), big * (2 * nq + 2 * heads)), device=dev)
    for n, seq in ((batch, False), (rows, True)):
        pos = torch.full((n,), 5, dtype=torch.int32, device=dev) if not seq else torch.arange(5, 5 + n, dtype=torch.int32, device=dev)
        slot = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
        runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [5]) if seq else None
        x = [rnd(n, C + 2 * heads + nv).to(BF) for _ in range(copies)]
        o32, o16, c16, gated = torch.empty(n, nv, device=dev), torch.empty(n, nv, dtype=BF, device=dev), torch.empty(n, C, dtype=BF, device=dev), torch.empty(n, nv, dtype=BF, device=dev)

        def mine(j):
            if not seq:
                return mx.linear_state(s, x[j], *st[j], slot, pos, out=gated)
            mx.linear_state(s, x[j], *st[j], slot, pos, runs=runs, prep=prep, o=o32)
            mx.gated_group_norm(o32, x[j][:, s.gate_off:], s.norm_w, gated, heads, dim, 1e-5, silu=True)

        def gdn(j):
            y, ab = ops.gdn_conv(x[j][:, :C], cw, None, conv[j], c16, None if seq else slot, 0, seq), x[j][:, C:]
            ops.gdn_recurrent(y[:, :nq], y[:, nq:2 * nq], y[:, 2 * nq:], ab[:, heads:2 * heads], ab[:, :heads], s.A_log, s.dt_bias, st[j][0], o16, hk, heads, dim, dim,
                              None if seq else slot, 0, seq, prep=prep)
            ops.gated_rmsnorm(o16, x[j][:, C + 2 * heads:], nw, gated, heads, dim)

        sio = (n if not seq else 1) * heads * dim * dim * 8
        roof = _roof(sio + n * (C + 2 * heads + 2 * nv) * 2, fp32_flops=n * heads * dim * dim * 8.0)
        out.append(_row(f"delta rule + gated norm, {'prefill' if seq else 'decode'}", [lambda j=j: mine(j) for j in range(copies)],
                        [lambda j=j: gdn(j) for j in range(copies)], roof, roof))
    return out


def _attention_rows(dev, batch: int, rows: int, heads: int = 32, kv: int = 8, dim: int = 128, ctx: int = 2048, chunk: int = 1024) -> List[dict]:
    """Full attention over ctx earlier keys; differential attention (heads / 2 output heads, kv / 2 value heads of twice the width) inside
    chunks, decode rows and prompt at a chunk's end; the like operator sees the same number of keys per row."""
    from ..engine.kv_cache import PagedKV
    from ..models.rows import RowRuns
    from ..ops import mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    nq, nk = heads * dim, kv * dim
    cols, out = nq + 2 * nk, []
    per = (ctx + rows) // 64 + 1
    w_row, w_krow, w_head = rnd(nq), rnd(nk), torch.ones(dim, device=dev)
    bias, freq = (rnd(nq), rnd(nk), rnd(nk)), mx.rotation_freqs(1e4, dim, dev)
    full = mx.WindowHeads(heads, kv, dim, dim, mx.NO_WINDOW, dim ** -0.5, 1e-5, 0, nq, nq + nk, norm="row", bias=bias, temp=(0.1, 1024), gate_off=cols)
    diff = mx.WindowHeads(heads // 2, kv // 2, dim, 2 * dim, chunk, dim ** -0.5, 1e-5, 0, nq, nq + nk, norm=None, bias=bias, freq=freq, rot=dim, maps=2, chunked=True)
    base = mx.WindowHeads(heads, kv, dim, dim, mx.NO_WINDOW, dim ** -0.5, 1e-5, 0, nq, nq + nk)
    part = mx.WindowHeads(heads, kv, dim, dim, chunk, dim ** -0.5, 1e-5, 0, nq, nq + nk)
    for name, g, like_g, wq, wk in (("full attention", full, base, w_row, w_krow), ("differential attention", diff, part, None, None)):
        span = ctx if g is full else chunk
        kvs = [[PagedKV(1, 0, 0, batch * (ctx // 64 + 1) + per, batch, per, 64, False, dev, shapes=[h.kv_shape]) for _ in range(2)] for h in (g, like_g)]
        for c in kvs[0] + kvs[1]:
            for s in range(batch):
                assert c.reserve(s, ctx + (rows if s == 0 else 0))
            for t in (c.layers[0].k, c.layers[0].v):
                t.copy_(rnd(*t.shape))
        for n, seq in ((batch, False), (8, False), (rows, True)):
            first = ctx if g is full else (ctx // chunk) * chunk
            pos = torch.full((n,), ctx - 1, dtype=torch.int32, device=dev) if not seq else torch.arange(first, first + n, dtype=torch.int32, device=dev)
            req = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
            x, gx = rnd(n, cols + nq).to(BF), rnd(n, cols + nq).to(BF)
            y = torch.empty(n, nq, dtype=BF, device=dev)
            runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [first])
            scratch = (torch.empty(n * heads * 32 * 2, device=dev), torch.empty(n * heads * (32 if not seq else 1) * g.DV, device=dev))

            def run(h, c, q, k, a):
                args = (h, a, q, k, c.layers[0], c.block_table, req, pos)
                if not seq:
                    sp = h.splits(n, ctx, 32)
                    mx.window_attn(*args, y, fused=True, splits=sp, scratch=scratch)
                    if h.maps == 2:
                        mx.diff_combine(h, scratch, a, cols, y, 0.3, 0.7, sp)
                    return
                mx.qk_norm_append(*args)
                mx.window_prefill(h, a, c.layers[0], c.block_table, req, pos, runs, y, raw=scratch[1] if h.maps == 2 else None)
                if h.maps == 2:
                    mx.diff_combine(h, scratch[1], a, cols, y, 0.3, 0.7, finished=True)

            keys = n * span if not seq else first + n - (0 if g is full else first)
            seen = span if not seq else (ctx + n / 2 if g is full else chunk / 2)
            like_seen = seen if not seq or g is full else chunk
            kb = 2 * nk * 2
            io = n * (cols + nq + (nq if g.maps == 2 else heads)) * 2
            fl = n * seen * heads * (dim + g.DV) * 2.0
            lfl, like_io = n * like_seen * heads * 2 * dim * 2.0, n * (cols + nq) * 2
            out.append(_row(f"{name}, {'prefill' if seq else 'decode'} {n} rows", [lambda c=c: run(g, c, wq, wk, x) for c in kvs[0]],
                            [lambda c=c: run(like_g, c, w_head, w_head, gx) for c in kvs[1]], _roof(keys * kb + io, fl),
                            _roof((keys if not seq or g is full else n + chunk) * kb + like_io, lfl)))
        del kvs
        torch.cuda.empty_cache()
    return out


def _expert_rows(dev, batch: int, rows: int, width: int = 2048, experts: int = 64, top: int = 8, ff: int = 1024) -> List[dict]:
    from ..models.row_moe import RowExperts, RowExpertsScratch, run_experts
    from ..ops import core as ops, mixers as mx
    from ..quant.formats import QuantLinear

    rnd = lambda *s: torch.randn(*s, device=dev).to(BF) * s[-1] ** -0.5
    first, gu, down = QuantLinear("bf16", experts, width, rnd(experts, width)), rnd(experts * 2 * ff, width), rnd(experts * width, ff)
    mine = RowExperts(experts, top, ff, float("inf"), first, gu, down, width, alpha=1.0, shift=0.0, score="chosen", weigh_out=True, router_b=torch.zeros(experts, device=dev))
    like = RowExperts(experts, top, ff, 7.0, first, gu, down, width)
    scratch = RowExpertsScratch([mine, like], max(rows, batch), BF, dev)
    x32, w, b = torch.randn(max(rows, batch), width, device=dev), torch.ones(width, device=dev), torch.zeros(width, device=dev)
    out = torch.empty(max(rows, batch), width, dtype=BF, device=dev)
    res = []
    for n in (8, batch, rows):
        x = [torch.randn(n, width, device=dev).to(BF) for _ in range(3)]
        pairs = n * top
        active = len(set((ops.gemm_tc(x[0], first, out32=torch.empty(n, experts, device=dev)) + mine.router_b).topk(top).indices.flatten().tolist()))
        run = lambda blk, j, post: mx.stream_norm(x32[:n], width, 1e-5, out[:n], run_experts(blk, scratch, x[j]), post, (None, None), 0.8)
        roof = _roof(active * 3 * ff * width * 2 + n * width * 2 + pairs * (width * 4 + ff * 6), pairs * 3.0 * ff * width * 2)
        res.append(_row(f"expert block + norm, {n} rows", [lambda j=j: run(mine, j, ("layer", w, b)) for j in range(3)],
                        [lambda j=j: run(like, j, ("layer", w)) for j in range(3)], roof, roof))
    return res


def _row_operators(dev, rows: int, width: int = 4096) -> List[dict]:
    from ..ops import core as ops, mixers as mx
    from ..quant.formats import QuantLinear

    rnd = lambda *s: torch.randn(*s, device=dev)
    x, d, xn = [rnd(rows, width) for _ in range(4)], [rnd(rows, width) for _ in range(4)], torch.empty(rows, width, dtype=BF, device=dev)
    w, b = rnd(width), rnd(width)
    out = [_row("norm, residual, norm with biases", [lambda j=j: mx.stream_norm(x[j], width, 1e-5, xn, d[j], ("layer", w, b), ("layer", w, b), 0.8, b) for j in range(4)],
                [lambda j=j: mx.stream_norm(x[j], width, 1e-5, xn, d[j], ("layer", w), ("layer", w)) for j in range(4)], _roof(rows * width * 14), _roof(rows * width * 14))]
    xx, m = [rnd(rows, 2 * width).to(BF) for _ in range(3)], QuantLinear("bf16", width, 2 * width, (rnd(width, 2 * width) * 0.01).to(BF))
    dx = torch.empty(rows, width, device=dev)

    def entry(j):
        mx.stream_norm(x[j], width, 1e-5, xx[j][:, :width], d[j], ("layer", w, b), (None, None), 0.8)
        ops.gemm_tc(xx[j], m, out32=dx)
        mx.stream_norm(dx, width, 1e-5, xn, None, (None, None), ("layer", w, b), vec=b)

    def plain_linear(j):
        mx.stream_norm(x[j], width, 1e-5, xn, d[j], ("layer", w), ("layer", w))
        ops.gemm_tc(xx[j], m, out32=dx)

    fl = rows * width * width * 4.0
    out.append(_row("entry of a loop's pass", [lambda j=j: entry(j) for j in range(3)], [lambda j=j: plain_linear(j) for j in range(3)],
                    _roof(rows * width * (14 + 4 + 14) + m.nbytes, fl), _roof(rows * width * (14 + 4 + 4) + m.nbytes, fl)))
    return out


def kernels(dev, batch: int = 64, rows: int = 2048) -> List[dict]:
    return _state_rows(dev, batch, rows) + _attention_rows(dev, batch, rows) + _expert_rows(dev, batch, rows) + _row_operators(dev, rows)


def _runners(width: int, layers: int, dev, slots: int, max_seq: int):
    """(name, runner, weight bytes) of the models at equal width and depth, one after the other."""
    from ..models.hybrid import HybridConfig, HybridModel, HybridRunner
    from ..models.moe import MoEConfig
    from ..models.potivik import ExpertsSpec as PExperts, FeedForward, LatentSpec, PotivikConfig, PotivikModel, PotivikRunner, StateSpaceSpec
    from ..models.vevapel import AttentionSpec, DeltaSpec, DiffSpec, ExpertsSpec, LoopSpec, VevapelConfig, VevapelModel, VevapelRunner

    h, vocab, rows = width // 128, 32768, 2048
    kv = max(h // 4, 1)
    mixers = (DeltaSpec(h, h // 2, 128, 128, 4), DiffSpec(h // 2, max(kv // 2, 1), 128, 256, 128 ** -0.5, 1024, 1e4, 128, 0.3),
              AttentionSpec(h, kv, 128, 128, 128 ** -0.5, 0.1, 1024))
    moe = ExpertsSpec(64, 8, width // 2)
    for name, n, loop in (("vevapel", layers, None), ("vevapel, two layers run twice", layers - 2, LoopSpec(2, 4, 2))):
        m = VevapelModel.random_init(VevapelConfig.cycle(n, width, vocab, mixers, moe, loop), dev, std=0.02)
        yield name, VevapelRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
        del m
        torch.cuda.empty_cache()
    c = PotivikConfig.uniform(layers, width, vocab, LatentSpec(h, 128, 64, 128, 512, 192 ** -0.5, 1024, 1e4, 64), StateSpaceSpec(width // 32, 1, 64, 128, 4, 8),
                              PExperts(64, 8, FeedForward(width // 2, 7.0), None), FeedForward(width // 2, 7.0), 256)
    c.plan = [type(L)(L.mixer, c.plan[1].mlp) for L in c.plan]
    m = PotivikModel.random_init(c, dev, std=0.02)
    yield "latent + state space, bf16 experts", PotivikRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
    del m
    torch.cuda.empty_cache()
    c = HybridConfig(layers=layers, hidden=width, full_every=2, q_heads=h, kv_heads=kv, head_dim=128, gdn_k_heads=h // 2, gdn_v_heads=h, vocab=vocab,
                     moe=MoEConfig(width, 64, 8, width // 2, width // 2, router="softmax"))
    m = HybridModel.random_init(c, dev, std=0.02, fmt="nvfp4")
    yield "delta rule + attention, NVFP4 experts", HybridRunner(m, max_rows=rows, slots=slots, max_seq_len=max_seq, device=dev), 0
    del m
    torch.cuda.empty_cache()


def models(width: int, dev, steps: int, warmup: int, layers: int = 8) -> List[dict]:
    res, gen, vocab = [], torch.Generator().manual_seed(0), 32768
    for name, r, wbytes in _runners(width, layers, dev, 64, 4608):
        row = {"model": name, "width": width, "layer_runs": layers}
        if wbytes:
            row["weight_gb"] = round(wbytes / 1e9, 3)
        _time_prefill(r, vocab, 0, 4096, gen, 2048)
        row["prefill_4096_tok_s"] = round(4096 / min(_time_prefill(r, vocab, 0, 4096, gen, 2048) for _ in range(3)))
        for s in range(1, 64):
            r.prefill(s, torch.randint(0, vocab, (64,), generator=gen).tolist(), chunk=2048)
        for b in (1, 8, 64):
            ms = _time_decode(r, vocab, list(range(b)), steps, warmup, gen)
            row[f"decode_{b}_ms"], row[f"decode_{b}_tok_s"] = round(ms, 3), round(1e3 * b / ms)
        print("# " + json.dumps(row), flush=True)
        res.append(row)
        del r
        torch.cuda.empty_cache()
    return res


def run(args) -> int:
    from ..ops import core as ops

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    with torch.no_grad():
        res = {"family": "vevapel", "dtype": "bf16", "data": "synthetic", "peaks": peaks(), "kernels": kernels(dev)}
        ops.check_status()
        for row in res["kernels"]:
            print("# " + json.dumps(row), flush=True)
        res["models"] = [row for w in args.sizes.split(",") if w for row in models(int(w), dev, max(args.steps, 1), max(args.warmup, 3))]
    ops.check_status()
    print(json.dumps(res))
    return 0
