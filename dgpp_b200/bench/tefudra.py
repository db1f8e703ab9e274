"""Tefudra at the sizes of a real model's layers, beside the closest families at equal size (random weights, one GPU).

    python bench.py --family tefudra [--sizes 2048,4096] [--steps K] [--warmup W]

Kernels: every attention, memory, expert and row operator of the family, decode (64 requests, also 8) and prefill (2048 tokens of one
request), next to the like operator of the family closest to it: for both attentions the sliding-window attention of
`models/sitirax.py` (norms, append, same window, same 16-bit cache; no convolution, rotation, cap, sink or kept tokens there); for the matrix
memory that family's lightning attention with its gated norm; for the convolution the one of `models/gdn.py` (with a silu); the bf16 experts
(gated, a gated shared expert) of `models/potivik.py`; the norms and activations of that family.  Inputs rotate over more than the 126 MB
L2.  `roofline_ms` is the larger of algorithmic bytes / measured copy bandwidth and FLOPs / measured bf16 throughput (fp32 work on the CUDA
cores: FLOPs / 2 x 128 x SMs x clock); `frac` = roofline_ms / measured.

Models: 8 layers of width W (attention and parallel layers in turn), dense feed-forwards of 4 W or 64 experts of W / 2 and 8 identity
experts, 8 per token, with a shared expert, against the family with window attention beside lightning attention (gated dense
feed-forwards of equal bytes) and the latent + state-space family with equal numbers of bf16 experts: decode tokens/s at 1, 8 and 64
requests and prefill tokens/s of one 4096-token prompt (2048-token passes).  A decode step includes the runner's host work and the
read-back of its tokens.
"""
from __future__ import annotations

import json
import math
from typing import List

import torch

from .configs import _time_decode, _time_prefill
from .micro import peaks
from .sitirax import _roof, _row

BF = torch.bfloat16


def _memory_rows(dev, batch: int, rows: int, heads: int = 32, dim: int = 128, copies: int = 3) -> List[dict]:
    from ..models.rows import RowRuns
    from ..ops import mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    out, K = [], heads * dim
    g = mx.MatrixHeads(heads, dim, dim, 0, 4 * K, 4 * K + heads, 3 * K, rnd(heads), rnd(heads) + 3, 15.0, rnd(K), 1e-5)
    light = mx.StateHeads(heads, heads, dim, dim, 0, eps=1e-5, decay=torch.rand(heads, device=dev))
    st, ls = [g.new_state(batch, dev) for _ in range(copies)], [light.new_state(batch, dev)[0] for _ in range(copies)]
    big = max(rows, batch)
    prep = torch.empty(max(g.prep_floats(big, 1), light.prep_floats(big, 1)), device=dev)
    w_all = rnd(K)
    for n, seq in ((batch, False), (8, False), (rows, True)):
        pos = torch.full((n,), 5, dtype=torch.int32, device=dev) if not seq else torch.arange(5, 5 + n, dtype=torch.int32, device=dev)
        slot = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
        runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [5]) if seq else None
        x = [rnd(n, 4 * K + 2 * heads).to(BF) for _ in range(copies)]
        o32, den, gated = torch.empty(n, K, device=dev), torch.empty(n, heads, device=dev), torch.empty(n, K, dtype=BF, device=dev)

        def mine(j):
            if not seq:
                return mx.matrix_memory(g, x[j], *st[j], slot, pos, out=gated)
            mx.matrix_memory(g, x[j], *st[j], slot, pos, runs=runs, prep=prep, o=o32, den=den)
            mx.gated_group_norm(o32, x[j][:, 3 * K:], g.norm_w, gated, heads, dim, 1e-5, den=den)

        def like(j):
            mx.linear_state(light, x[j], ls[j], None, slot, pos, runs=runs, prep=prep, o=o32)
            mx.gated_group_norm(o32, x[j][:, 3 * K:], w_all, gated, 1, K, 1e-5)

        state = (n if not seq else 1) * heads * dim * dim * 8
        roof = _roof(state + n * K * 10, fp32_flops=n * heads * dim * dim * 6.0)
        out.append(_row(f"matrix memory + gated norm, {'prefill' if seq else 'decode'} {n} rows", [lambda j=j: mine(j) for j in range(copies)],
                        [lambda j=j: like(j) for j in range(copies)], roof, roof))
    return out


def _attention_rows(dev, batch: int, rows: int, heads: int = 32, kv: int = 8, dim: int = 128, window: int = 1024, keep: int = 4) -> List[dict]:
    from ..engine.kv_cache import PagedKV
    from ..models.rows import RowRuns
    from ..ops import core as ops, mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    nq, nk, ctx, taps = heads * dim, kv * dim, 2 * window, 4
    cols, out, scale = nq + 2 * nk, [], dim ** -0.5
    per = (ctx + rows) // 64 + 1
    one, freq = torch.ones(dim, device=dev), mx.rotation_freqs(1e5, dim, dev)
    kept = mx.WindowHeads(heads, kv, dim, dim, window, scale, 1e-5, 0, nq, nq, norm="head", freq=mx.rotation_freqs(1e5, dim // 2, dev), rot=dim // 2,
                          keep_first=keep, sink=rnd(heads))
    turned = mx.WindowHeads(heads, kv, dim, dim, window, scale, 1e-5, 0, nq, nq + nk, norm=None, bias=(rnd(nq), rnd(nk), rnd(nk)), freq=freq, rot=dim, softcap=20.0,
                            conv_w=rnd(taps, cols), vnorm=True, vfreq=mx.value_freqs(1e5, dim, dim, dev))
    base = mx.WindowHeads(heads, kv, dim, dim, window, scale, 1e-5, 0, nq, nq + nk)
    for name, g, w in (("attention with kept tokens and sinks", kept, one), ("attention of convolved keys and rotated values", turned, None)):
        kvs = [[PagedKV(1, 0, 0, batch * (ctx // 64 + 1) + per, batch, per, 64, False, dev, shapes=[h.kv_shape]) for _ in range(2)] for h in (g, base)]
        for c in kvs[0] + kvs[1]:
            for s in range(batch):
                assert c.reserve(s, ctx + (rows if s == 0 else 0))
            for t in (c.layers[0].k, c.layers[0].v):
                t.copy_(rnd(*t.shape))
        ring = g.new_ring(batch, dev)
        for n, seq in ((batch, False), (8, False), (rows, True)):
            pos = torch.full((n,), ctx - 1, dtype=torch.int32, device=dev) if not seq else torch.arange(ctx, ctx + n, dtype=torch.int32, device=dev)
            req = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
            x, y = rnd(n, cols).to(BF), torch.empty(n, nq, dtype=BF, device=dev)
            runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [ctx])
            scratch = (torch.empty(n * heads * 32 * 2, device=dev), torch.empty(n * heads * (32 if not seq else 1) * dim, device=dev))
            conv, turn = torch.empty(n, cols, dtype=BF, device=dev), torch.empty(n * dim, device=dev)

            def run(h, c, w, ring):
                a, L, bt = x, c.layers[0], c.block_table
                if not seq:
                    return mx.window_attn(h, a, w, w, L, bt, req, pos, y, fused=True, splits=h.splits(n, ctx, 32), scratch=scratch, ring=ring)
                if h.taps:
                    a, h = mx.short_conv(a, h.stacked_bias, h.conv_w, ring, req, pos, runs, conv), h.after_conv
                mx.qk_norm_append(h, a, w, w, L, bt, req, pos, turn if h.vfreq is not None else None)
                mx.window_prefill(h, a, L, bt, req, pos, runs, y, turn=turn)

            keys = n * window if not seq else n + window
            io = lambda h: n * (cols if h is not kept else nq + nk) * 2 + n * nq * 2 + (0 if seq or not h.taps else n * taps * cols * 4)
            fl = n * window * heads * dim * 4.0
            out.append(_row(f"{name}, {'prefill' if seq else 'decode'} {n} rows", [lambda c=c: run(g, c, w, ring) for c in kvs[0]],
                            [lambda c=c: run(base, c, one, None) for c in kvs[1]], _roof(keys * nk * 4 + io(g), fl), _roof(keys * nk * 4 + io(base), fl)))
        del kvs
        torch.cuda.empty_cache()
    pos, req = torch.arange(ctx, ctx + rows, dtype=torch.int32, device=dev), torch.zeros(rows, dtype=torch.int32, device=dev)
    runs, ring = RowRuns(i32([0, rows]), i32([0] * rows), [rows], [0], [ctx]), turned.new_ring(1, dev)
    x, y = [rnd(rows, cols).to(BF) for _ in range(6)], torch.empty(rows, cols, dtype=BF, device=dev)
    cw, cs = rnd(cols, taps).to(BF), torch.zeros(1, taps - 1, cols, device=dev)
    out.append(_row(f"convolution, prefill {rows} rows", [lambda j=j: mx.short_conv(x[j], turned.stacked_bias, turned.conv_w, ring, req, pos, runs, y) for j in range(6)],
                    [lambda j=j: ops.gdn_conv(x[j], cw, None, cs, y, None, 0, True) for j in range(6)], _roof(rows * cols * 4), _roof(rows * cols * 4)))
    return out


def _expert_rows(dev, batch: int, rows: int, width: int = 2048, experts: int = 64, identity: int = 8, top: int = 8, ff: int = 1024, shared: int = 1024) -> List[dict]:
    from ..models.row_moe import RowExperts, RowExpertsScratch, run_experts
    from ..ops import core as ops, mixers as mx
    from ..quant.formats import QuantLinear

    rnd = lambda *s: torch.randn(*s, device=dev).to(BF) * s[-1] ** -0.5
    lin = lambda t: QuantLinear("bf16", *t.shape, t)
    n_out = experts + identity
    first, up, down, sdown = rnd(n_out + shared, width), rnd(experts * ff, width), rnd(experts * width, ff), rnd(width, shared)
    mine = RowExperts(experts, top, ff, math.inf, lin(first), up, down, width, shared_col=n_out, shared_ff=shared, shared_down=lin(sdown), score="softmax",
                      correction=torch.zeros(n_out, device=dev), norm_topk=True, identity=identity, act="gelu", shared_gated=False)
    like = RowExperts(experts, top, ff, 7.0, lin(rnd(experts + 8 + 2 * shared, width)), rnd(experts * 2 * ff, width), down, width, sg_col=experts,
                      shared_col=experts + 8, shared_ff=shared, shared_limit=7.0, shared_down=lin(sdown))
    scratch = RowExpertsScratch([mine, like], max(rows, batch), BF, dev)
    x32, w = torch.randn(max(rows, batch), width, device=dev), torch.ones(width, device=dev)
    out, res = torch.empty(max(rows, batch), width, dtype=BF, device=dev), []
    for n in (8, batch, rows):
        x = [torch.randn(n, width, device=dev).to(BF) for _ in range(3)]

        def roof(b, mats):
            best = ops.gemm_tc(x[0], b.w_first, out32=torch.empty(n, b.w_first.n, device=dev))[:, :b.outputs].topk(top).indices
            pairs, active = int((best < experts).sum()), len(set(best[best < experts].tolist()))
            bytes_ = active * mats * ff * width * 2 + b.w_first.nbytes + sdown.numel() * 2 + n * width * 2 + pairs * (width * 4 + ff * 2 * mats) + n * (shared * 6 + width * 14)
            return _roof(bytes_, (pairs * mats * ff + n * (b.w_first.n + shared)) * 2.0 * width)

        run = lambda blk, j, **kw: mx.stream_norm(x32[:n], width, 1e-5, out[:n], run_experts(blk, scratch, x[j]), **kw)
        res.append(_row(f"expert block + norms, {n} rows", [lambda j=j: run(mine, j, post=("parts", w), pre=("parts", w), parts=4) for j in range(3)],
                        [lambda j=j: run(like, j, post=("layer", w), pre=("layer", w)) for j in range(3)], roof(mine, 2), roof(like, 3)))
    return res


def _row_operators(dev, rows: int, width: int = 4096) -> List[dict]:
    from ..ops import mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    x, d, e = ([rnd(rows, width) for _ in range(4)] for _ in range(3))
    xn = torch.empty(rows, width, dtype=BF, device=dev)
    w, b = rnd(width), rnd(width)
    like = [lambda j=j: mx.stream_norm(x[j], width, 1e-5, xn, d[j], ("layer", w), ("layer", w)) for j in range(4)]
    parts = dict(post=("parts", w), pre=("parts", w), parts=4)
    out = [_row("norm, residual, norm over parts", [lambda j=j: mx.stream_norm(x[j], width, 1e-5, xn, d[j], **parts) for j in range(4)], like,
                _roof(rows * width * 14), _roof(rows * width * 14)),
           _row("two norms, mean, norm, residual, norm", [lambda j=j: mx.stream_norm(x[j], width, 1e-5, xn, mx.PairDelta(d[j], w, e[j], w, 0.5, b), **parts) for j in range(4)],
                like, _roof(rows * width * 18), _roof(rows * width * 14))]
    ff = 3 * width
    up, gu, act = [rnd(rows, ff).to(BF) for _ in range(4)], [rnd(rows, 2 * ff).to(BF) for _ in range(3)], torch.empty(rows, ff, dtype=BF, device=dev)
    glu = [lambda j=j: mx.clamped_glu(gu[j], act, 7.0) for j in range(3)]
    for name, kind in (("square of relu", "relu2"), ("erf gelu", "gelu")):
        out.append(_row(name, [lambda j=j: mx.act_rows(up[j], act, kind) for j in range(4)], glu, _roof(rows * ff * 4), _roof(rows * ff * 6)))
    return out


def kernels(dev, batch: int = 64, rows: int = 2048) -> List[dict]:
    return _memory_rows(dev, batch, rows) + _attention_rows(dev, batch, rows) + _expert_rows(dev, batch, rows) + _row_operators(dev, rows)


def _runners(width: int, layers: int, dev, slots: int, max_seq: int):
    """(name, runner, weight bytes) of the models at equal width and depth, one after the other."""
    from ..models import potivik as pv, sitirax as sx
    from ..models.tefudra import DenseSpec, ExpertsSpec, MatrixSpec, ParallelSpec, TefudraConfig, TefudraModel, TefudraRunner, WindowSpec

    h, vocab, rows = width // 128, 32768, 2048
    kv, scale = max(h // 4, 1), 128 ** -0.5
    mixers = (WindowSpec(h, kv, 128, 128, scale, 1024, 1e5, 64, 4),
              ParallelSpec(WindowSpec(h, kv, 128, 128, scale, 1024, 1e5, 128, softcap=20.0, taps=4), MatrixSpec(h // 2, 128, 128, 15.0)))
    for name, ff in (("tefudra, dense", DenseSpec(4 * width)), ("tefudra, experts", ExpertsSpec(64, 8, 8, width // 2, width // 2))):
        m = TefudraModel.random_init(TefudraConfig.cycle(layers, width, vocab, mixers, (ff,)), dev, std=0.02)
        yield name, TefudraRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
        del m
        torch.cuda.empty_cache()
    win, decay = sx.WindowSpec(h, kv, 128, 128, scale, 1024), tuple(1 - 2.0 ** -(1 + 10 * i / max(h // 2 - 1, 1)) for i in range(h // 2))
    both = sx.ParallelSpec(win, sx.LightningSpec(h // 2, 128, 128, decay), 0.7, 0.7)
    m = sx.SitiraxModel.random_init(sx.SitiraxConfig.uniform(layers, width, vocab, both, both, 8 * width // 3 // 8 * 8), dev, std=0.02)
    yield "window beside lightning attention, dense", sx.SitiraxRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
    del m
    torch.cuda.empty_cache()
    c = pv.PotivikConfig.uniform(layers, width, vocab, pv.LatentSpec(h, 128, 64, 128, 512, 192 ** -0.5, 1024, 1e4, 64), pv.StateSpaceSpec(width // 32, 1, 64, 128, 4, 8),
                                 pv.ExpertsSpec(64, 8, pv.FeedForward(width // 2, 7.0), pv.FeedForward(width // 2, 7.0)), pv.FeedForward(width // 2, 7.0), 256)
    c.plan = [type(L)(L.mixer, c.plan[1].mlp) for L in c.plan]
    m = pv.PotivikModel.random_init(c, dev, std=0.02)
    yield "latent + state space, experts", pv.PotivikRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
    del m
    torch.cuda.empty_cache()


def models(width: int, dev, steps: int, warmup: int, layers: int = 8) -> List[dict]:
    res, gen, vocab = [], torch.Generator().manual_seed(0), 32768
    for name, r, wbytes in _runners(width, layers, dev, 64, 4608):
        row = {"model": name, "width": width, "layers": layers, "weight_gb": round(wbytes / 1e9, 3)}
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
        res = {"family": "tefudra", "dtype": "bf16", "data": "synthetic", "peaks": peaks(), "kernels": kernels(dev)}
        ops.check_status()
        for row in res["kernels"]:
            print("# " + json.dumps(row), flush=True)
        res["models"] = [row for w in args.sizes.split(",") if w for row in models(int(w), dev, max(args.steps, 1), max(args.warmup, 3))]
    ops.check_status()
    print(json.dumps(res))
    return 0
