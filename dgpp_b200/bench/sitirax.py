"""Sitirax at the sizes of a real model's layers, beside the closest families at equal size (random weights, one GPU).

    python bench.py --family sitirax [--sizes 2048,4096] [--steps K] [--warmup W]

Kernels: every state, attention and row operator of the family, decode (64 requests) and prefill (2048 tokens of one
request), next to the like operator of the family closest to it: the per-channel-decay delta rule of `models/glm_flash.py`
(convolution + recurrence + gated norm), the gated delta rule of `models/gdn.py` for lightning attention, the sliding-window
attention of `models/mimo.py` (FP8 cache there, bf16 here).  Inputs rotate over more than the 126 MB L2.  `roofline_ms` is the
larger of algorithmic bytes / measured copy bandwidth and FLOPs / measured bf16 throughput (fp32 work on the CUDA cores: FLOPs
/ 2 x 128 x SMs x clock); `frac` = roofline_ms / measured.

Models: 8 layers of width W, parallel and delta layers in turn, against the sliding-window family and the delta-rule family
with dense feed-forward blocks of the same width and depth: decode tokens/s at 1, 8 and 64 requests and prefill tokens/s of
one 4096-token prompt (2048-token passes).  A decode step includes the runner's host work and the read-back of its tokens.
"""
from __future__ import annotations

import json
from typing import List

import torch

from .configs import _time_decode, _time_prefill
from .micro import graph_time, peaks

BF = torch.bfloat16
FP32_FLOPS = 2 * 128 * 148 * 1.85e9            # CUDA-core multiply-adds at the clock the GPU holds under such loads


def _roof(bytes_: float, tc_flops: float = 0.0, fp32_flops: float = 0.0) -> float:
    p = peaks()
    return 1e3 * max(bytes_ / (p["hbm_gbs"] * 1e9), tc_flops / (p["tflops"] * 1e12), fp32_flops / FP32_FLOPS)


def _row(name: str, fns: List, like: List, roof: float, like_roof: float, reps: int = 10) -> dict:
    ms, ref = graph_time(fns, reps), graph_time(like, reps)
    return {"kernel": name, "ms": round(ms, 4), "roofline_ms": round(roof, 4), "frac": round(roof / ms, 3),
            "like_ms": round(ref, 4), "like_roofline_ms": round(like_roof, 4), "like_frac": round(like_roof / ref, 3)}


def kernels(dev, heads: int = 32, kv: int = 8, dim: int = 128, window: int = 1024, batch: int = 64, rows: int = 2048) -> List[dict]:
    from ..engine.kv_cache import PagedKV
    from ..models.rows import RowRuns
    from ..ops import core as ops, mixers as mx, reference as ref

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    out = []
    hk, taps, ctx, copies = heads // 2, 4, 2 * window, 3
    # ---- the two state layers
    C, K = 2 * hk * dim + heads * dim, heads * dim
    delta = mx.StateHeads(heads, hk, dim, dim, 0, C, 1e-5, rnd(taps, C), rnd(heads) - 2, rnd(K) - 2, norm_w=rnd(dim))
    light = mx.StateHeads(heads, heads, dim, dim, 0, eps=1e-5, decay=torch.rand(heads, device=dev))
    st = [delta.new_state(batch, dev) for _ in range(copies)]
    A_log, dt, w_conv, nw = rnd(heads), rnd(K), rnd(C, taps).to(BF), rnd(dim).to(BF)
    like_conv = [torch.zeros(batch, taps - 1, C, device=dev) for _ in range(copies)]
    sbytes = batch * heads * dim * dim * 8

    def gate_rows(n):
        return rnd(n, C + 2 * K + heads).to(BF)

    def kda(x, state, conv, o, g, n, seq, slots):
        y = ops.gdn_conv(x[:, :C], w_conv, None, conv, o["conv"][:n], None if seq else slots, 0, seq)
        nq = hk * dim
        ops.kda_recurrent(y[:, :nq], y[:, nq:2 * nq], y[:, 2 * nq:], x[:, C:C + K], x[:, C + 2 * K:], A_log, dt, -5.0, state, o["o"][:n],
                          hk, heads, dim, dim, row_slot=None if seq else slots, slot=0, sequential=seq, prep=o["prep"])
        ops.gated_rmsnorm(o["o"][:n], x[:, C + K:C + 2 * K], nw, g[:n], heads, dim)

    def gdn(x, state, o, n, seq, slots):
        ab = x[:, :2 * heads]
        ops.gdn_recurrent(x[:, :K], x[:, K:2 * K], x[:, 2 * K:3 * K], ab[:, :heads], ab[:, heads:], A_log, A_log, state, o["o"][:n], heads,
                          heads, dim, dim, None if seq else slots, 0, seq)

    big = max(rows, batch)
    buf = {"conv": torch.empty(big, C, dtype=BF, device=dev), "o": torch.empty(big, K, dtype=BF, device=dev),
           "prep": torch.empty(max(delta.prep_floats(big, 1), light.prep_floats(big, 1)), device=dev)}
    o32, gated = torch.empty(big, K, device=dev), torch.empty(big, K, dtype=BF, device=dev)
    for n, seq in ((batch, False), (rows, True)):
        pos = torch.full((n,), 5, dtype=torch.int32, device=dev) if not seq else torch.arange(5, 5 + n, dtype=torch.int32, device=dev)
        slot = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
        runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [5]) if seq else None
        x = [gate_rows(n) for _ in range(copies)]
        xd = [rnd(n, (C + heads + 7) // 8 * 8).to(BF) for _ in range(copies)]
        xl = [rnd(n, 4 * K).to(BF) for _ in range(copies)]
        low = [rnd(n, 2 * K) for _ in range(copies)]

        def d_step(j):
            if not seq:
                return mx.linear_state(delta, xd[j], *st[j], slot, pos, low=low[j], out=gated[:n])
            mx.linear_state(delta, xd[j], *st[j], slot, pos, low=low[j], runs=runs, prep=buf["prep"], o=o32[:n])
            mx.gated_group_norm(o32[:n], low[j][:, K:], delta.norm_w, gated[:n], heads, dim, 1e-5)

        def l_step(j):
            mx.linear_state(light, xl[j], st[j][0], None, slot, pos, runs=runs, prep=buf["prep"], o=o32[:n])

        ops_tok = heads * dim * dim * 2.0 * 4                       # decay, two read-outs, one write per state element
        io = n * (C * 2 + K * 8 + K * 2)
        state_io = sbytes if not seq else heads * dim * dim * 8
        roof = _roof(state_io + io, fp32_flops=n * ops_tok)
        kind = "prefill" if seq else "decode"
        out.append(_row(f"channel delta {kind}", [lambda j=j: d_step(j) for j in range(copies)],
                        [lambda j=j: kda(x[j], st[j][0], like_conv[j], buf, gated, n, seq, slot) for j in range(copies)],
                        roof, _roof(state_io + n * (C + 2 * K) * 2 + n * K * 2, fp32_flops=n * ops_tok)))
        roof = _roof(state_io + n * K * (6 + 4), fp32_flops=n * ops_tok * 0.75)
        out.append(_row(f"lightning {kind}", [lambda j=j: l_step(j) for j in range(copies)],
                        [lambda j=j: gdn(xl[j], st[j][0], buf, n, seq, slot) for j in range(copies)], roof,
                        _roof(state_io + n * K * 8, fp32_flops=n * ops_tok)))
    del st, like_conv
    # ---- window attention
    page, per = 64, (ctx + rows) // 64 + 1
    mine = [PagedKV(1, kv, dim, batch * (ctx // page + 1) + per, batch, per, page, False, dev) for _ in range(2)]
    like = [PagedKV(1, kv, dim, batch * (ctx // page + 1) + per, batch, per, page, True, dev) for _ in range(2)]
    for c in mine + like:
        for s in range(batch):
            assert c.reserve(s, ctx + (rows if s == 0 else 0))
        for L in c.layers:
            for t in (L.k, L.v):
                t.copy_(torch.randint(0, 96, t.shape, device=dev) if t.dtype == torch.uint8 else rnd(*t.shape))
    g = mx.WindowHeads(heads, kv, dim, dim, window, dim ** -0.5, 1e-5, 0, heads * dim, (heads + kv) * dim)
    cols = (heads + 2 * kv) * dim
    wq = torch.ones(dim, device=dev)
    inv, _ = ref.rope_inv_freq(dim, 1e4, dev)
    for n, seq in ((batch, False), (rows, True)):
        pos = torch.full((n,), ctx - 1, dtype=torch.int32, device=dev) if not seq else torch.arange(ctx, ctx + n, dtype=torch.int32, device=dev)
        req = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
        x, y = rnd(n, cols).to(BF), torch.empty(n, heads * dim, dtype=BF, device=dev)
        runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [ctx])
        scratch = (torch.empty(n * heads * 2 * 2, device=dev), torch.empty(n * heads * 2 * dim, device=dev))

        def w_step(c):
            a = (g, x, wq, wq, c.layers[0], c.block_table, req, pos)
            if not seq:
                return mx.window_attn(*a, y, fused=True)
            mx.qk_norm_append(*a)
            mx.window_prefill(g, x, c.layers[0], c.block_table, req, pos, runs, y)

        def s_step(c):
            ops.rope_kv_write(x, pos, req, c.block_table, inv, c.layers[0], heads, kv, dim)
            ops.attn_decode(x, x.stride(0), c.layers[0], c.block_table, req, pos, heads, kv, dim, dim ** -0.5, out=y, window=window)

        keys = n * window * kv * dim * 2 if not seq else (n + window) * kv * dim * 2
        io, fl = n * (cols + heads * dim) * 2, n * window * heads * dim * 4.0
        out.append(_row(f"window attention {'prefill' if seq else 'decode'}", [lambda c=c: w_step(c) for c in mine],
                        [lambda c=c: s_step(c) for c in like], _roof(2 * keys + io, fl), _roof(keys + io, fl)))
    del mine, like
    # ---- row operators
    W, ff = heads * dim, 3 * heads * dim
    x32 = [rnd(rows, W) for _ in range(4)]
    d32, d16, xn = [rnd(rows, W) for _ in range(4)], [rnd(rows, W).to(BF) for _ in range(4)], torch.empty(rows, W, dtype=BF, device=dev)
    x16, w32, w16 = [rnd(rows, W).to(BF) for _ in range(4)], rnd(W), rnd(W).to(BF)
    out.append(_row("residual + norm", [lambda j=j: mx.resid_norm(x32[j], w32, W, 1e-5, xn, d32[j]) for j in range(4)],
                    [lambda j=j: ops.rmsnorm(x16[j], w16, 1e-5, delta=d16[j], out=xn) for j in range(4)],
                    _roof(rows * W * 14), _roof(rows * W * 8)))
    gu, act = [rnd(rows, 2 * ff).to(BF) for _ in range(3)], torch.empty(rows, ff, dtype=BF, device=dev)
    out.append(_row("gated activation", [lambda j=j: mx.geglu(gu[j], act) for j in range(3)],
                    [lambda j=j: ops.swiglu(gu[j], out=act) for j in range(3)], _roof(rows * ff * 6), _roof(rows * ff * 6)))
    return out


def _runners(width: int, layers: int, dev, slots: int, max_seq: int):
    """(name, runner, weight bytes) of the three models at equal width and depth, one after the other."""
    from ..models.glm_flash import GlmFlashConfig, GlmFlashModel, GlmFlashRunner
    from ..models.mimo import MimoConfig, MimoModel, MimoRunner
    from ..models.sitirax import DeltaSpec, LightningSpec, ParallelSpec, SitiraxConfig, SitiraxModel, SitiraxRunner, WindowSpec

    h, ff, vocab, rows = width // 128, 3 * width, 32768, 2048
    decay = tuple(1 - 2.0 ** -(1 + 10 * i / max(h // 2 - 1, 1)) for i in range(h // 2))
    c = SitiraxConfig.uniform(layers, width, vocab, ParallelSpec(WindowSpec(h, h // 4, 128, 128, 128 ** -0.5, 1024),
                                                                LightningSpec(h // 2, 128, 128, decay), 0.7, 0.7),
                              DeltaSpec(h, h // 2, 128, 128, 4), ff)
    m = SitiraxModel.random_init(c, dev, std=0.02)
    yield "sitirax", SitiraxRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
    m = MimoModel.random_init(MimoConfig(layers=layers, hidden=width, q_heads=h, swa_kv_heads=h // 4, kv_heads=h // 4, rotary_dim=128,
                                         window=1024, swa_layers=[True] * layers, ffn=ff, dense_layers=layers, draft=False, vocab=vocab),
                              dev, std=0.02)
    yield "sliding-window", MimoRunner(m, rows, slots, max_seq, dev), sum(w.nbytes for L in m.layers for w in (L.qkv, L.o, L.gate_up, L.down)) + m.head.nbytes
    m = GlmFlashModel.random_init(GlmFlashConfig(layers=layers, hidden=width, vocab=vocab, mla_every=layers + 1, streams=2, k_heads=h // 2,
                                                 v_heads=h, ffn=ff, dense_layers=layers), dev, std=0.02)
    yield "delta-rule", GlmFlashRunner(m, rows, slots, max_seq, dev), sum(w.nbytes for L in m.layers for w in (L.kda.in_proj, L.kda.out_proj, L.gate_up, L.down)) + m.head.nbytes


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
        res.append(row)
        del r
        torch.cuda.empty_cache()
    return res


def run(args) -> int:
    from ..ops import core as ops

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    with torch.no_grad():
        res = {"family": "sitirax", "dtype": "bf16", "data": "synthetic", "peaks": peaks(), "kernels": kernels(dev)}
        ops.check_status()
        res["models"] = [row for w in args.sizes.split(",") if w for row in models(int(w), dev, max(args.steps, 1), max(args.warmup, 3))]
    ops.check_status()
    for row in res["kernels"] + res["models"]:
        print("# " + json.dumps(row))
    print(json.dumps(res))
    return 0
