"""Potivik at the sizes of a real model's layers, beside the closest families at equal size (random weights, one GPU).

    python bench.py --family potivik [--sizes 2048,4096] [--steps K] [--warmup W]

Kernels: every state, attention, expert and row operator of the family, decode (64 requests, experts also 8) and prefill (2048
tokens of one request), next to the like operator of the family closest to it: the gated delta rule of `models/gdn.py` (convolution +
recurrence + gated norm) for the state-space recurrence, the absorbed latent attention of `models/mla.py` (full context there, a
window here, equal keys at decode), the NVFP4 expert block of `models/moe.py` for the bf16 one, `rmsnorm` / `swiglu`.  Inputs rotate
over more than the 126 MB L2.  `roofline_ms` is the larger of algorithmic bytes / measured copy bandwidth and FLOPs / measured bf16
throughput (fp32 work on the CUDA cores: FLOPs / 2 x 128 x SMs x clock); `frac` = roofline_ms / measured.

Models: 8 layers of width W, latent and state layers in turn, against the family with delta-rule and latent layers in turn, with dense
feed-forward blocks and with experts (bf16 here, NVFP4 there): decode tokens/s at 1, 8 and 64 requests and prefill tokens/s of one
4096-token prompt (2048-token passes).  A decode step includes the runner's host work and the read-back of its tokens.
"""
from __future__ import annotations

import json
from typing import List

import torch

from .configs import _time_decode, _time_prefill
from .micro import peaks
from .sitirax import _roof, _row

BF = torch.bfloat16


def _state_rows(dev, batch: int, rows: int, heads: int = 64, vdim: int = 64, state: int = 128, copies: int = 3) -> List[dict]:
    from ..models.rows import RowRuns
    from ..ops import core as ops, mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    out, inner, taps = [], heads * vdim, 4
    C = 2 * state + inner
    s = mx.StateHeads(heads, 1, state, vdim, 0, C, 1e-5, rnd(taps, C), rnd(heads), rnd(heads) - 3, conv_b=rnd(C), skip=rnd(heads))
    st = [s.new_state(batch, dev) for _ in range(copies)]
    gh, gd = heads * vdim // 128, 128                       # the delta rule at the same state size: heads of 128 x 128
    gc = 3 * gh * gd
    g_state, g_conv = [torch.zeros(batch, gh, gd, gd, device=dev) for _ in range(copies)], [torch.zeros(batch, taps - 1, gc, device=dev) for _ in range(copies)]
    A, dtb, cw, nw, pw = rnd(gh), rnd(gh), rnd(gc, taps).to(BF), rnd(gd).to(BF), rnd(inner)
    for n, seq in ((batch, False), (rows, True)):
        pos = torch.full((n,), 5, dtype=torch.int32, device=dev) if not seq else torch.arange(5, 5 + n, dtype=torch.int32, device=dev)
        slot = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
        runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [5]) if seq else None
        x = [rnd(n, C + heads + inner).to(BF) for _ in range(copies)]
        y = [rnd(n, gc + gh * gd + 2 * gh).to(BF) for _ in range(copies)]
        o, mixed = torch.empty(n, inner, device=dev), torch.empty(n, inner, dtype=BF, device=dev)
        co, go = torch.empty(n, gc, dtype=BF, device=dev), torch.empty(n, gh * gd, dtype=BF, device=dev)
        prep = torch.empty(max(s.prep_floats(n, 1), n * (2 * gh * gd + 2 * gh)), device=dev)

        def step(j):
            mx.linear_state(s, x[j], *st[j], slot, pos, runs=runs, prep=prep, o=o)

        def whole(j):
            step(j)
            mx.gated_part_norm(o, x[j][:, C + heads:], pw, mixed, 8, 1e-5)

        def gdn(j):
            c = ops.gdn_conv(y[j][:, :gc], cw, None, g_conv[j], co, None if seq else slot, 0, seq)
            k = gh * gd
            ab = y[j][:, gc + k:]
            ops.gdn_recurrent(c[:, :k], c[:, k:2 * k], c[:, 2 * k:], ab[:, :gh], ab[:, gh:], A, dtb, g_state[j], go, gh, gh, gd, gd, None if seq else slot, 0,
                              seq, prep=prep)
            ops.gated_rmsnorm(go, y[j][:, gc:gc + k], nw, mixed, gh, gd)

        kind = "prefill" if seq else "decode"
        sio = (n if not seq else 1) * heads * state * vdim * 8
        roof = _roof(sio + n * (C + heads) * 2 + n * inner * 4 + n * inner * 4, fp32_flops=n * heads * state * vdim * 5.0)
        like = _roof(sio + n * (gc + gh * gd) * 2 + n * gh * gd * 2, fp32_flops=n * gh * gd * gd * 8.0)
        out.append(_row(f"state space + gated norm, {kind}", [lambda j=j: whole(j) for j in range(copies)], [lambda j=j: gdn(j) for j in range(copies)], roof, like))
    return out


def _latent_rows(dev, batch: int, rows: int, heads: int = 32, dim: int = 128, rot: int = 64, vdim: int = 128, rank: int = 512,
                 window: int = 1024) -> List[dict]:
    from ..engine.kv_cache import PagedKV
    from ..models.potivik import LatentSpec, PotivikConfig, PotivikModel, PotivikRunner, StateSpaceSpec, FeedForward
    from ..models.rows import RowRuns
    from ..ops import core as ops, mixers as mx, reference as ref

    rnd = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    c = PotivikConfig.uniform(1, 1024, 64, LatentSpec(heads, dim, rot, vdim, rank, (dim + rot) ** -0.5, window, 1e4, rot), StateSpaceSpec(1, 1, 8, 8, 1, 1), None,
                              FeedForward(8, 1.0), 8)
    copies = 2
    runners = [PotivikRunner(PotivikModel.random_init(c, dev, seed=i), rows, batch, window + rows, dev, batch * (window + 64) + rows + window) for i in range(copies)]
    out, D = [], rank + rot
    like_kv = [PagedKV(1, 1, D, batch * (window // 64) + rows // 64 + 64, batch, (window + rows) // 64 + 1, 64, False, dev) for _ in range(copies)]
    for kv in [r.kv for r in runners] + like_kv:
        for s in range(batch):
            assert kv.reserve(s, window + (rows if s == 0 else 0))
        for L in kv.layers:
            L.k.copy_(rnd(*L.k.shape))
    w_uk, w_uv = rnd(heads, dim, rank).to(BF) * rank ** -0.5, rnd(heads, vdim, rank).to(BF) * rank ** -0.5
    inv, _ = ref.rope_inv_freq(rot, 1e4, dev)
    nw = rnd(rank).to(BF)
    g = runners[0].m.layers[0].latent
    cols = runners[0].m.layers[0].w_in.n
    for n, seq in ((batch, False), (rows, True)):
        pos = torch.full((n,), window - 1, dtype=torch.int32, device=dev) if not seq else torch.arange(window, window + n, dtype=torch.int32, device=dev)
        req = torch.arange(n, dtype=torch.int32, device=dev) if not seq else torch.zeros(n, dtype=torch.int32, device=dev)
        x = [rnd(n, cols).to(BF) for _ in range(copies)]
        mixed = torch.empty(n, heads * vdim, dtype=BF, device=dev)
        q, kvp = [rnd(n, heads, dim + rot).to(BF) for _ in range(copies)], [rnd(n, D).to(BF) for _ in range(copies)]
        qa, lat = torch.empty(n, heads, D, dtype=BF, device=dev), rnd(n, heads, rank).to(BF)
        runs = RowRuns(i32([0, n]), i32([0] * n), [n], [0], [window]) if seq else None
        plan = runners[0]._plan_runs(runs) if seq else None

        def whole(j):
            r = runners[j]
            r._latent(0, r.m.layers[0], x[j], mixed, pos, req, runs, plan)

        def prep(j):
            r = runners[j]
            mx.latent_absorb(r.m.layers[0].latent, x[j], pos, req, r.kv.block_table, r.kv.layers[0].k, 64, r.q_abs, n, None, True)

        def attn(j):
            r = runners[j]
            splits = mx.latent_splits(n, heads, window, r.max_splits)
            mx.latent_attn(r.m.layers[0].latent, r.q_abs, r.kv.layers[0].k, r.kv.block_table, req, pos, 64, r.lat, n, None, splits, r.scratch)

        def ups(j):
            r = runners[j]
            mx.latent_up(r.m.layers[0].latent, r.lat, x[j], mixed, n)

        def l_prep(j):
            ops.mla_kv_prep(kvp[j], nw, 1e-5, inv, pos, req, like_kv[j].block_table, like_kv[j].layers[0].k.view(-1, 64, D), rank, rot)
            ops.mla_q_absorb(q[j], w_uk, inv, pos, rank, rot, out=qa)

        def l_attn(j):
            splits = max(1, -(-148 // (n * -(-heads // 32))))
            ops.mla_decode(qa, like_kv[j].layers[0].k.view(-1, 64, D), like_kv[j].block_table, req, pos, (dim + rot) ** -0.5, rank, rot, splits=splits, out=lat)

        def l_ups(j):
            ops.mla_v_up(lat, w_uv, out=mixed)

        def l_whole(j):
            l_prep(j)
            l_attn(j)
            l_ups(j)

        r2 = range(copies)
        each = lambda f: [lambda j=j: f(j) for j in r2]
        wb, absorb = heads * rank * dim * 2, n * heads * rank * 2.0
        if not seq:
            keys, io = n * window * D * 2, n * heads * (D + rank)
            roofs = [(f"latent: queries absorbed, keys appended, {n} rows", prep, l_prep, _roof(wb + n * (cols * 2 + D * 2 + heads * D * 4), absorb * dim),
                      _roof(wb + n * (heads * (dim + rot) * 2 + D * 4 + heads * D * 2), absorb * dim)),
                     (f"latent attention decode, {n} rows", attn, l_attn, _roof(keys + io * 4, n * heads * window * (D + rank) * 2.0),
                      _roof(keys + io * 2, n * heads * window * (D + rank) * 2.0)),
                     (f"latent: values up, {n} rows", ups, l_ups, _roof(wb + n * heads * (rank * 4 + vdim * 2), absorb * vdim), _roof(wb + n * heads * (rank + vdim) * 2, absorb * vdim))]
            out += [_row(name, each(a), each(b), ra, rb) for name, a, b, ra, rb in roofs]
            full = sum(r[3] for r in roofs), sum(r[4] for r in roofs)
            out.append(_row("latent layer between its projections, decode", each(whole), each(l_whole), *full))
        else:
            keys = (n + window) * D * 2
            fl = (n + window) * rank * heads * (dim + vdim) * 2.0 + n * heads * window * (dim + rot + vdim) * 2.0
            lfl = n * heads * (rank * (dim + vdim) * 2.0 + (window + n / 2) * (D + rank) * 2.0)
            out.append(_row("latent layer between its projections, prefill", each(whole), each(l_whole),
                            _roof(2 * wb + keys + n * (cols + heads * vdim) * 2, fl), _roof(2 * wb + keys + n * heads * (dim + rot + vdim) * 2, lfl), reps=5))
    return out


def _expert_rows(dev, batch: int, rows: int, width: int = 2048, experts: int = 64, top: int = 8, ff: int = 1024) -> List[dict]:
    from ..models.moe import MoEBlock, MoEConfig, MoEWeights
    from ..models.row_moe import RowExperts, RowExpertsScratch, run_experts
    from ..ops import core as ops, mixers as mx
    from ..quant.formats import QuantLinear

    rnd = lambda *s: torch.randn(*s, device=dev).to(BF) * s[-1] ** -0.5
    lin = lambda n, k: QuantLinear("bf16", n, k, rnd(n, k))
    block = RowExperts(experts, top, ff, 7.0, lin(experts + 8 + 2 * ff, width), rnd(experts * 2 * ff, width), rnd(experts * width, ff), width, experts, experts + 8, ff, 7.0,
                       lin(width, ff))
    scratch = RowExpertsScratch([block], max(rows, batch), BF, dev)
    like_w = MoEWeights.random_init(MoEConfig(width, experts, top, ff, ff, norm_topk_prob=False, swiglu_limit=7.0, swiglu_alpha=1.702), dev)
    res = []
    x32, out, w = torch.randn(max(rows, batch), width, device=dev), torch.empty(max(rows, batch), width, dtype=BF, device=dev), torch.ones(width, device=dev)
    for n in (8, batch, rows):
        x = [torch.randn(n, width, device=dev).to(BF) for _ in range(3)]
        pairs, active = n * top, min(experts, n * top)
        b = MoEBlock(like_w, n if n <= 64 else 64, dev)
        wbytes = (active + 1) * 3 * ff * width
        io = n * width * 2 + pairs * (width * 4 + ff * 6)
        fl = (pairs + n) * 3.0 * ff * width * 2
        mine = lambda j: mx.stream_norm(x32[:n], width, 1e-5, out[:n], run_experts(block, scratch, x[j]), ("layer", w), (None, None))

        def like(j):
            y = b.forward(x[j], out[:n]) if n <= 64 else b.forward_gathered(x[j])
            ops.rmsnorm(x[j], w.to(BF), 1e-5, delta=y, out=out[:n])

        res.append(_row(f"expert block + norm, {n} rows", [lambda j=j: mine(j) for j in range(3)], [lambda j=j: like(j) for j in range(3)],
                        _roof(wbytes * 2 + io, fl), _roof(wbytes * 9 / 16 + io, fl)))
    return res


def _row_operators(dev, rows: int, width: int = 4096) -> List[dict]:
    from ..ops import core as ops, mixers as mx

    rnd = lambda *s: torch.randn(*s, device=dev)
    x, d, xn = [rnd(rows, width) for _ in range(4)], [rnd(rows, width) for _ in range(4)], torch.empty(rows, width, dtype=BF, device=dev)
    x16, d16, w, w16 = [rnd(rows, width).to(BF) for _ in range(4)], [rnd(rows, width).to(BF) for _ in range(4)], rnd(width), rnd(width).to(BF)
    out = [_row("norm, residual, norm", [lambda j=j: mx.stream_norm(x[j], width, 1e-5, xn, d[j], ("layer", w), ("layer", w)) for j in range(4)],
                [lambda j=j: ops.rmsnorm(x16[j], w16, 1e-5, delta=d16[j], out=xn) for j in range(4)], _roof(rows * width * 14), _roof(rows * width * 8))]
    ff = 3 * width
    gu, act = [rnd(rows, 2 * ff).to(BF) for _ in range(3)], torch.empty(rows, ff, dtype=BF, device=dev)
    out.append(_row("clamped activation", [lambda j=j: mx.clamped_glu(gu[j], act, 7.0) for j in range(3)],
                    [lambda j=j: ops.swiglu(gu[j], out=act, limit=7.0, alpha=1.702) for j in range(3)], _roof(rows * ff * 6), _roof(rows * ff * 6)))
    return out


def kernels(dev, batch: int = 64, rows: int = 2048) -> List[dict]:
    return _state_rows(dev, batch, rows) + _latent_rows(dev, batch, rows) + _expert_rows(dev, batch, rows) + _row_operators(dev, rows)


def _runners(width: int, layers: int, dev, slots: int, max_seq: int):
    """(name, runner, weight bytes) of the models at equal width and depth, one after the other."""
    from ..models.glm_flash import GlmFlashConfig, GlmFlashModel, GlmFlashRunner
    from ..models.moe import MoEConfig
    from ..models.potivik import ExpertsSpec, FeedForward, LatentSpec, PotivikConfig, PotivikModel, PotivikRunner, StateSpaceSpec

    h, ff, vocab, rows = width // 128, 3 * width, 32768, 2048
    latent = LatentSpec(h, 128, 64, 128, 512, 192 ** -0.5, 1024, 1e4, 64)
    state = StateSpaceSpec(width // 32, 1, 64, 128, 4, 8)
    for kind in ("dense", "experts"):
        moe = ExpertsSpec(64, 8, FeedForward(width // 2, 7.0), FeedForward(width // 2, 7.0)) if kind == "experts" else None
        m = PotivikModel.random_init(PotivikConfig.uniform(layers, width, vocab, latent, state, moe, FeedForward(ff, 7.0), 256), dev, std=0.02)
        yield f"potivik, {kind}", PotivikRunner(m, rows, slots, max_seq, dev), m.weight_bytes()
        del m
        torch.cuda.empty_cache()
        c = GlmFlashConfig(layers=layers, hidden=width, vocab=vocab, mla_every=2, streams=2, k_heads=h, v_heads=h, heads=h, q_lora=width, kv_lora=512, nope=128,
                           rope=64, v_dim=128, ffn=ff, dense_layers=layers if moe is None else 1,
                           moe=None if moe is None else MoEConfig(width, 64, 8, width // 2, width // 2, swiglu_limit=7.0, swiglu_alpha=1.702))
        m = GlmFlashModel.random_init(c, dev, std=0.02)
        yield f"delta-rule + latent, {kind}", GlmFlashRunner(m, rows, slots, max_seq, dev), 0
        del m
        torch.cuda.empty_cache()


def models(width: int, dev, steps: int, warmup: int, layers: int = 8) -> List[dict]:
    res, gen, vocab = [], torch.Generator().manual_seed(0), 32768
    for name, r, wbytes in _runners(width, layers, dev, 64, 4608):
        row = {"model": name, "width": width, "layers": layers}
        if wbytes:
            row["weight_gb"] = round(wbytes / 1e9, 3)
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
        res = {"family": "potivik", "dtype": "bf16", "data": "synthetic", "peaks": peaks(), "kernels": kernels(dev)}
        ops.check_status()
        for row in res["kernels"]:
            print("# " + json.dumps(row), flush=True)
        res["models"] = [row for w in args.sizes.split(",") if w for row in models(int(w), dev, max(args.steps, 1), max(args.warmup, 3))]
    ops.check_status()
    for row in res["models"]:
        print("# " + json.dumps(row))
    print(json.dumps(res))
    return 0
