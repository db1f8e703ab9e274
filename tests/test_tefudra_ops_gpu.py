"""The operators behind the Tefudra family on the GPU, each against its plain restatement, in bf16 and in true fp32."""
import math

import pytest
import torch
import torch.nn.functional as F

import tefudra_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def dev():
    if not torch.cuda.is_available():
        pytest.skip("needs a GPU")
    return torch.device("cuda:0")


def _close(got, want, dtype, fine=3e-5, coarse=2e-2):
    want = want.double().cpu()
    err = (got.double().cpu() - want).abs().max().item()
    assert err <= (fine if dtype == torch.float32 else coarse) * (want.abs().max().item() + 1e-6), err


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _runs(dev, lens, slots, pos0):
    from dgpp_b200.models.rows import RowRuns

    start = [0]
    for n in lens:
        start.append(start[-1] + n)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    run0 = [s for s, n in zip(start, lens) for _ in range(n)]
    rows = i32([s for s, n in zip(slots, lens) for _ in range(n)]), i32([p + k for p, n in zip(pos0, lens) for k in range(n)])
    return RowRuns(i32(start), i32(run0), list(lens), list(slots), list(pos0)), *rows


# ---------------------------------------------------------------------------------------------- rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,cols,parts", [(100, 104, 4), (90, 96, 6), (90, 96, 90), (1500, 1504, 1), (1500, 1504, 20), (5000, 5008, 8), (9000, 9000, 3),
                                          (16000, 16000, 64), (14, 16, 2)])
def test_norms_over_parts(dev, dtype, n, cols, parts):
    """x + norm(delta), then the next norm, every part by its own root mean square; padded columns stay zero."""
    from dgpp_b200.ops import mixers as mx

    g, rows, eps = _gen(n), 3, 1e-3
    pad = lambda t: F.pad(t, (0, cols - n)).to(dev)
    spread = torch.exp(torch.randn(parts, generator=g)).repeat_interleave(n // parts)      # parts of unlike sizes
    x0, d, wa, wb = torch.randn(rows, n, generator=g) * spread, torch.randn(rows, n, generator=g) * spread, torch.randn(n, generator=g), torch.randn(n, generator=g)
    norm = lambda v, w: plain.group_norm(v, parts, eps, w.double())
    for with_delta in (True, False):
        x, out = pad(x0), torch.full((rows, cols), 7.0, dtype=dtype, device=dev)
        mx.stream_norm(x, n, eps, out, pad(d) if with_delta else None, ("parts", pad(wa)), ("parts", pad(wb)), parts=parts)
        s = x0.double() + (norm(d.double(), wa) if with_delta else 0)
        _close(x[:, :n], s, torch.float32, 1e-6)
        _close(out[:, :n], norm(s, wb), dtype, 2e-6, 5e-3)
        assert x[:, n:].abs().sum() == 0 and out[:, n:].abs().sum() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,cols,parts", [(100, 104, 1), (90, 96, 6), (3000, 3000, 4), (9000, 9000, 8)])
def test_mean_of_two_normed_rows(dev, dtype, n, cols, parts):
    from dgpp_b200.ops import mixers as mx

    g, rows, eps = _gen(cols), 5, 1e-2
    pad = lambda t: F.pad(t, (0, cols - n)).to(dev)
    x0, a, b = torch.randn(rows, n, generator=g), 3 * torch.randn(rows, n, generator=g), 0.2 * torch.randn(rows, n, generator=g)
    wa, wb, ba, bb, post, pre = (torch.randn(n, generator=g) for _ in range(6))
    kind = "parts" if parts > 1 else "rms"
    for biases in ((ba, bb), (ba, None), (None, None)):
        A, B = (v.double() + (0 if c is None else c.double()) for v, c in zip((a, b), biases))
        x, out = pad(x0), torch.empty(rows, cols, dtype=dtype, device=dev)
        pair = mx.PairDelta(pad(a), pad(wa), pad(b), pad(wb), 0.5, *(None if c is None else pad(c) for c in biases))
        mx.stream_norm(x, n, eps, out, pair, (kind, pad(post)), (kind, pad(pre)), parts=parts)
        mean = (plain.rms(A, eps) * wa.double() + plain.rms(B, eps) * wb.double()) / 2
        s = x0.double() + plain.group_norm(mean, parts, eps, post.double())
        _close(x[:, :n], s, torch.float32, 2e-6)
        _close(out[:, :n], plain.group_norm(s, parts, eps, pre.double()), dtype, 3e-6, 5e-3)


def test_norms_refuse_what_they_cannot_do(dev):
    from dgpp_b200.ops import mixers as mx

    x, w = torch.zeros(1, 96, device=dev), torch.ones(96, device=dev)
    for pre, parts in ((("parts", w), 7), (("parts", w), 0)):
        with pytest.raises(RuntimeError):
            mx.stream_norm(x, 90, 1e-5, torch.empty_like(x), None, (None, None), pre, parts=parts)
    with pytest.raises(RuntimeError):
        mx.stream_norm(x, 90, 1e-5, torch.empty_like(x), x.clone(), ("rms", w), ("parts", w), parts=6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act,fn", [("relu2", plain.relu_squared), ("gelu", plain.gelu_erf)])
def test_plain_activations(dev, dtype, act, fn):
    """Strided rows, fp32 rows in front of 16-bit ones, weights per row, tiles that nobody reads."""
    from dgpp_b200.ops import mixers as mx

    g = _gen(3)
    x, w = 3 * torch.randn(32, 48, generator=g), torch.rand(32, generator=g)
    for src in {torch.float32, dtype}:
        v = x.to(src)
        out = mx.act_rows(v.to(dev)[:, :40], torch.empty(32, 40, dtype=dtype, device=dev), act)
        _close(out, fn(v.double()[:, :40]), dtype, 2e-6, 5e-3)
        out = torch.full((32, 40), 5.0, dtype=dtype, device=dev)
        mx.act_rows(v.to(dev)[:, :40], out, act, w.to(dev), torch.tensor([2, -1], dtype=torch.int32, device=dev), 16)
        _close(out[:16], (fn(v.double()[:, :40]) * w.double()[:, None])[:16], dtype, 2e-6, 5e-3)
        assert (out[16:] == 5).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vdim,dv", [(3, 20, 32), (4, 128, 128), (2, 600, 600)])
def test_head_norm_with_weights_of_its_own_and_denominators(dev, dtype, heads, vdim, dv):
    from dgpp_b200.ops import mixers as mx

    g, rows = _gen(dv), 5
    o, gate = torch.randn(rows, heads, vdim, generator=g), (3 * torch.randn(rows, heads, vdim, generator=g)).to(dtype)
    w, den = torch.randn(heads, vdim, generator=g), 0.01 + 30 * torch.rand(rows, heads, generator=g)
    pad = lambda t: F.pad(t, (0, dv - vdim)).reshape(*t.shape[:-2], -1).to(dev)
    out = torch.empty(rows, heads * dv, dtype=dtype, device=dev)
    mx.gated_group_norm(pad(o), pad(gate), pad(w), out, heads, vdim, 1e-2, den=den.to(dev))
    want = plain.rms(o.double() / den.double()[..., None], 1e-2) * w.double() * plain.sigmoid(gate.double())
    _close(out.view(rows, heads, dv)[..., :vdim], want, dtype, 3e-6, 8e-3)


# ---------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("experts,identity,top", [(1, 0, 1), (1, 1, 2), (7, 2, 5), (12, 20, 16), (33, 1, 4), (200, 56, 8), (500, 12, 3)])
def test_router_with_a_correction_and_identity_experts(dev, experts, identity, top):
    """Both routes; the correction decides who is chosen and leaves the weights alone; identity experts have no row."""
    from dgpp_b200.ops import core as ops, mixers as mx

    g, n = _gen(experts), experts + identity
    i32 = dict(dtype=torch.int32, device=dev)
    corr = torch.randn(n, generator=g) * 0.1
    for rows in (1, 16, 17, 90):
        logits = torch.randn(rows, n + 5, generator=g) * 2
        z = logits[:, :n].double()
        best, share = zip(*(plain.route(t, corr.double(), top) for t in z))
        best = torch.stack(best)
        order = best.argsort(-1)
        best, share = best.gather(1, order), torch.stack(share).gather(1, order)
        bn, nt = 16, min(experts, rows * top) + (0 if rows <= mx.SMALL_TOKENS else rows * top // 16)
        pair, tiles, row_w = torch.empty(rows * top, **i32), torch.empty(nt, **i32), torch.zeros(nt * bn, device=dev)
        wts = torch.empty(rows, top, device=dev)
        if rows <= mx.SMALL_TOKENS:
            mx.moe_route_small(logits.to(dev), experts, top, pair, tiles, row_w, "softmax", None, corr.to(dev), True, identity, wts)
        else:
            ids, x = torch.empty(rows, top, **i32), torch.zeros(rows, 8, device=dev)
            mx.moe_select(logits.to(dev), n, top, ids, wts, "softmax", True, correction=corr.to(dev))
            assert torch.equal(ids.cpu().long(), best)
            ops.moe_segment_sort(ids, bn, nt, 0, experts, pair, tiles, torch.empty(1, **i32))
            mx.moe_scatter_rows(x, pair, wts, torch.zeros(nt * bn, 8, device=dev), row_w, top)
        pair, tiles, row_w = pair.cpu().long().view(rows, top), tiles.cpu().long(), row_w.cpu()
        own = best >= experts
        assert (pair[own] == -1).all() and torch.equal(tiles[pair[~own] // bn], best[~own])
        assert (wts.cpu().double() - share).abs().max() < 2e-5 and (row_w[pair[~own]].double() - share[~own]).abs().max() < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 9, 40])
@pytest.mark.parametrize("identity,shared", [(3, 24), (0, 24), (2, 0)])
def test_expert_block(dev, dtype, rows, identity, shared):
    from dgpp_b200.models.row_moe import RowExperts, RowExpertsScratch, run_experts
    from dgpp_b200.ops import mixers as mx
    from dgpp_b200.quant.formats import QuantLinear

    g, H, ff, E, top = _gen(rows), 72, 40, 5, 3
    sizes = [(f"e{e}.", ff) for e in range(E)] + ([("shared.", shared)] if shared else [])
    w = {f"{p}{n}": (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype) for p, f in sizes for n, s in (("up", (f, H)), ("down", (H, f)))}
    w["router"], w["correction"] = (torch.randn(E + identity, H, generator=g) * 0.3).to(dtype), torch.randn(E + identity, generator=g) * 0.1
    fmt = "fp32" if dtype == torch.float32 else "bf16"
    lin = lambda t: QuantLinear(fmt, *t.shape, t.contiguous().to(dev))
    first = F.pad(w["router"], (0, 0, 0, -(E + identity) % 8))
    b = RowExperts(E, top, ff, math.inf, lin(torch.cat([first] + ([w["shared.up"]] if shared else []))), torch.cat([w[f"e{e}.up"] for e in range(E)]).to(dev),
                   torch.cat([w[f"e{e}.down"] for e in range(E)]).to(dev), H, shared_col=first.shape[0], shared_ff=shared,
                   shared_down=lin(w["shared.down"]) if shared else None, score="softmax", correction=w["correction"].to(dev), norm_topk=True,
                   identity=identity, act="gelu", shared_gated=False)
    h = torch.randn(rows, H, generator=g).to(dtype)
    x, out = torch.zeros(rows, H, device=dev), torch.empty(rows, H, dtype=dtype, device=dev)
    ones = torch.ones(H, device=dev)
    mx.stream_norm(x, H, 1e-5, out, run_experts(b, RowExpertsScratch([b], 64, dtype, dev), h.to(dev)), (None, None), ("parts", ones))
    cfg = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
    _close(x, plain.experts(h.double(), "", cfg, {k: v.double() for k, v in w.items()}), dtype, 5e-6, 1.5e-2)


# ---------------------------------------------------------------------------------------------- convolution
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
@pytest.mark.parametrize("bias", [True, False])
def test_short_convolution_in_portions_over_reused_rings(dev, dtype, taps, bias):
    from dgpp_b200.ops import mixers as mx

    g, C, T = _gen(taps), 520, 60
    x, w, b = torch.randn(T, C, generator=g).to(dtype), torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    want = plain.causal_conv(x.double() + (b.double() if bias else 0), w.double())
    wide = F.pad(x, (8, 16)).to(dev)[:, 8:8 + C]
    ring = torch.full((4, taps, C), 50.0, device=dev)               # what earlier requests left

    def run(*parts):
        runs, req, pos = _runs(dev, [n for _, _, n in parts], [s for s, _, _ in parts], [p for _, p, _ in parts])
        rows = torch.cat([wide[p:p + n] for _, p, n in parts])
        rows = F.pad(rows, (0, 8))[:, :C]                           # a stride of its own
        out = mx.short_conv(rows, b.to(dev) if bias else None, w.T.contiguous().to(dev), ring, req, pos, runs, torch.empty(len(rows), C, dtype=dtype, device=dev))
        _close(out, torch.cat([want[p:p + n] for _, p, n in parts]), dtype, 3e-6, 6e-3)

    run((2, 0, T))
    run((2, 0, 1), (0, 0, 37), (3, 0, 2))
    run((3, 2, 1), (2, 1, 1), (0, 37, 1), (1, 0, 3))
    run((0, 38, 2), (3, 3, 33), (1, 3, 20))
    run((3, 36, 24), (0, 40, 20), (2, 2, 58), (1, 23, 1))


# ---------------------------------------------------------------------------------------------- attention
class Attention:
    """One attention layer between its projections: raw rows of a sequence, the kernels over a paged cache whose pages are handed out in
    a scrambled order, and the plain restatement.  stand_out: positions whose keys draw every query that sees them (through columns that
    are not rotated).  own_values False: values are the raw keys."""

    def __init__(self, dev, dtype, T, H, G, d, e, scale, size, keep=0, rot=0, base=1000.0, norm=False, cap=None, sink=False, taps=0, values=False,
                 own_values=True, stand_out=(), seed=0, eps=1e-3):
        from dgpp_b200.ops import mixers as mx

        g = _gen(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        q, k, v = rnd(T, H, d), rnd(T, G, d), rnd(T, G, e)
        if stand_out:
            u = F.pad(torch.ones(d - rot), (rot, 0)) * (24 / scale / (d - rot)) ** 0.5
            q = q * 0.2 + u
            k[list(stand_out)] = k[list(stand_out)] * 0.2 + u
            v[list(stand_out)] = 4 * v[list(stand_out)]
        bias = [0.3 * rnd(H, d), 0.3 * rnd(G, d), 0.3 * rnd(G, e)] if taps else [None] * 3
        q, k, v = (a.to(dtype) for a in (q, k, v))
        conv = [0.6 * rnd(h * n, taps) for h, n in ((H, d), (G, d), (G, e))] if taps else None
        if taps and stand_out:
            for c in conv:                                          # the current token passes, the past hardly
                c *= 0.02
                c[:, -1] = 1.0
        wq, wk = (1 + 0.2 * rnd(d), 1 + 0.2 * rnd(d)) if norm else (None, None)
        sinks = (2 * rnd(H) + (20 if stand_out else 0)) if sink else None
        # ---- plain
        Q, K, V = (a.double() + (0 if b is None else b.double()) for a, b in zip((q, k, v), bias))
        if not own_values:
            V = K
        if taps:
            Q, K, V = (plain.causal_conv(x.flatten(1), c.double()).view(x.shape) for x, c in zip((Q, K, V), conv))
        if norm:
            Q, K = plain.rms(Q, eps) * wq.double(), plain.rms(K, eps) * wk.double()
        if rot:
            Q, K = plain.rotate_halves(Q, base, rot), plain.rotate_halves(K, base, rot)
        if values:
            V = plain.left_values(V, base, eps)
        o = plain.attention(Q, K, V, scale, size, keep, cap, None if sinks is None else sinks.double())
        self.want = plain.rotate_halves(o, base, e, -1) if values else o
        # ---- rows for the kernels
        self.dtype, self.T, self.H, self.e, self.dev = dtype, T, H, e, dev
        D, DV = mx.pad_to(d, mx.ATTN_WIDTHS), mx.pad_to(e, mx.ATTN_WIDTHS)
        pad = lambda x, n: F.pad(x, (0, n - x.shape[-1])).flatten(-2)
        half = lambda x: F.pad(x.unflatten(-1, (2, -1)), (0, (DV - e) // 2)).flatten(-3) if values else pad(x, DV)     # [..., G, e] -> [..., G * DV]
        cols = [pad(q, D), pad(k, D)] + ([half(v)] if own_values else [])
        off = [0]
        for c in cols:
            off.append(off[-1] + c.shape[1])
        self.proj = torch.cat(cols, 1).to(dtype).to(dev)
        cw = torch.cat([f(c.T.reshape(taps, h, n)) for f, c, h, n in zip((lambda x: pad(x, D), lambda x: pad(x, D), half), conv, (H, G, G), (d, d, e))], 1) if taps else None
        self.g = mx.WindowHeads(H, G, d, e, size, scale, eps, 0, off[1], off[2] if own_values else off[1], norm="head" if norm else None,
                                bias=tuple(None if b is None else f(b).contiguous().to(dev) for f, b in zip((lambda x: pad(x, D), lambda x: pad(x, D), half), bias)),
                                freq=mx.rotation_freqs(base, rot, dev) if rot else None, rot=rot, keep_first=keep, softcap=cap or 0.0,
                                sink=None if sinks is None else sinks.to(dev), conv_w=None if cw is None else cw.contiguous().to(dev), vnorm=values,
                                vfreq=mx.value_freqs(base, e, DV, dev) if values else None)
        self.norms = tuple(None if w is None else F.pad(w, (0, D - d)).to(dev) for w in (wq, wk))
        self.values = values

    def cache(self, slots, pages, seed=0):
        from dgpp_b200.engine.kv_cache import PagedKV

        kv = PagedKV(1, 0, 0, pages, slots, pages, 64, False, self.dev, shapes=[self.g.kv_shape], dtype=self.dtype)
        order = torch.randperm(pages, generator=_gen(seed)).tolist()
        taken = [kv.alloc.alloc() for _ in range(pages)]
        assert sorted(taken) == list(range(pages))
        for b in order:
            kv.alloc.release(b)
        for t in (kv.layers[0].k, kv.layers[0].v):
            t.fill_(100.0)                                          # what earlier requests left
        kv.ring = self.g.new_ring(slots, self.dev)
        if kv.ring is not None:
            kv.ring.fill_(50.0)
        return kv

    def run(self, kv, parts, splits=1, tc=True, fused=None):
        """parts: [(slot, first position, tokens)] as one pass -> rows in order."""
        from dgpp_b200.ops import mixers as mx

        assert all(kv.reserve(s, p + n) for s, p, n in parts)
        runs, req, pos = _runs(self.dev, [n for *_, n in parts], [s for s, *_ in parts], [p for _, p, _ in parts])
        proj = torch.cat([self.proj[p:p + n] for _, p, n in parts]).contiguous()
        rows, g, L, bt = proj.shape[0], self.g, kv.layers[0], kv.block_table
        out = torch.full((rows, self.H * g.DV), 9.0, dtype=self.dtype, device=self.dev)
        scratch = torch.empty(rows * g.hq * splits * 2, device=self.dev), torch.empty(rows * g.hq * splits * g.DV, device=self.dev)
        fused = all(n == 1 for *_, n in parts) if fused is None else fused
        turn = torch.empty(rows * g.DV, device=self.dev)
        if not fused:
            if g.taps:
                proj = mx.short_conv(proj, g.stacked_bias, g.conv_w, kv.ring, req, pos, runs, torch.empty(rows, g.channels, dtype=self.dtype, device=self.dev))
                g = g.after_conv
            mx.qk_norm_append(g, proj, *self.norms, L, bt, req, pos, turn)
        if tc and not fused and mx.window_prefill_usable(g, proj):
            mx.window_prefill(g, proj, L, bt, req, pos, runs, out, turn=turn)
        else:
            mx.window_attn(g, proj, *self.norms, L, bt, req, pos, out, fused=fused, splits=splits, scratch=scratch, ring=kv.ring)
        out = out.view(rows, self.H, g.DV)
        return torch.cat([out[..., :self.e // 2], out[..., g.DV // 2:g.DV // 2 + self.e // 2]], -1) if self.values else out[..., :self.e]

    def check(self, got, rows):
        from dgpp_b200.ops import core as ops

        ops.check_status()
        want = self.want[rows]
        _close(got, want, self.dtype, 8e-5, 8e-2)                   # bf16: single places where rounded scores stand close
        assert (got.double().cpu() - want).pow(2).mean().sqrt() <= (1e-5 if self.dtype == torch.float32 else 8e-3) * want.abs().max()


SHAPES = [dict(H=4, G=2, d=24, e=40, scale=0.4), dict(H=6, G=6, d=64, e=20, scale=0.2), dict(H=12, G=1, d=100, e=130, scale=0.15),
          dict(H=1, G=1, d=8, e=8, scale=1.0), dict(H=20, G=2, d=72, e=200, scale=0.1), dict(H=16, G=2, d=200, e=250, scale=0.07)]
KINDS = {"kept": dict(size=40, keep=5, sink=True, norm=True, rot=4, own_values=False), "turned": dict(size=33, taps=4, values=True, rot=8, cap=6.0),
         "long taps": dict(size=100, taps=7, values=True, rot=0), "all at once": dict(size=70, keep=66, sink=True, norm=True, rot=8, taps=3, values=True, cap=4.0),
         "cap": dict(size=64, keep=1, cap=2.0), "plain": dict(size=1000)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(KINDS))
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_attention_prompts_portions_and_decoding(dev, dtype, kind, shape):
    """A prompt in one run, in portions, and token by token with and without splits give the plain result."""
    T, sizes = 140, dict(SHAPES[shape])
    if not KINDS[kind].get("own_values", True):
        sizes["e"] = sizes["d"]
    a = Attention(dev, dtype, T, **sizes, **KINDS[kind], seed=shape)
    kv = a.cache(2, 7)
    for tc in (True, False):
        a.check(a.run(kv, [(0, 0, T)], tc=tc), slice(0, T))
        kv.release(0)
    parts, o = [], 0
    for n in (2, 47, 1, 2, 14, 33, 21):
        parts.append(a.run(kv, [(1, o, n)], fused=False))
        o += n
    for splits in (1, 3) * 10:
        parts.append(a.run(kv, [(1, o, 1)], splits=splits))
        o += 1
    assert o == T
    a.check(torch.cat(parts), slice(0, T))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("extra", [dict(), dict(norm=False, taps=3, values=True, cap=40.0), dict(sink=True, own_values=False)])
@pytest.mark.parametrize("size,keep", [(1, 0), (1, 3), (33, 5), (64, 64), (65, 1), (100, 65), (128, 130)])
def test_keys_on_both_sides_of_an_edge(dev, dtype, size, keep, extra):
    """The last kept key, the first that is not kept, and keys at page borders and inside the window draw every query that sees them:
    prompts cut anywhere, and decoding."""
    T, edges = 300, sorted({x for x in (keep - 1, keep, 63, 64, 127, 150, 192) if x >= 0})
    a = Attention(dev, dtype, T, 4, 2, 32, 32, 0.3, size, keep, rot=16, stand_out=edges, seed=size + keep, **extra)
    kv = a.cache(2, 12)
    a.check(a.run(kv, [(0, 0, T)]), slice(0, T))
    at = {x + size + k for x in edges for k in (-1, 0, 1)} | {x + k for x in edges for k in (0, 1)}
    cuts, parts = sorted({0, T} | {x for x in at if 0 < x < T}), []
    for lo, hi in zip(cuts, cuts[1:]):
        parts.append(a.run(kv, [(1, lo, hi - lo)], splits=2 if hi - lo == 1 else 1))
    a.check(torch.cat(parts), slice(0, T))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("extra", [dict(), dict(taps=4, values=True, cap=50.0)])
def test_one_far_key_among_hundreds(dev, dtype, extra):
    """Single keys that stand out at page borders, hundreds of positions back, inside the window or kept, found by prompts and by decoded tokens."""
    T = 700
    for far, size, keep in (((0,), 650, 0), ((0,), 100, 1), ((63,), 90, 64), ((64,), 130, 65), ((127, 320), 600, 0), ((1, 447), 260, 2)):
        a = Attention(dev, dtype, T, 4, 2, 40, 24, 0.3, size, keep, stand_out=far, seed=far[0], **extra)
        kv = a.cache(2, 22)
        got = [a.run(kv, [(0, 0, 640)]), a.run(kv, [(0, 640, 3)], fused=False)]
        got += [a.run(kv, [(0, o, 1)], splits=s) for o, s in zip(range(643, 649), (1, 2, 5, 8, 1, 3))] + [a.run(kv, [(0, 649, T - 649)])]
        a.check(torch.cat(got), slice(0, T))


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_far_above_and_far_below_the_scores(dev, dtype):
    for level in (-90.0, 0.0, 90.0):
        a = Attention(dev, dtype, 90, 4, 2, 32, 32, 0.3, 40, sink=True)
        a.g.sink.add_(level)
        kv = a.cache(1, 3)
        got = torch.cat([a.run(kv, [(0, 0, 70)])] + [a.run(kv, [(0, t, 1)], splits=1 + t % 2) for t in range(70, 90)])
        if level == 0:
            a.check(got, slice(0, 90))
        elif level > 0:
            assert got.abs().max() < 1e-20
        else:
            b = Attention(dev, dtype, 90, 4, 2, 32, 32, 0.3, 40)
            _close(got, b.want, dtype, 8e-5, 8e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["kept", "turned", "all at once"])
def test_attention_of_unequal_requests_side_by_side(dev, dtype, kind):
    """Portions beside single tokens over reused pages and rings."""
    T = 130
    sizes = dict(e=40 if kind == "kept" else 72)
    a = Attention(dev, dtype, T, 6, 2, 40, scale=0.3, **sizes, **KINDS[kind], seed=5)
    kv = a.cache(4, 9)
    a.run(kv, [(2, 0, 100)])
    kv.release(2)
    a.check(a.run(kv, [(0, 0, 70), (3, 0, 1), (1, 0, 3)]), list(range(70)) + [0, 0, 1, 2])
    a.check(a.run(kv, [(3, 1, 90), (0, 70, 1), (1, 3, 1)]), list(range(1, 91)) + [70, 3])
    a.check(a.run(kv, [(1, 4, 1), (0, 71, 1), (3, 91, 1)], splits=2), [4, 71, 91])
    a.check(a.run(kv, [(0, 72, 2), (1, 5, 60), (3, 92, 1)]), [72, 73] + list(range(5, 65)) + [92])


def test_attention_refuses_what_it_cannot_do(dev):
    a = Attention(dev, torch.float32, 4, 4, 2, 24, 40, 0.4, **KINDS["all at once"])
    kv = a.cache(1, 2)
    for change in (dict(rot=26), dict(hq=5), dict(window=0), dict(keep_first=-1), dict(softcap=-1.0), dict(vdim=300), dict(norm="row"), dict(chunked=True)):
        old = {k: getattr(a.g, k) for k in change}
        for k, v in change.items():
            setattr(a.g, k, v)
        with pytest.raises((RuntimeError, AssertionError)):
            a.run(kv, [(0, 0, 1)])
        for k, v in old.items():
            setattr(a.g, k, v)


# ---------------------------------------------------------------------------------------------- matrix memory
class Memory:
    """The recurrent mixer between its projections, and its plain restatement."""

    def __init__(self, dev, dtype, T, H, d, e, cap=6.0, keep=2.0, write=0.0, seed=0, eps=1e-3):
        from dgpp_b200.ops import mixers as mx

        g = _gen(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        q, k, v, gate = (rnd(T, H, n).to(dtype) for n in (d, d, e, e))
        i, f = (2 * rnd(T, H)).to(dtype), (2 * rnd(T, H)).to(dtype)
        ib, fb, nw = write + rnd(H), keep + rnd(H), 1 + 0.2 * rnd(H, e)
        I, Fg = plain.soft_cap(i.double() + ib.double(), cap), plain.log_sigmoid(plain.soft_cap(f.double() + fb.double(), cap))
        o = plain.matrix_memory(q.double() * d ** -0.5, k.double(), v.double(), I, Fg)
        self.want = plain.rms(o, eps) * nw.double() * plain.sigmoid(gate.double())
        DK, DV = mx.pad_to(d, mx.STATE_WIDTHS), mx.pad_to(e, mx.STATE_WIDTHS)
        pad = lambda x, n: F.pad(x, (0, n - x.shape[-1])).flatten(1)
        up = lambda x: F.pad(x, (0, -x.shape[1] % 8))
        cols = [up(f), pad(q, DK), pad(k, DK), pad(v, DV), up(i), pad(gate, DV)]
        off = [0]
        for c in cols:
            off.append(off[-1] + c.shape[1])
        self.proj = torch.cat(cols, 1).to(dev).contiguous()
        self.g = mx.MatrixHeads(H, d, e, off[1], off[4], off[0], off[5], ib.to(dev), fb.to(dev), cap, pad(nw[None], DV)[0].contiguous().to(dev), eps)
        self.dev, self.dtype, self.e, self.T = dev, dtype, e, T

    def state(self, slots):
        st = self.g.new_state(slots, self.dev)
        for t in st:
            t.fill_(50.0)                                           # what earlier requests left
        return st

    def run(self, st, *parts):
        from dgpp_b200.ops import mixers as mx

        runs, req, pos = _runs(self.dev, [n for *_, n in parts], [s for s, *_ in parts], [p for _, p, _ in parts])
        proj, g = torch.cat([self.proj[p:p + n] for _, p, n in parts]).contiguous(), self.g
        rows = proj.shape[0]
        out = torch.empty(rows, g.heads * g.DV, dtype=self.dtype, device=self.dev)
        if all(n == 1 for *_, n in parts):
            mx.matrix_memory(g, proj, *st, req, pos, out=out)
        else:
            o, den = torch.empty(rows, g.heads * g.DV, device=self.dev), torch.empty(rows, g.heads, device=self.dev)
            mx.matrix_memory(g, proj, *st, req, pos, runs=runs, prep=torch.empty(g.prep_floats(rows, len(parts)), device=self.dev), o=o, den=den)
            mx.gated_group_norm(o, proj[:, g.gate_off:], g.norm_w, out, g.heads, g.vdim, g.eps, den=den)
        return out.view(rows, g.heads, g.DV)[..., :self.e]


MEMORIES = [(4, 32, 64), (3, 20, 24), (2, 130, 40), (9, 64, 130), (1, 8, 8), (4, 256, 32), (5, 100, 256), (2, 128, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MEMORIES)
def test_matrix_memory_prompts_portions_and_decoding(dev, dtype, shape):
    T = 110
    a = Memory(dev, dtype, T, *shape, seed=shape[1])
    st = a.state(3)
    fine = dict(fine=1e-4, coarse=3e-2)
    _close(a.run(st, (1, 0, T)), a.want, dtype, **fine)
    parts, o = [], 0
    for n in (1, 2, 2, 16, 17, 3, 1, 1, 35, 20) + (1,) * 12:
        parts.append(a.run(st, (2, o, n)))
        o += n
    assert o == T
    _close(torch.cat(parts), a.want, dtype, **fine)
    _close(torch.cat([a.run(st, (1, t, 1)) for t in range(40)]), a.want[:40], dtype, **fine)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap,keep,write", [(30.0, 12.0, 0.0), (40.0, -25.0, 0.0), (40.0, 3.0, -30.0), (60.0, 8.0, 40.0), (0.5, 0.0, 0.0), (15.0, 30.0, -9.0)])
def test_matrix_memory_with_extreme_gates(dev, dtype, cap, keep, write):
    """Memories that last and that vanish at once, writes that dwarf all before them or hardly show: where the running maximum, the floor of
    the denominator and the start from zero decide."""
    a = Memory(dev, dtype, 75, 4, 32, 32, cap, keep, write)
    st = a.state(1)
    got = torch.cat([a.run(st, (0, 0, 50)), a.run(st, (0, 50, 1)), a.run(st, (0, 51, 19))] + [a.run(st, (0, t, 1)) for t in range(70, 75)])
    assert torch.isfinite(got).all()
    _close(got, a.want, dtype, 3e-4, 3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_in_unequal_batches_with_reused_slots(dev, dtype):
    a = Memory(dev, dtype, 80, 6, 48, 32)
    st = a.state(4)
    at = lambda *r: torch.cat([a.want[p:p + n] for p, n in r])
    a.run(st, *((s, 0, 33) for s in range(4)))
    _close(a.run(st, (2, 0, 40), (0, 0, 1), (3, 0, 2), (1, 0, 17)), at((0, 40), (0, 1), (0, 2), (0, 17)), dtype, 1e-4, 3e-2)
    _close(a.run(st, (0, 1, 1), (3, 2, 1), (2, 40, 1)), at((1, 1), (2, 1), (40, 1)), dtype, 1e-4, 3e-2)
    _close(a.run(st, (1, 17, 1), (0, 2, 50), (3, 3, 3)), at((17, 1), (2, 50), (3, 3)), dtype, 1e-4, 3e-2)
