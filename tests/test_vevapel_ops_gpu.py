"""The operators behind the Vevapel family on the GPU, each against its plain restatement, in bf16 and in true fp32."""
import math

import pytest
import torch
import torch.nn.functional as F

import vevapel_plain as plain

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
@pytest.mark.parametrize("n,cols", [(100, 104), (1500, 1504), (5000, 5008), (9000, 9000)])
def test_norms_with_biases_factor_and_row_vector(dev, dtype, n, cols):
    """x + m norm(delta + b) + vec, then the next norm into rows with a stride of their own; padded columns stay zero."""
    from dgpp_b200.ops import mixers as mx

    g, rows, eps, m = _gen(n), 3, 1e-3, 0.37
    pad = lambda t: F.pad(t, (0, cols - n)).to(dev)
    x0, d = torch.randn(rows, n, generator=g) + 3, torch.randn(rows, n, generator=g) - 2
    wa, ba, wb, bb, db, vec = (torch.randn(n, generator=g) for _ in range(6))
    big = torch.full((rows, 2 * cols), 7.0, dtype=dtype, device=dev)
    ln = lambda v, w, b: plain.layer_norm(v, eps, w.double(), b.double())
    for with_delta in (True, False):
        x = pad(x0)
        mx.stream_norm(x, n, eps, big[:, cols:], pad(d) if with_delta else None, ("layer", pad(wa), pad(ba)), ("layer", pad(wb), pad(bb)), m,
                       pad(db) if with_delta else None, pad(vec))
        s = x0.double() + vec.double() + (m * ln(d.double() + db.double(), wa, ba) if with_delta else 0)
        _close(x[:, :n], s, torch.float32, 1e-6)
        _close(big[:, cols:cols + n], ln(s, wb, bb), dtype, 2e-6, 5e-3)
        assert x[:, n:].abs().sum() == 0 and big[:, cols + n:].abs().sum() == 0 and (big[:, :cols] == 7).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_scaled_embedding_rows_and_their_copy(dev, dtype):
    from dgpp_b200.ops import mixers as mx

    table, ids = torch.randn(11, 104, generator=_gen(1)).to(dtype).to(dev), torch.tensor([3, 10, 0, 3], dtype=torch.int32, device=dev)
    x, both = torch.empty(4, 104, device=dev), torch.full((4, 208), 5.0, dtype=dtype, device=dev)
    mx.embed_rows(ids, table, x, 2.7, both[:, 104:])
    want = table.float()[ids.long()] * 2.7
    assert torch.allclose(x, want, rtol=1e-6) and torch.equal(both[:, 104:], want.to(dtype)) and (both[:, :104] == 5).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vdim,dv", [(3, 20, 32), (4, 128, 128), (2, 600, 600)])
def test_head_norm_with_a_silu_gate(dev, dtype, heads, vdim, dv):
    from dgpp_b200.ops import mixers as mx

    g, rows = _gen(dv), 5
    o, gate, w = torch.randn(rows, heads, vdim, generator=g), (3 * torch.randn(rows, heads, vdim, generator=g)).to(dtype), torch.randn(vdim, generator=g)
    pad = lambda t: F.pad(t, (0, dv - vdim)).reshape(rows, -1).to(dev)
    out = torch.empty(rows, heads * dv, dtype=dtype, device=dev)
    mx.gated_group_norm(pad(o), pad(gate), F.pad(w, (0, dv - vdim)).to(dev), out, heads, vdim, 1e-2, silu=True)
    _close(out.view(rows, heads, dv)[..., :vdim], plain.rms(o.double(), 1e-2) * w.double() * plain.silu(gate.double()), dtype, 3e-6, 8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_expert_activation_weighs_the_output(dev, dtype):
    from dgpp_b200.ops import mixers as mx

    g, rows, ff = _gen(7), 6, 40
    gu, w = (2 * torch.randn(rows, 2 * ff, generator=g)).to(dtype), torch.rand(rows, generator=g)
    out = mx.clamped_glu(gu.to(dev), torch.empty(rows, ff, dtype=dtype, device=dev), math.inf, 1.0, w.to(dev), shift=0.0, weigh_out=True)
    a, b = gu.double().chunk(2, 1)
    _close(out, plain.silu(a) * b * w.double()[:, None], dtype, 2e-6, 8e-3)


@pytest.mark.parametrize("experts,top", [(1, 1), (7, 2), (16, 16), (33, 5), (200, 8), (512, 3)])
def test_router_bias_and_softmax_over_the_chosen(dev, experts, top):
    """Both routes; logits so far apart that scores over all experts would vanish; ties go to the lower ids."""
    from dgpp_b200.ops import core as ops, mixers as mx

    g = _gen(experts)
    i32 = dict(dtype=torch.int32, device=dev)
    bias = torch.randn(experts, generator=g) * 2
    for rows in (1, 16, 17, 90):
        logits = torch.randn(rows, experts + 5, generator=g) * 2
        if experts > 2:
            logits[0, :experts] = -bias                             # all the same with the bias
        logits[rows // 2, :experts] *= 150
        z = (logits[:, :experts] + bias).double()
        best = torch.argsort(-z, dim=-1, stable=True)[:, :top].sort(-1).values
        share = z.gather(1, best).softmax(-1)
        small = rows <= mx.SMALL_TOKENS
        bn, nt = 16, min(experts, rows * top) + (0 if rows <= mx.SMALL_TOKENS else rows * top // 16)
        pair, tiles, row_w = torch.empty(rows * top, **i32), torch.empty(nt, **i32), torch.zeros(nt * bn, device=dev)
        if small:
            mx.moe_route_small(logits.to(dev), experts, top, pair, tiles, row_w, "chosen", bias.to(dev))
        else:
            ids, wts, x = torch.empty(rows, top, **i32), torch.empty(rows, top, device=dev), torch.zeros(rows, 8, device=dev)
            mx.moe_select(logits.to(dev), experts, top, ids, wts, "chosen", bias=bias.to(dev))
            ops.moe_segment_sort(ids, bn, nt, 0, experts, pair, tiles, torch.empty(1, **i32))
            mx.moe_scatter_rows(x, pair, wts, torch.zeros(nt * bn, 8, device=dev), row_w, top)
        pair, tiles, row_w = pair.cpu().long(), tiles.cpu().long(), row_w.cpu()
        assert torch.equal(tiles[pair // bn].view(rows, top), best)
        assert (row_w[pair].view(rows, top).double() - share).abs().max() < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 9, 40])
def test_expert_block(dev, dtype, rows):
    from dgpp_b200.models.row_moe import RowExperts, RowExpertsScratch, run_experts
    from dgpp_b200.ops import mixers as mx
    from dgpp_b200.quant.formats import QuantLinear

    g, H, ff, E, top = _gen(rows), 72, 40, 6, 3
    w = {f"e{e}.{n}": (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype) for e in range(E) for n, s in (("gate", (ff, H)), ("up", (ff, H)), ("down", (H, ff)))}
    w["router"], w["router.b"] = (torch.randn(E, H, generator=g) * 0.3).to(dtype), torch.randn(E, generator=g)
    gu = torch.cat([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).to(dev)
    down = torch.cat([w[f"e{e}.down"] for e in range(E)]).to(dev)
    first = QuantLinear("fp32" if dtype == torch.float32 else "bf16", 8, H, F.pad(w["router"], (0, 0, 0, 2)).to(dev))
    b = RowExperts(E, top, ff, math.inf, first, gu, down, H, alpha=1.0, shift=0.0, score="chosen", weigh_out=True, router_b=w["router.b"].to(dev))
    h = torch.randn(rows, H, generator=g).to(dtype)
    x, out = torch.zeros(rows, H, device=dev), torch.empty(rows, H, dtype=dtype, device=dev)
    mx.stream_norm(x, H, 1e-5, out, run_experts(b, RowExpertsScratch([b], 64, dtype, dev), h.to(dev)))
    _close(x, plain.experts(h.double(), "", {"router": {"top": top}}, {k: v.double() for k, v in w.items()}), dtype, 5e-6, 1.5e-2)


# ---------------------------------------------------------------------------------------------- attention
class Attention:
    """One attention layer between its projections: raw rows of a sequence, the kernels over a paged cache whose pages are handed out
    in a scrambled order, and the plain restatement.  stand_out: positions whose keys draw every query that sees them (through columns
    that are not rotated)."""

    def __init__(self, dev, dtype, T, H, G, d, e, scale, maps=1, chunk=None, rot=0, base=1000.0, temp=(0.0, 1), norm=False, stand_out=(), seed=0,
                 lam=0.6, eps=1e-3):
        from dgpp_b200.ops import mixers as mx

        g = _gen(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        q, k, v = rnd(T, H, maps, d), rnd(T, G, maps, d), rnd(T, G, e)
        if stand_out:
            u = F.pad(torch.ones(d - rot), (rot, 0)) * (24 / scale / (d - rot)) ** 0.5
            q = q * 0.2 + u
            k[list(stand_out)] = k[list(stand_out)] * 0.2 + u
            v[list(stand_out)] = 4 * v[list(stand_out)]
        bias = [0.3 * rnd(H, maps, d), 0.3 * rnd(G, maps, d), 0.3 * rnd(G, e)]
        q, k, v = ((a - b).to(dtype) for a, b in zip((q, k, v), bias))
        wq, wk = (1 + 0.2 * rnd(H * maps * d), 1 + 0.2 * rnd(G * maps * d)) if norm else (None, None)
        gate = rnd(T, H, 1 if maps == 1 else e).to(dtype)
        self.dtype, self.T, self.H, self.maps, self.chunk, self.eps, self.dev, self.e = dtype, T, H, maps, chunk, eps, dev, e
        # ---- plain
        Q, K, V = (a.double() + b.double() for a, b in zip((q, k, v), bias))
        if norm:
            Q = (plain.rms(Q.view(T, -1), eps) * wq.double()).view(Q.shape)
            K = (plain.rms(K.view(T, -1), eps) * wk.double()).view(K.shape)
        Q = Q * torch.tensor([plain.temperature(t, *temp) for t in range(T)]).view(T, 1, 1, 1)
        if rot:
            Q, K = plain.rotate_halves(Q, base, rot), plain.rotate_halves(K, base, rot)
        a = [plain.attention(Q[:, :, m], K[:, :, m], V, scale, chunk) for m in range(maps)]
        self.diff, lq = 0.25, torch.tensor([1.0, 0.0])
        self.lam = lam
        if maps == 1:
            self.want = a[0] * plain.sigmoid(gate.double())
        else:
            lk = torch.tensor([math.log(lam - self.diff + 1.0), 0.0])
            self.want = plain.differential(a[0], a[1], lq, lk, lq * 0, lq, self.diff, eps) * plain.sigmoid(gate.double())
        # ---- rows for the kernels
        self.g = mx.WindowHeads(H, G, d, e, chunk or mx.NO_WINDOW, scale, eps, 0, 0, 0, norm="row" if norm else None, rot=rot, temp=temp, maps=maps,
                                chunked=chunk is not None, freq=mx.rotation_freqs(base, rot, dev) if rot else None)
        D, DV, grp = self.g.D, self.g.DV, H // G
        pad = lambda x, n: F.pad(x, (0, n - x.shape[-1]))
        by_map = lambda x: x.reshape(*x.shape[:-3], G, grp, maps, d).transpose(-3, -2).flatten(-4, -2)
        row = lambda x, n: pad(x, n).flatten(-2).float().contiguous().to(dev)
        cols = [row(by_map(q), D), row(k.flatten(-3, -2), D), row(v, DV), row(gate, DV) if maps == 2 else pad(gate[..., 0].float(), (H + 7) // 8 * 8).to(dev)]
        off = [0]
        for c in cols:
            off.append(off[-1] + c.shape[1])
        self.proj = torch.cat(cols, 1).to(dtype)
        self.g.q_off, self.g.k_off, self.g.v_off, self.gate_off = off[:4]
        self.g.gate_off = off[3] if maps == 1 else -1
        self.g.bias = row(by_map(bias[0]), D), row(bias[1].flatten(-3, -2), D), row(bias[2], DV)
        self.wq, self.wk = (row(by_map(wq.view(H, maps, d)), D), row(wk.view(G * maps, d), D)) if norm else (None, None)

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
        return kv

    def run(self, kv, parts, splits=1, tc=True, fused=None):
        """parts: [(slot, first row of `proj`, first position, tokens)] as one pass -> rows in order."""
        from dgpp_b200.ops import mixers as mx

        assert all(kv.reserve(s, p + n) for s, _, p, n in parts)
        runs, req, pos = _runs(self.dev, [n for *_, n in parts], [s for s, *_ in parts], [p for _, _, p, _ in parts])
        proj = torch.cat([self.proj[a:a + n] for _, a, _, n in parts]).contiguous()
        rows, g, L, bt = proj.shape[0], self.g, kv.layers[0], kv.block_table
        out = torch.full((rows, self.H * g.DV), 9.0, dtype=self.dtype, device=self.dev)
        scratch = torch.empty(rows * g.hq * splits * 2, device=self.dev), torch.empty(rows * g.hq * splits * g.DV, device=self.dev)
        fused = all(n == 1 for *_, n in parts) if fused is None else fused
        finish = lambda s, **kw: mx.diff_combine(g, s, proj, self.gate_off, out, self.lam, 1 - self.diff, **kw) if self.maps == 2 else None
        if not fused:
            mx.qk_norm_append(g, proj, self.wq, self.wk, L, bt, req, pos)
        if tc and not fused and mx.window_prefill_usable(g, proj):
            mx.window_prefill(g, proj, L, bt, req, pos, runs, out, raw=scratch[1] if self.maps == 2 else None)
            finish(scratch[1], finished=True)
        else:
            mx.window_attn(g, proj, self.wq, self.wk, L, bt, req, pos, out, fused=fused, splits=splits, scratch=scratch)
            finish(scratch, splits=splits)
        return out.view(rows, self.H, g.DV)[..., :self.e]

    def check(self, got, rows):
        from dgpp_b200.ops import core as ops

        ops.check_status()
        want = self.want[rows]
        _close(got, want, self.dtype, 5e-5, 8e-2)                   # bf16: single places where rounded scores stand close
        assert (got.double().cpu() - want).pow(2).mean().sqrt() <= (1e-5 if self.dtype == torch.float32 else 6e-3) * want.abs().max()


SHAPES = [dict(H=4, G=2, d=24, e=40, scale=0.4), dict(H=6, G=6, d=64, e=20, scale=0.2), dict(H=12, G=1, d=100, e=130, scale=0.15),
          dict(H=1, G=1, d=8, e=8, scale=1.0), dict(H=20, G=2, d=72, e=200, scale=0.1)]
KINDS = {"full": dict(norm=True, temp=(0.7, 9)), "diff": dict(maps=2, chunk=50, rot=8), "diff all": dict(maps=2, chunk=1000, rot=0),
         "all at once": dict(maps=2, chunk=70, rot=4, norm=True, temp=(1.1, 5)), "plain": dict()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(KINDS))
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_attention_prompts_portions_and_decoding(dev, dtype, kind, shape):
    """A prompt in one run, in portions, and token by token with and without splits give the plain result."""
    T = 140
    a = Attention(dev, dtype, T, **SHAPES[shape], **KINDS[kind], seed=shape)
    kv = a.cache(2, 7)
    for tc in (True, False):
        a.check(a.run(kv, [(0, 0, 0, T)], tc=tc), slice(0, T))
        kv.release(0)
    parts, o = [], 0
    for n in (2, 47, 1, 2, 14, 33, 21):
        parts.append(a.run(kv, [(1, o, o, n)], fused=False))
        o += n
    for splits in (1, 3) * 10:
        parts.append(a.run(kv, [(1, o, o, 1)], splits=splits))
        o += 1
    assert o == T
    a.check(torch.cat(parts), slice(0, T))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [1, 33, 64, 128, 129])
def test_keys_on_both_sides_of_a_chunks_edge(dev, dtype, chunk):
    """The last key of a chunk and the first of the next one draw every query that sees them: prompts cut anywhere, and decoding."""
    T, edges = 300, sorted({x for c in range(0, 300, chunk) for x in (c, c + chunk - 1) if x < 300}) if chunk > 1 else (0, 63, 64, 299)
    a = Attention(dev, dtype, T, 4, 2, 32, 32, 0.3, maps=2, chunk=chunk, rot=16, stand_out=edges, seed=chunk)
    kv = a.cache(2, 12)
    a.check(a.run(kv, [(0, 0, 0, T)]), slice(0, T))
    at = {x + k for x in edges for k in (-1, 0, 1)}
    cuts, o, parts = sorted({0, T} | {x for x in at if 0 < x < T and x % 3}), 0, []
    for lo, hi in zip(cuts, cuts[1:]):
        parts.append(a.run(kv, [(1, lo, lo, hi - lo)], splits=2 if hi - lo == 1 else 1))
    a.check(torch.cat(parts), slice(0, T))


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_key_among_hundreds(dev, dtype):
    """Single keys that stand out at page borders, hundreds of positions back, found by prompts and by decoded tokens."""
    T = 700
    for far in ((0,), (63,), (64,), (127, 320), (1, 447)):
        a = Attention(dev, dtype, T, 4, 2, 40, 24, 0.3, norm=True, temp=(0.5, 64), stand_out=far, seed=far[0])
        kv = a.cache(2, 22)
        got = [a.run(kv, [(0, 0, 0, 640)]), a.run(kv, [(0, 640, 640, 3)], fused=False)]
        got += [a.run(kv, [(0, o, o, 1)], splits=s) for o, s in zip(range(643, 649), (1, 2, 5, 8, 1, 3))] + [a.run(kv, [(0, 649, 649, T - 649)])]
        a.check(torch.cat(got), slice(0, T))
        assert a.want[600:].std() > 0.5 * a.want[:2].std()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["full", "all at once"])
def test_attention_of_unequal_requests_side_by_side(dev, dtype, kind):
    """Portions beside single tokens over reused pages, and the rows of the short runs alone (row lists, splits)."""
    from dgpp_b200.ops import mixers as mx

    T = 130
    a = Attention(dev, dtype, T, 6, 2, 40, 72, 0.3, **KINDS[kind], seed=5)
    kv = a.cache(4, 9)
    a.run(kv, [(2, 0, 0, 100)])
    kv.release(2)
    a.check(a.run(kv, [(0, 0, 0, 70), (3, 0, 0, 1), (1, 0, 0, 3)]), list(range(70)) + [0, 0, 1, 2])
    a.check(a.run(kv, [(3, 1, 1, 90), (0, 70, 70, 1), (1, 3, 3, 1)]), list(range(1, 91)) + [70, 3])
    a.check(a.run(kv, [(1, 4, 4, 1), (0, 71, 71, 1), (3, 91, 91, 1)], splits=2), [4, 71, 91])
    # a pass whose long run takes the prompt kernel and whose short runs go row by row
    parts = [(0, 72, 72, 2), (1, 5, 5, 60), (3, 92, 92, 1)]
    assert all(kv.reserve(s, p + n) for s, _, p, n in parts)
    runs, req, pos = _runs(dev, [2, 60, 1], [0, 1, 3], [72, 5, 92])
    proj = torch.cat([a.proj[o:o + n] for _, o, _, n in parts]).contiguous()
    g, L, bt, rows = a.g, kv.layers[0], kv.block_table, 63
    out = torch.full((rows, a.H * g.DV), 9.0, dtype=dtype, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    short, long = i32([0, 1, 62]), list(range(2, 62))
    mx.qk_norm_append(g, proj, a.wq, a.wk, L, bt, req, pos)
    finish = lambda s, **kw: mx.diff_combine(g, s, proj, a.gate_off, out, a.lam, 1 - a.diff, **kw) if a.maps == 2 else None
    if mx.window_prefill_usable(g, proj):
        raw = torch.empty(rows * g.hq * g.DV, device=dev) if a.maps == 2 else None
        mx.window_prefill(g, proj, L, bt, req, pos, runs, out, raw=raw, some=(i32([2]), i32([60]), [60]))
        finish(raw, row_list=i32(long), finished=True)
        assert (out[[0, 1, 62]] == 9).all()
    scratch = torch.empty(3 * g.hq * 3 * 2, device=dev), torch.empty(3 * g.hq * 3 * g.DV, device=dev)
    mx.window_attn(g, proj, a.wq, a.wk, L, bt, req, pos, out, splits=3, scratch=scratch, row_list=short)
    finish(scratch, splits=3, row_list=short)
    pick = [0, 1, 62] + (long if mx.window_prefill_usable(g, proj) else [])
    at = torch.tensor([72, 73] + list(range(5, 65)) + [92])
    a.check(out.view(rows, a.H, g.DV)[..., :a.e][pick], at[pick])


def test_attention_refuses_what_it_cannot_do(dev):
    a = Attention(dev, torch.float32, 4, 4, 2, 24, 40, 0.4, **KINDS["full"])
    kv = a.cache(1, 2)
    for change in (dict(rot=26), dict(rot=3), dict(hq=5), dict(window=0), dict(temp=(0.1, 0))):
        old = {k: getattr(a.g, k) for k in change}
        for k, v in change.items():
            setattr(a.g, k, v)
        with pytest.raises(RuntimeError):
            a.run(kv, [(0, 0, 0, 1)])
        for k, v in old.items():
            setattr(a.g, k, v)


# ---------------------------------------------------------------------------------------------- delta rule
class Delta:
    """The recurrent layer between its projections, and its plain restatement."""

    def __init__(self, dev, dtype, T, H, G, d, e, taps, decay=1.0, seed=0, eps=1e-3):
        from dgpp_b200.ops import mixers as mx

        g = _gen(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        q, k, v = rnd(T, G, d).to(dtype), rnd(T, G, d).to(dtype), rnd(T, H, e).to(dtype)
        b, a, gate = (2 * rnd(T, H)).to(dtype), rnd(T, H).to(dtype), rnd(T, H, e).to(dtype)
        conv = [0.6 * rnd(n, taps) for n in (G * d, G * d, H * e)]
        A, dt, nw = rnd(H), rnd(H) - 3 + decay, 1 + 0.2 * rnd(e)
        Q, K, V = (plain.causal_conv(x.double().flatten(1), c.double()) for x, c in zip((q, k, v), conv))
        grp = torch.arange(H) // (H // G)
        Q, K = plain.unit(Q.view(T, G, d))[:, grp] * d ** -0.5, plain.unit(K.view(T, G, d))[:, grp]
        f = torch.exp(-torch.exp(A.double()) * plain.softplus(a.double() + dt.double()))
        o = plain.delta_rule(Q, K, V.view(T, H, e), plain.sigmoid(b.double()), f)
        self.want = plain.rms(o, eps) * nw.double() * plain.silu(gate.double())
        DK, DV = mx.pad_to(d, mx.STATE_WIDTHS), mx.pad_to(e, mx.STATE_WIDTHS)
        pad = lambda x, n: F.pad(x, (0, n - x.shape[-1])).flatten(1)
        up = lambda x: F.pad(x, (0, -x.shape[1] % 8))
        cols = [pad(q, DK), pad(k, DK), pad(v, DV), up(b), up(a), pad(gate, DV)]
        off = [0]
        for c in cols:
            off.append(off[-1] + c.shape[1])
        self.proj = torch.cat(cols, 1).to(dev).contiguous()
        cw = torch.cat([F.pad(c.view(h, n, taps), (0, 0, 0, p - n)).reshape(-1, taps) for c, h, n, p in zip(conv, (G, G, H), (d, d, e), (DK, DK, DV))])
        self.s = mx.StateHeads(H, G, d, e, 0, off[3], eps, cw.T.contiguous().to(dev), A.to(dev), dt.to(dev), norm_w=F.pad(nw, (0, DV - e)).to(dev),
                               a_off=off[4], gate_off=off[5])
        self.dev, self.dtype, self.e, self.T = dev, dtype, e, T

    def state(self, slots):
        st = self.s.new_state(slots, self.dev)
        for t in st:
            t.fill_(50.0)                                           # what earlier requests left
        return st

    def run(self, st, parts):
        from dgpp_b200.ops import mixers as mx

        runs, req, pos = _runs(self.dev, [n for *_, n in parts], [s for s, *_ in parts], [p for _, p, _ in parts])
        proj, s = torch.cat([self.proj[p:p + n] for _, p, n in parts]).contiguous(), self.s
        rows = proj.shape[0]
        out = torch.empty(rows, s.hv * s.DV, dtype=self.dtype, device=self.dev)
        if all(n == 1 for *_, n in parts):
            mx.linear_state(s, proj, *st, req, pos, out=out)
        else:
            o, prep = torch.empty(rows, s.hv * s.DV, device=self.dev), torch.empty(s.prep_floats(rows, len(parts)), device=self.dev)
            mx.linear_state(s, proj, *st, req, pos, runs=runs, prep=prep, o=o)
            mx.gated_group_norm(o, proj[:, s.gate_off:], s.norm_w, out, s.hv, s.vdim, s.eps, silu=True)
        return out.view(rows, s.hv, s.DV)[..., :self.e]


DELTAS = [(4, 2, 32, 64, 4), (3, 1, 20, 24, 2), (2, 2, 130, 40, 3), (12, 1, 64, 130, 6), (1, 1, 8, 8, 1), (4, 4, 256, 32, 5), (20, 2, 100, 200, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", DELTAS)
def test_delta_rule_prompts_portions_and_decoding(dev, dtype, shape):
    T = 90
    a = Delta(dev, dtype, T, *shape, seed=shape[2])
    st = a.state(3)
    fine = dict(fine=1e-4, coarse=3e-2)
    _close(a.run(st, [(1, 0, T)]), a.want, dtype, **fine)
    parts, o = [], 0
    for n in (1, 2, 2, 16, 17, 3, 1, 1, 30, 5) + (1,) * 12:
        parts.append(a.run(st, [(2, o, n)]))
        o += n
    assert o == T
    _close(torch.cat(parts), a.want, dtype, **fine)
    _close(torch.cat([a.run(st, [(1, t, 1)]) for t in range(40)]), a.want[:40], dtype, **fine)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", [-6.0, 8.0, 60.0])
def test_delta_rule_with_extreme_decays(dev, dtype, decay):
    """Memories that last, and decays so strong that quotients of them would overflow."""
    a = Delta(dev, dtype, 70, 4, 2, 32, 32, 3, decay=decay)
    st = a.state(1)
    got = torch.cat([a.run(st, [(0, 0, 50)]), a.run(st, [(0, 50, 1)]), a.run(st, [(0, 51, 19)])])
    assert torch.isfinite(got).all()
    _close(got, a.want, dtype, 2e-4, 3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_in_unequal_batches_with_reused_slots(dev, dtype):
    a = Delta(dev, dtype, 80, 6, 3, 48, 32, 4)
    st = a.state(4)
    at = lambda *r: torch.cat([a.want[p:p + n] for p, n in r])
    a.run(st, [(s, 0, 33) for s in range(4)])
    _close(a.run(st, [(2, 0, 40), (0, 0, 1), (3, 0, 2), (1, 0, 17)]), at((0, 40), (0, 1), (0, 2), (0, 17)), dtype, 1e-4, 3e-2)
    _close(a.run(st, [(0, 1, 1), (3, 2, 1), (2, 40, 1)]), at((1, 1), (2, 1), (40, 1)), dtype, 1e-4, 3e-2)
    _close(a.run(st, [(1, 17, 1), (0, 2, 50), (3, 3, 3)]), at((17, 1), (2, 50), (3, 3)), dtype, 1e-4, 3e-2)
