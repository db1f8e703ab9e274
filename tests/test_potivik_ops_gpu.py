"""The operators behind the Potivik family on the GPU, each against its plain restatement, in bf16 and in true fp32."""

import pytest
import torch
import torch.nn.functional as F

import potivik_plain as plain

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


# ---------------------------------------------------------------------------------------------- rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,cols", [(100, 104), (1500, 1504), (2600, 2600), (5000, 5008), (9000, 9000)])
def test_norms_before_and_after_a_sublayer(dev, dtype, n, cols):
    """x takes in the normed delta in fp32, the next norm reads the sum; every kind of norm on either side; padded columns stay zero.
    The mean of the rows is far from zero, so a layer norm that is not centred shows."""
    from dgpp_b200.ops import mixers as mx

    g, rows, eps = _gen(n), 3, 1e-3
    pad = lambda t: F.pad(t, (0, cols - n))
    x0, d = torch.randn(rows, n, generator=g) + 3, torch.randn(rows, n, generator=g) - 2
    wa, wb = 1 + 0.3 * torch.randn(n, generator=g), 1 + 0.3 * torch.randn(n, generator=g)
    kinds = {None: lambda v, w: v, "rms": lambda v, w: plain.rms(v, eps) * w.double(), "layer": lambda v, w: plain.layer_norm(v, eps) * w.double()}
    out = torch.empty(rows, cols, dtype=dtype, device=dev)
    dev_w = [pad(w).to(dev) for w in (wa, wb)]
    for post in kinds:
        for pre in kinds:
            x = pad(x0).to(dev)
            mx.stream_norm(x, n, eps, out, pad(d).to(dev), (post, dev_w[0] if post else None), (pre, dev_w[1] if pre else None))
            s = x0.double() + kinds[post](d.double(), wa)
            _close(x[:, :n], s, torch.float32, 1e-6)
            _close(out[:, :n], kinds[pre](s, wb), dtype, 2e-6, 5e-3)
            assert x[:, n:].abs().sum() == 0 and out[:, n:].abs().sum() == 0
    x = pad(x0).to(dev)
    mx.stream_norm(x, n, eps, out, None, (None, None), ("layer", dev_w[1]))
    assert torch.equal(x, pad(x0).to(dev))
    _close(out[:, :n], kinds["layer"](x0.double(), wb), dtype, 2e-6, 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_expert_rows_enter_the_stream(dev, dtype):
    from dgpp_b200.ops import mixers as mx

    g, rows, n, top = _gen(2), 5, 104, 3
    y, sh = (torch.randn(20, n, generator=g)).to(dtype), torch.randn(rows, n, generator=g).to(dtype)
    pair, gate = torch.randint(0, 20, (rows * top,), generator=g, dtype=torch.int32), torch.randn(rows, 6, generator=g)
    x0, w = torch.randn(rows, n, generator=g), torch.randn(n, generator=g)
    out = torch.empty(rows, n, dtype=dtype, device=dev)
    routed = y.double()[pair.long()].view(rows, top, n).sum(1)
    for shared in (False, True):
        m = mx.MoeDelta(y.to(dev), pair.to(dev), top, *((sh.to(dev), gate.to(dev)[:, 2:]) if shared else ()))
        x = x0.to(dev)
        mx.stream_norm(x, n, 1e-5, out, m, ("layer", w.to(dev)), (None, None))
        d = routed + (plain.sigmoid(gate[:, 2:3].double()) * sh.double() if shared else 0)
        want = x0.double() + plain.layer_norm(d, 1e-5) * w.double()
        _close(x, want, torch.float32, 2e-6)
        _close(out, want, dtype, 2e-6, 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gate_then_norm_by_parts(dev, dtype):
    """Parts that are no multiple of four columns, one part, a part per column; columns behind the last are cleared."""
    from dgpp_b200.ops import mixers as mx

    g, rows = _gen(3), 4
    for n, parts in ((120, 5), (132, 6), (132, 44), (288, 1), (30, 30), (4096, 8), (9000, 1)):
        y, z, w = torch.randn(rows, n, generator=g) * 2, torch.randn(rows, n + 11, generator=g).to(dtype), torch.randn(n, generator=g)
        z = F.pad(z, (0, (-z.shape[1]) % 8))
        y[:, :n // 2] *= 8                                                  # parts of unlike size
        out = torch.full((rows, (n + 7) // 8 * 8 + 8), 9.0, dtype=dtype, device=dev)
        mx.gated_part_norm(y.to(dev), z.to(dev)[:, 8:], w.to(dev), out, parts, 1e-2)
        _close(out[:, :n], plain.gated_part_norm(y.double(), z[:, 8:8 + n].double(), parts, w.double(), 1e-2), dtype, 2e-6, 5e-3)
        assert out[:, n:].abs().sum() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_activation(dev, dtype):
    """Values on both sides of both limits; the row factor acts before the clamps; dead tiles are left alone; fp32 input."""
    from dgpp_b200.ops import mixers as mx

    g, rows, inter, limit = _gen(4), 8, 72, 1.3
    gu, rw = torch.randn(rows, 2 * inter + 8, generator=g) * 3, torch.rand(rows, generator=g)

    def want(a, s):
        gate, up = (a[:, k * inter:(k + 1) * inter].double() * s for k in (0, 1))
        gate, up = gate.clamp(max=limit), up.clamp(-limit, limit)
        return gate * plain.sigmoid(1.702 * gate) * (up + 1)

    for t in {dtype, torch.float32}:
        a = gu.to(t)
        _close(mx.clamped_glu(a.to(dev), torch.empty(rows, inter, dtype=dtype, device=dev), limit), want(a, 1), dtype, 2e-6, 5e-3)
    a = gu.to(dtype)
    tiles = torch.tensor([3, -1, 0, -1], dtype=torch.int32, device=dev)
    out = torch.full((rows, inter), 5.0, dtype=dtype, device=dev)
    mx.clamped_glu(a.to(dev), out, limit, row_w=rw.to(dev), tiles=tiles, bn=2)
    live = [0, 1, 4, 5]
    _close(out[live], want(a, rw.double()[:, None])[live], dtype, 2e-6, 5e-3)
    assert (out[[2, 3, 6, 7]] == 5).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_token_gate_and_softcap(dev, dtype):
    from dgpp_b200.ops import mixers as mx

    g, rows, dim, layers = _gen(5), 6, 24, 3
    table, gate = torch.randn(11, layers * dim, generator=g).to(dtype), torch.randn(rows, dim, generator=g) * 2
    ids = torch.tensor([0, 10, 4, 4, 1, 9], dtype=torch.int32)
    for i in range(layers):
        out = mx.token_gate(gate.to(dev), ids.to(dev), table.to(dev), i * dim, torch.empty(rows, dim, dtype=dtype, device=dev))
        _close(out, plain.gelu_tanh(gate.double()) * table.double()[ids.long(), i * dim:(i + 1) * dim], dtype, 2e-6, 5e-3)
    x = torch.randn(7, 333, generator=g) * 30
    _close(mx.softcap(x.to(dev), 12.5), 12.5 * torch.tanh(x.double() / 12.5), torch.float32, 1e-6)


# ---------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("experts,top", [(1, 1), (7, 2), (16, 16), (33, 5), (200, 8), (512, 3)])
def test_routing_small_and_sorted(dev, experts, top):
    """Both routes pick the experts with the largest scores, put every pair into a tile of its expert, and leave its weight there."""
    from dgpp_b200.ops import core as ops, mixers as mx

    g = _gen(experts)
    i32 = dict(dtype=torch.int32, device=dev)
    for rows in (1, 3, 16, 17, 90):
        logits = torch.randn(rows, experts + 5, generator=g) * 2
        if experts > 2 and top < experts:
            logits[0, :experts] = logits[0, 0]                             # ties go to the lower ids
        score = plain.sigmoid(logits[:, :experts].double())
        best = torch.argsort(-score, dim=-1, stable=True)[:, :top].sort(-1).values
        small = rows <= mx.SMALL_TOKENS
        bn = 16
        nt = min(experts, rows * top) + (0 if small else rows * top // bn)
        pair, tiles, row_w = torch.full((rows * top,), -7, **i32), torch.full((nt,), -7, **i32), torch.zeros(nt * bn, device=dev)
        if small:
            mx.moe_route_small(logits.to(dev), experts, top, pair, tiles, row_w)
        else:
            ids, wts = torch.empty(rows, top, **i32), torch.empty(rows, top, device=dev)
            mx.moe_select(logits.to(dev), experts, top, ids, wts)
            ops.moe_segment_sort(ids, bn, nt, 0, experts, pair, tiles, torch.empty(1, **i32))
            x = torch.randn(rows, 24, generator=g)
            xs = torch.zeros(nt * bn, 24, device=dev)
            mx.moe_scatter_rows(x.to(dev), pair, wts, xs, row_w, top)
            assert torch.equal(xs.cpu()[pair.long().cpu()], x.repeat_interleave(top, 0))
        pair, tiles, row_w = pair.cpu().long(), tiles.cpu().long(), row_w.cpu()
        assert torch.equal(tiles[pair // bn].view(rows, top), best) and len(set(pair.tolist())) == rows * top
        _close(row_w[pair], score.gather(1, best).reshape(-1), torch.float32, 1e-6)
        if small:
            used = sorted(set(best.flatten().tolist()))
            assert tiles.tolist() == used + [-1] * (nt - len(used)) and (pair % 16 == torch.arange(rows).repeat_interleave(top)).all()
            assert int((row_w != 0).sum()) == rows * top


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bn", [16, 32, 64, 128])
def test_grouped_linear(dev, dtype, bn):
    """Widths that end inside a tile (the next expert's rows follow), K beyond one block and no multiple of it, dead tiles, shared rows."""
    from dgpp_b200.ops import core as ops, mixers as mx

    if dtype == torch.float32 and bn > 64:
        pytest.skip("fp32 tiles have at most 64 rows")
    g = _gen(bn)
    for n, k, experts in ((72, 40, 3), (256, 200, 5), (136, 520, 2)):
        w = torch.randn(experts * n, k, generator=g).to(dtype)
        tiles = torch.tensor([experts - 1, 0, -1, experts - 1, 1 % experts], dtype=torch.int32)
        x = torch.randn(5 * bn, k, generator=g).to(dtype)
        out = torch.full((5 * bn, n), 3.0, dtype=dtype, device=dev)
        mx.grouped_linear(x.to(dev), w.to(dev), n, tiles.to(dev), bn, out)
        for t, e in enumerate(tiles.tolist()):
            rows = slice(t * bn, (t + 1) * bn)
            if e < 0:
                assert (out[rows] == 3).all()
            else:
                _close(out[rows], x[rows].double() @ w[e * n:(e + 1) * n].double().T, dtype, 2e-6, 5e-3)
        few = x[:bn - 3]
        mx.grouped_linear(few.to(dev), w.to(dev), n, tiles.to(dev), bn, out, shared_rows=True)
        for t, e in enumerate(tiles.tolist()):
            if e >= 0:
                _close(out[t * bn:(t + 1) * bn - 3], few.double() @ w[e * n:(e + 1) * n].double().T, dtype, 2e-6, 5e-3)
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top,shared", [(6, 2, True), (9, 1, False), (4, 4, True)])
def test_expert_block(dev, dtype, experts, top, shared):
    """The whole block at every kind of row count; the routing weight acts on the input: with limits this tight an output weight
    would be far off.  Scores are spread, so 16-bit rounding moves no choice."""
    from dgpp_b200.models.row_moe import RowExperts, RowExpertsScratch, run_experts
    from dgpp_b200.ops import core as ops, mixers as mx
    from dgpp_b200.quant.formats import QuantLinear

    g, H, ff, fs, limit = _gen(experts), 128, 40, 24, 0.8
    rnd = lambda *s: (torch.randn(*s, generator=g) * s[-1] ** -0.5 * 1.5).to(torch.bfloat16)
    w = {f"e{e}.{n}": rnd(*s) for e in range(experts) for n, s in (("gate", (ff, H)), ("up", (ff, H)), ("down", (H, ff)))}
    w.update({"shared.gate": rnd(fs, H), "shared.up": rnd(fs, H), "shared.down": rnd(H, fs), "shared.sg": rnd(1, H)})
    basis = torch.linalg.qr(torch.randn(H, H, generator=g))[0]
    w["router"] = (basis[:experts] * 2).to(torch.bfloat16)
    lin = lambda t: QuantLinear("fp32" if dtype == torch.float32 else "bf16", *t.shape, t.to(dtype).to(dev).contiguous())
    pad8 = lambda t: F.pad(t, (0, 0, 0, -t.shape[0] % 8))
    first = [pad8(w["router"])] + ([pad8(w["shared.sg"]), w["shared.gate"], w["shared.up"]] if shared else [])
    e8 = (experts + 7) // 8 * 8
    kw = dict(sg_col=e8, shared_col=e8 + 8, shared_ff=fs, shared_limit=0.5, shared_down=lin(w["shared.down"])) if shared else {}
    cat = lambda names: torch.cat([w[f"e{e}.{n}"] for e in range(experts) for n in names]).to(dtype).to(dev).contiguous()
    b = RowExperts(experts, top, ff, limit, lin(torch.cat(first)), cat(("gate", "up")), cat(("down",)), H, **kw)
    s = RowExpertsScratch([b], 300, dtype, dev)
    c = {"router": {"top": top}, "expert": {"limit": limit}, "shared": {"limit": 0.5} if shared else None}
    for rows in (1, 5, 16, 17, 64, 300):
        order = torch.stack([torch.randperm(experts, generator=g) for _ in range(rows)]).float() - experts / 2
        x = order @ basis[:experts] * 0.5 + 0.5 * torch.randn(rows, H - experts, generator=g) @ basis[experts:]
        x = x.to(dtype)
        out = torch.empty(rows, H, dtype=dtype, device=dev)
        acc = torch.zeros(rows, H, device=dev)
        mx.stream_norm(acc, H, 1e-5, out, run_experts(b, s, x.to(dev)), (None, None), (None, None))
        want = plain.experts(x.double(), "", c, {k: v.double() for k, v in w.items()})
        _close(acc, want, dtype, 1e-5, 1.5e-2)
    ops.check_status()


# ---------------------------------------------------------------------------------------------- state space
class StateRig:
    """One state-space block; projection rows are made from x, B, C, raw steps directly."""

    def __init__(self, dev, dtype, heads, groups, vdim, state, taps, slots=3, seed=0, A=(-2.0, 2.0), dt=(-4.0, 1.0)):
        from dgpp_b200.ops import mixers as mx

        g = _gen(seed)
        self.mx, self.dev, self.dtype, self.heads, self.groups, self.vdim, self.N, self.taps = mx, dev, dtype, heads, groups, vdim, state, taps
        uni = lambda n, lo, hi: lo + (hi - lo) * torch.rand(n, generator=g)
        inner, gn = heads * vdim, groups * state
        self.conv, self.conv_b = torch.randn(inner + 2 * gn, taps, generator=g) * 0.7, torch.randn(inner + 2 * gn, generator=g) * 0.3
        self.A_log, self.dt_bias, self.D = uni(heads, *A), uni(heads, *dt), torch.randn(heads, generator=g)
        conv = torch.cat([self._channels(self.conv.T), self._channels(self.conv_b[None])])
        d = lambda t: t.contiguous().to(dev)
        K, V = mx.pad_to(state, mx.STATE_WIDTHS), mx.pad_to(vdim, mx.STATE_WIDTHS)
        self.C = 2 * groups * K + heads * V
        self.s = mx.StateHeads(heads, groups, state, vdim, 8, 8 + self.C, 1e-5, d(conv[:taps]), d(self.A_log), d(self.dt_bias), conv_b=d(conv[taps]), skip=d(self.D))
        assert self.s.channels == self.C
        self.state, self.ring = self.s.new_state(slots, dev)
        self.state.fill_(float("nan"))                                     # a request's first token clears nothing by itself
        self.ring.fill_(float("nan"))
        self.at = [0] * slots

    def _channels(self, t):
        """[n, x | B | C] -> [n, C | B | x], padded per head and group."""
        mx, n, inner, gn = self.mx, t.shape[0], self.heads * self.vdim, self.groups * self.N
        pad = lambda a, h, w: F.pad(a.reshape(n, h, -1), (0, mx.pad_to(w, mx.STATE_WIDTHS) - w)).reshape(n, -1)
        x, B, C = t.split([inner, gn, gn], -1)
        return torch.cat([pad(C, self.groups, self.N), pad(B, self.groups, self.N), pad(x, self.heads, self.vdim)], -1)

    def random(self, n, seed):
        g = _gen(seed)
        return torch.randn(n, self.conv.shape[0], generator=g).to(self.dtype), torch.randn(n, self.heads, generator=g).to(self.dtype)

    def want(self, xbc, dt):
        T = xbc.shape[0]
        a = plain.causal_conv(xbc.double(), self.conv.double(), self.conv_b.double())
        x, B, C = a.split([self.heads * self.vdim, self.groups * self.N, self.groups * self.N], -1)
        y = plain.state_space(x.view(T, self.heads, -1), B.view(T, self.groups, -1), C.view(T, self.groups, -1),
                              plain.softplus(dt.double() + self.dt_bias.double()), self.A_log.double(), self.D.double())
        return y.reshape(T, -1)

    def run(self, batch, decode=False):
        """batch: [(slot, xbc, dt)] next tokens -> outputs."""
        from dgpp_b200.models.rows import RowRuns

        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=self.dev)
        lens, slots = [b[1].shape[0] for b in batch], [b[0] for b in batch]
        start = [0]
        for n in lens:
            start.append(start[-1] + n)
        pos = i32([self.at[s] + k for s, n in zip(slots, lens) for k in range(n)])
        row_slot = i32([s for s, n in zip(slots, lens) for _ in range(n)])
        run0 = i32([a for a, n in zip(start, lens) for _ in range(n)])
        body = torch.cat([torch.cat([self._channels(x), F.pad(d, (0, -d.shape[1] % 8))], 1) for _, x, d in batch])
        proj = F.pad(body, (8, 0)).to(self.dtype).to(self.dev)
        o = torch.full((start[-1], self.heads * self.vdim), float("nan"), device=self.dev)
        runs = None if decode else RowRuns(i32(start), run0, lens, slots, [self.at[s] for s in slots])
        prep = torch.empty(self.s.prep_floats(start[-1], len(lens)), device=self.dev)
        self.mx.linear_state(self.s, proj, self.state, self.ring, row_slot, pos, runs=runs, prep=prep, o=o)
        for s, n in zip(slots, lens):
            self.at[s] += n
        return [o[a:a + n].cpu() for a, n in zip(start, lens)]


STATES = [(4, 2, 48, 40, 4), (6, 1, 20, 24, 2), (3, 3, 64, 128, 3), (1, 1, 8, 8, 1), (20, 2, 16, 64, 4), (2, 1, 130, 200, 6)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", STATES)
def test_state_space_portions_and_decoding(dev, dtype, shape):
    rig, n = StateRig(dev, dtype, *shape), 100
    xbc, dt = rig.random(n, 1)
    want = rig.want(xbc, dt)
    for sizes in ([n], [2, 3, 16, 17, 31, 2, 29], [1] * 5 + [33, 1, 1, 60], [1] * 40 + [2] * 30):
        got, o = [], 0
        for s in sizes:
            got += rig.run([(1, xbc[o:o + s], dt[o:o + s])], decode=s == 1)
            o += s
        _close(torch.cat(got), want, torch.float32, 2e-5)                  # bf16 inputs are exact here: the recurrence itself is fp32
        rig.at[1] = 0


@pytest.mark.parametrize("A,dt", [((3.0, 5.0), (2.0, 4.0)), ((-9.0, -7.0), (-6.0, -4.0)), ((-1.0, 1.0), (15.0, 25.0))])
def test_state_space_extreme_decays(dev, A, dt):
    """Memories of a fraction of a token, of thousands of tokens, and steps where softplus is the identity."""
    rig, n = StateRig(dev, torch.float32, 4, 2, 32, 32, 4, A=A, dt=dt), 400
    xbc, raw = rig.random(n, 2)
    want = rig.want(xbc, raw)
    got = rig.run([(0, xbc[:250], raw[:250])]) + [rig.run([(0, xbc[t:t + 1], raw[t:t + 1])], decode=True)[0] for t in range(250, n)]
    _close(torch.cat(got), want, torch.float32, 3e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_space_unequal_batches_and_reused_slots(dev, dtype):
    """Runs of unlike lengths of several requests in one pass, single tokens beside them, slots taken over by other requests."""
    rig = StateRig(dev, dtype, 6, 3, 40, 24, 4)
    data = [rig.random(120, 10 + i) for i in range(4)]
    want = [rig.want(*d) for d in data]
    at = [0] * 4
    slot = {0: 0, 1: 1, 2: 2}

    def step(parts, decode=False):
        batch = [(slot[i], data[i][0][at[i]:at[i] + n], data[i][1][at[i]:at[i] + n]) for i, n in parts]
        for (i, n), o in zip(parts, rig.run(batch, decode)):
            _close(o, want[i][at[i]:at[i] + n], torch.float32, 2e-5)
            at[i] += n

    for parts in ([(0, 50), (1, 2)], [(0, 1), (2, 1), (1, 1)], [(2, 33), (0, 1), (1, 16)], [(1, 1), (0, 17)]):
        step(parts, decode=all(n == 1 for _, n in parts))
    slot[3] = slot.pop(0)
    rig.at[slot[3]] = 0
    for parts in ([(3, 1), (1, 1)], [(3, 20), (2, 2)], [(3, 1)], [(3, 80), (1, 1), (2, 40)]):
        step(parts, decode=all(n == 1 for _, n in parts))


# ---------------------------------------------------------------------------------------------- latent attention
class LatentRig:
    """One latent-attention block over a paged cache whose pages are handed out in a scrambled order."""

    def __init__(self, dev, dtype, heads, dim, rot_dim, vdim, rank, window, scale, base=10000.0, rot=None, max_tokens=512, page=64, reqs=3, seed=0):
        from dgpp_b200.engine.kv_cache import PagedKV
        from dgpp_b200.ops import mixers as mx

        self.mx, self.dev, self.dtype, self.window, self.scale, self.eps, self.base = mx, dev, dtype, window, scale, 1e-4, base
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank, self.page = heads, dim, rot_dim, vdim, rank, page
        self.rot = rot_dim if rot is None else rot
        DN, DV, KC, RP = mx.latent_widths(dim, rot_dim, vdim, rank)
        g = _gen(seed)
        self.norm_w = 1 + 0.2 * torch.randn(rank, generator=g)
        self.uk = (torch.randn(heads * dim, rank, generator=g) * rank ** -0.5 * 1.3).to(torch.bfloat16)
        self.uv = (torch.randn(heads * vdim, rank, generator=g) * rank ** -0.5 * 1.3).to(torch.bfloat16)
        pad = lambda w, n, npad: F.pad(F.pad(w.float().view(heads, n, rank), (0, 0, 0, npad - n)).reshape(heads * npad, rank), (0, KC - rank))
        self.w_up = torch.cat([pad(self.uk, dim, DN), pad(self.uv, vdim, DV)]).to(dtype).to(dev).contiguous()
        q_cols = heads * (DN + RP)
        self.g = mx.LatentHeads(heads, dim, rot_dim, vdim, rank, window, scale, self.eps, base, self.rot, 8, 8 + q_cols, 8 + q_cols + KC + RP,
                                self.norm_w.to(dev), self.w_up)
        self.cols = 8 + q_cols + KC + RP + (heads + 7) // 8 * 8
        per = max_tokens // page
        self.kv = PagedKV(1, 0, 0, reqs * per, reqs, per, page, False, dev, shapes=[(1, KC + RP, 0)], dtype=dtype)
        order = torch.randperm(reqs * per, generator=_gen(seed + 9)).tolist()
        for _ in order:
            self.kv.alloc.alloc()
        for b in order:
            self.kv.alloc.release(b)
        self.at = [0] * reqs

    def random(self, n, seed):
        """q [n, H, dim + rot_dim], down [n, rank + rot_dim], gates [n, H]"""
        g = _gen(seed)
        return (torch.randn(n, self.heads, self.dim + self.rot_dim, generator=g).to(self.dtype),
                torch.randn(n, self.rank + self.rot_dim, generator=g).to(self.dtype), torch.randn(n, self.heads, generator=g).to(self.dtype))

    def parts(self, q, down, first=0):
        q, down, T = q.double(), down.double(), q.shape[0]
        lat = plain.rms(down[:, :self.rank], self.eps) * self.norm_w.double()
        kr = plain.rotate_pairs(down[:, self.rank:], self.base, self.rot, first)
        k = torch.cat([(lat @ self.uk.double().T).view(T, self.heads, self.dim), kr[:, None].expand(T, self.heads, self.rot_dim)], -1)
        qq = torch.cat([q[:, :, :self.dim], plain.rotate_pairs(q[:, :, self.dim:], self.base, self.rot, first)], -1)
        return qq, k, (lat @ self.uv.double().T).view(T, self.heads, self.vdim)

    def want(self, q, down, gate, first=0):
        out = plain.window_attention(*self.parts(q, down, first), self.scale, self.window)
        return out * plain.sigmoid(gate.double())[:, :, None]

    def rows(self, q, down, gate):
        g, n = self.g, q.shape[0]
        qp = torch.cat([F.pad(q[:, :, :self.dim], (0, g.DN - self.dim)), F.pad(q[:, :, self.dim:], (0, g.RP - self.rot_dim))], -1).reshape(n, -1)
        body = torch.cat([qp, F.pad(down[:, :self.rank], (0, g.KC - self.rank)), F.pad(down[:, self.rank:], (0, g.RP - self.rot_dim)),
                          F.pad(gate, (0, -self.heads % 8))], 1)
        return F.pad(body, (8, 0)).to(self.dtype).to(self.dev).contiguous()

    def run(self, batch, how, splits=1):
        """batch: [(request, q, down, gate)] next tokens; how: "fused" (single tokens), "absorbed", "expanded", or "both" (runs of at
        most 8 tokens absorbed by list, the others expanded)."""
        mx, g, page = self.mx, self.g, self.page
        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=self.dev)
        lens, reqs = [b[1].shape[0] for b in batch], [b[0] for b in batch]
        start = [0]
        for r, n in zip(reqs, lens):
            assert self.kv.reserve(r, self.at[r] + n)
            start.append(start[-1] + n)
        pos, req = i32([self.at[r] + k for r, n in zip(reqs, lens) for k in range(n)]), i32([r for r, n in zip(reqs, lens) for _ in range(n)])
        x = torch.cat([self.rows(*b[1:]) for b in batch])
        rows, bt, cache = x.shape[0], self.kv.block_table, self.kv.layers[0].k
        out = torch.full((rows, self.heads * g.DV), 7.0, dtype=self.dtype, device=self.dev)

        def absorbed(n, row_list, fused):
            q_abs = torch.empty(n * self.heads * g.cache_cols, device=self.dev)
            lat = torch.empty(n * self.heads * g.KC, device=self.dev)
            scratch = (torch.empty(n * self.heads * splits * 2, device=self.dev), torch.empty(n * self.heads * splits * g.KC, device=self.dev))
            mx.latent_absorb(g, x, pos, req, bt, cache, page, q_abs, n, row_list, fused)
            mx.latent_attn(g, q_abs, cache, bt, req, pos, page, lat, n, row_list, splits, scratch)
            mx.latent_up(g, lat, x, out, n, row_list)

        if how == "fused":
            absorbed(rows, None, True)
        else:
            mx.latent_append(g, x, pos, req, bt, cache, page)
            long = [] if how == "absorbed" else [r for r, n in enumerate(lens) if how == "expanded" or n > 8]
            short = [start[r] + k for r, n in enumerate(lens) if r not in long for k in range(n)]
            if long:
                base, pages = [], []
                for r in long:
                    first = max(0, self.at[reqs[r]] + 1 - self.window) // page
                    base.append((len(pages) - first) * page)
                    pages += self.kv.req_blocks[reqs[r]][first:(self.at[reqs[r]] + lens[r] - 1) // page + 1]
                from dgpp_b200.ops import core as ops
                from dgpp_b200.quant.formats import QuantLinear
                got = mx.latent_gather(cache, i32(pages), torch.empty(len(pages) * page, g.cache_cols, dtype=self.dtype, device=self.dev), page)
                flat = ops.linear(got[:, :g.KC], QuantLinear("bf16", g.flat_cols, g.KC, self.w_up))
                lr = mx.LatentRuns(i32([start[r] for r in long]), i32([lens[r] for r in long]), i32(base), i32(pages), sum(-(-lens[r] // 128) for r in long))
                mx.latent_prefill(g, x, flat, got, req, pos, lr, out)
            if short:
                absorbed(len(short), i32(short) if long else None, False)
        res = []
        for a, r, n in zip(start, reqs, lens):
            y = out[a:a + n].view(n, self.heads, g.DV)
            assert self.vdim == g.DV or y[:, :, self.vdim:].abs().sum().item() == 0
            res.append(y[:, :, :self.vdim].float().cpu())
            self.at[r] += n
        return res

    def release(self, r):
        self.kv.release(r)
        self.at[r] = 0

    def hows(self):
        return ["absorbed"] + (["expanded"] if self.g.tc_runs(self.dtype) else [])


#          heads dim rot vdim rank window scale
LATENTS = [(6, 32, 16, 40, 64, 48, 0.15), (5, 24, 10, 72, 52, 17, 0.3), (20, 64, 64, 128, 200, 100, 0.09), (3, 128, 32, 64, 300, 70, 0.07),
           (2, 16, 2, 16, 16, 1, 1.0), (16, 128, 64, 128, 512, 200, 0.07), (3, 40, 80, 30, 520, 33, 0.1), (1, 200, 48, 260, 128, 129, 0.06)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LATENTS)
def test_latent_attention_portions_and_decoding(dev, dtype, shape):
    from dgpp_b200.ops import core as ops

    rig, n = LatentRig(dev, dtype, *shape), 220
    q, down, gate = rig.random(n, 3)
    want = rig.want(q, down, gate)
    part = lambda a, b: (q[a:b], down[a:b], gate[a:b])
    for how in rig.hows():
        for sizes, splits in (([n], 1), ([2, 130, 61], 1), ([3] + [1] * 40 + [9, 90], 3)):
            got, o = [], 0
            for s in sizes + [1] * (n - sum(sizes)):
                got += rig.run([(1, *part(o, o + s))], "fused" if s == 1 else how, splits if s == 1 else 1)
                o += s
            _close(torch.cat(got), want, dtype, 1e-5, 1.5e-2)
            rig.release(1)
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,page", [(48, 64), (64, 64), (129, 64), (1, 64), (200, 64), (50, 16)])
def test_a_latent_that_stands_out_is_seen_just_inside_the_window_only(dev, dtype, window, page):
    """Every query asks for one token's key so loudly that it takes the whole softmax: its value is the output while it is at most
    window - 1 tokens back, and leaves no trace one token later, for prompt rows and decoded rows alike."""
    n = window + page + 60
    for at in (0, page - 1, page, 7):                                      # the key's place: first token, around a page border
        rig = LatentRig(dev, dtype, 4, 64, 16, 32, 128, window, 0.5, base=1e7, page=page, seed=at)
        q, down, gate = rig.random(n, at)
        down[:, rig.rank:] *= 0.02                                         # the rotated part stays out of the way
        q[:, :, rig.dim:] *= 0.02
        lat = plain.rms(down[at:at + 1, :rig.rank].double(), rig.eps) * rig.norm_w.double()
        key = (lat @ rig.uk.double().T).view(rig.heads, rig.dim)
        q[:, :, :rig.dim] = (key / key.norm(dim=-1, keepdim=True) * 14).to(dtype)
        gate[:] = 4.0
        want = rig.want(q, down, gate)
        value = (lat @ rig.uv.double().T).view(rig.heads, rig.vdim)
        near = lambda rows: ((rows - value).norm(dim=-1) / value.norm(dim=-1)).flatten()
        assert (near(want[at:at + window]) < 0.05).all() and (near(want[at + window:]) > 0.3).all()
        edge = at + window
        for how in (rig.hows() if page == 64 else ["absorbed"]) + ["fused"]:
            sizes = [s for s in ([edge - 3, 1, 1, 1, 1, 1] if how == "fused" else [max(1, edge - 20), 40]) if s > 0]
            got, o = [], 0
            for s in sizes:
                mode = "fused" if s == 1 else ("absorbed" if how == "fused" else how)
                got += rig.run([(0, q[o:o + s], down[o:o + s], gate[o:o + s])], mode, 2 if s == 1 else 1)
                o += s
            _close(torch.cat(got), want[:o], dtype, 2e-5, 3e-2)            # (scores near 70: the rounding of a 16-bit key shows)
            rig.release(0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_in_unequal_batches_with_reused_pages(dev, dtype):
    """Portions of several requests in one pass, single tokens and short runs beside them, requests that end and others that take over
    their pages: each request gets what it gets alone."""
    rig = LatentRig(dev, dtype, 6, 40, 24, 64, 96, 71, 0.2, max_tokens=320)
    data = [rig.random(300, 10 + i) for i in range(4)]
    want = [rig.want(*d) for d in data]
    mixed = "both" if rig.g.tc_runs(dtype) else "absorbed"
    at, req = [0] * 4, {0: 0, 1: 1, 2: 2}

    def step(parts):
        how = "fused" if all(n == 1 for _, n in parts) else mixed
        outs = rig.run([(req[i], *(t[at[i]:at[i] + n] for t in data[i])) for i, n in parts], how, 2 if how == "fused" else 1)
        for (i, n), o in zip(parts, outs):
            _close(o, want[i][at[i]:at[i] + n], dtype, 1e-5, 1.5e-2)
            at[i] += n

    for parts in ([(0, 150), (1, 3)], [(0, 1), (1, 130), (2, 2)], [(0, 1), (1, 1), (2, 1)], [(2, 140), (0, 2), (1, 9)], [(1, 1), (2, 70), (0, 129)]):
        step(parts)
    rig.release(req[0])
    rig.release(req[1])
    req[3] = req.pop(0)
    for parts in ([(3, 65), (2, 1)], [(3, 1), (2, 1)], [(3, 200), (2, 8)], [(2, 70), (3, 1)]):
        step(parts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_of_far_positions_and_partial_rotation(dev, dtype):
    """Neighbouring pairs turn by position * base^(-2 i / dims) also far out; columns behind the rotated ones pass unchanged."""
    first = 100_000
    for rot in (20, 12, 0):
        rig = LatentRig(dev, dtype, 2, 16, 20, 16, 32, 24, 0.25, base=50.0, rot=rot, max_tokens=first + 192, reqs=1)
        q, down, gate = rig.random(90, 4)
        q[:, :, :rig.dim] *= 0.1                                           # the rotated part decides
        want = rig.want(q, down, gate, first)
        assert rig.kv.reserve(0, first)
        rig.at[0], o, got = first, 0, []
        for s in (60, 1, 1, 28):
            got += rig.run([(0, q[o:o + s], down[o:o + s], gate[o:o + s])], "fused" if s == 1 else rig.hows()[-1])
            o += s
        _close(torch.cat(got)[rig.window:], want[rig.window:], dtype, 3e-5, 2e-2)
        if dtype == torch.float32 and rot == 20:
            _close(torch.cat(got)[rig.window:], rig.want(q, down, gate, 7)[rig.window:], dtype, 3e-5)     # only distances matter


def test_operators_refuse_what_they_do_not_take(dev):
    from dgpp_b200.ops import mixers as mx

    with pytest.raises(ValueError):
        StateRig(dev, torch.float32, 1, 1, 300, 16, 2)
    rig = LatentRig(dev, torch.bfloat16, 4, 32, 16, 32, 64, 20, 0.2)
    rig.g.rot = 15
    with pytest.raises(RuntimeError, match="rotated"):
        rig.run([(0, *rig.random(1, 0))], "fused")
    i32 = dict(dtype=torch.int32, device=dev)
    with pytest.raises(RuntimeError, match="moe_route_small"):
        mx.moe_route_small(torch.zeros(17, 8, device=dev), 8, 2, torch.zeros(34, **i32), torch.zeros(8, **i32), torch.zeros(128, device=dev))
    with pytest.raises(RuntimeError, match="softcap"):
        mx.softcap(torch.zeros(4, device=dev), 0.0)
