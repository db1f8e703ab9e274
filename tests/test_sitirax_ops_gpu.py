"""The operators behind the Sitirax family on the GPU, each against its plain restatement, in bf16 and in true fp32."""
import pytest
import torch

import sitirax_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def dev():
    if not torch.cuda.is_available():
        pytest.skip("needs a GPU")
    return torch.device("cuda:0")


def _tol(dtype, fine=3e-5, coarse=2e-2):
    return fine if dtype == torch.float32 else coarse


def _close(got, want, dtype, fine=3e-5, coarse=2e-2):
    want = want.double().cpu()
    err = (got.double().cpu() - want).abs().max().item()
    assert err <= _tol(dtype, fine, coarse) * (want.abs().max().item() + 1e-6), err


def _gen(seed):
    return torch.Generator().manual_seed(seed)


@pytest.mark.parametrize("dtype", DTYPES)
def test_row_operators(dev, dtype):
    from dgpp_b200.ops import mixers as mx

    g = _gen(1)
    rows, n, cols, vocab = 5, 100, 104, 37
    pad = lambda t: torch.nn.functional.pad(t, (0, cols - n))
    table = pad(torch.randn(vocab, n, generator=g)).to(dtype)
    ids = torch.tensor([0, 36, 5, 5, 11], dtype=torch.int32)
    x = mx.embed_rows(ids.to(dev), table.to(dev), torch.empty(rows, cols, device=dev))
    assert torch.equal(x.cpu(), table.float()[ids.long()])
    d, w = pad(torch.randn(rows, n, generator=g)), pad(torch.randn(1, n, generator=g))[0]
    out = mx.resid_norm(x, w.to(dev), n, 1e-3, torch.empty(rows, cols, dtype=dtype, device=dev), d.to(dev))
    s = table.float()[ids.long()] + d
    assert torch.equal(x.cpu(), s)                                    # the sum stays in fp32
    _close(out[:, :n], plain.rms(s[:, :n].double(), 1e-3) * w[:n].double(), dtype, 1e-6, 5e-3)
    assert out[:, n:].abs().max().item() == 0
    for groups, gp, true in ((3, 64, 40), (1, 192, 120)):
        o = torch.randn(rows, groups, gp, generator=g)
        if groups > 1:
            o[:, :, true:] = 0
        else:
            o.view(rows, 3, 64)[:, :, 40:] = 0
        ww, gate = torch.randn(gp, generator=g), torch.randn(rows, groups * gp + 8, generator=g).to(dtype)
        dst = torch.empty(rows, groups * gp + 16, dtype=dtype, device=dev)
        mx.gated_group_norm(o.view(rows, -1).contiguous().to(dev), gate.to(dev)[:, 8:], ww.to(dev), dst[:, 16:], groups, true, 1e-2, 0.6)
        od = o.double()
        want = od / torch.sqrt((od ** 2).sum(-1, keepdim=True) / true + 1e-2) * ww.double()
        _close(dst[:, 16:], 0.6 * want.reshape(rows, -1) * plain.sigmoid(gate[:, 8:].double()), dtype, 2e-6, 5e-3)
    gu = (torch.randn(rows, 2 * 72, generator=g) * 3).to(dtype)
    got = mx.geglu(gu.to(dev), torch.empty(rows, 72, dtype=dtype, device=dev))
    _close(got, plain.gelu_tanh(gu[:, :72].double()) * gu[:, 72:].double(), dtype, 2e-6, 5e-3)


@pytest.mark.parametrize("rows,n,k", [(1, 100, 24), (3, 320, 200), (70, 131, 104), (300, 257, 1000), (17, 128, 64)])
def test_linears_of_any_width(dev, rows, n, k):
    """bf16 weights whose K is a multiple of 8 but not of the MMA block, split K included, and the fp32 linear."""
    from dgpp_b200.ops import core as ops
    from dgpp_b200.quant.formats import QuantLinear

    g = _gen(rows)
    x, w = torch.randn(rows, k + 16, generator=g), torch.randn(n, k, generator=g)
    xb, wb = x.bfloat16(), w.bfloat16()
    want = xb[:, 8:8 + k].double() @ wb.double().T * 0.5
    q = QuantLinear("bf16", n, k, wb.to(dev), None, 0.5)
    _close(ops.gemm_tc(xb.to(dev)[:, 8:8 + k], q, out32=torch.empty(rows, n, device=dev)), want, torch.float32, 1e-5)
    _close(ops.linear(xb.to(dev)[:, 8:8 + k], q), want, torch.bfloat16, coarse=5e-3)
    if k > 64:
        _close(ops.gemm_tc(xb.to(dev)[:, 8:8 + k], q, out32=torch.empty(rows, n, device=dev), splits=2), want, torch.float32, 1e-5)
    f = QuantLinear("fp32", n, k, w.to(dev), None, 0.5)
    _close(ops.linear(x.to(dev)[:, 8:8 + k], f), x[:, 8:8 + k].double() @ w.double().T * 0.5, torch.float32, 2e-6)
    ops.check_status()


# ---------------------------------------------------------------------------------------------- window attention
class WindowRig:
    """One window-attention block over a paged cache whose pages are handed out in a scrambled order."""

    def __init__(self, dev, dtype, heads, kv, dim, vdim, window, scale, max_tokens=512, page=16, reqs=3, sharp=1.0, seed=0):
        from dgpp_b200.engine.kv_cache import PagedKV
        from dgpp_b200.ops import mixers as mx

        self.mx, self.dev, self.dtype, self.heads, self.kvh, self.dim, self.vdim = mx, dev, dtype, heads, kv, dim, vdim
        self.window, self.scale, self.eps = window, scale, 1e-5
        D, DV = mx.pad_to(dim, mx.ATTN_WIDTHS), mx.pad_to(vdim, mx.ATTN_WIDTHS)
        off = [8, 8 + heads * D, 8 + (heads + kv) * D]
        self.g = mx.WindowHeads(heads, kv, dim, vdim, window, scale, self.eps, *off)
        self.cols = off[2] + kv * DV
        per = max_tokens // page
        self.kv = PagedKV(1, 0, 0, reqs * per, reqs, per, page, False, dev, shapes=[(kv, D, DV)], dtype=dtype)
        order = torch.randperm(reqs * per, generator=_gen(seed + 9)).tolist()
        for i in order:                                   # scramble the free list
            self.kv.alloc.alloc()
        for b in order:
            self.kv.alloc.release(b)
        g = _gen(seed)
        self.wq = (1 + 0.2 * torch.randn(dim, generator=g)) * sharp
        self.wk = (1 + 0.2 * torch.randn(dim, generator=g)) * sharp
        vec = lambda w: torch.nn.functional.pad(w, (0, D - dim)).to(dev)
        self.wq_d, self.wk_d = vec(self.wq), vec(self.wk)
        self.lengths = [0] * reqs

    def rows(self, q, k, v):
        """[n, H, dim], [n, G, dim], [n, G, vdim] -> padded projection rows."""
        pad = lambda t, w: torch.nn.functional.pad(t, (0, w - t.shape[2])).reshape(t.shape[0], -1)
        body = torch.cat([pad(q, self.g.D), pad(k, self.g.D), pad(v, self.g.DV)], 1)
        return torch.nn.functional.pad(body, (8, 0)).to(self.dtype).to(self.dev)

    def run(self, batch, splits=1, fused=None, row_list=None, tc=True):
        """batch: [(request, q, k, v)] next tokens of every request -> [outputs [n, H, vdim]] x 0.7."""
        pos, req = [], []
        for r, q, _, _ in batch:
            n = q.shape[0]
            assert self.kv.reserve(r, self.lengths[r] + n)
            pos += range(self.lengths[r], self.lengths[r] + n)
            req += [r] * n
        x = torch.cat([self.rows(q, k, v) for _, q, k, v in batch])
        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=self.dev)
        pos, req = i32(pos), i32(req)
        fused = all(q.shape[0] == 1 for _, q, _, _ in batch) if fused is None else fused
        out = torch.zeros(x.shape[0], self.heads * self.g.DV + 8, dtype=self.dtype, device=self.dev)
        args = (self.wq_d, self.wk_d, self.kv.layers[0], self.kv.block_table, req, pos)
        if not fused:
            self.mx.qk_norm_append(self.g, x, *args)
        scratch = (torch.empty(x.shape[0] * self.heads * splits * 2, device=self.dev),
                   torch.empty(x.shape[0] * self.heads * splits * self.g.DV, device=self.dev))
        starts = [0]
        for _, q, _, _ in batch:
            starts.append(starts[-1] + q.shape[0])
        runs = type("Runs", (), dict(start=i32(starts), lens=[q.shape[0] for _, q, _, _ in batch], slots=[r for r, _, _, _ in batch],
                                     pos0=[self.lengths[r] for r, _, _, _ in batch]))
        if not fused and tc and self.mx.window_prefill_usable(self.g, x, self.kv.page):
            self.mx.window_prefill(self.g, x, *args[2:], runs, out, 0.7)
        else:
            self.mx.window_attn(self.g, x, *args, out, 0.7, fused=fused, splits=splits, scratch=scratch, row_list=row_list)
        res, o = [], 0
        for r, q, _, _ in batch:
            n = q.shape[0]
            y = out[o:o + n, :self.heads * self.g.DV].reshape(n, self.heads, self.g.DV)
            assert y[:, :, self.vdim:].abs().max().item() == 0 if self.vdim < self.g.DV else True
            res.append(y[:, :, :self.vdim].float().cpu())
            self.lengths[r] += n
            o += n
        return res

    def release(self, r):
        self.kv.release(r)
        self.lengths[r] = 0

    def want(self, q, k, v):
        r = lambda t: t.to(self.dtype).double()
        qn = plain.rms(r(q), self.eps) * self.wq.double()
        kn = plain.rms(r(k), self.eps) * self.wk.double()
        return 0.7 * plain.window_attention(qn, kn, r(v), self.scale, self.window)

    def random(self, n, seed):
        g = _gen(seed)
        return (torch.randn(n, self.heads, self.dim, generator=g), torch.randn(n, self.kvh, self.dim, generator=g),
                torch.randn(n, self.kvh, self.vdim, generator=g))


SHAPES = [(6, 2, 64, 64, 40, 0.2), (5, 1, 24, 72, 17, 0.4), (4, 4, 128, 128, 100, 0.09), (12, 1, 100, 200, 33, 0.15),
          (2, 1, 192, 64, 64, 0.1), (3, 3, 16, 136, 1, 1.0), (8, 8, 256, 256, 300, 0.06), (32, 2, 64, 128, 70, 0.1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page", [64, 16])              # pages of 64 tokens: bf16 prompt rows take the tensor-core kernel
@pytest.mark.parametrize("shape", SHAPES)
def test_window_attention_prompt_portions_and_decoding(dev, dtype, shape, page):
    rig = WindowRig(dev, dtype, *shape, page=page)
    n = 150
    q, k, v = rig.random(n, 3)
    want = rig.want(q, k, v)
    for sizes, splits in (([n], 1), ([2, 30, 61, 40], 1), ([3] + [1] * 40 + [2, 90], 3)):
        got, o = [], 0
        for s in sizes + [1] * (n - sum(sizes)):
            got += rig.run([(1, q[o:o + s], k[o:o + s], v[o:o + s])], splits=splits if s == 1 else 1)
            o += s
        _close(torch.cat(got), want, dtype, 1e-5, 1.5e-2)
        rig.release(1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,page", [(48, 16), (50, 16), (129, 64), (1, 16), (128, 64), (200, 64)])
def test_a_key_that_stands_out_is_seen_just_inside_the_window_only(dev, dtype, window, page):
    """Sharp norms make one aligned key win the softmax outright: its value is the output while it is at most window - 1
    tokens back, and leaves no trace one token later, for prompt rows and decoded rows alike."""
    n = window + page + 60
    for at in (0, page - 1, page, 7):                                # the key's place: first token, around a page border
        rig = WindowRig(dev, dtype, 4, 2, 64, 64, window, 0.25, page=page, sharp=4.0, seed=at)
        q, k, v = rig.random(n, at)
        q[:] = q[:1, :1]                                             # every query asks for the same direction
        k[at] = q[0, :1] * 3
        v[at] = 50.0
        want = rig.want(q, k, v)
        assert (want[at:at + window] > 25).all() and (want[at + window:] < 25).all() and (want[:at] < 25).all()
        for lone in (False, True):                                   # the edge in a prompt portion, and decoded
            edge = at + window
            sizes = [edge - 3, 1, 1, 1, 1, 1] if lone else [max(1, edge - 20), 40]
            sizes = [s for s in sizes if s > 0]
            got, o = [], 0
            for s in sizes:
                got += rig.run([(0, q[o:o + s], k[o:o + s], v[o:o + s])], splits=2 if s == 1 else 1)
                o += s
            _close(torch.cat(got), want[:o], dtype, 1e-5, 1.5e-2)
            rig.release(0)


@pytest.mark.parametrize("page", [64, 16])
@pytest.mark.parametrize("dtype", DTYPES)
def test_window_attention_in_unequal_batches_with_reused_pages(dev, dtype, page):
    """Portions of several requests in one pass, single tokens beside them, requests that end and others that take over their
    pages: each request gets what it gets alone."""
    rig = WindowRig(dev, dtype, 6, 3, 40, 64, 37, 0.3, max_tokens=192, page=page)
    data = [rig.random(160, 10 + i) for i in range(4)]
    want = [rig.want(*d) for d in data]
    part = lambda i, a, b: tuple(t[a:b] for t in data[i])
    plan = [[(0, 0, 50), (1, 0, 3)], [(0, 50, 51), (1, 3, 130), (2, 0, 2)], [(0, 51, 52), (1, 130, 131), (2, 2, 3)],
            [(2, 3, 140), (0, 52, 54)]]
    for step in plan:
        outs = rig.run([(r, *part(r, a, b)) for r, a, b in step], splits=2 if all(b - a == 1 for _, a, b in step) else 1)
        for (r, a, b), o in zip(step, outs):
            _close(o, want[r][a:b], dtype, 1e-5, 1.5e-2)
    rig.release(1)
    rig.release(0)
    for a, b, r0 in ((0, 70, (54, 60)), (70, 71, (60, 61)), (71, 160, (61, 62))):
        d0 = part(2, 140 + (a > 0) + (a > 70), 141 + (a > 0) + (a > 70))
        outs = rig.run([(1, *part(3, a, b)), (2, *d0)])
        _close(outs[0], want[3][a:b], dtype, 1e-5, 1.5e-2)
    # a subset of rows by list
    rig.release(1)
    full = rig.run([(1, *part(3, 0, 90))], tc=False)[0]
    rig.release(1)
    rows = torch.tensor([3, 50, 89], dtype=torch.int32, device=dev)
    some = rig.run([(1, *part(3, 0, 90))], tc=False, row_list=rows)[0]
    assert torch.equal(some[[3, 50, 89]], full[[3, 50, 89]]) and some[[0, 4, 88]].abs().max() == 0


def test_window_operators_refuse_what_they_do_not_take(dev):
    from dgpp_b200.ops import mixers as mx

    with pytest.raises(ValueError):
        mx.WindowHeads(2, 1, 300, 64, 8, 0.1, 1e-5, 0, 64, 128)
    rig = WindowRig(dev, torch.bfloat16, 4, 2, 64, 64, 8, 0.2)
    rig.g.hkv = 3
    with pytest.raises(RuntimeError, match="query heads"):
        rig.run([(0, *WindowRig(dev, torch.bfloat16, 4, 2, 64, 64, 8, 0.2).random(1, 0))], fused=True)


# ---------------------------------------------------------------------------------------------- linear-attention states
class StateRig:
    """One linear-attention block with its state slots; the rows it is given are projections, as the mixer's matrix makes
    them."""

    def __init__(self, dev, dtype, heads, kheads, dim, vdim, taps=0, decay=None, slots=3, seed=0, decay_bias=-1.0):
        from dgpp_b200.ops import mixers as mx

        self.mx, self.dev, self.dtype = mx, dev, dtype
        self.hv, self.hk, self.dim, self.vdim, self.taps = heads, kheads, dim, vdim, taps
        g = _gen(seed)
        K, V = mx.pad_to(dim, mx.STATE_WIDTHS), mx.pad_to(vdim, mx.STATE_WIDTHS)
        self.K, self.V, self.eps = K, V, 1e-4
        self.delta = decay is None
        c, b = 8, 8 + 2 * kheads * K + heads * V
        self.cols = b + (heads + 7) // 8 * 8
        if self.delta:
            self.conv = {n: 0.7 * torch.randn(h, w, taps, generator=g) for n, h, w in (("q", kheads, dim), ("k", kheads, dim), ("v", heads, vdim))}
            self.A_log = torch.rand(heads, generator=g) * 3 - 2.5
            self.dt = torch.randn(heads, dim, generator=g) + decay_bias
            self.nw = 1 + 0.3 * torch.randn(vdim, generator=g)
            pad = lambda t, w: torch.nn.functional.pad(t, (0, 0, 0, w - t.shape[1])).reshape(-1, taps)
            conv = torch.cat([pad(self.conv["q"], K), pad(self.conv["k"], K), pad(self.conv["v"], V)]).T.contiguous().to(dev)
            self.g = mx.StateHeads(heads, kheads, dim, vdim, c, b, self.eps, conv, self.A_log.to(dev),
                                   torch.nn.functional.pad(self.dt, (0, K - dim)).reshape(-1).to(dev),
                                   norm_w=torch.nn.functional.pad(self.nw, (0, V - vdim)).to(dev))
        else:
            self.decay = torch.tensor(decay)
            self.g = mx.StateHeads(heads, kheads, dim, vdim, c, eps=self.eps, decay=self.decay.to(dev))
        self.state, self.ring = self.g.new_state(slots, dev)
        self.state.fill_(7.0)                              # what an earlier request might have left
        if self.ring is not None:
            self.ring.fill_(5.0)
        self.lengths = [0] * slots

    def random(self, n, seed):
        g = _gen(seed)
        r = lambda *s: torch.randn(n, *s, generator=g)
        return dict(q=r(self.hk, self.dim), k=r(self.hk, self.dim), v=r(self.hv, self.vdim), b=r(self.hv), a=r(self.hv, self.dim),
                    gate=r(self.hv, self.vdim))

    def run(self, batch):
        """batch [(slot, inputs)] -> outputs [n, hv, vdim] per entry; single tokens for all entries take the decode kernel."""
        pad = lambda t, w: torch.nn.functional.pad(t, (0, w - t.shape[2])).reshape(t.shape[0], -1)
        x, low, pos, slot, starts = [], [], [], [], [0]
        for s, d in batch:
            n = d["q"].shape[0]
            row = torch.cat([torch.zeros(n, 8), pad(d["q"], self.K), pad(d["k"], self.K), pad(d["v"], self.V), d["b"]], 1)
            x.append(torch.nn.functional.pad(row, (0, self.cols - row.shape[1])))
            low.append(torch.cat([pad(d["a"], self.K), pad(d["gate"], self.V)], 1))
            pos += range(self.lengths[s], self.lengths[s] + n)
            slot += [s] * n
            starts.append(starts[-1] + n)
            self.lengths[s] += n
        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=self.dev)
        x, low = torch.cat(x).to(self.dtype).to(self.dev), torch.cat(low).to(self.dev)
        rows = x.shape[0]
        lens = [d["q"].shape[0] for _, d in batch]
        o = torch.zeros(rows, self.hv * self.V, device=self.dev)
        out = torch.zeros(rows, self.hv * self.V, dtype=self.dtype, device=self.dev)
        low = low if self.delta else None
        if all(n == 1 for n in lens):
            self.mx.linear_state(self.g, x, self.state, self.ring, i32(slot), i32(pos), low=low, o=o, out=out)
        else:
            runs = type("Runs", (), dict(start=i32(starts), row_run0=i32([starts[i] for i, n in enumerate(lens) for _ in range(n)]), lens=lens))
            prep = torch.empty(self.g.prep_floats(rows, len(lens)), device=self.dev)
            self.mx.linear_state(self.g, x, self.state, self.ring, i32(slot), i32(pos), low=low, runs=runs, prep=prep, o=o)
            if self.delta:
                self.mx.gated_group_norm(o, low[:, self.hv * self.K:], self.g.norm_w, out, self.hv, self.vdim, self.eps)
        y = (out if self.delta else o).float().cpu().view(rows, self.hv, self.V)
        assert self.vdim == self.V or y[:, :, self.vdim:].abs().max().item() == 0
        return [y[a:b, :, :self.vdim] for a, b in zip(starts, starts[1:])]

    def want(self, d):
        r = lambda t: t.to(self.dtype).double()
        n = d["q"].shape[0]
        if not self.delta:
            return plain.lightning(plain.silu(r(d["q"])), plain.silu(r(d["k"])), plain.silu(r(d["v"])), self.decay.double())
        conv = lambda t, name: plain.causal_conv(r(d[name]).reshape(n, -1), t[name].double().reshape(-1, self.taps)).view(d[name].shape)
        q, k, v = conv(self.conv, "q"), conv(self.conv, "k"), conv(self.conv, "v")
        g = torch.exp(-torch.exp(self.A_log.double())[:, None] * plain.softplus(d["a"].double() + self.dt.double()))
        o = plain.delta_rule(plain.unit(q) * self.dim ** -0.5, plain.unit(k), v, plain.sigmoid(r(d["b"])), g)
        return plain.rms(o, self.eps) * self.nw.double() * plain.sigmoid(d["gate"].double())


STATES = [dict(heads=4, kheads=2, dim=64, vdim=64, taps=4), dict(heads=3, kheads=1, dim=20, vdim=40, taps=2),
          dict(heads=2, kheads=2, dim=128, vdim=128, taps=1), dict(heads=2, kheads=1, dim=32, vdim=200, taps=7),
          dict(heads=1, kheads=1, dim=256, vdim=32, taps=3), dict(heads=2, kheads=2, dim=250, vdim=256, taps=4),
          dict(heads=3, kheads=3, dim=64, vdim=64, decay=(0.5, 1.0, 0.99)), dict(heads=2, kheads=2, dim=40, vdim=128, decay=(0.9, 0.0)),
          dict(heads=1, kheads=1, dim=128, vdim=24, decay=(0.999,))]


def _cut(d, a, b):
    return {k: t[a:b] for k, t in d.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", STATES, ids=str)
def test_states_in_portions_and_decoding(dev, dtype, shape):
    """One request as a whole, in portions down to two tokens, and token by token; slots are not cleared in between."""
    rig = StateRig(dev, dtype, **shape)
    n = 133
    d = rig.random(n, 4)
    want = rig.want(d)
    for sizes in ([n], [2, 3, 30, 64, 2, 32], [1, 1, 1, 2, 17, 1, 2, 1] + [16, 17]):
        rig.lengths[1] = 0
        got, o = [], 0
        for s in sizes + [1] * (n - sum(sizes)):
            got += rig.run([(1, _cut(d, o, o + s))])
            o += s
        _close(torch.cat(got), want, dtype, 2e-5, 8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [STATES[0], STATES[3], STATES[6]], ids=str)
def test_states_of_unequal_batches(dev, dtype, shape):
    rig = StateRig(dev, dtype, **shape)
    data = [rig.random(90, 20 + i) for i in range(4)]
    want = [rig.want(d) for d in data]
    for step in ([(0, 0, 40), (1, 0, 2)], [(0, 40, 41), (1, 2, 77), (2, 0, 3)], [(2, 3, 4), (0, 41, 42), (1, 77, 78)], [(1, 78, 80), (2, 4, 90)]):
        for (r, a, b), o in zip(step, rig.run([(r, _cut(data[r], a, b)) for r, a, b in step])):
            _close(o, want[r][a:b], dtype, 2e-5, 8e-3)
    rig.lengths[1] = 0                                     # slot 1 goes to another request
    for (a, b), (c, e) in (((0, 1), (42, 43)), ((1, 60), (43, 44)), ((60, 90), (44, 45))):
        outs = rig.run([(1, _cut(data[3], a, b)), (0, _cut(data[0], c, e))])
        _close(outs[0], want[3][a:b], dtype, 2e-5, 8e-3)
        _close(outs[1], want[0][c:e], dtype, 2e-5, 8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("split", [2, 150, 203, 204])
def test_a_far_write_is_still_read_from_the_state(dev, dtype, split):
    """One token writes a value under a key nobody else uses; 200 tokens later a query for that key returns it, whether the
    portions are cut between them or not.  (Slow decays; the other tokens' keys leave that channel alone.)"""
    for shape in (dict(heads=2, kheads=1, dim=64, vdim=64, taps=4), dict(heads=2, kheads=2, dim=64, vdim=64, decay=(1.0, 0.999))):
        rig = StateRig(dev, dtype, decay_bias=-9.0, **shape)
        n = 206
        d = rig.random(n, 6)
        for t in ("q", "k"):
            d[t][:, :, 11] = -40.0 if not rig.delta else 0.0          # silu(-40) = 0: the channel stays out of all other tokens
        d["k"][2, :, :] = -40.0 if not rig.delta else 0.0
        d["k"][2, :, 11] = 6.0
        d["v"][2] = 9.0
        d["b"][2] = 9.0
        for t in range(203, n):
            d["q"][t] = -40.0 if not rig.delta else 0.0
            d["q"][t, :, 11] = 6.0
        if rig.delta:
            for name in ("q", "k"):
                rig.conv[name][:, 11, :] = 0
                rig.conv[name][:, 11, -1] = 1.0
            C = torch.cat([torch.nn.functional.pad(rig.conv[nm], (0, 0, 0, w - rig.conv[nm].shape[1])).reshape(-1, rig.taps)
                           for nm, w in (("q", rig.K), ("k", rig.K), ("v", rig.V))])
            rig.g.conv_w.copy_(C.T)
        want = rig.want(d)
        alone = dict(d, v=d["v"].clone())
        alone["v"][2] = -3.0
        assert (rig.want(alone)[205] - want[205]).abs().mean() > 0.2 * want[205].abs().mean()      # the write shows
        got = []
        for a, b in ((0, split), (split, n - 1), (n - 1, n)):
            if b > a:
                got += rig.run([(0, _cut(d, a, b))])
        _close(torch.cat(got), want, dtype, 3e-5, 1e-2)
