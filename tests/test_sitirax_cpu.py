"""Sitirax family without a GPU: configuration, packing (against the plain restatement), checkpoints, the mixed pass's
bookkeeping and its engine behind the scheduler."""
import copy
import json

import pytest
import torch

import sitirax_cases as sc
import sitirax_plain as plain
from dgpp_b200.models.rows import RowRunner
from dgpp_b200.models.sitirax import SitiraxConfig, SitiraxModel
from dgpp_b200.runtime import rt


@pytest.mark.parametrize("name", sorted(sc.CONFIGS))
def test_packed_model_matches_the_plain_restatement(name):
    cfg = sc.CONFIGS[name]
    c = SitiraxConfig.from_dict(cfg)
    assert SitiraxConfig.from_dict(c.to_dict()) == c
    w = sc.tensors(cfg, 1)
    toks = sc.token_ids(cfg, 83)
    want = plain.forward(cfg, sc.doubles(w), toks)
    for dtype in (torch.float32, torch.bfloat16):
        m = SitiraxModel.from_tensors(c, w.__getitem__, "cpu", dtype)
        assert (m.forward_reference(torch.tensor(toks)) - want).abs().max() <= 3e-5 * want.abs().max()


def test_refused_configurations():
    base = sc.CONFIGS["mixed"]

    def broken(change):
        d = copy.deepcopy(base)
        change(d["layers"])
        with pytest.raises(ValueError):
            SitiraxConfig.from_dict(d)

    broken(lambda L: L[1].update(type="something_else"))
    broken(lambda L: L[0]["mlp"].update(kind="sparse"))
    broken(lambda L: L[0]["mixer"]["right"]["decay"].pop())
    broken(lambda L: L[0]["mixer"]["left"].update(kv_heads=3))
    broken(lambda L: L[3]["mixer"].update(left_scale=0.5))          # shares weights but differs from its source
    broken(lambda L: L[1].update(weights_of=4))                     # 4 takes them from 1
    broken(lambda L: L[1].update(weights_of=9))
    broken(lambda L: L[1]["mixer"].update(bias=True))


def test_checkpoint_round_trip_and_refusals(tmp_path):
    from dgpp_b200.loaders.checkpoint import open_checkpoint, write_safetensors
    from dgpp_b200.loaders.family_io import load_family, save_published

    cfg = sc.CONFIGS["odd"]
    c, w = SitiraxConfig.from_dict(cfg), sc.tensors(cfg, 2)
    out = str(tmp_path / "ck")
    save_published(c, w, out)
    assert open_checkpoint(out).family == "sitirax"
    assert json.load(open(out + "/config.json")) == cfg
    toks = torch.tensor(sc.token_ids(cfg, 20))
    m = SitiraxModel.from_tensors(c, w.__getitem__, "cpu")
    back = load_family(out, "cpu")
    assert back.cfg == c and torch.equal(back.forward_reference(toks), m.forward_reference(toks))
    assert load_family(out, "cpu", torch.float32).embed.dtype == torch.float32
    for change, word in ((lambda t: t.pop("l0.mix.A_log"), "l0.mix.A_log"), (lambda t: t.update(extra=t["embed"]), "extra"),
                         (lambda t: t.update({"l0.mix.b": t["l0.mix.b"][:2]}), "l0.mix.b")):
        t = dict(w)
        change(t)
        write_safetensors(out + "/model.safetensors", t)
        with pytest.raises(ValueError, match=word):
            load_family(out, "cpu")


class FakeRunner(RowRunner):
    """A mixed-pass runner without a model: logits row = one-hot of (sum of the request's tokens so far) % vocab, carried as the
    request's state; records every pass."""
    mixed_runs = True
    VOCAB = 50

    class c:
        vocab = 50

    def __init__(self, max_rows=8, slots=3, pool_tokens=256, max_seq=128):
        self._init_pool(slots, "cpu", [], torch.float32, 16, max_seq, max_rows, pool_tokens)
        self.sums, self.passes = [0] * slots, []

    def _reset_state(self, slot):
        self.sums[slot] = 0

    def _row(self, slot, tok):
        self.sums[slot] += tok
        return torch.nn.functional.one_hot(torch.tensor(self.sums[slot] % self.VOCAB), self.VOCAB).float()

    def forward(self, tokens, positions, row_req, chunk_slot=None, all_logits=True, pos0=None, extra=None):
        self.passes.append(("decode", tokens.tolist(), positions.tolist(), row_req.tolist()))
        return torch.stack([self._row(int(s), int(t)) for s, t in zip(row_req, tokens)])

    def forward_runs(self, tokens, positions, row_req, runs, logit_rows):
        st = runs.start.tolist()
        assert st[-1] == len(tokens) <= self.max_rows and len(st) == len(runs.lens) + 1
        for r, (n, s, p0) in enumerate(zip(runs.lens, runs.slots, runs.pos0)):
            assert st[r + 1] - st[r] == n and row_req[st[r]:st[r + 1]].tolist() == [s] * n
            assert positions[st[r]:st[r + 1]].tolist() == list(range(p0, p0 + n))
            assert runs.row_run0[st[r]:st[r + 1]].tolist() == [st[r]] * n
        self.passes.append(("runs", tokens.tolist(), positions.tolist(), row_req.tolist()))
        rows = torch.stack([self._row(int(s), int(t)) for s, t in zip(row_req, tokens)])
        return rows[logit_rows]


def test_mixed_pass_cuts_orders_and_gives_back():
    r = FakeRunner()
    got = r.step([(2, [1, 2, 3], [2, 0]), (0, list(range(1, 14)), [0, 12, 5]), (1, [9], [0])])
    assert got.argmax(-1).tolist() == [6, 1, 1, 91 % 50, 21, 9]
    assert [len(p[1]) for p in r.passes] == [8, 8, 1] and r.lengths == [13, 1, 3]
    assert r.step([(1, [4], []), (0, [5], [0])]).argmax(-1).tolist() == [96 % 50]
    assert r.passes[-1][0] == "decode" and r.passes[-1][2] == [1, 13]
    free = r.kv.free_blocks()
    r.reset(0)
    assert r.kv.free_blocks() == free + 1 and r.lengths[0] == 0
    assert r.step([(0, [7, 8], [])]).numel() == 0
    with pytest.raises(RuntimeError, match="pool"):
        r.step([(0, [1] * 200, [])])


@pytest.mark.parametrize("mixed_pass", [False, True])
def test_runner_engine_with_a_shared_pool(mixed_pass):
    """More requests than slots over a pool smaller than all of them: the scheduler admits against the runner's own blocks,
    groups readers and mixes them with decoders; every request gets the tokens it would get alone."""
    from dgpp_b200.engine.adapters import RunnerEngine

    r = FakeRunner(max_rows=64, slots=3, pool_tokens=128)
    r.use_graphs = False
    cfg = rt.SchedulerConfig()
    cfg.prefix_cache, cfg.prefill_chunk, cfg.mixed_pass, cfg.prefill_group_max = False, 16, mixed_pass, 4
    cfg.prefill_budget_busy = 16
    s = rt.Scheduler(RunnerEngine(r, max_context=96), cfg)
    g = torch.Generator().manual_seed(3)
    reqs = {f"r{i}": torch.randint(0, 50, (5 + 11 * i,), generator=g).tolist() for i in range(6)}
    for rid, p in reqs.items():
        s.submit(rid, p, 8)
    s.run(10000)
    got = {}
    for kind, x, a, b in s.events():
        if kind == "token":
            got.setdefault(x, []).append(a)
    for rid, p in reqs.items():
        total, want = sum(p), []
        for _ in range(8):
            want.append(total % 50)
            total += want[-1]
        assert got[rid] == want
    assert r.kv.free_blocks() == 8 and r.lengths == [0, 0, 0]
    assert any(k == "runs" and len(set(q)) > 1 for k, _, _, q in r.passes)


def test_fixture_writer(tmp_path, capsys):
    from dgpp_b200.loaders.family_io import main

    assert main(["--family", "sitirax", "--out", str(tmp_path / "ck"), "--vocab", "300", "--check"]) == 0
    report = json.loads(capsys.readouterr().out)
    assert report["round_trip_equal"] and report["tensors"] == len(sc.tensor_shapes(SitiraxConfig.from_dict(
        json.load(open(tmp_path / "ck" / "config.json")))))
