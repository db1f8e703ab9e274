"""Vevapel family without a GPU: configuration, packing (against the plain restatement), checkpoints, the plan of a mixed pass."""
import copy
import json
import math

import pytest
import torch

import vevapel_cases as vc
import vevapel_plain as plain
from dgpp_b200.models.vevapel import VevapelConfig, VevapelModel, tensor_shapes


@pytest.mark.parametrize("name", sorted(vc.CONFIGS))
def test_packed_model_matches_the_plain_restatement(name):
    cfg = vc.CONFIGS[name]
    c = VevapelConfig.from_dict(cfg)
    assert VevapelConfig.from_dict(c.to_dict()) == c and c.to_dict() == cfg
    assert c.runs() == plain.schedule(cfg)
    w = vc.tensors(cfg, 1)
    toks = vc.token_ids(cfg, 83)
    want = plain.forward(cfg, vc.doubles(w), toks)
    for dtype in (torch.float32, torch.bfloat16):
        m = VevapelModel.from_tensors(c, w.__getitem__, "cpu", dtype)
        assert (m.forward_reference(torch.tensor(toks)) - want).abs().max() <= 1e-4 * want.abs().max()


def test_order_of_a_loop():
    c = VevapelConfig.from_dict(vc.CONFIGS["mixed"])
    assert c.runs() == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None), (5, None)]
    assert VevapelConfig.from_dict(vc.CONFIGS["keys"]).runs() == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None)]


def test_plain_mechanisms_by_hand():
    """The restatement itself, where a slip would go unnoticed by everything compared with it."""
    d = torch.float64
    t = lambda *v: torch.tensor(v, dtype=d)
    assert torch.allclose(plain.layer_norm(t(3, 5, 7)[None], 4.0 / 3, t(1, 2, 3), t(0, 0, 5)), t(-1, 0, 8)[None])
    x = plain.rotate_halves(t(2, 9, 1, 8)[None].expand(2, 4), 1.0, 2)[1]             # columns 0 and 1 are the pair
    c, s = math.cos(1.0), math.sin(1.0)
    assert torch.allclose(x, t(2 * c - 9 * s, 9 * c + 2 * s, 1, 8))
    x = plain.rotate_halves(t(2, 9, 1, 8)[None].expand(3, 4), 100.0, 4)[2]           # columns 0 and 2, 1 and 3; the second pair turns slower
    c1, s1, c2, s2 = math.cos(2.0), math.sin(2.0), math.cos(0.2), math.sin(0.2)
    assert torch.allclose(x, t(2 * c1 - s1, 9 * c2 - 8 * s2, c1 + 2 * s1, 8 * c2 + 9 * s2))
    assert plain.temperature(0, 0.5, 3) == 1 and plain.temperature(1, 0.5, 3) == 1 and plain.temperature(2, 0.5, 3) == 1 + 0.5 * math.log(2)
    one = torch.ones(4, 1, 1, dtype=d)
    v = t(1, 10, 100, 1000).view(4, 1, 1)
    assert torch.allclose(plain.attention(one * 0, one, v, 1.0).flatten(), t(1, 5.5, 37, 277.75))
    assert torch.allclose(plain.attention(one * 0, one, v, 1.0, 3).flatten(), t(1, 5.5, 37, 1000))
    zero = t(0, 0)
    o = plain.differential(t(3, 5), t(2, 2), zero, zero, zero, zero, 0.5, 0.0)       # lambda = 1 - 1 + 0.5
    assert torch.allclose(o, t(2, 4) / 10 ** 0.5 * 0.5)
    # two tokens along the same key: the second write is what the first one left to correct; the read-out sees it
    got = plain.delta_rule(torch.ones(2, 1, 1, dtype=d), torch.ones(2, 1, 1, dtype=d), t(4, 10).view(2, 1, 1), t(0.5, 0.25).view(2, 1), t(1, 0.5).view(2, 1))
    assert got.flatten().tolist() == [2.0, 1.0 + 0.25 * (10 - 1.0)]
    w = {"e0.gate": t(1)[None], "e0.up": t(1)[None], "e0.down": t(1)[None], "e1.gate": t(2)[None], "e1.up": t(1)[None], "e1.down": t(1)[None],
         "e2.gate": t(9)[None], "e2.up": t(9)[None], "e2.down": t(9)[None], "router": t(0, 0, 0)[:, None], "router.b": t(0, math.log(3), -1)}
    got = plain.experts(t(0.3)[None], "", {"router": {"top": 2}}, w)                 # weights 1/4 and 3/4
    assert torch.allclose(got, 0.3 * (plain.silu(t(0.3)) / 4 + 0.75 * plain.silu(t(0.6)))[None])


def test_refused_configurations():
    def broken(change):
        d = copy.deepcopy(vc.CONFIGS["mixed"])
        change(d)
        with pytest.raises((ValueError, KeyError)):
            VevapelConfig.from_dict(d)

    broken(lambda d: d["layers"][1].update(type="something_else"))
    broken(lambda d: d["layers"][1].update(weights_of=0))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="dense"))
    broken(lambda d: d["layers"][1]["mlp"].update(shared=None))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(top=7))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(scale=2.0))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][0]["mixer"].update(sink=1))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=33))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=34))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][2]["mixer"]["q_temp"].update(every=0))
    broken(lambda d: d["layers"][2]["mixer"].pop("q_temp"))
    broken(lambda d: d["loop"].update(stop=7))
    broken(lambda d: d["loop"].update(stop=1))
    broken(lambda d: d["loop"].update(times=0))
    broken(lambda d: d.pop("residual_mult"))


def test_checkpoint_round_trip_and_refusals(tmp_path):
    from dgpp_b200.loaders.checkpoint import open_checkpoint, write_safetensors
    from dgpp_b200.loaders.family_io import load_family, save_published

    cfg = vc.CONFIGS["odd"]
    c, w = VevapelConfig.from_dict(cfg), vc.tensors(cfg, 2)
    out = str(tmp_path / "ck")
    save_published(c, w, out)
    assert open_checkpoint(out).family == "vevapel"
    assert json.load(open(out + "/config.json")) == cfg
    toks = torch.tensor(vc.token_ids(cfg, 20))
    m = VevapelModel.from_tensors(c, w.__getitem__, "cpu")
    back = load_family(out, "cpu")
    assert back.cfg == c and torch.equal(back.forward_reference(toks), m.forward_reference(toks))
    assert load_family(out, "cpu", torch.float32).embed.dtype == torch.float32
    for change, word in ((lambda t: t.pop("l1.mix.A_log"), "l1.mix.A_log"), (lambda t: t.update(extra=t["embed"]), "extra"),
                         (lambda t: t.pop("loop.step"), "loop.step"), (lambda t: t.update({"l0.mix.g": t["l0.mix.g"][:2]}), "l0.mix.g")):
        t = dict(w)
        change(t)
        write_safetensors(out + "/model.safetensors", t)
        with pytest.raises(ValueError, match=word):
            load_family(out, "cpu")


def test_cache_planes_and_plan_of_a_mixed_pass():
    """Every run of a looped layer has planes of its own; differential layers keep two key heads per value head.  Short runs become
    single rows, the rows of the longer ones are listed beside them."""
    from dgpp_b200.loaders.family_io import runner_for
    from dgpp_b200.models.rows import RowRuns

    cfg = vc.CONFIGS["mixed"]
    m = VevapelModel.from_tensors(VevapelConfig.from_dict(cfg), vc.tensors(cfg, 1).__getitem__, "cpu")
    r = runner_for(m, 256, 4, 512, "cpu", 640)
    assert sorted(r.kv_index) == [0, 2, 3, 5, 6, 8] and sorted(r.states) == [1, 4, 7]
    assert [tuple(L.k.shape) for L in r.kv.layers] == [(10, 4, 64, 64), (10, 2, 64, 64), (10, 4, 64, 64), (10, 2, 64, 64), (10, 4, 64, 64), (10, 8, 64, 64)]
    assert [tuple(L.v.shape[:2]) for L in r.kv.layers] == [(10, 2), (10, 2), (10, 2), (10, 2), (10, 2), (10, 8)]
    assert len({t.data_ptr() for L in r.kv.layers for t in (L.k, L.v)}) == 12
    short, (start, lens, host), rows = r._plan(RowRuns(None, None, [20, 3, 1, 9], [2, 0, 1, 3], [0, 37, 1, 5]))
    assert short.tolist() == [20, 21, 22, 23] and start.tolist() == [0, 24] and lens.tolist() == host == [20, 9]
    assert rows.tolist() == list(range(20)) + list(range(24, 33))
    whole = RowRuns("starts", None, [20, 9], [2, 3], [0, 5])
    assert r._plan(whole) == (None, ("starts", None, [20, 9]), None)
    short, long, _ = r._plan(RowRuns(None, None, [2, 1], [2, 0], [0, 37]))
    assert short.tolist() == [0, 1, 2] and long is None


def test_fixture_writer(tmp_path, capsys):
    from dgpp_b200.loaders.family_io import main

    assert main(["--family", "vevapel", "--out", str(tmp_path / "ck"), "--vocab", "300", "--check"]) == 0
    report = json.loads(capsys.readouterr().out)
    assert report["round_trip_equal"] and report["tensors"] == len(tensor_shapes(VevapelConfig.from_dict(
        json.load(open(tmp_path / "ck" / "config.json")))))
