"""Tefudra family without a GPU: configuration, packing (against the plain restatement), checkpoints, the runner's buffers."""
import json
import math

import pytest
import torch

import tefudra_cases as tc
import tefudra_plain as plain
from dgpp_b200.models.tefudra import TefudraConfig, TefudraModel, tensor_shapes


@pytest.mark.parametrize("name", sorted(tc.CONFIGS))
def test_packed_model_matches_the_plain_restatement(name):
    cfg = tc.CONFIGS[name]
    c = TefudraConfig.from_dict(cfg)
    assert TefudraConfig.from_dict(c.to_dict()) == c and c.to_dict() == cfg
    w = tc.tensors(cfg, 1)
    toks = tc.token_ids(cfg, 83)
    want = plain.forward(cfg, tc.doubles(w), toks)
    for dtype in (torch.float32, torch.bfloat16):
        m = TefudraModel.from_tensors(c, w.__getitem__, "cpu", dtype)
        assert (m.forward_reference(torch.tensor(toks)) - want).abs().max() <= 1e-4 * want.abs().max()


def test_plain_mechanisms_by_hand():
    """The restatement itself, where a slip would go unnoticed by everything compared with it."""
    d = torch.float64
    t = lambda *v: torch.tensor(v, dtype=d)
    assert torch.allclose(plain.group_norm(t(3, 4, 0, 10), 2, 0.0, t(1, 1, 1, 2)), t(3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 0, 20 / 50 ** 0.5))
    x = plain.rotate_halves(t(2, 9, 1, 8)[None].expand(3, 4), 100.0, 4)[2]           # columns 0 and 2, 1 and 3; the second pair turns slower
    c1, s1, c2, s2 = math.cos(2.0), math.sin(2.0), math.cos(0.2), math.sin(0.2)
    assert torch.allclose(x, t(2 * c1 - s1, 9 * c2 - 8 * s2, c1 + 2 * s1, 8 * c2 + 9 * s2))
    assert torch.allclose(plain.rotate_halves(x[None].expand(3, 4), 100.0, 4, -1)[2], t(2, 9, 1, 8))
    assert plain.causal_conv(t(1, 2, 4)[:, None], t(10, 1)[None]).flatten().tolist() == [1, 12, 24]
    one, v = torch.ones(4, 1, 1, dtype=d), t(1, 10, 100, 1000).view(4, 1, 1)
    assert torch.allclose(plain.attention(one * 0, one, v, 1.0, 2).flatten(), t(1, 5.5, 55, 550))
    assert torch.allclose(plain.attention(one * 0, one, v, 1.0, 2, 1).flatten(), t(1, 5.5, 37, 1101 / 3))
    assert torch.allclose(plain.attention(one * 0, one, v, 1.0, 1, 2).flatten(), t(1, 5.5, 37, 1011 / 3))
    assert torch.allclose(plain.attention(one * 0, one, v, 1.0, 2, sink=t(math.log(2))).flatten(), t(1 / 3, 11 / 4, 110 / 4, 1100 / 4))
    two = plain.attention(one, t(0, 3, 0, 0).view(4, 1, 1), v, 1.0, 4, cap=2.0).flatten()[1]
    a = math.exp(2 * math.tanh(1.5))
    assert torch.allclose(two, t((1 + 10 * a) / (1 + a))[0])
    # one token: the memory is the write itself, the floor is exp(-m) with m = max(f, i)
    got = plain.matrix_memory(t(2).view(1, 1, 1), t(3).view(1, 1, 1), t(5).view(1, 1, 1), t(-1).view(1, 1), t(-0.5).view(1, 1))
    w = math.exp(-0.5)
    assert torch.allclose(got.flatten(), t(2 * 3 * 5 * w / (max(6 * w, math.exp(0.5)) + 1e-6)))
    got = plain.matrix_memory(t(1, 1).view(2, 1, 1), t(1, 2).view(2, 1, 1), t(4, 8).view(2, 1, 1), t(0, 0).view(2, 1), t(-9, math.log(0.5)).view(2, 1))
    assert torch.allclose(got.flatten(), t(4 / (1 + 1e-6), (0.5 * 4 + 16) / (2.5 + 1e-6)))
    best, share = plain.route(t(0, math.log(2), math.log(5)), t(1, 0, 0), 2)         # the correction lifts the smallest score in
    assert best.tolist() == [0, 2] and torch.allclose(share, t(1, 5) / 6)
    eye = {"e0.up": t(1)[None], "e0.down": t(2)[None], "router": t(0, 0)[:, None], "correction": t(0, 0), "shared.up": t(3)[None], "shared.down": t(1)[None]}
    got = plain.experts(t(0.4)[None], "", {"router": {"experts": 1, "top": 2}, "shared": {"ff": 1}}, eye)
    assert torch.allclose(got, (0.5 * 2 * plain.gelu_erf(t(0.4)) + 0.5 * 0.4 + plain.gelu_erf(t(1.2)))[None])
    assert plain.relu_squared(t(-2, 3)).tolist() == [0, 9] and abs(plain.gelu_erf(t(1.0)).item() - 0.8413447460685429) < 1e-12


def test_refused_configurations():
    def broken(change):
        d = json.loads(json.dumps(tc.CONFIGS["mixed"]))
        change(d)
        with pytest.raises((ValueError, KeyError)):
            TefudraConfig.from_dict(d)

    broken(lambda d: d["layers"][1].update(type="something_else"))
    broken(lambda d: d["layers"][1].update(loop=2))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="other"))
    broken(lambda d: d["layers"][1]["mlp"].update(gate=True))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=9))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(scale=2.0))
    broken(lambda d: d["layers"][0]["mlp"]["shared"].update(act="silu"))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][0]["mixer"].update(vdim=64))
    broken(lambda d: d["layers"][0]["mixer"].update(softcap=3.0))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=33))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(stride=2))
    broken(lambda d: d["layers"][1]["mixer"]["left"].update(vdim=33))
    broken(lambda d: d["layers"][1]["mixer"]["left"].update(conv=0))
    broken(lambda d: d["layers"][1]["mixer"]["right"].update(gate_cap=0))
    broken(lambda d: d["layers"][1]["mixer"].pop("right"))
    broken(lambda d: d["layers"][2].update(weights_of=9))
    broken(lambda d: d["layers"][2].update(weights_of=2))
    broken(lambda d: d["layers"][0].update(weights_of=2))
    broken(lambda d: d["layers"][2].update(weights_of=1))
    broken(lambda d: d["layers"][2]["mixer"].update(scale=7.0))
    broken(lambda d: d["norm"].update(groups=3))


def test_layers_that_borrow_weights_have_no_tensors():
    for name in ("mixed", "odd"):
        cfg = tc.CONFIGS[name]
        names = set(tensor_shapes(TefudraConfig.from_dict(cfg)))
        for i, L in enumerate(cfg["layers"]):
            assert any(n.startswith(f"l{i}.") for n in names) == ("weights_of" not in L)


def test_checkpoint_round_trip_and_refusals(tmp_path):
    from dgpp_b200.loaders.checkpoint import open_checkpoint, write_safetensors
    from dgpp_b200.loaders.family_io import load_family, save_published

    cfg = tc.CONFIGS["odd"]
    c, w = TefudraConfig.from_dict(cfg), tc.tensors(cfg, 2)
    out = str(tmp_path / "ck")
    save_published(c, w, out)
    assert open_checkpoint(out).family == "tefudra"
    assert json.load(open(out + "/config.json")) == cfg
    toks = torch.tensor(tc.token_ids(cfg, 20))
    m = TefudraModel.from_tensors(c, w.__getitem__, "cpu")
    back = load_family(out, "cpu")
    assert back.cfg == c and torch.equal(back.forward_reference(toks), m.forward_reference(toks))
    assert load_family(out, "cpu", torch.float32).embed.dtype == torch.float32
    for change, word in ((lambda t: t.pop("l0.mix.left.q.conv"), "l0.mix.left.q.conv"), (lambda t: t.update({"l1.norm1": t["l0.norm1"]}), "l1.norm1"),
                         (lambda t: t.pop("l3.mix.sink"), "l3.mix.sink"), (lambda t: t.update({"l0.mix.right.g": t["l0.mix.right.g"][:2]}), "l0.mix.right.g")):
        t = dict(w)
        change(t)
        write_safetensors(out + "/model.safetensors", t)
        with pytest.raises(ValueError, match=word):
            load_family(out, "cpu")


def test_planes_rings_and_memories_per_layer():
    """A layer with borrowed weights shares the packed matrices and nothing else; values that are keys take the keys' columns."""
    from dgpp_b200.loaders.family_io import runner_for

    cfg = tc.CONFIGS["mixed"]
    m = TefudraModel.from_tensors(TefudraConfig.from_dict(cfg), tc.tensors(cfg, 1).__getitem__, "cpu")
    r = runner_for(m, 256, 4, 512, "cpu", 640)
    assert [tuple(L.k.shape[1:]) for L in r.kv.layers] == [(2, 64, 64), (2, 64, 64), (2, 64, 64), (4, 64, 64), (2, 64, 64), (2, 64, 64)]
    assert len({t.data_ptr() for L in r.kv.layers for t in (L.k, L.v)}) == 12
    assert m.layers[5] is m.layers[1] and r.rings[5].data_ptr() != r.rings[1].data_ptr() and r.memories[5][0].data_ptr() != r.memories[1][0].data_ptr()
    assert [x is None for x in r.rings] == [x is None for x in r.memories] == [True, False, True, False, True, False]
    assert tuple(r.rings[1].shape) == (4, 4, 4 * 64 + 2 * 64 + 2 * 64) and tuple(r.memories[3][1].shape) == (4, 4, 64 + 4)
    assert m.layers[0].heads.v_off == m.layers[0].heads.k_off and m.layers[0].w_in.n == 4 * 64 + 2 * 64
    assert len(r._state_tensors()) == 9


def test_packed_values_are_padded_half_by_half():
    cfg = tc.CONFIGS["odd"]
    w = tc.tensors(cfg, 1)
    P = TefudraModel.from_tensors(TefudraConfig.from_dict(cfg), w.__getitem__, "cpu", torch.float32).layers[0]
    g = P.heads
    assert (g.DV, g.vdim) == (64, 44) and g.vfreq.shape == (2, 32) and (g.vfreq[:, 22:] == 0).all()
    v = P.w_in.payload[g.v_off:g.v_off + 3 * 64, :90].view(3, 2, 32, 90)
    assert torch.equal(v[:, :, :22], w["l0.mix.left.v"].float().view(3, 2, 22, 90)) and v[:, :, 22:].abs().sum() == 0


def test_fixture_writer(tmp_path, capsys):
    from dgpp_b200.loaders.family_io import main

    assert main(["--family", "tefudra", "--out", str(tmp_path / "ck"), "--vocab", "300", "--check"]) == 0
    report = json.loads(capsys.readouterr().out)
    assert report["round_trip_equal"] and report["tensors"] == len(tensor_shapes(TefudraConfig.from_dict(
        json.load(open(tmp_path / "ck" / "config.json")))))
