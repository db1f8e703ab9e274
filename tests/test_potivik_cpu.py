"""Potivik family without a GPU: configuration, packing (against the plain restatement), checkpoints, the plan of a mixed pass."""
import copy
import json

import pytest
import torch

import potivik_cases as pc
import potivik_plain as plain
from dgpp_b200.models.potivik import PotivikConfig, PotivikModel, tensor_shapes


@pytest.mark.parametrize("name", sorted(pc.CONFIGS))
def test_packed_model_matches_the_plain_restatement(name):
    cfg = pc.CONFIGS[name]
    c = PotivikConfig.from_dict(cfg)
    assert PotivikConfig.from_dict(c.to_dict()) == c
    w = pc.tensors(cfg, 1)
    toks = pc.token_ids(cfg, 83)
    want = plain.forward(cfg, pc.doubles(w), toks)
    for dtype in (torch.float32, torch.bfloat16):
        m = PotivikModel.from_tensors(c, w.__getitem__, "cpu", dtype)
        assert (m.forward_reference(torch.tensor(toks)) - want).abs().max() <= 5e-5 * want.abs().max()


def test_plain_mechanisms_by_hand():
    """The restatement itself, where a slip would go unnoticed by everything compared with it."""
    d = torch.float64
    x = torch.tensor([[3.0, 5.0, 7.0]], dtype=d)
    assert torch.allclose(plain.layer_norm(x, 0.0), torch.tensor([[-1.0, 0.0, 1.0]], dtype=d) * 1.5 ** 0.5)
    assert torch.allclose(plain.layer_norm(x, 4.0 / 3), torch.tensor([[-1.0, 0.0, 1.0]], dtype=d))
    quarter = plain.rotate_pairs(torch.tensor([[0.0, 0, 0], [2.0, 1.0, 9.0]], dtype=d), 1.0, 2)[1]
    c, s = torch.cos(torch.tensor(1.0, dtype=d)), torch.sin(torch.tensor(1.0, dtype=d))
    assert torch.allclose(quarter, torch.stack([2 * c - s, c + 2 * s, torch.tensor(9.0, dtype=d)]))
    one = torch.ones(3, 1, 1, dtype=d)
    v = torch.tensor([1.0, 10.0, 100.0], dtype=d).view(3, 1, 1)
    assert plain.window_attention(one * 0, one, v, 1.0, 2).flatten().tolist() == [1.0, 5.5, 55.0]
    y = plain.causal_conv(torch.tensor([[1.0], [2.0]], dtype=d), torch.tensor([[10.0, 1.0]], dtype=d), torch.tensor([0.5], dtype=d))
    assert torch.allclose(y[:, 0], plain.silu(torch.tensor([1.5, 12.5], dtype=d)))
    # two tokens: S1 = dt B x, S2 = exp(-dt) S1 + dt B x; y = C S + D x
    B, C, X, dt = 2.0, 3.0, 5.0, 0.5
    e = torch.exp(torch.tensor(-dt, dtype=d))
    got = plain.state_space(torch.full((2, 1, 1), X, dtype=d), torch.full((2, 1, 1), B, dtype=d), torch.full((2, 1, 1), C, dtype=d),
                            torch.full((2, 1), dt, dtype=d), torch.zeros(1, dtype=d), torch.tensor([7.0], dtype=d)).flatten()
    assert torch.allclose(got, torch.stack([C * dt * B * X + 7 * X + 0 * e, C * (e + 1) * dt * B * X + 7 * X]))
    a = plain.gated_part_norm(torch.tensor([3.0, 4.0, 1.0, 1.0], dtype=d)[None], torch.full((1, 4), 60.0, dtype=d), 2, torch.ones(4, dtype=d), 0.0)
    assert torch.allclose(a, torch.tensor([[3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 1.0, 1.0]], dtype=d))
    # a routed expert sees score * input: with one expert and a linear regime that is not score * output
    w = {"gate": torch.eye(1, dtype=d), "up": torch.eye(1, dtype=d), "down": torch.eye(1, dtype=d)}
    h = torch.tensor([[0.3]], dtype=d)
    r = {**{f"e0.{k}": t for k, t in w.items()}, "router": torch.zeros(1, 1, dtype=d)}
    got = plain.experts(h, "", {"router": {"top": 1}, "expert": {"limit": 9.0}}, r)
    assert torch.allclose(got, plain.clamped_glu(h / 2, "", w, 9.0)) and not torch.allclose(got, plain.clamped_glu(h, "", w, 9.0) / 2)


def test_refused_configurations():
    base = pc.CONFIGS["mixed"]

    def broken(change):
        d = copy.deepcopy(base)
        change(d)
        with pytest.raises((ValueError, KeyError)):
            PotivikConfig.from_dict(d)

    broken(lambda d: d["layers"][1].update(type="something_else"))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda d: d["layers"][1]["mlp"].update(bias=True))
    broken(lambda d: d["layers"][0]["mixer"].update(groups=3))
    broken(lambda d: d["layers"][0]["mixer"].update(norm_groups=7))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=33))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=34))
    broken(lambda d: d["layers"][1]["mixer"].update(sink=1))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=9))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(scale=2.0))
    broken(lambda d: d.pop("logit_softcap"))
    broken(lambda d: d["token_side"].update(layers=3))


def test_checkpoint_round_trip_and_refusals(tmp_path):
    from dgpp_b200.loaders.checkpoint import open_checkpoint, write_safetensors
    from dgpp_b200.loaders.family_io import load_family, save_published

    cfg = pc.CONFIGS["odd"]
    c, w = PotivikConfig.from_dict(cfg), pc.tensors(cfg, 2)
    out = str(tmp_path / "ck")
    save_published(c, w, out)
    assert open_checkpoint(out).family == "potivik"
    assert json.load(open(out + "/config.json")) == cfg
    toks = torch.tensor(pc.token_ids(cfg, 20))
    m = PotivikModel.from_tensors(c, w.__getitem__, "cpu")
    back = load_family(out, "cpu")
    assert back.cfg == c and torch.equal(back.forward_reference(toks), m.forward_reference(toks))
    assert load_family(out, "cpu", torch.float32).embed.dtype == torch.float32
    for change, word in ((lambda t: t.pop("l1.mix.A_log"), "l1.mix.A_log"), (lambda t: t.update(extra=t["embed"]), "extra"),
                         (lambda t: t.update({"l0.mix.g": t["l0.mix.g"][:2]}), "l0.mix.g")):
        t = dict(w)
        change(t)
        write_safetensors(out + "/model.safetensors", t)
        with pytest.raises(ValueError, match=word):
            load_family(out, "cpu")


def test_plan_of_a_mixed_pass():
    """Long runs are expanded from the page of the first key they see, per window; short runs become single rows."""
    from dgpp_b200.loaders.family_io import runner_for
    from dgpp_b200.models.rows import RowRuns

    cfg = pc.CONFIGS["mixed"]                                              # windows 48 and 100
    m = PotivikModel.from_tensors(PotivikConfig.from_dict(cfg), pc.tensors(cfg, 1).__getitem__, "cpu")
    r = runner_for(m, 256, 4, 512, "cpu", 2048)
    for slot, n in ((2, 300), (0, 40), (1, 130)):
        assert r.kv.reserve(slot, n)
    lens, slots, pos0 = [100, 3, 129], [2, 0, 1], [200, 37, 1]
    short, by_window = r._plan_runs(RowRuns(None, None, lens, slots, pos0))
    assert short.tolist() == [100, 101, 102] and sorted(by_window) == [48, 100]
    for w, lr in by_window.items():
        assert lr.start.tolist() == [0, 103] and lr.lens.tolist() == [100, 129] and lr.tiles == 3
        pages = lr.pages.tolist()
        for base, slot, p0, n in zip(lr.base.tolist(), (2, 1), (200, 1), (100, 129)):
            for p in range(max(0, p0 + 1 - w), p0 + n):                    # every key that the run sees is where the kernel looks
                assert pages[(base + p // 64 * 64) // 64] == r.kv.req_blocks[slot][p // 64]
    assert r._plan_runs(RowRuns(None, None, [4], [2], [296]))[1] == {}
    assert r._plan_runs(RowRuns(None, None, [40], [2], [260]))[0] is None


def test_scratch_of_the_experts_holds_every_row_count():
    from dgpp_b200.models.row_moe import RowExperts, RowExpertsScratch
    from dgpp_b200.quant.formats import QuantLinear

    t = torch.empty(0)
    for experts, top in ((16, 1), (64, 8), (5, 5), (1, 1), (33, 4)):
        b = RowExperts(experts, top, 8, 1.0, QuantLinear("bf16", 8, 8, t), t, t, 8)
        for f32 in (False, True):
            s = RowExpertsScratch([b], 1200, torch.float32 if f32 else torch.bfloat16, "cpu")
            for n in range(1, 1201):
                bn = b.tile_rows(n, f32)
                nt = b.max_tiles(n, bn)
                assert s.tiles.numel() >= nt and s.xs.numel() >= nt * bn * 8 and s.row_w.numel() >= nt * bn and s.pair_row.numel() >= n * top


def test_fixture_writer(tmp_path, capsys):
    from dgpp_b200.loaders.family_io import main

    assert main(["--family", "potivik", "--out", str(tmp_path / "ck"), "--vocab", "300", "--check"]) == 0
    report = json.loads(capsys.readouterr().out)
    assert report["round_trip_equal"] and report["tensors"] == len(tensor_shapes(PotivikConfig.from_dict(
        json.load(open(tmp_path / "ck" / "config.json")))))
