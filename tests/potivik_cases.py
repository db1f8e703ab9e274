"""Small random Potivik models for the tests: configurations in the published form and tensors to go with them."""
import torch

from dgpp_b200.models.potivik import PotivikConfig, tensor_shapes


def latent(heads, dim, rot_dim, vdim, rank, window, scale, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "mask": {"size": window},
            "rot": {"base": base, "dims": rot_dim}}


def mamba(heads, groups, vdim, state, conv, parts):
    return {"heads": heads, "groups": groups, "vdim": vdim, "state": state, "conv": conv, "norm_groups": parts}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, limit, shared=None):
    e = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        e["shared"] = {"ff": shared[0], "limit": shared[1]}
    return e


def layer(mixer, mlp=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "mamba2", "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, side=16, eps=1e-5, cap=20.0):
    return {"architecture": "Potivik", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side},
            "logit_softcap": cap}


CONFIGS = {
    # grouped state heads, several norm parts, several experts per token, unlike windows, a layer without a feed-forward
    "mixed": config(128, 320, [
        layer(mamba(4, 2, 32, 64, 4, 2), moe(8, 3, 64, 3.0, (96, 2.0))), layer(latent(8, 64, 32, 64, 128, 48, 0.11), dense(192, 1.5)),
        layer(latent(4, 32, 64, 32, 64, 100, 0.1, 500.0)), layer(mamba(8, 1, 16, 32, 3, 4), moe(12, 2, 40, 1.0)),
        layer(latent(8, 64, 32, 64, 128, 48, 0.11), moe(5, 5, 32, 2.0, (32, 4.0)))]),
    # sizes that fit no tile: width, ranks, head widths and counts, side input, norm parts that cut heads; a window of a page and a bit
    "odd": config(100, 131, [
        layer(latent(5, 24, 12, 40, 52, 70, 0.31, 100.0), moe(7, 2, 44, 1.7, (28, 0.9))), layer(mamba(6, 3, 20, 24, 2, 5), dense(52, 2.2)),
        layer(mamba(3, 1, 44, 40, 6, 6)), layer(latent(3, 40, 20, 24, 100, 9, 0.2), moe(9, 1, 36, 0.8, (20, 3.0)))], side=10, eps=1e-3, cap=7.0),
    # single heads, one tap, one expert, a window of one token, one pair of rotated columns
    "ones": config(64, 96, [
        layer(mamba(1, 1, 16, 16, 1, 1), moe(1, 1, 16, 1.0, (8, 1.0))), layer(latent(1, 16, 2, 16, 16, 1, 1.0), dense(40, 3.0)),
        layer(mamba(1, 1, 8, 8, 1, 8))], side=8),
    # no attention at all
    "states": config(72, 80, [layer(mamba(4, 4, 32, 32, 4, 1), dense(64, 2.0)), layer(mamba(4, 2, 32, 32, 4, 4), dense(64, 2.0))], side=24),
    # only attention
    "windows": config(72, 80, [layer(latent(4, 32, 16, 32, 48, 65, 0.2), dense(64, 2.0)), layer(latent(2, 16, 16, 48, 32, 33, 0.3))]),
    # widths beyond a tile: a wide latent, a rotated part of more than one block, values of more than one, wide states
    "wide": config(256, 512, [
        layer(latent(20, 100, 60, 130, 300, 130, 0.08), moe(16, 4, 128, 2.0, (256, 2.0))), layer(mamba(3, 1, 130, 200, 4, 2), dense(512, 2.0)),
        layer(latent(3, 200, 96, 40, 520, 40, 0.06), dense(128, 2.0))], side=40),
}


def tensors(cfg, seed=0, alike=False):
    """bf16 tensors; decays from short to long, norms, biases and step sizes away from their neutral values.  alike: a layer's
    experts are variations of one another, so a routing decision that 16-bit rounding tips over moves the result little."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in tensor_shapes(PotivikConfig.from_dict(cfg)).items():
        r = torch.randn(*s, generator=g)
        if name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 1 + 0.3 * r
            if name.endswith(("1b", "2b", "side.norm")):
                t = t * 0.7
        elif name.endswith("A_log"):
            t = torch.rand(*s, generator=g) * 4 - 2
        elif name.endswith("dt_bias"):
            t = torch.rand(*s, generator=g) * 4 - 4
        elif name.endswith(".conv"):
            t = 0.7 * r
        elif name.endswith((".conv.b", ".D")):
            t = 0.4 * r
        elif name == "embed":
            t = 0.8 * r
        elif name == "side.embed":
            t = r
        elif name.endswith("router"):
            t = r * s[1] ** -0.5 * 2
        else:
            t = r * s[1] ** -0.5 * 1.3
        out[name] = t.to(torch.bfloat16)
    for name, t in out.items() if alike else ():
        layer, _, rest = name.partition(".mlp.e")
        if rest:
            first = out[f"{layer}.mlp.e0.{rest.partition('.')[2]}"]
            out[name] = (first.float() + 0.1 * (t.float() - first.float())).to(torch.bfloat16)
    return out


def doubles(w):
    return {k: v.double() for k, v in w.items()}


def token_ids(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()
