"""Small random Sitirax models for the tests: configurations in the published form and tensors to go with them."""
import torch

from dgpp_b200.models.sitirax import SitiraxConfig, tensor_shapes


def parallel(heads, kv, dim, vdim, window, scale, rheads, rdim, rvdim, decay, ls=0.8, rs=0.5):
    return {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}},
            "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": list(decay)}, "left_scale": ls, "right_scale": rs}


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def layer(mixer, ff=None, of=None):
    e = {"type": "parallel" if "left" in mixer else "channel_delta", "mixer": mixer,
         "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if of is not None:
        e["weights_of"] = of
    return e


def config(width, vocab, layers, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Sitirax", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "logit_scale": logit_scale}


CONFIGS = {
    # grouped heads, values narrower than keys, a shared parallel layer, delta layers with and without a feed-forward
    "mixed": config(128, 320, [
        layer(parallel(8, 2, 64, 32, 48, 0.2, 2, 32, 64, (0.7, 0.99)), 256), layer(delta(4, 2, 64, 32, 4)),
        layer(delta(2, 2, 32, 128, 3), 128), layer(parallel(8, 2, 64, 32, 48, 0.2, 2, 32, 64, (0.7, 0.99)), 256, of=0),
        layer(delta(4, 2, 64, 32, 4), of=1)]),
    # weights of a layer further on
    "ahead": config(64, 80, [layer(delta(2, 1, 32, 32, 3), of=2), layer(parallel(2, 1, 32, 32, 20, 0.3, 2, 16, 32, (0.9, 0.6)), 64),
                             layer(delta(2, 1, 32, 32, 3)), layer(delta(2, 1, 32, 32, 3), of=2)]),
    # sizes that fit no tile: width, ranks, head widths and counts; one kv head; a window of one page and a bit; decay one
    "odd": config(100, 131, [
        layer(delta(3, 1, 20, 40, 2), 52), layer(parallel(5, 1, 24, 72, 70, 0.31, 3, 40, 20, (0.5, 1.0, 0.9), 1.2, 0.4)),
        layer(parallel(3, 3, 40, 24, 9, 0.5, 1, 20, 44, (0.97,), 0.3, 0.9), 36), layer(delta(2, 1, 48, 16, 6))], eps=1e-3, logit_scale=1.3),
    # single heads, one tap, a window of one token, no parallel feed-forward, delta layers last and first
    "ones": config(64, 96, [
        layer(parallel(1, 1, 16, 16, 1, 1.0, 1, 16, 16, (0.8,), 1.0, 1.0)), layer(delta(1, 1, 16, 16, 1), 40),
        layer(delta(1, 1, 16, 16, 1), 40, of=1)], logit_scale=1.0),
    # no attention at all
    "states": config(72, 80, [layer(delta(4, 4, 32, 32, 4), 64), layer(delta(4, 4, 32, 32, 4), 64, of=0)]),
    # wide heads and groups
    "wide": config(256, 512, [
        layer(parallel(12, 1, 160, 200, 130, 0.1, 2, 100, 130, (0.9, 0.995)), 512), layer(delta(2, 1, 130, 100, 4), 512)]),
}


def tensors(cfg, seed=0, rank_a=10, rank_g=12):
    """bf16 tensors; decays from short to long, norms and step sizes away from their neutral values."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in tensor_shapes(SitiraxConfig.from_dict(cfg), rank_a, rank_g).items():
        r = torch.randn(*s, generator=g)
        if name.endswith(("norm", "norm1", "norm2")):
            t = 1 + 0.3 * r
        elif name.endswith("A_log"):
            t = torch.rand(*s, generator=g) * 4 - 3.5
        elif name.endswith("dt_bias"):
            t = torch.rand(*s, generator=g) * 4 - 3
        elif name.endswith(".conv"):
            t = 0.7 * r
        elif name == "embed":
            t = 0.15 * r                     # small: the layers, not the tied embedding, decide the logits
        else:
            t = r * s[1] ** -0.5 * 1.3
        out[name] = t.to(torch.bfloat16)
    return out


def doubles(w):
    return {k: v.double() for k, v in w.items()}


def token_ids(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()
