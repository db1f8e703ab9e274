"""Small random Vevapel models for the tests: configurations in the published form and tensors to go with them."""
import torch

from dgpp_b200.models.vevapel import VevapelConfig, tensor_shapes


def full(heads, kv_heads, dim, vdim, scale, coef=0.4, every=20):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "q_temp": {"coef": coef, "every": every}}


def diff(heads, kv_heads, dim, vdim, scale, size, rot, base=1000.0, lam=0.3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
            "rot": {"base": base, "dims": rot}, "diff": lam}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp=None):
    return {"type": "delta" if "conv" in mixer else "attention_2" if "diff" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, loop=(0, 1, 1), eps=1e-5, scale=2.0, mult=0.8):
    c = {"architecture": "Vevapel", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": scale},
         "residual_mult": mult}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # every kind of layer inside and outside of the loop, unlike chunks, a layer without a feed-forward
    "mixed": config(128, 320, [
        layer(diff(4, 2, 32, 64, 0.3, 40, 32), moe(8, 3, 64)), layer(delta(4, 2, 32, 64, 4), moe(6, 2, 40)),
        layer(full(4, 2, 64, 32, 0.2)), layer(diff(6, 2, 64, 32, 0.2, 100, 24, 500.0, 0.6), moe(12, 2, 40)),
        layer(delta(4, 4, 64, 32, 3), moe(5, 5, 32)), layer(full(8, 8, 32, 64, 0.25, 0.9, 7), moe(8, 1, 64))], (1, 4, 2)),
    # sizes that fit no tile: width, head widths and counts, chunks, experts; a convolution beyond four taps
    "odd": config(100, 131, [
        layer(full(5, 5, 24, 40, 0.3, 0.7, 13), moe(7, 2, 44)), layer(delta(6, 3, 20, 24, 2), moe(9, 4, 36)),
        layer(diff(6, 3, 20, 44, 0.3, 37, 12, 100.0, 0.15)), layer(delta(3, 1, 44, 36, 6), moe(3, 2, 28)),
        layer(full(6, 2, 36, 20, 0.25, 1.3, 5))], (2, 5, 3), 1e-3, 0.7, 1.3),
    # single heads, one tap, one expert, chunks of one token, no rotation, no temperature, one pass of one layer
    "ones": config(64, 96, [
        layer(delta(1, 1, 16, 16, 1), moe(1, 1, 16)), layer(diff(1, 1, 16, 16, 1.0, 1, 0), moe(2, 1, 40)),
        layer(full(1, 1, 8, 8, 1.0, 0.0, 1), moe(1, 1, 8))], (1, 2, 1), mult=1.0, scale=1.0),
    # no loop; no attention at all
    "states": config(72, 80, [layer(delta(4, 4, 32, 32, 4), moe(4, 2, 24)), layer(delta(4, 2, 32, 32, 4))], None),
    # only attention; the loop takes the whole model
    "keys": config(72, 80, [layer(diff(4, 4, 32, 32, 0.25, 65, 32), moe(4, 2, 24)), layer(full(4, 1, 32, 32, 0.25))], (0, 2, 3)),
    # widths beyond a tile, many heads per key head, wide states
    "wide": config(256, 512, [
        layer(full(20, 2, 100, 130, 0.1), moe(16, 4, 128)), layer(diff(10, 1, 130, 200, 0.09, 129, 80, 5e4, 0.8), moe(4, 2, 256)),
        layer(delta(18, 2, 130, 200, 4))], (1, 3, 2)),
}


def tensors(cfg, seed=0, alike=False):
    """bf16 tensors; decays from short to long, norms, biases and step sizes away from their neutral values.  alike: a layer's
    experts are variations of one another, so a routing decision that 16-bit rounding tips over moves the result little."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in tensor_shapes(VevapelConfig.from_dict(cfg)).items():
        r = torch.randn(*s, generator=g)
        if name.endswith((".b", "loop.step")) and not name.endswith("mix.b"):
            t = 0.4 * r
        elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 1 + 0.3 * r
        elif name.endswith("A_log"):
            t = torch.rand(*s, generator=g) * 4 - 2
        elif name.endswith("dt_bias"):
            t = torch.rand(*s, generator=g) * 4 - 4
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = r * 0.8 * s[0] ** -0.25
        elif name.endswith(".conv"):
            t = 0.7 * r
        elif name == "embed":
            t = 0.8 * r
        elif name.endswith("router"):
            t = r * s[1] ** -0.5 * 2
        elif name == "loop.in":
            t = r * s[1] ** -0.5
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
