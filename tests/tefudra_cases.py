"""Small random Tefudra models for the tests: configurations in the published form and tensors to go with them."""
import torch

from dgpp_b200.models.tefudra import TefudraConfig, tensor_shapes


def window(heads, kv_heads, dim, size, keep, rot, base=1000.0, scale=0.3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": size, "keep_first": keep},
            "rot": {"base": base, "dims": rot}}


def left(heads, kv_heads, dim, vdim, size, rot, conv, cap=8.0, base=1000.0, scale=0.3):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}, "rot": {"base": base, "dims": rot},
         "conv": conv}
    return m if cap is None else {**m, "softcap": cap}


def right(heads, dim, vdim, cap=6.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def moe(experts, identity, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    return m if shared is None else {**m, "shared": {"ff": shared}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def layer(mixer, mlp=None, of=None):
    e = {"type": "attention", "mixer": mixer, "mlp": mlp} if not isinstance(mixer, tuple) else \
        {"type": "parallel", "mixer": dict(zip(("left", "right"), mixer)), "mlp": mlp}
    return e if of is None else {**e, "weights_of": of}


def config(width, vocab, layers, groups=1, eps=1e-5):
    return {"architecture": "Tefudra", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps, "groups": groups}}


_A = layer(window(4, 2, 32, 40, 3, 16), moe(6, 2, 3, 40, 48))
_P = layer((left(4, 2, 32, 64, 24, 32, 4), right(2, 32, 64)), dense(96))
_ODD_A = layer(window(6, 2, 36, 37, 5, 12, 500.0), moe(7, 3, 2, 44, 20))
_ODD_P = layer((left(6, 3, 20, 44, 50, 12, 3, 5.0, 100.0), right(3, 20, 24, 3.0)), moe(5, 1, 4, 28, 36))

CONFIGS = {
    # every branch; layers that borrow weights, also from a layer behind them
    "mixed": config(128, 320, [_A, _P, {**_A, "weights_of": 0}, layer((left(4, 4, 64, 32, 70, 64, 4), right(4, 64, 32)), moe(8, 2, 2, 64, 32)),
                               layer(window(8, 2, 64, 100, 70, 64), None), {**_P, "weights_of": 1}], 4),
    # sizes that fit no tile: width, parts of a norm, head widths and counts, windows, experts
    "odd": config(90, 131, [_ODD_P, {**_ODD_A, "weights_of": 3}, layer(window(5, 5, 24, 65, 1, 4), dense(52)), _ODD_A, {**_ODD_P, "weights_of": 0}], 6, 1e-3),
    # single heads, one tap, one expert, a window of one token, nothing kept, nothing rotated, one part
    "ones": config(64, 96, [layer((left(1, 1, 16, 16, 1, 0, 1, None), right(1, 16, 16)), moe(1, 0, 1, 16)),
                            layer(window(1, 1, 8, 1, 0, 0, scale=1.0), moe(1, 1, 1, 8, 8)), layer(window(2, 1, 16, 1, 2, 16), moe(3, 0, 3, 24))], 1),
    # no attention but the parallel layers'; six taps, a part per eight columns
    "memories": config(72, 80, [layer((left(2, 1, 32, 32, 16, 8, 6, 3.0), right(4, 32, 32, 2.0))), layer((left(4, 2, 24, 40, 64, 24, 2), right(2, 32, 40)), dense(64))], 9),
    # only attention, one of it without any token kept, the other with more kept than fit a page
    "keys": config(72, 80, [layer(window(4, 4, 32, 65, 0, 32), moe(4, 1, 2, 24)), layer(window(4, 1, 32, 30, 130, 20), moe(4, 4, 4, 24, 16))], 3),
    # widths beyond a tile, many heads per key head, wide memories
    "wide": config(256, 512, [layer(window(20, 2, 100, 129, 9, 50), dense(200)), layer((left(10, 1, 130, 200, 90, 80, 4, 20.0, 5e4, 0.1), right(3, 130, 200)),
                                                                                       moe(16, 4, 4, 64, 96))], 2),
}


def tensors(cfg, seed=0, alike=False):
    """bf16 tensors; norms, biases, sinks and corrections away from their neutral values, gates that remember and gates that forget.  alike:
    a layer's experts are variations of one another, and which identity experts are chosen is beyond doubt, so a routing decision that
    16-bit rounding tips over moves the result little."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in tensor_shapes(TefudraConfig.from_dict(cfg)).items():
        r, last = torch.randn(*s, generator=g), name.rpartition(".")[2]
        if name.endswith("f.b"):
            t = 2 + 1.5 * r
        elif name.endswith("i.b"):
            t = 0.7 * r
        elif last == "b":
            t = 0.4 * r
        elif last == "correction":
            t = 0.1 * r
        elif last in ("norm", "norm1", "norm2", "norm1b", "norm2b", "out"):
            t = 1 + 0.3 * r
        elif last == "sink":
            t = 1 + r
        elif last == "conv":
            t = 0.7 * r
        elif name == "embed":
            t = 0.1 * r
        elif last == "router":
            t = r * s[1] ** -0.5 * 2
        else:
            t = r * s[1] ** -0.5 * 1.3
        out[name] = t.to(torch.bfloat16)
    for name, t in out.items() if alike else ():
        layer_, _, rest = name.partition(".mlp.e")
        if rest:
            first = out[f"{layer_}.mlp.e0.{rest.partition('.')[2]}"]
            out[name] = (first.float() + 0.1 * (t.float() - first.float())).to(torch.bfloat16)
        elif name.endswith("correction"):
            f = cfg["layers"][int(layer_.split(".")[0][1:])]["mlp"]["router"]
            t[f["experts"]:] = -2
            if f["top"] > 1:
                t[f["experts"]:f["experts"] + 1] = 2
    return out


def doubles(w):
    return {k: v.double() for k, v in w.items()}


def token_ids(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()
