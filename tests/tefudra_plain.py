"""Plain, slow restatement of the Tefudra design on the CPU: one function per mechanism, whole sequences, no cache, no kernels.
`cfg` is the parsed config.json, `w` maps tensor names to tensors.  Every function takes the working dtype from its inputs (the
tests run it in float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, groups, eps, weight):
    """Every one of `groups` equal parts by its own root mean square, then one weight per column."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def gelu_erf(z):
    return z * 0.5 * (1 + torch.erf(z / math.sqrt(2)))


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def linear(h, w, name):
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def rotate_halves(x, base, dims, sign=1):
    """x [T, ..., d], row t at position t: column i < dims / 2 is turned with column i + dims / 2 (sign -1: backwards)."""
    out, half = x.clone(), dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = sign * t * base ** (-2 * i / dims)
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def causal_conv(x, taps):
    """x [T, C], taps [C, n] (last column: the current token) with zeros before the start."""
    n = taps.shape[1]
    pad = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return sum(pad[j:j + x.shape[0]] * taps[:, j] for j in range(n))


def visible(i, j, size, keep_first=0):
    return j <= i and (i - j < size or j < keep_first)


def attention(q, k, v, scale, size, keep_first=0, cap=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]."""
    T, H = q.shape[:2]
    group = torch.arange(H) // (H // k.shape[1])
    k, v, out = k[:, group], v[:, group], q.new_zeros(T, H, v.shape[2])
    for i in range(T):
        see = torch.tensor([j for j in range(i + 1) if visible(i, j, size, keep_first)])
        s = torch.einsum("jhd,hd->hj", k[see], q[i]) * scale
        if cap is not None:
            s = soft_cap(s, cap)
        if sink is not None:
            s = torch.cat([s, sink[:, None]], 1)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        p = p / p.sum(-1, keepdim=True)
        out[i] = torch.einsum("hj,jhe->he", p[:, :len(see)], v[see])
    return out


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, e], log gates i, f [T, H] -> [T, H, e]."""
    T, H, d = q.shape
    S, n, m, out = q.new_zeros(H, d, v.shape[2]), q.new_zeros(H, d), q.new_zeros(H), []
    for t in range(T):
        top = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = top
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / den[:, None])
    return torch.stack(out)


def mixer_attention(h, p, c, w, eps):
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    raw = linear(h, w, p + "k").view(T, G, d)
    turn = lambda x: rotate_halves(x, c["rot"]["base"], c["rot"]["dims"])
    q = turn(rms(linear(h, w, p + "q").view(T, H, d), eps) * w[p + "q.norm"])
    k = turn(rms(raw, eps) * w[p + "k.norm"])
    o = attention(q, k, raw, c["scale"], c["mask"]["size"], c["mask"].get("keep_first", 0), None, w[p + "sink"])
    return linear(o.reshape(T, -1), w, p + "o")


def left_values(v, base, eps):
    """v [T, G, e]: unit root mean square, turned by the position over the whole head."""
    return rotate_halves(rms(v, eps), base, v.shape[-1])


def mixer_left(h, p, c, w, eps):
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q, k, v = (causal_conv(linear(h, w, p + n), w[p + n + ".conv"]) for n in "qkv")
    base = c["rot"]["base"]
    turn = lambda x: rotate_halves(x, base, c["rot"]["dims"])
    o = attention(turn(q.view(T, H, d)), turn(k.view(T, G, d)), left_values(v.view(T, G, -1), base, eps), c["scale"], c["mask"]["size"],
                  cap=c.get("softcap"))
    return linear(rotate_halves(o, base, c["vdim"], -1).reshape(T, -1), w, p + "o")


def mixer_right(h, p, c, w, eps):
    T, H, d = h.shape[0], c["heads"], c["dim"]
    split = lambda n: linear(h, w, p + n).view(T, H, -1)
    cap = c["gate_cap"]
    o = matrix_memory(split("q") * d ** -0.5, split("k"), split("v"), soft_cap(linear(h, w, p + "i"), cap), log_sigmoid(soft_cap(linear(h, w, p + "f"), cap)))
    return (rms(o, eps).reshape(T, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer_parallel(h, p, c, w, eps):
    left = rms(mixer_left(h, p + "left.", c["left"], w, eps), eps) * w[p + "left.out"]
    right = rms(mixer_right(h, p + "right.", c["right"], w, eps), eps) * w[p + "right.out"]
    return (left + right) / 2


def route(z, correction, top):
    """One token's logits -> (chosen outputs, their weights)."""
    s = torch.softmax(z, -1)
    best = torch.argsort(-(s + correction), stable=True)[:top]
    return best, s[best] / (s[best].sum() + 1e-20)


def plain_ff(h, p, w, act):
    return act(h @ w[p + "up"].T) @ w[p + "down"].T


def experts(h, p, c, w):
    n, z, out = c["router"]["experts"], h @ w[p + "router"].T, torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(*route(z[t], w[p + "correction"], c["router"]["top"])):
            out[t] += a * (plain_ff(h[t][None], f"{p}e{e}.", w, gelu_erf)[0] if e < n else h[t])
    return out + plain_ff(h, p + "shared.", w, gelu_erf) if c.get("shared") else out


def feed_forward(h, p, c, w):
    return plain_ff(h, p, w, relu_squared) if c["kind"] == "dense" else experts(h, p, c, w)


MIXERS = {"attention": mixer_attention, "parallel": mixer_parallel}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    norm = lambda v, name: group_norm(v, cfg["norm"]["groups"], eps, w[name])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{L.get('weights_of', i)}."
        x = x + norm(MIXERS[L["type"]](norm(x, p + "norm1"), p + "mix.", L["mixer"], w, eps), p + "norm1b")
        if L["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, p + "norm2"), p + "mlp.", L["mlp"], w), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ w["embed"].T
