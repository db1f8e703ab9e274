"""Plain, slow restatement of the Vevapel design on the CPU: one function per mechanism, whole sequences, no cache, no kernels.
`cfg` is the parsed config.json, `w` maps tensor names to tensors.  Every function takes the working dtype from its inputs (the
tests run it in float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, eps, weight, bias):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def linear(h, w, name):
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def rotate_halves(x, base, dims, first=0):
    """x [T, ..., d], row t at position first + t: column i < dims / 2 is turned with column i + dims / 2."""
    out, half = x.clone(), dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = (first + t) * base ** (-2 * i / dims)
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def temperature(p, coef, every):
    return 1 + coef * math.log((p + 1) // every + 1)


def attention(q, k, v, scale, chunk=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; query i sees keys j <= i, of its own chunk where there are chunks."""
    T, H = q.shape[:2]
    group = torch.arange(H) // (H // k.shape[1])
    k, v, out = k[:, group], v[:, group], q.new_zeros(T, H, v.shape[2])
    for i in range(T):
        lo = 0 if chunk is None else i // chunk * chunk
        s = torch.einsum("jhd,hd->hj", k[lo:i + 1], q[i]) * scale
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhe->he", p / p.sum(-1, keepdim=True), v[lo:i + 1])
    return out


def differential(a1, a2, lq1, lk1, lq2, lk2, diff, eps):
    lam = torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff
    return rms(a1 - lam * a2, eps) * (1 - diff)


def causal_conv(x, taps):
    """x [T, C], taps [C, n] (last column: the current token) with zeros before the start, then silu."""
    n = taps.shape[1]
    pad = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return silu(sum(pad[j:j + x.shape[0]] * taps[:, j] for j in range(n)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, decay):
    """q, k [T, H, d], v [T, H, e], beta, decay [T, H] -> [T, H, e]."""
    S, out = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
    for t in range(q.shape[0]):
        S = S * decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def mixer_attention(h, p, c, w, eps):
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q = rms(linear(h, w, p + "q"), eps) * w[p + "q.norm"]
    k = rms(linear(h, w, p + "k"), eps) * w[p + "k.norm"]
    q = q * q.new_tensor([temperature(t, c["q_temp"]["coef"], c["q_temp"]["every"]) for t in range(T)])[:, None]
    o = attention(q.view(T, H, d), k.view(T, G, d), linear(h, w, p + "v").view(T, G, -1), c["scale"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return linear(o.reshape(T, -1), w, p + "o")


def mixer_attention_2(h, p, c, w, eps):
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    turn = lambda x: rotate_halves(x, c["rot"]["base"], c["rot"]["dims"])
    q, k = turn(linear(h, w, p + "q").view(T, H, 2, d)), turn(linear(h, w, p + "k").view(T, G, 2, d))
    v = linear(h, w, p + "v").view(T, G, -1)
    a1, a2 = (attention(q[:, :, m], k[:, :, m], v, c["scale"], c["mask"]["size"]) for m in (0, 1))
    o = differential(a1, a2, w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], c["diff"], eps)
    return linear(o.reshape(T, -1) * sigmoid(h @ w[p + "g"].T), w, p + "o")


def mixer_delta(h, p, c, w, eps):
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q, k, v = (causal_conv(h @ w[p + n].T, w[p + n + ".conv"]) for n in "qkv")
    group = torch.arange(H) // (H // G)
    q, k = unit(q.view(T, G, d))[:, group] * d ** -0.5, unit(k.view(T, G, d))[:, group]
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = delta_rule(q, k, v.view(T, H, -1), sigmoid(h @ w[p + "b"].T), g)
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(o.shape)
    return o.reshape(T, -1) @ w[p + "o"].T


def expert(h, p, w):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def experts(h, p, c, w):
    z = linear(h, w, p + "router")
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = torch.argsort(-z[t], stable=True)[:c["router"]["top"]]
        for e, a in zip(best.tolist(), torch.softmax(z[t][best], 0)):
            out[t] += a * expert(h[t][None], f"{p}e{e}.", w)[0]
    return out


def loop_entry(x, x0, t, w):
    """What comes before a pass: the stream and the embedding output mixed, then the vector of the pass."""
    return torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]


MIXERS = {"attention": mixer_attention, "attention_2": mixer_attention_2, "delta": mixer_delta}


def schedule(cfg):
    """[(layer, pass or None)] in the order they run; the pass where a layer is the first of one."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if lp is None:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        order += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return order + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    norm = lambda v, name: layer_norm(v, eps, w[name], w[name + ".b"])
    x = x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, t in schedule(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = loop_entry(x, x0, t, w)
        x = x + m * norm(MIXERS[L["type"]](norm(x, p + "norm1"), p + "mix.", L["mixer"], w, eps), p + "norm1b")
        if L["mlp"] is not None:
            x = x + m * norm(experts(norm(x, p + "norm2"), p + "mlp.", L["mlp"], w), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ w["embed"].T
