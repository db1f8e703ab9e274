"""Plain, slow restatement of the Sitirax design on the CPU: one function per mechanism, whole sequences, no cache, no
kernels.  `cfg` is the parsed config.json, `w` maps tensor names to tensors.  Every function takes the working dtype
from its inputs (the tests run it in float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def window_attention(q, k, v, scale, size):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; query i sees keys i - size + 1 .. i."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = q.new_zeros(T, H, v.shape[2])
    for i in range(T):
        lo = max(0, i - size + 1)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, g]
    return out


def lightning(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], decay [H] -> outputs [T, H, e] of S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[2])
    out = []
    for t in range(T):
        S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def causal_conv(x, taps):
    """x [T, C], taps [C, n] (last column: the current token) with zeros before the start, then silu."""
    n = taps.shape[1]
    pad = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    y = sum(pad[j:j + x.shape[0]] * taps[:, j] for j in range(n))
    return silu(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """q, k [T, G, d] (unit, q scaled), v [T, H, e], beta [T, H], g [T, H, d] decays in (0, 1] -> [T, H, e]."""
    T, H = beta.shape
    G = q.shape[1]
    head = torch.arange(H) // (H // G)
    S = v.new_zeros(H, q.shape[2], v.shape[2])
    out = []
    for t in range(T):
        kt, qt = k[t][head], q[t][head]
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - (S * kt[:, :, None]).sum(1))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append((S * qt[:, :, None]).sum(1))
    return torch.stack(out)


def mixer_left(h, p, c, w, eps):
    T = h.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d)
    k = (h @ w[p + "k"].T).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, e)
    q, k = rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"]
    return window_attention(q, k, v, c["scale"], c["mask"]["size"]).reshape(T, H * e) @ w[p + "o"].T


def mixer_right(h, p, c, w, eps):
    T = h.shape[0]
    H, d, e = c["heads"], c["dim"], c["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, d)
    k = silu(h @ w[p + "k"].T).view(T, H, d)
    v = silu(h @ w[p + "v"].T).view(T, H, e)
    o = lightning(q, k, v, torch.tensor(c["decay"], dtype=h.dtype)).reshape(T, H * e)
    return (rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer_parallel(h, p, c, w, eps):
    return (c["left_scale"] * mixer_left(h, p + "left.", c["left"], w, eps)
            + c["right_scale"] * mixer_right(h, p + "right.", c["right"], w, eps))


def mixer_channel_delta(h, p, c, w, eps):
    T = h.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = unit(causal_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, G, d)) * d ** -0.5
    k = unit(causal_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, d))
    v = causal_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(T, H, e)
    beta = sigmoid(h @ w[p + "b"].T)
    a = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, d)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * softplus(a))
    o = delta_rule(q, k, v, beta, g)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, e)
    return (rms(o, eps) * w[p + "norm"] * gate).reshape(T, H * e) @ w[p + "o"].T


MIXERS = {"parallel": mixer_parallel, "channel_delta": mixer_channel_delta}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % L.get("weights_of", i)
        x = x + MIXERS[L["type"]](rms(x, eps) * w[p + "norm1"], p + "mix.", L["mixer"], w, eps)
        if L["mlp"] is not None:
            h = rms(x, eps) * w[p + "norm2"]
            x = x + (gelu_tanh(h @ w[p + "mlp.gate"].T) * (h @ w[p + "mlp.up"].T)) @ w[p + "mlp.down"].T
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T * cfg["logit_scale"]
