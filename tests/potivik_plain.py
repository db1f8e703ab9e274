"""Plain, slow restatement of the Potivik design on the CPU: one function per mechanism, whole sequences, no cache, no
kernels.  `cfg` is the parsed config.json, `w` maps tensor names to tensors.  Every function takes the working dtype
from its inputs (the tests run it in float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_pairs(x, base, dims, first=0):
    """x [T, ..., d], row t at position first + t: the first `dims` columns turned as neighbouring pairs (0, 1), (2, 3), ..."""
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = (first + t) * base ** (-2 * i / dims)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def window_attention(q, k, v, scale, size):
    """q, k [T, H, d], v [T, H, e] -> [T, H, e]; query i sees keys i - size + 1 .. i."""
    out = q.new_zeros(q.shape[0], q.shape[1], v.shape[2])
    for i in range(q.shape[0]):
        lo = max(0, i - size + 1)
        s = torch.einsum("jhd,hd->hj", k[lo:i + 1], q[i]) * scale
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhe->he", p / p.sum(-1, keepdim=True), v[lo:i + 1])
    return out


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n] (last column: the current token) with zeros before the start, plus bias, then silu."""
    n = taps.shape[1]
    pad = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return silu(sum(pad[j:j + x.shape[0]] * taps[:, j] for j in range(n)) + bias)


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, e], B, C [T, G, n], dt [T, H] (already positive) -> [T, H, e]."""
    T, H, e = x.shape
    group = torch.arange(H) // (H // B.shape[1])
    S, out = x.new_zeros(H, B.shape[2], e), []
    for t in range(T):
        S = S * torch.exp(-torch.exp(A_log) * dt[t])[:, None, None] + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        out.append((S * C[t][group][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(out)


def gated_part_norm(y, z, parts, w, eps):
    """The gate first, then every one of `parts` equal runs of columns by its own root mean square."""
    a = y * silu(z)
    return rms(a.reshape(*a.shape[:-1], parts, -1), eps).reshape(a.shape) * w


def mixer_latent_attention(h, p, c, w, eps):
    T, H, d, r = h.shape[0], c["heads"], c["dim"], c["rot_dim"]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    down = h @ w[p + "dkv"].T
    lat = rms(down[:, :c["kv_rank"]], eps) * w[p + "dkv.norm"]
    base, dims = c["rot"]["base"], c["rot"]["dims"]
    qr = rotate_pairs(q[:, :, d:], base, dims)
    kr = rotate_pairs(down[:, c["kv_rank"]:], base, dims)
    k = torch.cat([(lat @ w[p + "uk"].T).view(T, H, d), kr[:, None].expand(T, H, r)], -1)
    v = (lat @ w[p + "uv"].T).view(T, H, c["vdim"])
    o = window_attention(torch.cat([q[:, :, :d], qr], -1), k, v, c["scale"], c["mask"]["size"])
    return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, -1) @ w[p + "o"].T


def mixer_mamba2(h, p, c, w, eps):
    T, H, G, N, e = h.shape[0], c["heads"], c["groups"], c["state"], c["vdim"]
    inner = H * e
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], -1)
    x, B, C = causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]).split([inner, G * N, G * N], -1)
    y = state_space(x.view(T, H, e), B.view(T, G, N), C.view(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_part_norm(y.reshape(T, inner), z, c["norm_groups"], w[p + "norm"], eps) @ w[p + "o"].T


def clamped_glu(h, p, w, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def experts(h, p, c, w):
    """Input-weighted routing: an expert gets its token times the token's score for it."""
    score = sigmoid(h @ w[p + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.argsort(-score[t], stable=True)[:c["router"]["top"]].tolist():
            out[t] += clamped_glu((score[t, e] * h[t])[None], f"{p}e{e}.", w, c["expert"]["limit"])[0]
    if c.get("shared") is not None:
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * clamped_glu(h, p + "shared.", w, c["shared"]["limit"])
    return out


def feed_forward(h, p, c, w):
    return clamped_glu(h, p, w, c["limit"]) if c["kind"] == "dense" else experts(h, p, c, w)


def token_side(x, tokens, i, p, dim, w, eps):
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms(y, eps) * w[p + "side.norm"]


MIXERS = {"latent_attention": mixer_latent_attention, "mamba2": mixer_mamba2}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer."""
    eps, tokens = cfg["norm"]["eps"], torch.as_tensor(tokens, dtype=torch.long)
    norm = lambda v, name: layer_norm(v, eps) * w[name]
    x = w["embed"][tokens]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm(MIXERS[L["type"]](norm(x, p + "norm1"), p + "mix.", L["mixer"], w, eps), p + "norm1b")
        if L["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, p + "norm2"), p + "mlp.", L["mlp"], w), p + "norm2b")
        x = x + token_side(x, tokens, i, p, cfg["token_side"]["dim"], w, eps)
        if layers_out is not None:
            layers_out.append(x)
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(norm(x, "final.norm") @ w["head"].T / cap)
