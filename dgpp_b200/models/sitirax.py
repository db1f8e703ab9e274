"""Sitirax decoder family: layers of two kinds in any order, each a pre-norm mixer sublayer and, where the configuration
names one, a gated feed-forward sublayer (tanh-gelu).

  parallel        two mixers side by side on the same input, their outputs scaled and added:
                  left   sliding-window GQA, per-head query / key norms, no rotation, value heads of their own width
                  right  lightning attention (constant decay per head), normed over all heads together and gated
  channel_delta   gated delta rule with a decay per key channel, a causal depthwise convolution in front, low-rank decay and
                  output-gate projections, a per-head norm behind

A layer may take its weights from another one (`weights_of`); it still has a cache or state of its own.  The head is the
embedding table.  The residual stream, norms, scores, gates, decays and states are fp32; projections and activations are
bf16 (or everything fp32 with dtype float32).

Weights are packed for the kernels when they are loaded: all projections of a mixer that read its input form one matrix,
the two output projections of a parallel layer another (the mixers write their scaled outputs side by side), the low-rank
pairs of the delta rule a block-diagonal one.  Head widths are padded with zero rows and columns to what the kernels take,
rows of every matrix to multiples of 8 columns.

``SitiraxModel.forward_reference`` restates the packed model in PyTorch; ``SitiraxRunner`` runs it on the sm_100a kernels
(`ops/mixers.py`), prompt portions and decoded tokens of several requests in one pass.
"""
from __future__ import annotations

import math
from dataclasses import asdict, dataclass
from typing import Callable, Dict, List, Optional, Tuple, Union

import torch
import torch.nn.functional as F

from ..ops import core as ops
from ..ops import mixers as mx
from ..quant.formats import QuantLinear
from .packing import only_keys as _only, pad_cols as _pad_cols, pad_rows as _pad_rows, pad_vec as _pad_vec, up8
from .rows import RowRunner, RowRuns

BF = torch.bfloat16
UNIT_EPS = 1e-6                 # inside the root of the delta rule's unit vectors


# ---------------------------------------------------------------------------------------------- configuration
@dataclass(frozen=True)
class WindowSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int


@dataclass(frozen=True)
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class ParallelSpec:
    left: WindowSpec
    right: LightningSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[ParallelSpec, DeltaSpec]
    ff: Optional[int]            # None: the layer has no feed-forward sublayer
    source: int                  # the layer whose tensors it uses (itself, unless it shares)


@dataclass
class SitiraxConfig:
    width: int
    vocab: int
    plan: List[LayerSpec]
    eps: float
    logit_scale: float
    page: int = 64

    @staticmethod
    def from_dict(d: dict) -> "SitiraxConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, kind = e["mixer"], e["type"]
            if kind == "parallel":
                _only(m, ("left", "right", "left_scale", "right_scale"), f"layer {i} mixer")
                _only(m["left"], ("heads", "kv_heads", "dim", "vdim", "scale", "mask"), f"layer {i} left mixer")
                _only(m["left"]["mask"], ("size",), f"layer {i} mask")
                _only(m["right"], ("heads", "dim", "vdim", "decay"), f"layer {i} right mixer")
                a, b = m["left"], m["right"]
                decay = tuple(float(x) for x in b["decay"])
                if len(decay) != b["heads"] or a["heads"] % a["kv_heads"]:
                    raise ValueError(f"layer {i}: {b['heads']} heads with {len(decay)} decays, {a['heads']} over {a['kv_heads']} heads")
                spec = ParallelSpec(WindowSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                                               int(a["mask"]["size"])),
                                    LightningSpec(int(b["heads"]), int(b["dim"]), int(b["vdim"]), decay),
                                    float(m["left_scale"]), float(m["right_scale"]))
            elif kind == "channel_delta":
                _only(m, ("heads", "kv_heads", "dim", "vdim", "conv"), f"layer {i} mixer")
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"layer {i}: {m['heads']} heads over {m['kv_heads']} key heads")
                spec = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            ff = None
            if e.get("mlp") is not None:
                if e["mlp"].get("kind") != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {e['mlp'].get('kind')!r}")
                ff = int(e["mlp"]["ff"])
            layers.append(LayerSpec(spec, ff, int(e.get("weights_of", i))))
        for i, L in enumerate(layers):
            src = L.source
            if not 0 <= src < len(layers) or layers[src].source != src:
                raise ValueError(f"layer {i}: weights_of names no layer with weights of its own")
            if (layers[src].mixer, layers[src].ff) != (L.mixer, L.ff):
                raise ValueError(f"layer {i} shares the weights of layer {src} but is described differently")
        return SitiraxConfig(int(d["width"]), int(d["vocab"]), layers, float(d["norm"]["eps"]), float(d["logit_scale"]))

    def to_dict(self) -> dict:
        out = []
        for i, L in enumerate(self.plan):
            m = L.mixer
            if isinstance(m, ParallelSpec):
                left, right = asdict(m.left), asdict(m.right)
                left["mask"] = {"size": left.pop("window")}
                right["decay"] = list(right["decay"])
                e = {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}}
            else:
                mixer = asdict(m)
                mixer["conv"] = mixer.pop("taps")
                e = {"type": "channel_delta", "mixer": mixer}
            e["mlp"] = None if L.ff is None else {"kind": "dense", "ff": L.ff}
            if L.source != i:
                e["weights_of"] = L.source
            out.append(e)
        return {"architecture": "Sitirax", "width": self.width, "vocab": self.vocab, "layers": out, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale}

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def layers(self) -> int:
        return len(self.plan)

    @staticmethod
    def uniform(layers: int, width: int, vocab: int, parallel: ParallelSpec, delta: DeltaSpec, ff: int, every: int = 2,
                eps: float = 1e-5, logit_scale: float = 1.0) -> "SitiraxConfig":
        """`layers` layers, every `every`-th (from the first) parallel with a feed-forward of width ff, the others delta layers
        with one too."""
        return SitiraxConfig(width, vocab, [LayerSpec(parallel if i % every == 0 else delta, ff, i) for i in range(layers)], eps,
                             logit_scale)


def tensor_shapes(cfg: SitiraxConfig, rank_a: int = 0, rank_g: int = 0) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint of `cfg`.  The ranks of the low-rank pairs are not part of a configuration: loading
    takes them from the tensors, the default here is the key / value head width."""
    H, out = cfg.width, {"embed": (cfg.vocab, cfg.width)}
    for i, L in enumerate(cfg.plan):
        if L.source != i:
            continue
        p, m = f"l{i}.", L.mixer
        out[p + "norm1"] = (H,)
        if isinstance(m, ParallelSpec):
            a, b = m.left, m.right
            lp, rp = p + "mix.left.", p + "mix.right."
            out.update({lp + "q": (a.heads * a.dim, H), lp + "k": (a.kv_heads * a.dim, H), lp + "v": (a.kv_heads * a.vdim, H),
                        lp + "q.norm": (a.dim,), lp + "k.norm": (a.dim,), lp + "o": (H, a.heads * a.vdim),
                        rp + "q": (b.heads * b.dim, H), rp + "k": (b.heads * b.dim, H), rp + "v": (b.heads * b.vdim, H),
                        rp + "g": (b.heads * b.vdim, H), rp + "o": (H, b.heads * b.vdim), rp + "norm": (b.heads * b.vdim,)})
        else:
            ra, rg = rank_a or m.dim, rank_g or m.vdim
            mp, nk, nv = p + "mix.", m.kv_heads * m.dim, m.heads * m.vdim
            out.update({mp + "q": (nk, H), mp + "k": (nk, H), mp + "v": (nv, H), mp + "q.conv": (nk, m.taps), mp + "k.conv": (nk, m.taps),
                        mp + "v.conv": (nv, m.taps), mp + "b": (m.heads, H), mp + "A_log": (m.heads,), mp + "norm": (m.vdim,),
                        mp + "a1": (ra, H), mp + "a2": (m.heads * m.dim, ra), mp + "dt_bias": (m.heads * m.dim,),
                        mp + "g1": (rg, H), mp + "g2": (nv, rg), mp + "o": (H, nv)})
        if L.ff is not None:
            out.update({p + "norm2": (H,), p + "mlp.gate": (L.ff, H), p + "mlp.up": (L.ff, H), p + "mlp.down": (H, L.ff)})
    out["final.norm"] = (H,)
    return out


def random_tensors(cfg: SitiraxConfig, seed: int = 0, rank_a: int = 0, rank_g: int = 0, std: Optional[float] = None,
                   device="cpu") -> Dict[str, torch.Tensor]:
    """bf16 tensors of a random-init checkpoint: N(0, 1 / fan-in) matrices (or N(0, std^2)), norm weights around one, decays
    spread from short to long memories."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)
    uni = lambda n, lo, hi: lo + (hi - lo) * torch.rand(n, device=device, generator=g)
    out = {}
    for name, s in tensor_shapes(cfg, rank_a, rank_g).items():
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            t = 1 + 0.2 * rnd(*s)
        elif name.endswith("A_log"):
            t = uni(s[0], -4.0, 0.0)
        elif name.endswith("dt_bias"):
            t = uni(s[0], -4.0, -1.0)
        elif name.endswith(".conv"):
            t = 0.6 * rnd(*s)
        elif name == "embed":
            t = rnd(*s) * (std * 4 if std else 0.25)
        else:
            t = rnd(*s) * (std or s[1] ** -0.5)
        out[name] = t.to(BF)
    return out


# ---------------------------------------------------------------------------------------------- packed weights
@dataclass
class Packed:
    """Kernel-ready weights of one layer (shared by the layers that use them)."""
    norm1: torch.Tensor                        # fp32 [Hp]
    w_in: QuantLinear                          # every projection of the mixer's input
    w_out: QuantLinear                         # [Hp, outputs of the mixer(s)]
    n_out: int
    window: Optional[mx.WindowHeads] = None
    q_norm: Optional[torch.Tensor] = None      # fp32 [D]
    k_norm: Optional[torch.Tensor] = None
    state: Optional[mx.StateHeads] = None
    gate_off: int = 0                          # parallel: the lightning gate's columns of w_in; delta: a1's columns
    right_norm: Optional[torch.Tensor] = None  # parallel: fp32 [heads * DV]
    w_low: Optional[QuantLinear] = None        # delta: block-diagonal [decays | gates] over [a1 | g1]
    norm2: Optional[torch.Tensor] = None
    gate_up: Optional[QuantLinear] = None
    down: Optional[QuantLinear] = None

    def matrices(self) -> List[QuantLinear]:
        return [w for w in (self.w_in, self.w_out, self.w_low, self.gate_up, self.down) if w is not None]


class SitiraxModel:
    def __init__(self, cfg: SitiraxConfig, embed: torch.Tensor, layers: List[Packed], final_norm: torch.Tensor, dtype: torch.dtype):
        self.cfg, self.embed, self.layers, self.final_norm, self.dtype = cfg, embed, layers, final_norm, dtype
        fmt = "fp32" if dtype == torch.float32 else "bf16"
        self.head = QuantLinear(fmt, cfg.vocab, embed.shape[1], embed, None, cfg.logit_scale)
        self.tp_size, self.tp_rank = 1, 0

    @property
    def hp(self) -> int:
        return self.embed.shape[1]

    @staticmethod
    def from_tensors(cfg: SitiraxConfig, get: Callable[[str], torch.Tensor], device="cuda", dtype: torch.dtype = BF) -> "SitiraxModel":
        """Packs the checkpoint tensors `get(name)` returns; shapes are checked against the configuration."""
        shapes = tensor_shapes(cfg)
        H, Hp = cfg.width, up8(cfg.width)
        fmt = "fp32" if dtype == torch.float32 else "bf16"

        def t(name: str) -> torch.Tensor:
            v, want = get(name), shapes[name]
            low = name.endswith((".a1", ".g1", ".a2", ".g2"))       # their rank is the tensor's own
            ok = len(v.shape) == len(want) and all(a == b for k, (a, b) in enumerate(zip(v.shape, want))
                                                   if not (low and k == (0 if name.endswith("1") else 1)))
            if not ok:
                raise ValueError(f"{name} is {tuple(v.shape)}, the configuration wants {want}")
            return v.to(device=device, dtype=torch.float32)

        def lin(w: torch.Tensor) -> QuantLinear:
            return QuantLinear(fmt, w.shape[0], w.shape[1], w.to(dtype).contiguous())

        vec = lambda v: v.contiguous()
        hid = lambda w: _pad_cols(w, 1, H, Hp)                      # matrices that read the stream
        hout = lambda w: _pad_rows(w, 1, H, Hp)                     # matrices that write it
        hvec = lambda name: vec(_pad_vec(t(name), 1, H, Hp))

        def parallel(p: str, m: ParallelSpec) -> Packed:
            a, b = m.left, m.right
            D, DV = mx.pad_to(a.dim, mx.ATTN_WIDTHS), mx.pad_to(a.vdim, mx.ATTN_WIDTHS)
            RK, RV = mx.pad_to(b.dim, mx.STATE_WIDTHS), mx.pad_to(b.vdim, mx.STATE_WIDTHS)
            lp, rp = p + "left.", p + "right."
            blocks = [_pad_rows(t(lp + "q"), a.heads, a.dim, D), _pad_rows(t(lp + "k"), a.kv_heads, a.dim, D),
                      _pad_rows(t(lp + "v"), a.kv_heads, a.vdim, DV), _pad_rows(t(rp + "q"), b.heads, b.dim, RK),
                      _pad_rows(t(rp + "k"), b.heads, b.dim, RK), _pad_rows(t(rp + "v"), b.heads, b.vdim, RV),
                      _pad_rows(t(rp + "g"), b.heads, b.vdim, RV)]
            off = [0]
            for w in blocks:
                off.append(off[-1] + w.shape[0])
            w_o = torch.cat([_pad_cols(t(lp + "o"), a.heads, a.vdim, DV), _pad_cols(t(rp + "o"), b.heads, b.vdim, RV)], 1)
            return Packed(hvec(p[:-4] + "norm1"), lin(hid(torch.cat(blocks))), lin(hout(w_o)), w_o.shape[1],
                          window=mx.WindowHeads(a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, cfg.eps, off[0], off[1], off[2]),
                          q_norm=vec(_pad_vec(t(lp + "q.norm"), 1, a.dim, D)), k_norm=vec(_pad_vec(t(lp + "k.norm"), 1, a.dim, D)),
                          state=mx.StateHeads(b.heads, b.heads, b.dim, b.vdim, off[3], eps=cfg.eps,
                                              decay=torch.tensor(b.decay, dtype=torch.float32, device=device)),
                          gate_off=off[6], right_norm=vec(_pad_vec(t(rp + "norm"), b.heads, b.vdim, RV)))

        def delta(p: str, m: DeltaSpec) -> Packed:
            K, V = mx.pad_to(m.dim, mx.STATE_WIDTHS), mx.pad_to(m.vdim, mx.STATE_WIDTHS)
            q, k, v = (_pad_rows(t(p + n), g, d, dp) for n, g, d, dp in
                       (("q", m.kv_heads, m.dim, K), ("k", m.kv_heads, m.dim, K), ("v", m.heads, m.vdim, V)))
            a1, g1, a2, g2 = t(p + "a1"), t(p + "g1"), t(p + "a2"), t(p + "g2")
            ra, rg = a1.shape[0], g1.shape[0]
            if a2.shape[1] != ra or g2.shape[1] != rg:
                raise ValueError(f"{p}a1 / a2 or {p}g1 / g2 differ in rank")
            blocks = [q, k, v, _pad_rows(t(p + "b"), 1, m.heads, up8(m.heads)), _pad_rows(a1, 1, ra, up8(ra)), _pad_rows(g1, 1, rg, up8(rg))]
            off = [0]
            for w in blocks:
                off.append(off[-1] + w.shape[0])
            low = torch.zeros(m.heads * (K + V), up8(ra) + up8(rg), device=device)
            low[:m.heads * K, :ra] = _pad_rows(a2, m.heads, m.dim, K)
            low[m.heads * K:, up8(ra):up8(ra) + rg] = _pad_rows(g2, m.heads, m.vdim, V)
            conv = torch.cat([_pad_rows(t(p + n + ".conv"), g, d, dp) for n, g, d, dp in
                              (("q", m.kv_heads, m.dim, K), ("k", m.kv_heads, m.dim, K), ("v", m.heads, m.vdim, V))])
            w_o = _pad_cols(t(p + "o"), m.heads, m.vdim, V)
            return Packed(hvec(p[:-4] + "norm1"), lin(hid(torch.cat(blocks))), lin(hout(w_o)), w_o.shape[1],
                          state=mx.StateHeads(m.heads, m.kv_heads, m.dim, m.vdim, off[0], off[3], cfg.eps, vec(conv.T),
                                              vec(t(p + "A_log")), vec(_pad_vec(t(p + "dt_bias"), m.heads, m.dim, K)),
                                              norm_w=vec(_pad_vec(t(p + "norm"), 1, m.vdim, V))),
                          gate_off=off[4], w_low=lin(low))

        own: Dict[int, Packed] = {}
        for i in sorted({L.source for L in cfg.plan}):
            L, p = cfg.plan[i], f"l{i}."
            w = parallel(p + "mix.", L.mixer) if isinstance(L.mixer, ParallelSpec) else delta(p + "mix.", L.mixer)
            if L.ff is not None:
                fp = up8(L.ff)
                w.norm2 = hvec(p + "norm2")
                w.gate_up = lin(hid(torch.cat([_pad_rows(t(p + "mlp.gate"), 1, L.ff, fp), _pad_rows(t(p + "mlp.up"), 1, L.ff, fp)])))
                w.down = lin(hout(_pad_cols(t(p + "mlp.down"), 1, L.ff, fp)))
            own[i] = w
        layers = [own[L.source] for L in cfg.plan]
        embed = hid(t("embed")).to(dtype).contiguous()
        return SitiraxModel(cfg, embed, layers, hvec("final.norm"), dtype)

    @staticmethod
    def random_init(cfg: SitiraxConfig, device="cuda", seed: int = 0, std: Optional[float] = None, dtype: torch.dtype = BF,
                    rank_a: int = 0, rank_g: int = 0) -> "SitiraxModel":
        w = random_tensors(cfg, seed, rank_a, rank_g, std, device)
        return SitiraxModel.from_tensors(cfg, w.__getitem__, device, dtype)

    def weight_bytes(self) -> int:
        seen = {id(w): w.nbytes for L in self.layers for w in L.matrices()}
        return self.head.nbytes + sum(seen.values())

    # ------------------------------------------------------------------ oracle
    @torch.no_grad()
    def forward_reference(self, tokens: torch.Tensor) -> torch.Tensor:
        """fp32 logits [T, V] of one request from position 0, on the packed weights (fp32 arithmetic, any device)."""
        c = self.cfg
        x = self.embed.float()[tokens.to(self.embed.device).long()]
        norm = lambda v, w, n: v * torch.rsqrt(v.pow(2).sum(-1, keepdim=True) / n + c.eps) * w
        mm = lambda v, w: v @ w.payload.float().T
        T = x.shape[0]
        for L, P in zip(c.plan, self.layers):
            proj = mm(norm(x, P.norm1, c.width), P.w_in)
            mixed = self._parallel_reference(L.mixer, P, proj, norm) if P.window is not None else self._delta_reference(P, proj, norm)
            x = x + mm(mixed, P.w_out)
            if P.gate_up is not None:
                g, u = mm(norm(x, P.norm2, c.width), P.gate_up).chunk(2, -1)
                x = x + mm(F.gelu(g, approximate="tanh") * u, P.down)
        return mm(norm(x, self.final_norm, c.width), self.head) * c.logit_scale

    def _parallel_reference(self, m: ParallelSpec, P: Packed, proj, norm):
        T, g, s = proj.shape[0], P.window, P.state
        q = norm(proj[:, g.q_off:g.k_off].view(T, g.hq, g.D), P.q_norm, g.dim)
        k = norm(proj[:, g.k_off:g.v_off].view(T, g.hkv, g.D), P.k_norm, g.dim).repeat_interleave(g.hq // g.hkv, 1)
        v = proj[:, g.v_off:g.v_off + g.hkv * g.DV].view(T, g.hkv, g.DV).repeat_interleave(g.hq // g.hkv, 1)
        i = torch.arange(T, device=proj.device)
        dist = i[:, None] - i[None, :]
        score = torch.einsum("ihd,jhd->hij", q, k) * g.scale
        score = score.masked_fill((dist < 0) | (dist >= g.window), float("-inf"))
        left = torch.einsum("hij,jhd->ihd", score.softmax(-1), v).reshape(T, -1) * m.left_scale
        n = s.hv * s.DK
        q, k = (F.silu(proj[:, s.c_off + a:s.c_off + a + n]).view(T, s.hv, s.DK) for a in (0, n))
        v = F.silu(proj[:, s.c_off + 2 * n:P.gate_off]).view(T, s.hv, s.DV)
        S, outs = proj.new_zeros(s.hv, s.DK, s.DV), []
        for t in range(T):
            S = S * s.decay[:, None, None] + k[t, :, :, None] * v[t, :, None, :]
            outs.append(torch.einsum("hkv,hk->hv", S, q[t]))
        o = norm(torch.stack(outs).reshape(T, -1), P.right_norm, s.hv * s.vdim)
        return torch.cat([left, o * torch.sigmoid(proj[:, P.gate_off:P.gate_off + s.hv * s.DV]) * m.right_scale], 1)

    def _delta_reference(self, P: Packed, proj, norm):
        T, s = proj.shape[0], P.state
        nk, nv, ratio = s.hk * s.DK, s.hv * s.DV, s.hv // s.hk
        hist = F.pad(proj[:, s.c_off:s.c_off + s.channels], (0, 0, s.taps - 1, 0))
        act = F.silu(sum(hist[j:j + T] * s.conv_w[j] for j in range(s.taps)))
        unit = lambda a: a * torch.rsqrt(a.pow(2).sum(-1, keepdim=True) + UNIT_EPS)
        q = (unit(act[:, :nk].view(T, s.hk, s.DK)) * s.dim ** -0.5).repeat_interleave(ratio, 1)
        k = unit(act[:, nk:2 * nk].view(T, s.hk, s.DK)).repeat_interleave(ratio, 1)
        v = act[:, 2 * nk:].view(T, s.hv, s.DV)
        beta = torch.sigmoid(proj[:, s.b_off:s.b_off + s.hv])
        low = proj[:, P.gate_off:P.gate_off + P.w_low.k] @ P.w_low.payload.float().T
        g = torch.exp(-torch.exp(s.A_log)[:, None] * F.softplus((low[:, :s.hv * s.DK] + s.dt_bias).view(T, s.hv, s.DK)))
        S, outs = proj.new_zeros(s.hv, s.DK, s.DV), []
        for t in range(T):
            S = S * g[t, :, :, None]
            u = beta[t, :, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
            S = S + k[t, :, :, None] * u[:, None, :]
            outs.append(torch.einsum("hkv,hk->hv", S, q[t]))
        o = norm(torch.stack(outs), s.norm_w, s.vdim) * torch.sigmoid(low[:, s.hv * s.DK:]).view(T, s.hv, s.DV)
        return o.reshape(T, nv)


# ---------------------------------------------------------------------------------------------- kernel runner
class SitiraxRunner(RowRunner):
    """Executes the model on the sm_100a kernels.  A request holds pages of the shared key / value pool (one table for all
    attention layers) and one slot of every layer's fp32 state; both are reused without clearing (a request's first token
    starts from zero states)."""

    mixed_runs = True

    def __init__(self, model: SitiraxModel, max_rows: int, slots: int, max_seq_len: int, device, pool_tokens: int = 0):
        c = model.cfg
        self.m, self.model, self.c = model, model, c
        max_rows = max(max_rows, slots)
        T = model.dtype
        self.kv_index = {i: j for j, i in enumerate(i for i, P in enumerate(model.layers) if P.window is not None)}
        heads = [model.layers[i].window for i in self.kv_index]
        self._init_pool(slots, device, [g.kv_shape for g in heads], T, c.page, max_seq_len, max_rows, pool_tokens)
        self.states = [P.state.new_state(slots, device) for P in model.layers]
        e = lambda n, dt: torch.empty(n, dtype=dt, device=device)
        R, Hp = max_rows, model.hp
        self.x, self.dx, self.xn = e(R * Hp, torch.float32).view(R, Hp), e(R * Hp, torch.float32).view(R, Hp), e(R * Hp, T).view(R, Hp)
        big = lambda vals: max(list(vals) + [1])
        self.proj = e(R * big(P.w_in.n for P in model.layers), T)
        self.mixed = e(R * big(P.n_out for P in model.layers), T)
        self.low = e(R * big(P.w_low.n for P in model.layers if P.w_low is not None), torch.float32)
        self.o = e(R * big(P.state.hv * P.state.DV for P in model.layers), torch.float32)
        self.gu = e(R * big(P.gate_up.n for P in model.layers if P.gate_up is not None), T)
        self.act = e(R * big(P.down.k for P in model.layers if P.down is not None), T)
        self.prep = e(big(P.state.prep_floats(R, slots) for P in model.layers), torch.float32)
        self.tc_prefill = True                     # prompt rows' window attention on the tensor cores where the kernel takes them
        self.max_splits = 32
        self.scratch = (e(slots * big(g.hq for g in heads) * self.max_splits * 2, torch.float32),
                        e(slots * big(g.hq * g.DV for g in heads) * self.max_splits, torch.float32))
        self.max_span = self.kv.max_blocks * c.page
        self.capture: Optional[list] = None        # a list: receives the residual stream after every layer (tests, debugging)

    def _state_tensors(self):
        return [t for pair in self.states for t in pair if t is not None]

    def _lin(self, x: torch.Tensor, w: QuantLinear, out: torch.Tensor) -> torch.Tensor:
        if w.fmt == "bf16" and out.dtype == torch.float32:
            return ops.gemm_tc(x, w, out32=out)
        return ops.linear(x, w, out=out)

    def _parallel(self, i: int, P: Packed, proj, mixed, positions, row_req, runs: Optional[RowRuns]) -> None:
        m, g, s = self.c.plan[i].mixer, P.window, P.state
        rows, n_left = proj.shape[0], g.hq * g.DV
        cache, bt = self.kv.layers[self.kv_index[i]], self.kv.block_table
        o = self.o[:rows * s.hv * s.DV].view(rows, s.hv * s.DV)
        if runs is None:
            mx.window_attn(g, proj, P.q_norm, P.k_norm, cache, bt, row_req, positions, mixed, m.left_scale, fused=True,
                           splits=g.splits(rows, self.max_span, self.max_splits), scratch=self.scratch)
            mx.linear_state(s, proj, *self.states[i], row_req, positions, o=o)
        else:
            mx.qk_norm_append(g, proj, P.q_norm, P.k_norm, cache, bt, row_req, positions)
            if self.tc_prefill and mx.window_prefill_usable(g, proj, cache.page):
                mx.window_prefill(g, proj, cache, bt, row_req, positions, runs, mixed, m.left_scale)
            else:
                mx.window_attn(g, proj, P.q_norm, P.k_norm, cache, bt, row_req, positions, mixed, m.left_scale)
            mx.linear_state(s, proj, *self.states[i], row_req, positions, runs=runs, prep=self.prep, o=o)
        mx.gated_group_norm(o, proj[:, P.gate_off:], P.right_norm, mixed[:, n_left:], 1, s.hv * s.vdim, self.c.eps, m.right_scale)

    def _delta(self, i: int, P: Packed, proj, mixed, positions, row_req, runs: Optional[RowRuns]) -> None:
        s, rows = P.state, proj.shape[0]
        low = self._lin(proj[:, P.gate_off:P.gate_off + P.w_low.k], P.w_low, self.low[:rows * P.w_low.n].view(rows, P.w_low.n))
        if runs is None:
            mx.linear_state(s, proj, *self.states[i], row_req, positions, low=low, out=mixed)
            return
        o = self.o[:rows * s.hv * s.DV].view(rows, s.hv * s.DV)
        mx.linear_state(s, proj, *self.states[i], row_req, positions, low=low, runs=runs, prep=self.prep, o=o)
        mx.gated_group_norm(o, low[:, s.hv * s.DK:], s.norm_w, mixed, s.hv, s.vdim, self.c.eps)

    def _layers(self, tokens, positions, row_req, runs: Optional[RowRuns]) -> torch.Tensor:
        """-> the final norm's rows."""
        m, c, rows = self.m, self.c, tokens.shape[0]
        x, xn, dx = self.x[:rows], self.xn[:rows], self.dx[:rows]
        mx.embed_rows(tokens, m.embed, x)
        view = lambda buf, n: buf[:rows * n].view(rows, n)
        delta = None
        for i, P in enumerate(m.layers):
            mx.resid_norm(x, P.norm1, c.width, c.eps, xn, delta)
            proj, mixed = self._lin(xn, P.w_in, view(self.proj, P.w_in.n)), view(self.mixed, P.n_out)
            (self._parallel if P.window is not None else self._delta)(i, P, proj, mixed, positions, row_req, runs)
            delta = self._lin(mixed, P.w_out, dx)
            if P.gate_up is not None:
                mx.resid_norm(x, P.norm2, c.width, c.eps, xn, delta)
                gu = self._lin(xn, P.gate_up, view(self.gu, P.gate_up.n))
                delta = self._lin(mx.geglu(gu, view(self.act, P.down.k)), P.down, dx)
            if self.capture is not None:
                self.capture.append((x + delta)[:, :c.width])
        return mx.resid_norm(x, m.final_norm, c.width, c.eps, xn, delta)

    def _head(self, rows: torch.Tensor) -> torch.Tensor:
        return self._lin(rows, self.m.head, torch.empty(rows.shape[0], self.c.vocab, dtype=torch.float32, device=self.dev))

    @torch.no_grad()
    def forward(self, tokens, positions, row_req, chunk_slot=None, all_logits=True, pos0=None, extra=None):
        """One new token per row (distinct requests) -> fp32 logits [rows, V]."""
        assert chunk_slot is None, "prompt portions go through forward_runs"
        return self._head(self._layers(tokens, positions, row_req, None))

    @torch.no_grad()
    def forward_runs(self, tokens, positions, row_req, runs: RowRuns, logit_rows: torch.Tensor):
        xn = self._layers(tokens, positions, row_req, runs)
        return self._head(xn.index_select(0, logit_rows)) if logit_rows.numel() else None
