"""Vevapel decoder family: layers of three kinds in any order, some of them run several times in a row with the same weights.

  attention     full causal attention, query and key norms over the whole projection, a query temperature that grows with the position,
                an output gate per head; no rotation
  attention_2   differential attention (two attentions over the same values, one subtracted from the other) inside chunks of positions,
                rotated halves, an output gate per column
  delta         gated delta rule with one decay per head, a causal depthwise convolution in front, a per-head norm and a gate behind

  x <- x + m norm1b(mixer(norm1(x)));  x <- x + m norm2b(ff(norm2(x)))  (where the layer has a feed-forward: routed experts, weighed by
  the softmax over the chosen logits);  before every pass of the loop x <- W_in [x; embedding output] + step[pass]

Norms are layer norms with weight and bias.  The head is the embedding table.  Every pass of a looped layer has its own cache or state.
The residual stream, norms, angles, scores, router, gates of the recurrence, decays and states are fp32; projections and activations are
bf16 (or everything fp32 with dtype float32).

Weights are packed for the kernels when they are loaded: every reader of a mixer's input is one matrix (q | k | v | gates; q | k | v |
strengths | decays | gates), the experts two stacks.  Head widths are padded with zeros to what the kernels take, rows of every matrix
to multiples of 8 columns; the query heads of a differential layer are laid out [key head][map][head of the group].

``VevapelModel.forward_reference`` restates the packed model in PyTorch; ``VevapelRunner`` runs it on the sm_100a kernels
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
from .packing import only_keys, pad_cols, pad_rows, pad_vec, up8
from .row_moe import RowExperts, RowExpertsScratch, run_experts
from .rows import RowRuns
from .window_rows import WindowRowRunner

BF = torch.bfloat16
UNIT_EPS = 1e-6                 # inside the root of the delta rule's unit vectors


# ---------------------------------------------------------------------------------------------- configuration
@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float
    temp_every: int


@dataclass(frozen=True)
class DiffSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    base: float
    rot: int                     # rotated columns of every map, column i with column i + rot / 2
    diff: float


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, DiffSpec, DeltaSpec]
    mlp: Optional[ExpertsSpec]


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


def _mixer(kind: str, m: dict, what: str):
    heads = ("heads", "kv_heads", "dim", "vdim")
    if kind == "attention":
        only_keys(m, heads + ("scale", "q_temp"), what)
        only_keys(m["q_temp"], ("coef", "every"), f"{what} temperature")
        if m["q_temp"]["every"] != int(m["q_temp"]["every"]) or m["q_temp"]["every"] < 1:
            raise ValueError(f"{what}: temperature every {m['q_temp']['every']} positions")
        spec = AttentionSpec(*(int(m[k]) for k in heads), float(m["scale"]), float(m["q_temp"]["coef"]), int(m["q_temp"]["every"]))
    elif kind == "attention_2":
        only_keys(m, heads + ("scale", "mask", "rot", "diff"), what)
        only_keys(m["mask"], ("size",), f"{what} mask")
        only_keys(m["rot"], ("base", "dims"), f"{what} rotation")
        spec = DiffSpec(*(int(m[k]) for k in heads), float(m["scale"]), int(m["mask"]["size"]), float(m["rot"]["base"]), int(m["rot"]["dims"]),
                        float(m["diff"]))
        if spec.rot % 2 or not 0 <= spec.rot <= spec.dim or spec.chunk < 1:
            raise ValueError(f"{what}: {spec.rot} of {spec.dim} columns rotated, chunks of {spec.chunk}")
    elif kind == "delta":
        only_keys(m, heads + ("conv",), what)
        spec = DeltaSpec(*(int(m[k]) for k in heads + ("conv",)))
    else:
        raise ValueError(f"{what}: unknown type {kind!r}")
    if spec.kv_heads < 1 or spec.heads % spec.kv_heads:
        raise ValueError(f"{what}: {spec.heads} heads over {spec.kv_heads} key heads")
    return spec


@dataclass
class VevapelConfig:
    width: int
    vocab: int
    plan: List[LayerSpec]
    loop: Optional[LoopSpec]
    eps: float
    embed_scale: float
    residual: float              # factor of what a sublayer adds to the stream
    page: int = 64

    def __post_init__(self):
        L = self.loop
        if L is not None and not (0 <= L.start < L.stop <= len(self.plan) and L.times >= 1):
            raise ValueError(f"layers {L.start} .. {L.stop - 1} of {len(self.plan)} run {L.times} times")

    @staticmethod
    def from_dict(d: dict) -> "VevapelConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            only_keys(e, ("type", "mixer"), f"layer {i}", ("mlp",))
            mlp, ff = e.get("mlp"), None
            if mlp is not None:
                if mlp.get("kind") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
                only_keys(mlp, ("kind", "expert", "router"), f"layer {i} experts")
                only_keys(mlp["expert"], ("ff",), f"layer {i} expert")
                only_keys(mlp["router"], ("experts", "top"), f"layer {i} router")
                ff = ExpertsSpec(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]))
                if not 1 <= ff.top <= min(ff.experts, mx.MAX_TOP) or ff.experts > mx.MAX_EXPERTS:
                    raise ValueError(f"layer {i}: {ff.top} of {ff.experts} experts")
            layers.append(LayerSpec(_mixer(e["type"], e["mixer"], f"layer {i} mixer"), ff))
        loop = d.get("loop")
        if loop is not None:
            only_keys(loop, ("start", "stop", "times"), "loop")
            loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        only_keys(d["embedding"], ("scale",), "embedding")
        return VevapelConfig(int(d["width"]), int(d["vocab"]), layers, loop, float(d["norm"]["eps"]), float(d["embedding"]["scale"]),
                             float(d["residual_mult"]))

    def to_dict(self) -> dict:
        out = []
        for L in self.plan:
            m = asdict(L.mixer)
            if isinstance(L.mixer, AttentionSpec):
                kind, m["q_temp"] = "attention", {"coef": m.pop("temp_coef"), "every": m.pop("temp_every")}
            elif isinstance(L.mixer, DiffSpec):
                kind, m["mask"], m["rot"] = "attention_2", {"size": m.pop("chunk")}, {"base": m.pop("base"), "dims": m["rot"]}
            else:
                kind, m["conv"] = "delta", m.pop("taps")
            ff = L.mlp
            out.append({"type": kind, "mixer": m, "mlp": None if ff is None else
                        {"kind": "moe", "expert": {"ff": ff.ff}, "router": {"experts": ff.experts, "top": ff.top}}})
        d = {"architecture": "Vevapel", "width": self.width, "vocab": self.vocab, "layers": out, "norm": {"eps": self.eps},
             "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual}
        if self.loop is not None:
            d["loop"] = asdict(self.loop)
        return d

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def layers(self) -> int:
        return len(self.plan)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, number of the pass that begins here or None) in the order of execution."""
        n, L = len(self.plan), self.loop
        if L is None:
            return [(i, None) for i in range(n)]
        out = [(i, None) for i in range(L.start)]
        for t in range(L.times):
            out += [(i, t if i == L.start else None) for i in range(L.start, L.stop)]
        return out + [(i, None) for i in range(L.stop, n)]

    @staticmethod
    def cycle(layers: int, width: int, vocab: int, mixers, moe: Optional[ExpertsSpec], loop: Optional[LoopSpec] = None, eps: float = 1e-5,
              embed_scale: float = 1.0, residual: float = 1.0) -> "VevapelConfig":
        """`layers` layers that take the given mixers in turn, all with the same experts."""
        return VevapelConfig(width, vocab, [LayerSpec(mixers[i % len(mixers)], moe) for i in range(layers)], loop, eps, embed_scale, residual)


def tensor_shapes(cfg: VevapelConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint of `cfg`."""
    H = cfg.width
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H)}

    def norm(name: str) -> None:
        out.update({name: (H,), name + ".b": (H,)})

    def biased(name: str, n: int, k: int) -> None:
        out.update({name: (n, k), name + ".b": (n,)})

    if cfg.loop is not None:
        out.update({"loop.in": (H, 2 * H), "loop.step": (cfg.loop.times, H)})
    for i, L in enumerate(cfg.plan):
        p, m = f"l{i}.", L.mixer
        mp = p + "mix."
        nq, nk, nv, no = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim, m.heads * m.vdim
        norm(p + "norm1")
        norm(p + "norm1b")
        if isinstance(m, DeltaSpec):
            out.update({mp + "q": (nk, H), mp + "k": (nk, H), mp + "v": (no, H), mp + "q.conv": (nk, m.taps), mp + "k.conv": (nk, m.taps),
                        mp + "v.conv": (no, m.taps), mp + "b": (m.heads, H), mp + "a": (m.heads, H), mp + "A_log": (m.heads,),
                        mp + "dt_bias": (m.heads,), mp + "norm": (m.vdim,), mp + "g": (no, H), mp + "o": (H, no)})
        elif isinstance(m, AttentionSpec):
            for name, n in (("q", nq), ("k", nk), ("v", nv)):
                biased(mp + name, n, H)
            biased(mp + "o", H, no)
            out.update({mp + "q.norm": (nq,), mp + "k.norm": (nk,), mp + "g": (m.heads, H)})
        else:
            for name, n in (("q", 2 * nq), ("k", 2 * nk), ("v", nv)):
                biased(mp + name, n, H)
            out.update({mp + n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
            out.update({mp + "g": (no, H), mp + "o": (H, no)})
        if L.mlp is not None:
            norm(p + "norm2")
            norm(p + "norm2b")
            for e in range(L.mlp.experts):
                q = f"{p}mlp.e{e}."
                out.update({q + "gate": (L.mlp.ff, H), q + "up": (L.mlp.ff, H), q + "down": (H, L.mlp.ff)})
            biased(p + "mlp.router", L.mlp.experts, H)
    norm("final.norm")
    return out


def random_tensors(cfg: VevapelConfig, seed: int = 0, std: Optional[float] = None, device="cpu") -> Dict[str, torch.Tensor]:
    """bf16 tensors of a random-init checkpoint: N(0, 1 / fan-in) matrices (or N(0, std^2)), norm weights around one, small biases,
    decays spread from short to long memories."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)
    uni = lambda n, lo, hi: lo + (hi - lo) * torch.rand(n, device=device, generator=g)
    out = {}
    for name, s in tensor_shapes(cfg).items():
        if name.endswith((".b", "loop.step")) and not name.endswith("mix.b"):
            t = 0.1 * rnd(*s)
        elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 1 + 0.2 * rnd(*s)
        elif name.endswith("A_log"):
            t = uni(s[0], -4.0, 0.0)
        elif name.endswith("dt_bias"):
            t = uni(s[0], -4.0, -1.0)
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = rnd(*s) * 0.3 * s[0] ** -0.5
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
    """Kernel-ready weights of one layer.  Norms are (weight, bias) rows, fp32 [Hp]."""
    norm1: Tuple[torch.Tensor, torch.Tensor]
    norm1b: Tuple[torch.Tensor, torch.Tensor]
    w_in: QuantLinear                          # every projection of the mixer's input
    w_out: QuantLinear                         # [Hp, mixer outputs]
    out_b: Optional[torch.Tensor] = None       # fp32 [Hp]
    heads: Optional[mx.WindowHeads] = None     # both attentions
    q_norm: Optional[torch.Tensor] = None      # fp32 [hq * D]
    k_norm: Optional[torch.Tensor] = None
    gate_off: int = 0                          # differential: the gate's columns of w_in
    lam: float = 0.0                           # differential: factor of the second map; factor behind the norm
    factor: float = 1.0
    state: Optional[mx.StateHeads] = None
    norm2: Optional[Tuple[torch.Tensor, torch.Tensor]] = None
    norm2b: Optional[Tuple[torch.Tensor, torch.Tensor]] = None
    moe: Optional[RowExperts] = None

    @property
    def n_out(self) -> int:
        return self.w_out.k


class VevapelModel:
    def __init__(self, cfg: VevapelConfig, embed: torch.Tensor, layers: List[Packed], final_norm, loop_in: Optional[QuantLinear],
                 loop_step: Optional[torch.Tensor], dtype: torch.dtype):
        self.cfg, self.embed, self.layers, self.final_norm, self.dtype = cfg, embed, layers, final_norm, dtype
        self.loop_in, self.loop_step = loop_in, loop_step
        self.head = QuantLinear("fp32" if dtype == torch.float32 else "bf16", cfg.vocab, embed.shape[1], embed)
        self.tp_size, self.tp_rank = 1, 0

    @property
    def hp(self) -> int:
        return self.embed.shape[1]

    @staticmethod
    def from_tensors(cfg: VevapelConfig, get: Callable[[str], torch.Tensor], device="cuda", dtype: torch.dtype = BF) -> "VevapelModel":
        """Packs the checkpoint tensors `get(name)` returns; shapes are checked against the configuration."""
        shapes = tensor_shapes(cfg)
        H, Hp = cfg.width, up8(cfg.width)
        fmt = "fp32" if dtype == torch.float32 else "bf16"

        def t(name: str) -> torch.Tensor:
            v, want = get(name), shapes[name]
            if tuple(v.shape) != want:
                raise ValueError(f"{name} is {tuple(v.shape)}, the configuration wants {want}")
            return v.to(device=device, dtype=torch.float32)

        def lin(w: torch.Tensor) -> QuantLinear:
            return QuantLinear(fmt, w.shape[0], w.shape[1], w.to(dtype).contiguous())

        hid = lambda w: pad_cols(w, 1, H, Hp)                       # matrices that read the stream
        hout = lambda w: pad_rows(w, 1, H, Hp)                      # matrices that write it
        hvec = lambda name: pad_vec(t(name), 1, H, Hp).contiguous()
        norm = lambda name: (hvec(name), hvec(name + ".b"))

        def stack(blocks):
            off = [0]
            for w in blocks:
                off.append(off[-1] + w.shape[0])
            return lin(hid(torch.cat(blocks))), off

        def attention(p: str, m: AttentionSpec) -> dict:
            D, DV = mx.pad_to(m.dim, mx.ATTN_WIDTHS), mx.pad_to(m.vdim, mx.ATTN_WIDTHS)
            parts = (("q", m.heads, m.dim, D), ("k", m.kv_heads, m.dim, D), ("v", m.kv_heads, m.vdim, DV))
            w_in, off = stack([pad_rows(t(p + n), g, d, dp) for n, g, d, dp in parts] + [pad_rows(t(p + "g"), 1, m.heads, up8(m.heads))])
            row = lambda name, g, d, dp: pad_vec(t(p + name), g, d, dp).contiguous()
            heads = mx.WindowHeads(m.heads, m.kv_heads, m.dim, m.vdim, mx.NO_WINDOW, m.scale, cfg.eps, *off[:3], norm="row",
                                   bias=tuple(row(n + ".b", g, d, dp) for n, g, d, dp in parts), temp=(m.temp_coef, m.temp_every), gate_off=off[3])
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(p + "o"), m.heads, m.vdim, DV))), out_b=hvec(p + "o.b"), heads=heads,
                        q_norm=row("q.norm", *parts[0][1:]), k_norm=row("k.norm", *parts[1][1:]))

        def differential(p: str, m: DiffSpec) -> dict:
            D, DV = mx.pad_to(m.dim, mx.ATTN_WIDTHS), mx.pad_to(m.vdim, mx.ATTN_WIDTHS)
            G, group = m.kv_heads, m.heads // m.kv_heads

            def by_map(w):                                          # rows [kv head, head of the group, map, dim] -> [kv head, map, head, dim]
                return w.reshape(G, group, 2, m.dim, -1).transpose(1, 2).reshape(2 * m.heads * m.dim, -1)

            parts = lambda f: [pad_rows(by_map(f("q")), 2 * m.heads, m.dim, D), pad_rows(f("k"), 2 * G, m.dim, D), pad_rows(f("v"), G, m.vdim, DV)]
            w_in, off = stack(parts(lambda n: t(p + n)) + [pad_rows(t(p + "g"), m.heads, m.vdim, DV)])
            bias = tuple(b.reshape(-1).contiguous() for b in parts(lambda n: t(p + n + ".b")[:, None]))
            heads = mx.WindowHeads(m.heads, G, m.dim, m.vdim, m.chunk, m.scale, cfg.eps, *off[:3], norm=None, bias=bias,
                                   freq=mx.rotation_freqs(m.base, m.rot, device) if m.rot else None, rot=m.rot, maps=2, chunked=True)
            dot = lambda a, b: math.exp(float((t(p + a).double() * t(p + b).double()).sum()))
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(p + "o"), m.heads, m.vdim, DV))), heads=heads, gate_off=off[3],
                        lam=dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff, factor=1.0 - m.diff)

        def delta(p: str, m: DeltaSpec) -> dict:
            K, V = mx.pad_to(m.dim, mx.STATE_WIDTHS), mx.pad_to(m.vdim, mx.STATE_WIDTHS)
            parts = (("q", m.kv_heads, m.dim, K), ("k", m.kv_heads, m.dim, K), ("v", m.heads, m.vdim, V))
            one = lambda n: pad_rows(t(p + n), 1, m.heads, up8(m.heads))
            w_in, off = stack([pad_rows(t(p + n), g, d, dp) for n, g, d, dp in parts] + [one("b"), one("a"), pad_rows(t(p + "g"), m.heads, m.vdim, V)])
            conv = torch.cat([pad_rows(t(p + n + ".conv"), g, d, dp) for n, g, d, dp in parts])
            vec = lambda n: t(p + n).contiguous()
            state = mx.StateHeads(m.heads, m.kv_heads, m.dim, m.vdim, off[0], off[3], cfg.eps, conv.T.contiguous(), vec("A_log"), vec("dt_bias"),
                                  norm_w=pad_vec(t(p + "norm"), 1, m.vdim, V).contiguous(), a_off=off[4], gate_off=off[5])
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(p + "o"), m.heads, m.vdim, V))), state=state)

        def experts(p: str, m: ExpertsSpec) -> RowExperts:
            fp = up8(m.ff)
            cat = lambda f: torch.cat([f(f"{p}e{e}.").to(dtype) for e in range(m.experts)]).contiguous()
            gu = cat(lambda q: hid(torch.cat([pad_rows(t(q + n), 1, m.ff, fp) for n in ("gate", "up")])))
            down = cat(lambda q: hout(pad_cols(t(q + "down"), 1, m.ff, fp)))
            return RowExperts(m.experts, m.top, fp, math.inf, lin(hid(pad_rows(t(p + "router"), 1, m.experts, up8(m.experts)))), gu, down, Hp,
                              alpha=1.0, shift=0.0, score="chosen", weigh_out=True, router_b=t(p + "router.b").contiguous())

        layers = []
        for i, L in enumerate(cfg.plan):
            p = f"l{i}."
            pack = {AttentionSpec: attention, DiffSpec: differential, DeltaSpec: delta}[type(L.mixer)]
            w = Packed(norm(p + "norm1"), norm(p + "norm1b"), **pack(p + "mix.", L.mixer))
            if L.mlp is not None:
                w.norm2, w.norm2b, w.moe = norm(p + "norm2"), norm(p + "norm2b"), experts(p + "mlp.", L.mlp)
            layers.append(w)
        loop_in = loop_step = None
        if cfg.loop is not None:
            loop_in, loop_step = lin(hout(pad_cols(t("loop.in"), 2, H, Hp))), hid(t("loop.step")).contiguous()
        return VevapelModel(cfg, hid(t("embed")).to(dtype).contiguous(), layers, norm("final.norm"), loop_in, loop_step, dtype)

    @staticmethod
    def random_init(cfg: VevapelConfig, device="cuda", seed: int = 0, std: Optional[float] = None, dtype: torch.dtype = BF) -> "VevapelModel":
        w = random_tensors(cfg, seed, std, device)
        return VevapelModel.from_tensors(cfg, w.__getitem__, device, dtype)

    def weight_bytes(self) -> int:
        """Bytes that one pass reads (a looped layer's matrices once per pass of the loop)."""
        runs = [self.layers[i] for i, _ in self.cfg.runs()]
        entries = sum(t is not None for _, t in self.cfg.runs())
        return (self.head.nbytes + (self.loop_in.nbytes * entries if entries else 0) +
                sum(L.w_in.nbytes + L.w_out.nbytes + (L.moe.nbytes if L.moe is not None else 0) for L in runs))

    # ------------------------------------------------------------------ oracle
    @torch.no_grad()
    def forward_reference(self, tokens: torch.Tensor) -> torch.Tensor:
        """fp32 logits [T, V] of one request from position 0, on the packed weights (fp32 arithmetic, any device)."""
        c, n = self.cfg, self.cfg.width
        x = x0 = self.embed.float()[tokens.to(self.embed.device).long()] * c.embed_scale
        mm = lambda v, w: v @ w.payload.float().T

        def norm(v, wb):
            d = torch.cat([v[:, :n] - v[:, :n].mean(-1, keepdim=True), v[:, n:]], 1)
            return d * torch.rsqrt(d.pow(2).sum(-1, keepdim=True) / n + c.eps) * wb[0] + wb[1]

        def experts(b: RowExperts, h):
            z = mm(h, b.w_first)[:, :b.experts] + b.router_b
            best = torch.argsort(-z, dim=-1, stable=True)[:, :b.top]
            share = z.gather(1, best).softmax(-1)
            gu, down = b.w_gu.float().view(b.experts, 2 * b.ff, -1), b.w_down.float().view(b.experts, b.hidden, -1)
            out = torch.zeros_like(h)
            for r in range(h.shape[0]):
                for a, e in zip(share[r], best[r].tolist()):
                    g, u = (h[r] @ gu[e].T).chunk(2)
                    out[r] += (F.silu(g) * u * a) @ down[e].T
            return out

        for i, t in c.runs():
            P, m = self.layers[i], c.plan[i].mixer
            if t is not None:
                x = mm(torch.cat([x, x0], 1), self.loop_in) + self.loop_step[t]
            proj = mm(norm(x, P.norm1), P.w_in)
            mixed = self._delta_reference(P, proj) if P.state is not None else self._attention_reference(m, P, proj)
            y = mm(mixed, P.w_out)
            x = x + c.residual * norm(y if P.out_b is None else y + P.out_b, P.norm1b)
            if P.moe is not None:
                x = x + c.residual * norm(experts(P.moe, norm(x, P.norm2)), P.norm2b)
        return mm(norm(x, self.final_norm), self.head)

    def _attention_reference(self, m, P: Packed, proj):
        T, g = proj.shape[0], P.heads
        i = torch.arange(T, device=proj.device)
        q, k, v = (proj[:, a:a + n] + b for a, n, b in zip((g.q_off, g.k_off, g.v_off), (g.hq * g.D, g.hkv * g.maps * g.D, g.hkv * g.DV), g.bias))
        if g.norm == "row":
            rms = lambda x, heads, w: x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / (heads * g.dim) + g.eps) * w
            coef, every = g.temp
            q, k = rms(q, g.hq, P.q_norm) * (1 + coef * torch.log((i + 1) // every + 1.0))[:, None], rms(k, g.hkv, P.k_norm)

        def turn(x):                                                # [T, heads, D]
            if not g.rot:
                return x
            ang = i[:, None] * g.freq.double().sum(0)
            cos, sin, half = ang.cos().float()[:, None], ang.sin().float()[:, None], g.rot // 2
            a, b = x[..., :half], x[..., half:g.rot]
            return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., g.rot:]], -1)

        shape = (T, g.hkv, g.maps, g.group, g.D)
        q, k, v = turn(q.view(T, g.hq, g.D)).view(shape), turn(k.view(T, -1, g.D)).view(T, g.hkv, g.maps, g.D), v.view(T, g.hkv, g.DV)
        seen = i[:, None] >= i[None, :]
        seen &= (i[:, None] // g.window == i[None, :] // g.window) if g.chunked else (i[:, None] - i[None, :] < g.window)
        p = (torch.einsum("ikmgd,jkmd->kmgij", q, k) * g.scale).masked_fill(~seen, float("-inf")).softmax(-1)
        o = torch.einsum("kmgij,jke->ikmge", p, v)
        if g.maps == 1:
            o = o.reshape(T, g.hq, g.DV) * torch.sigmoid(proj[:, g.gate_off:g.gate_off + g.hq])[:, :, None]
            return o.reshape(T, -1)
        o = (o[:, :, 0] - P.lam * o[:, :, 1]).reshape(T, g.hq // 2, g.DV)
        o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / g.vdim + g.eps) * P.factor
        return o.reshape(T, -1) * torch.sigmoid(proj[:, P.gate_off:P.gate_off + P.n_out])

    def _delta_reference(self, P: Packed, proj):
        T, s = proj.shape[0], P.state
        nk, ratio = s.hk * s.DK, s.hv // s.hk
        hist = F.pad(proj[:, s.c_off:s.c_off + s.channels], (0, 0, s.taps - 1, 0))
        act = F.silu(sum(hist[j:j + T] * s.conv_w[j] for j in range(s.taps)))
        unit = lambda a: a * torch.rsqrt(a.pow(2).sum(-1, keepdim=True) + UNIT_EPS)
        q = (unit(act[:, :nk].view(T, s.hk, s.DK)) * s.dim ** -0.5).repeat_interleave(ratio, 1)
        k = unit(act[:, nk:2 * nk].view(T, s.hk, s.DK)).repeat_interleave(ratio, 1)
        v = act[:, 2 * nk:].view(T, s.hv, s.DV)
        beta = torch.sigmoid(proj[:, s.b_off:s.b_off + s.hv])
        g = torch.exp(-torch.exp(s.A_log) * F.softplus(proj[:, s.a_off:s.a_off + s.hv] + s.dt_bias))
        S, outs = proj.new_zeros(s.hv, s.DK, s.DV), []
        for t in range(T):
            S = S * g[t, :, None, None]
            u = beta[t, :, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
            S = S + k[t, :, :, None] * u[:, None, :]
            outs.append(torch.einsum("hkv,hk->hv", S, q[t]))
        o = torch.stack(outs)
        o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / s.vdim + s.eps) * s.norm_w
        return o.reshape(T, -1) * F.silu(proj[:, s.gate_off:s.gate_off + s.hv * s.DV])


# ---------------------------------------------------------------------------------------------- kernel runner
class VevapelRunner(WindowRowRunner):
    """Executes the model on the sm_100a kernels.  A request holds pages of the shared key / value pool (one table for every run of an
    attention layer, each with planes of its own) and one slot of the fp32 state of every run of a delta layer; both are reused without
    clearing (a request's first token starts from zero states)."""

    mixed_runs = True

    def __init__(self, model: VevapelModel, max_rows: int, slots: int, max_seq_len: int, device, pool_tokens: int = 0):
        c = model.cfg
        self.m, self.model, self.c = model, model, c
        max_rows = max(max_rows, slots)
        T = model.dtype
        self.runs = c.runs()
        of = [model.layers[i] for i, _ in self.runs]
        self.kv_index = {r: j for j, r in enumerate(r for r, P in enumerate(of) if P.heads is not None)}
        heads = [P.heads for P in of if P.heads is not None]
        self._init_pool(slots, device, [g.kv_shape for g in heads], T, c.page, max_seq_len, max_rows, pool_tokens)
        self.states = {r: P.state.new_state(slots, device) for r, P in enumerate(of) if P.state is not None}
        e = lambda n, dt: torch.empty(n, dtype=dt, device=device)
        R, Hp = max_rows, model.hp
        big = lambda vals: max(list(vals) + [1])
        stream = lambda dt, n=Hp: e(R * n, dt).view(R, n)
        self.x, self.dx, self.xn = stream(torch.float32), stream(torch.float32), stream(T)
        self.xx = stream(T, 2 * Hp) if c.loop is not None else None       # [stream | embedding output] in front of a pass of the loop
        self.proj = e(R * big(P.w_in.n for P in of), T)
        self.mixed = e(R * big(P.n_out for P in of), T)
        states = [P.state for P in of if P.state is not None]
        self.o = e(R * big(s.hv * s.DV for s in states), torch.float32)
        self.prep = e(big(s.prep_floats(R, slots) for s in states), torch.float32)
        self.moe = RowExpertsScratch([P.moe for P in model.layers if P.moe is not None], R, T, device)
        self._init_attention(heads, R, slots, c.page, T, device)
        self.capture: Optional[list] = None        # a list: receives the residual stream after every layer run (tests, debugging)

    def _state_tensors(self):
        return [t for pair in self.states.values() for t in pair if t is not None]

    def _lin(self, x: torch.Tensor, w: QuantLinear, out: torch.Tensor) -> torch.Tensor:
        if w.fmt == "bf16" and out.dtype == torch.float32:
            return ops.gemm_tc(x, w, out32=out)
        return ops.linear(x, w, out=out)

    def _attention(self, r: int, P: Packed, proj, mixed, positions, row_req, runs: Optional[RowRuns], plan) -> None:
        diff = (proj, P.gate_off, P.lam, P.factor) if P.heads.maps == 2 else None
        self._attend(P.heads, (P.q_norm, P.k_norm), self.kv.layers[self.kv_index[r]], proj, mixed, positions, row_req, runs, plan, diff)

    def _delta(self, r: int, P: Packed, proj, mixed, positions, row_req, runs: Optional[RowRuns]) -> None:
        s, rows = P.state, proj.shape[0]
        if runs is None:
            return mx.linear_state(s, proj, *self.states[r], row_req, positions, out=mixed)
        o = self.o[:rows * s.hv * s.DV].view(rows, s.hv * s.DV)
        mx.linear_state(s, proj, *self.states[r], row_req, positions, runs=runs, prep=self.prep, o=o)
        mx.gated_group_norm(o, proj[:, s.gate_off:], s.norm_w, mixed, s.hv, s.vdim, self.c.eps, silu=True)

    def _layers(self, tokens, positions, row_req, runs: Optional[RowRuns]) -> torch.Tensor:
        """-> the final norm's rows."""
        m, c, rows, Hp = self.m, self.c, tokens.shape[0], self.m.hp
        x, xn, dx = self.x[:rows], self.xn[:rows], self.dx[:rows]
        xx = self.xx[:rows] if self.xx is not None else None
        view = lambda buf, n: buf[:rows * n].view(rows, n)
        step = lambda out, pre, delta=None, post=(None, None), b=None, vec=None: mx.stream_norm(x, c.width, c.eps, out, delta, post, pre, c.residual, b, vec)
        plan = self._plan(runs) if runs is not None and self.kv_index else None
        mx.embed_rows(tokens, m.embed, x, c.embed_scale, None if xx is None else xx[:, Hp:])
        last = (None, (None, None), None)                           # what the stream has still to take in: delta, its norm, its bias

        def take(out, pre):
            step(out, pre, *last)
            if self.capture is not None and last[0] is not None:
                self.capture.append(x[:, :c.width].clone())

        for r, (i, t) in enumerate(self.runs):
            P = m.layers[i]
            if t is not None:
                take(xx[:, :Hp], (None, None))
                self._lin(xx, m.loop_in, x)
                step(xn, ("layer", *P.norm1), vec=m.loop_step[t])
            else:
                take(xn, ("layer", *P.norm1))
            proj, mixed = self._lin(xn, P.w_in, view(self.proj, P.w_in.n)), view(self.mixed, P.n_out)
            if P.heads is not None:
                self._attention(r, P, proj, mixed, positions, row_req, runs, plan)
            else:
                self._delta(r, P, proj, mixed, positions, row_req, runs)
            last = self._lin(mixed, P.w_out, dx), ("layer", *P.norm1b), P.out_b
            if P.moe is not None:
                step(xn, ("layer", *P.norm2), *last)
                last = run_experts(P.moe, self.moe, xn), ("layer", *P.norm2b), None
        take(xn, ("layer", *m.final_norm))
        return xn

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
