"""Tefudra decoder family: layers of two kinds in any order, some of which use the weights of another layer.

  attention   sliding-window attention that also sees the first tokens of the sequence, values = the raw keys, query and key norms per
              head, rotated halves, a sink per head
  parallel    two mixers of one input, their outputs normed and averaged:
                left   sliding-window attention behind a causal depthwise convolution of q, k and v; rotated halves, normed and rotated values
                       (outputs are turned back), capped scores
                right  matrix memory with exponential gates (mLSTM), a norm per head, a gate per column

  x <- x + norm1b(mixer(norm1(x)));  x <- x + norm2b(ff(norm2(x)))

Feed-forward: none, dense (square of relu), or routed experts (erf gelu) of which some outputs are the input itself, chosen by softmax
score plus a correction and weighed by their normalised scores, beside a shared expert.  Norms are RMS norms over equal parts of the
vector.  The head is the embedding table.  A layer that uses another one's weights keeps its own cache and states.  The residual stream,
norms, angles, scores, router, gates of the recurrence and states are fp32; projections and activations are bf16 (or everything fp32 with
dtype float32).

Weights are packed for the kernels when they are loaded: every reader of a mixer's input is one matrix (q | k; left q | k | v, right q | k |
v | output gates | input gates | forget gates), the experts two stacks, the router and the shared expert's up matrix one.  Head widths are
padded with zeros to what the kernels take (rotated values half by half), rows of every matrix to multiples of 8 columns.

``TefudraModel.forward_reference`` restates the packed model in PyTorch; ``TefudraRunner`` runs it on the sm_100a kernels
(`ops/mixers.py`), prompt portions and decoded tokens of several requests in one pass.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
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
DENSE_ACT, EXPERT_ACT = "relu2", "gelu"
DEN_EPS = 1e-6                  # behind the matrix memory's denominator


# ---------------------------------------------------------------------------------------------- configuration
@dataclass(frozen=True)
class WindowSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    base: float
    rot: int                     # rotated columns of queries and keys, column i with column i + rot / 2
    keep_first: int = 0
    softcap: float = 0.0         # 0: scores are not capped
    taps: int = 0                # of the convolution (left mixers)


@dataclass(frozen=True)
class MatrixSpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelSpec:
    left: WindowSpec
    right: MatrixSpec


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    identity: int
    top: int
    ff: int
    shared_ff: int               # 0: no shared expert


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[WindowSpec, ParallelSpec]
    mlp: Union[DenseSpec, ExpertsSpec, None]
    weights_of: Optional[int] = None


def _window(m: dict, what: str, left: bool) -> WindowSpec:
    heads = ("heads", "kv_heads", "dim", "vdim")
    only_keys(m, heads + ("scale", "mask", "rot") + (("conv",) if left else ()), what, ("softcap",) if left else ())
    only_keys(m["mask"], ("size",), f"{what} mask", ("keep_first",))
    only_keys(m["rot"], ("base", "dims"), f"{what} rotation")
    spec = WindowSpec(*(int(m[k]) for k in heads), float(m["scale"]), int(m["mask"]["size"]), float(m["rot"]["base"]), int(m["rot"]["dims"]),
                      int(m["mask"].get("keep_first") or 0), float(m.get("softcap") or 0.0), int(m["conv"]) if left else 0)
    if spec.kv_heads < 1 or spec.heads % spec.kv_heads:
        raise ValueError(f"{what}: {spec.heads} heads over {spec.kv_heads} key heads")
    if spec.rot % 2 or not 0 <= spec.rot <= spec.dim or spec.window < 1 or spec.keep_first < 0:
        raise ValueError(f"{what}: {spec.rot} of {spec.dim} columns rotated, a window of {spec.window}, {spec.keep_first} kept tokens")
    if left and (spec.taps < 1 or spec.vdim % 2 or spec.softcap < 0):
        raise ValueError(f"{what}: {spec.taps} taps, values of {spec.vdim} columns, cap {spec.softcap}")
    if not left and spec.vdim != spec.dim:
        raise ValueError(f"{what}: values are the keys, but {spec.vdim} columns differ from {spec.dim}")
    return spec


def _mixer(kind: str, m: dict, what: str):
    if kind == "attention":
        return _window(m, what, False)
    if kind != "parallel":
        raise ValueError(f"{what}: unknown type {kind!r}")
    only_keys(m, ("left", "right"), what)
    only_keys(m["right"], ("heads", "dim", "vdim", "gate_cap"), f"{what} right")
    right = MatrixSpec(*(int(m["right"][k]) for k in ("heads", "dim", "vdim")), float(m["right"]["gate_cap"]))
    if right.heads < 1 or right.gate_cap <= 0:
        raise ValueError(f"{what} right: {right.heads} heads, gate cap {right.gate_cap}")
    return ParallelSpec(_window(m["left"], f"{what} left", True), right)


def _feed_forward(f: Optional[dict], what: str):
    if f is None:
        return None
    if f.get("kind") == "dense":
        only_keys(f, ("kind", "ff"), what)
        return DenseSpec(int(f["ff"]))
    if f.get("kind") != "moe":
        raise ValueError(f"{what}: unknown kind {f.get('kind')!r}")
    only_keys(f, ("kind", "expert", "router"), what, ("shared",))
    only_keys(f["expert"], ("ff",), f"{what} expert")
    only_keys(f["router"], ("experts", "top"), f"{what} router", ("identity",))
    shared = f.get("shared")
    if shared is not None:
        only_keys(shared, ("ff",), f"{what} shared expert")
    r = f["router"]
    spec = ExpertsSpec(int(r["experts"]), int(r.get("identity") or 0), int(r["top"]), int(f["expert"]["ff"]), int(shared["ff"]) if shared else 0)
    n = spec.experts + spec.identity
    if spec.experts < 1 or spec.identity < 0 or not 1 <= spec.top <= min(n, mx.MAX_TOP) or n > mx.MAX_EXPERTS:
        raise ValueError(f"{what}: {spec.top} of {spec.experts} experts and {spec.identity} identity experts")
    return spec


@dataclass
class TefudraConfig:
    width: int
    vocab: int
    plan: List[LayerSpec]
    eps: float
    groups: int                  # equal parts that the layers' norms take on their own
    page: int = 64

    def __post_init__(self):
        if self.groups < 1 or self.width % self.groups:
            raise ValueError(f"norms over {self.groups} parts of {self.width} columns")
        for i in range(len(self.plan)):
            L = self.plan[self.source(i)]
            if (L.mixer, L.mlp) != (self.plan[i].mixer, self.plan[i].mlp):
                raise ValueError(f"layer {i} differs from layer {self.source(i)}, whose weights it uses")

    def source(self, i: int) -> int:
        """The layer whose weights layer i uses."""
        j, seen = i, {i}
        while self.plan[j].weights_of is not None:
            j = self.plan[j].weights_of
            if not 0 <= j < len(self.plan) or j in seen:
                raise ValueError(f"layer {i} uses the weights of a layer that has none")
            seen.add(j)
        return j

    @staticmethod
    def from_dict(d: dict) -> "TefudraConfig":
        only_keys(d["norm"], ("eps",), "norm", ("groups",))
        layers = []
        for i, e in enumerate(d["layers"]):
            only_keys(e, ("type", "mixer"), f"layer {i}", ("mlp", "weights_of"))
            of = e.get("weights_of")
            layers.append(LayerSpec(_mixer(e["type"], e["mixer"], f"layer {i} mixer"), _feed_forward(e.get("mlp"), f"layer {i} feed-forward"),
                                    None if of is None else int(of)))
        return TefudraConfig(int(d["width"]), int(d["vocab"]), layers, float(d["norm"]["eps"]), int(d["norm"].get("groups") or 1))

    def to_dict(self) -> dict:
        def window(m: WindowSpec, left: bool) -> dict:
            out = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "mask": {"size": m.window},
                   "rot": {"base": m.base, "dims": m.rot}}
            if m.keep_first or not left:
                out["mask"]["keep_first"] = m.keep_first
            if left:
                out["conv"] = m.taps
            if m.softcap:
                out["softcap"] = m.softcap
            return out

        def feed_forward(f) -> Optional[dict]:
            if f is None:
                return None
            if isinstance(f, DenseSpec):
                return {"kind": "dense", "ff": f.ff}
            out = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "identity": f.identity, "top": f.top}}
            if f.shared_ff:
                out["shared"] = {"ff": f.shared_ff}
            return out

        layers = []
        for L in self.plan:
            if isinstance(L.mixer, ParallelSpec):
                r = L.mixer.right
                e = {"type": "parallel", "mixer": {"left": window(L.mixer.left, True),
                                                   "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "gate_cap": r.gate_cap}}}
            else:
                e = {"type": "attention", "mixer": window(L.mixer, False)}
            e["mlp"] = feed_forward(L.mlp)
            if L.weights_of is not None:
                e["weights_of"] = L.weights_of
            layers.append(e)
        return {"architecture": "Tefudra", "width": self.width, "vocab": self.vocab, "layers": layers, "norm": {"eps": self.eps, "groups": self.groups}}

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def layers(self) -> int:
        return len(self.plan)

    @staticmethod
    def cycle(layers: int, width: int, vocab: int, mixers, mlps, groups: int = 4, eps: float = 1e-5, shared: Tuple[Tuple[int, int], ...] = ()) -> "TefudraConfig":
        """`layers` layers that take the given mixers and feed-forwards in turn; shared: (layer, layer whose weights it uses)."""
        of = dict(shared)
        return TefudraConfig(width, vocab, [LayerSpec(mixers[i % len(mixers)], mlps[i % len(mlps)], of.get(i)) for i in range(layers)], eps, groups)


def tensor_shapes(cfg: TefudraConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint of `cfg`."""
    H = cfg.width
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H), "final.norm": (H,)}

    def biased(name: str, n: int, k: int) -> None:
        out.update({name: (n, k), name + ".b": (n,)})

    for i, L in enumerate(cfg.plan):
        if L.weights_of is not None:
            continue
        p, m = f"l{i}.", L.mixer
        mp, fp = p + "mix.", p + "mlp."
        out.update({p + n: (H,) for n in ("norm1", "norm1b")})
        if isinstance(m, ParallelSpec):
            a, r = m.left, m.right
            for name, n in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                biased(mp + "left." + name, n, H)
                out[mp + f"left.{name}.conv"] = (n, a.taps)
            biased(mp + "left.o", H, a.heads * a.vdim)
            nk, nv, q = r.heads * r.dim, r.heads * r.vdim, mp + "right."
            out.update({q + "q": (nk, H), q + "k": (nk, H), q + "v": (nv, H), q + "g": (nv, H), q + "o": (H, nv), q + "norm": (nv,)})
            biased(q + "i", r.heads, H)
            biased(q + "f", r.heads, H)
            out.update({mp + "left.out": (H,), mp + "right.out": (H,)})
        else:
            out.update({mp + "q": (m.heads * m.dim, H), mp + "k": (m.kv_heads * m.dim, H), mp + "q.norm": (m.dim,), mp + "k.norm": (m.dim,),
                        mp + "sink": (m.heads,), mp + "o": (H, m.heads * m.vdim)})
        f = L.mlp
        if f is None:
            continue
        out.update({p + n: (H,) for n in ("norm2", "norm2b")})
        ups = lambda name, ff: out.update({name + "up": (ff, H), name + "down": (H, ff)})
        if isinstance(f, DenseSpec):
            ups(fp, f.ff)
            continue
        for e in range(f.experts):
            ups(f"{fp}e{e}.", f.ff)
        out.update({fp + "router": (f.experts + f.identity, H), fp + "correction": (f.experts + f.identity,)})
        if f.shared_ff:
            ups(fp + "shared.", f.shared_ff)
    return out


def random_tensors(cfg: TefudraConfig, seed: int = 0, std: Optional[float] = None, device="cpu") -> Dict[str, torch.Tensor]:
    """bf16 tensors of a random-init checkpoint: N(0, 1 / fan-in) matrices (or N(0, std^2)), norm weights around one, small biases, sinks
    and corrections, forget gates that remember."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)
    out = {}
    for name, s in tensor_shapes(cfg).items():
        last = name.rpartition(".")[2]
        if name.endswith("f.b"):
            t = 2 + rnd(*s)
        elif last == "b":
            t = 0.1 * rnd(*s)
        elif last == "correction":
            t = 0.02 * rnd(*s)
        elif last in ("norm", "norm1", "norm2", "norm1b", "norm2b", "out"):
            t = 1 + 0.2 * rnd(*s)
        elif last == "sink":
            t = rnd(*s)
        elif last == "conv":
            t = 0.6 * rnd(*s)
        elif name == "embed":
            t = rnd(*s) * (std * 4 if std else 1.0)
        else:
            t = rnd(*s) * (std or s[1] ** -0.5)
        out[name] = t.to(BF)
    return out


# ---------------------------------------------------------------------------------------------- packed weights
@dataclass
class Packed:
    """Kernel-ready weights of one layer.  Norm weights are fp32 rows [Hp]."""
    norm1: torch.Tensor
    norm1b: torch.Tensor
    w_in: QuantLinear                          # every projection of the mixer's input
    w_out: QuantLinear                         # [Hp, heads * DV] (parallel: of the left mixer)
    heads: mx.WindowHeads
    q_norm: Optional[torch.Tensor] = None      # fp32 [D]
    k_norm: Optional[torch.Tensor] = None
    memory: Optional[mx.MatrixHeads] = None    # parallel: the right mixer
    right_out: Optional[QuantLinear] = None
    out_b: Optional[torch.Tensor] = None       # fp32 [Hp], of the left mixer
    mix: Optional[Tuple[torch.Tensor, torch.Tensor]] = None    # weights of the norms behind the two mixers
    norm2: Optional[torch.Tensor] = None
    norm2b: Optional[torch.Tensor] = None
    up: Optional[QuantLinear] = None           # dense feed-forward
    down: Optional[QuantLinear] = None
    moe: Optional[RowExperts] = None

    @property
    def nbytes(self) -> int:
        linears = (self.w_in, self.w_out, self.right_out, self.up, self.down, self.moe)
        return sum(w.nbytes for w in linears if w is not None)


class TefudraModel:
    def __init__(self, cfg: TefudraConfig, embed: torch.Tensor, layers: List[Packed], final_norm: torch.Tensor, dtype: torch.dtype):
        self.cfg, self.embed, self.layers, self.final_norm, self.dtype = cfg, embed, layers, final_norm, dtype
        self.head = QuantLinear("fp32" if dtype == torch.float32 else "bf16", cfg.vocab, embed.shape[1], embed)
        self.tp_size, self.tp_rank = 1, 0

    @property
    def hp(self) -> int:
        return self.embed.shape[1]

    @staticmethod
    def from_tensors(cfg: TefudraConfig, get: Callable[[str], torch.Tensor], device="cuda", dtype: torch.dtype = BF) -> "TefudraModel":
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

        def stack(blocks):
            off = [0]
            for w in blocks:
                off.append(off[-1] + w.shape[0])
            return lin(hid(torch.cat(blocks))), off

        freqs = lambda m: mx.rotation_freqs(m.base, m.rot, device) if m.rot else None

        def attention(p: str, m: WindowSpec) -> dict:
            D = mx.pad_to(m.dim, mx.ATTN_WIDTHS)
            w_in, off = stack([pad_rows(t(p + "q"), m.heads, m.dim, D), pad_rows(t(p + "k"), m.kv_heads, m.dim, D)])
            heads = mx.WindowHeads(m.heads, m.kv_heads, m.dim, m.dim, m.window, m.scale, cfg.eps, off[0], off[1], off[1], norm="head", freq=freqs(m), rot=m.rot,
                                   keep_first=m.keep_first, sink=t(p + "sink").contiguous())
            row = lambda n: pad_vec(t(p + n), 1, m.dim, D).contiguous()
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(p + "o"), m.heads, m.dim, D))), heads=heads, q_norm=row("q.norm"), k_norm=row("k.norm"))

        def parallel(p: str, m: ParallelSpec) -> dict:
            a, r, lp, rp = m.left, m.right, p + "left.", p + "right."
            D, DV = mx.pad_to(a.dim, mx.ATTN_WIDTHS), mx.pad_to(a.vdim, mx.ATTN_WIDTHS)
            K, V = mx.pad_to(r.dim, mx.STATE_WIDTHS), mx.pad_to(r.vdim, mx.STATE_WIDTHS)
            left = (("q", a.heads, a.dim, D), ("k", a.kv_heads, a.dim, D), ("v", 2 * a.kv_heads, a.vdim // 2, DV // 2))    # values half by half
            right = (("q", r.heads, r.dim, K), ("k", r.heads, r.dim, K), ("v", r.heads, r.vdim, V), ("g", r.heads, r.vdim, V), ("i", 1, r.heads, up8(r.heads)),
                     ("f", 1, r.heads, up8(r.heads)))
            w_in, off = stack([pad_rows(t(lp + n), g, d, dp) for n, g, d, dp in left] + [pad_rows(t(rp + n), g, d, dp) for n, g, d, dp in right])
            bias = tuple(pad_vec(t(f"{lp}{n}.b"), g, d, dp).contiguous() for n, g, d, dp in left)
            conv = torch.cat([pad_rows(t(f"{lp}{n}.conv"), g, d, dp) for n, g, d, dp in left]).T.contiguous()
            heads = mx.WindowHeads(a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, cfg.eps, *off[:3], norm=None, bias=bias, freq=freqs(a), rot=a.rot,
                                   keep_first=a.keep_first, softcap=a.softcap, conv_w=conv, vnorm=True, vfreq=mx.value_freqs(a.base, a.vdim, DV, device))
            vec = lambda n: t(rp + n).contiguous()
            memory = mx.MatrixHeads(r.heads, r.dim, r.vdim, off[3], off[7], off[8], off[6], vec("i.b"), vec("f.b"), r.gate_cap,
                                    pad_vec(t(rp + "norm"), r.heads, r.vdim, V).contiguous(), cfg.eps)
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(lp + "o"), 2 * a.heads, a.vdim // 2, DV // 2))), heads=heads, memory=memory,
                        right_out=lin(hout(pad_cols(t(rp + "o"), r.heads, r.vdim, V))), out_b=hvec(lp + "o.b"), mix=(hvec(lp + "out"), hvec(rp + "out")))

        def experts(p: str, f: ExpertsSpec) -> RowExperts:
            fp, sp, n = up8(f.ff), up8(f.shared_ff), f.experts + f.identity
            cat = lambda g: torch.cat([g(f"{p}e{e}.").to(dtype) for e in range(f.experts)]).contiguous()
            first = [pad_rows(t(p + "router"), 1, n, up8(n))] + ([pad_rows(t(p + "shared.up"), 1, f.shared_ff, sp)] if sp else [])
            return RowExperts(f.experts, f.top, fp, math.inf, lin(hid(torch.cat(first))), cat(lambda q: hid(pad_rows(t(q + "up"), 1, f.ff, fp))),
                              cat(lambda q: hout(pad_cols(t(q + "down"), 1, f.ff, fp))), Hp, shared_col=up8(n), shared_ff=sp, shared_gated=False,
                              shared_down=lin(hout(pad_cols(t(p + "shared.down"), 1, f.shared_ff, sp))) if sp else None, score="softmax",
                              correction=t(p + "correction").contiguous(), norm_topk=True, identity=f.identity, act=EXPERT_ACT)

        layers: List[Optional[Packed]] = []
        for i, L in enumerate(cfg.plan):
            p, f = f"l{i}.", L.mlp
            if L.weights_of is not None:
                layers.append(None)
                continue
            w = Packed(hvec(p + "norm1"), hvec(p + "norm1b"), **(parallel if isinstance(L.mixer, ParallelSpec) else attention)(p + "mix.", L.mixer))
            if f is not None:
                w.norm2, w.norm2b = hvec(p + "norm2"), hvec(p + "norm2b")
            if isinstance(f, DenseSpec):
                fp = up8(f.ff)
                w.up, w.down = lin(hid(pad_rows(t(p + "mlp.up"), 1, f.ff, fp))), lin(hout(pad_cols(t(p + "mlp.down"), 1, f.ff, fp)))
            elif f is not None:
                w.moe = experts(p + "mlp.", f)
            layers.append(w)
        layers = [layers[cfg.source(i)] for i in range(cfg.layers)]
        return TefudraModel(cfg, hid(t("embed")).to(dtype).contiguous(), layers, hvec("final.norm"), dtype)

    @staticmethod
    def random_init(cfg: TefudraConfig, device="cuda", seed: int = 0, std: Optional[float] = None, dtype: torch.dtype = BF) -> "TefudraModel":
        w = random_tensors(cfg, seed, std, device)
        return TefudraModel.from_tensors(cfg, w.__getitem__, device, dtype)

    def weight_bytes(self) -> int:
        """Bytes that one pass reads (weights that several layers use once per layer)."""
        return self.head.nbytes + sum(L.nbytes for L in self.layers)

    # ------------------------------------------------------------------ oracle
    @torch.no_grad()
    def forward_reference(self, tokens: torch.Tensor) -> torch.Tensor:
        """fp32 logits [T, V] of one request from position 0, on the packed weights (fp32 arithmetic, any device)."""
        c, n = self.cfg, self.cfg.width
        x = self.embed.float()[tokens.to(self.embed.device).long()]
        mm = lambda v, w: v @ w.payload.float().T

        def norm(v, w):
            parts = v[:, :n].reshape(v.shape[0], c.groups, -1)
            return F.pad((parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + c.eps)).reshape(v.shape[0], n), (0, v.shape[1] - n)) * w

        rms = lambda v, w: v * torch.rsqrt(v.pow(2).sum(-1, keepdim=True) / n + c.eps) * w

        def experts(b: RowExperts, h):
            first = mm(h, b.w_first)
            s = first[:, :b.outputs].softmax(-1)
            best = torch.argsort(-(s + b.correction), dim=-1, stable=True)[:, :b.top]
            share = s.gather(1, best)
            share = share / (share.sum(-1, keepdim=True) + 1e-20)
            up, down = b.w_gu.float().view(b.experts, b.ff, -1), b.w_down.float().view(b.experts, b.hidden, -1)
            out = mm(F.gelu(first[:, b.shared_col:]), b.shared_down) if b.shared_ff else torch.zeros_like(h)
            for r in range(h.shape[0]):
                for a, e in zip(share[r], best[r].tolist()):
                    out[r] += a * (F.gelu(h[r] @ up[e].T) @ down[e].T if e < b.experts else h[r])
            return out

        for P in self.layers:
            proj = mm(norm(x, P.norm1), P.w_in)
            y = mm(self._window_reference(P, proj), P.w_out)
            if P.memory is not None:
                y = (rms(y + P.out_b, P.mix[0]) + rms(mm(self._memory_reference(P.memory, proj), P.right_out), P.mix[1])) / 2
            x = x + norm(y, P.norm1b)
            if P.norm2 is not None:
                h = norm(x, P.norm2)
                x = x + norm(experts(P.moe, h) if P.moe is not None else mm(F.relu(mm(h, P.up)).square(), P.down), P.norm2b)
        return mm(norm(x, self.final_norm), self.head)

    @staticmethod
    def _window_reference(P: Packed, proj):
        T, g = proj.shape[0], P.heads
        i = torch.arange(T, device=proj.device)
        q, k, v = (proj[:, a:a + n] for a, n in zip((g.q_off, g.k_off, g.v_off), (g.hq * g.D, g.hkv * g.D, g.hkv * g.DV)))
        if g.taps:
            u = torch.cat([x + b for x, b in zip((q, k, v), g.bias)], 1)
            hist = F.pad(u, (0, 0, g.taps - 1, 0))
            q, k, v = sum(hist[j:j + T] * g.conv_w[j] for j in range(g.taps)).split([q.shape[1], k.shape[1], v.shape[1]], 1)
        q, k, v = q.view(T, g.hq, g.D), k.view(T, g.hkv, g.D), v.view(T, g.hkv, g.DV)
        rms = lambda x, m: x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / m + g.eps)
        if g.norm == "head":
            q, k = rms(q, g.dim) * P.q_norm, rms(k, g.dim) * P.k_norm

        def turn(x, freq, rot, sign=1.0):
            if not rot:
                return x
            ang = i[:, None] * freq.double().sum(0)
            cos, sin, half = ang.cos().float()[:, None], sign * ang.sin().float()[:, None], rot // 2
            a, b = x[..., :half], x[..., half:rot]
            return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., rot:]], -1)

        q, k = turn(q, g.freq, g.rot), turn(k, g.freq, g.rot)
        if g.vnorm:
            v = rms(v, g.vdim)
        if g.vfreq is not None:
            v = turn(v, g.vfreq, g.DV)
        s = torch.einsum("ikgd,jkd->kgij", q.view(T, g.hkv, g.group, g.D), k) * g.scale
        if g.softcap:
            s = g.softcap * torch.tanh(s / g.softcap)
        back = i[:, None] - i[None, :]
        s = s.masked_fill(~((back >= 0) & ((back < g.window) | (i[None, :] < g.keep_first))), float("-inf"))
        if g.sink is not None:
            s = torch.cat([s, g.sink.view(g.hkv, g.group, 1, 1).expand(-1, -1, T, 1)], -1)
        o = torch.einsum("kgij,jke->ikge", s.softmax(-1)[..., :T], v).reshape(T, g.hq, g.DV)
        return (turn(o, g.vfreq, g.DV, -1.0) if g.vfreq is not None else o).reshape(T, -1)

    @staticmethod
    def _memory_reference(g: mx.MatrixHeads, proj):
        T, H = proj.shape[0], g.heads
        nk, nv = H * g.DK, H * g.DV
        q, k, v = (x.reshape(T, H, -1) for x in proj[:, g.c_off:g.c_off + 2 * nk + nv].split([nk, nk, nv], 1))
        cap = lambda z: g.gate_cap * torch.tanh(z / g.gate_cap)
        i, f = cap(proj[:, g.i_off:g.i_off + H] + g.i_bias), F.logsigmoid(cap(proj[:, g.f_off:g.f_off + H] + g.f_bias))
        q = q * g.dim ** -0.5
        S, n, m, outs = proj.new_zeros(H, g.DK, g.DV), proj.new_zeros(H, g.DK), proj.new_zeros(H), []
        for t in range(T):
            top = torch.maximum(f[t] + m, i[t])
            keep, write = torch.exp(f[t] + m - top)[:, None], torch.exp(i[t] - top)[:, None]
            S = keep[..., None] * S + (write * k[t])[:, :, None] * v[t][:, None, :]
            n, m = keep * n + write * k[t], top
            outs.append(torch.einsum("hkv,hk->hv", S, q[t]) / (torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + DEN_EPS)[:, None])
        o = torch.stack(outs)
        o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / g.vdim + g.eps)
        return o.reshape(T, -1) * g.norm_w * torch.sigmoid(proj[:, g.gate_off:g.gate_off + nv])


# ---------------------------------------------------------------------------------------------- kernel runner
class TefudraRunner(WindowRowRunner):
    """Executes the model on the sm_100a kernels.  A request holds pages of the shared key / value pool (one table for every layer, each
    with planes of its own) and one slot of the convolution rings and fp32 memories of the parallel layers; all are reused without clearing
    (a request's first token starts from zeros)."""

    mixed_runs = True

    def __init__(self, model: TefudraModel, max_rows: int, slots: int, max_seq_len: int, device, pool_tokens: int = 0):
        c = model.cfg
        self.m, self.model, self.c = model, model, c
        max_rows = max(max_rows, slots)
        T, layers = model.dtype, model.layers
        self._init_pool(slots, device, [P.heads.kv_shape for P in layers], T, c.page, max_seq_len, max_rows, pool_tokens)
        self.rings = [P.heads.new_ring(slots, device) for P in layers]
        self.memories = [P.memory.new_state(slots, device) if P.memory is not None else None for P in layers]
        e = lambda n, dt: torch.empty(n, dtype=dt, device=device)
        R, Hp = max_rows, model.hp
        big = lambda vals: max(list(vals) + [1])
        stream = lambda dt: e(R * Hp, dt).view(R, Hp)
        self.x, self.dx, self.dx2 = stream(torch.float32), stream(torch.float32), stream(torch.float32)
        self.xn, self.xf = stream(T), stream(T)                   # inputs of the mixers and of the feed-forwards
        self.proj = e(R * big(P.w_in.n for P in layers), T)
        self.mixed = e(R * big(P.w_out.k for P in layers), T)
        memories = [P.memory for P in layers if P.memory is not None]
        self.mixed2 = e(R * big(g.heads * g.DV for g in memories), T)
        self.o, self.den = e(R * big(g.heads * g.DV for g in memories), torch.float32), e(R * big(g.heads for g in memories), torch.float32)
        self.prep = e(big(g.prep_floats(R, slots) for g in memories), torch.float32)
        dense = big(P.up.n for P in layers if P.up is not None)
        self.up, self.act = e(R * dense, T), e(R * dense, T)
        self.moe = RowExpertsScratch([P.moe for P in layers if P.moe is not None], R, T, device)
        self._init_attention([P.heads for P in layers], R, slots, c.page, T, device)
        self.capture: Optional[list] = None        # a list: receives the residual stream after every layer (tests, debugging)

    def _state_tensors(self):
        return [r for r in self.rings if r is not None] + [t for pair in self.memories if pair is not None for t in pair]

    def _lin(self, x: torch.Tensor, w: QuantLinear, out: torch.Tensor) -> torch.Tensor:
        if w.fmt == "bf16" and out.dtype == torch.float32:
            return ops.gemm_tc(x, w, out32=out)
        return ops.linear(x, w, out=out)

    def _memory(self, i: int, g: mx.MatrixHeads, proj, mixed, positions, row_req, runs: Optional[RowRuns]) -> None:
        rows = proj.shape[0]
        if runs is None:
            return mx.matrix_memory(g, proj, *self.memories[i], row_req, positions, out=mixed)
        o, den = self.o[:rows * g.heads * g.DV].view(rows, -1), self.den[:rows * g.heads].view(rows, -1)
        mx.matrix_memory(g, proj, *self.memories[i], row_req, positions, runs=runs, prep=self.prep, o=o, den=den)
        mx.gated_group_norm(o, proj[:, g.gate_off:], g.norm_w, mixed, g.heads, g.vdim, g.eps, den=den)

    def _layers(self, tokens, positions, row_req, runs: Optional[RowRuns]) -> torch.Tensor:
        """-> the final norm's rows."""
        m, c, rows = self.m, self.c, tokens.shape[0]
        x, xn, xf, dx, dx2 = (t[:rows] for t in (self.x, self.xn, self.xf, self.dx, self.dx2))
        view = lambda buf, n: buf[:rows * n].view(rows, n)
        plan = self._plan(runs) if runs is not None else None
        mx.embed_rows(tokens, m.embed, x)
        last = (None, (None, None))                                 # what the stream has still to take in: delta and its norm

        def take(out, w):
            mx.stream_norm(x, c.width, c.eps, out, *last, ("parts", w), parts=c.groups)

        for i, P in enumerate(m.layers):
            take(xn, P.norm1)
            if self.capture is not None and i:
                self.capture.append(x[:, :c.width].clone())
            proj, mixed = self._lin(xn, P.w_in, view(self.proj, P.w_in.n)), view(self.mixed, P.w_out.k)
            self._attend(P.heads, (P.q_norm, P.k_norm), self.kv.layers[i], proj, mixed, positions, row_req, runs, plan, ring=self.rings[i])
            delta = self._lin(mixed, P.w_out, dx)
            if P.memory is not None:
                mixed2 = view(self.mixed2, P.right_out.k)
                self._memory(i, P.memory, proj, mixed2, positions, row_req, runs)
                delta = mx.PairDelta(delta, P.mix[0], self._lin(mixed2, P.right_out, dx2), P.mix[1], 0.5, P.out_b)
            last = delta, ("parts", P.norm1b)
            if P.norm2 is None:
                continue
            take(xf, P.norm2)
            if P.moe is not None:
                delta = run_experts(P.moe, self.moe, xf)
            else:
                up = self._lin(xf, P.up, view(self.up, P.up.n))
                delta = self._lin(mx.act_rows(up, view(self.act, P.up.n), DENSE_ACT), P.down, dx)
            last = delta, ("parts", P.norm2b)
        take(xn, m.final_norm)
        if self.capture is not None:
            self.capture.append(x[:, :c.width].clone())
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
