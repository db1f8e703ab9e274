"""Potivik decoder family: layers of two kinds in any order, norms before and after every sublayer, a per-layer input of the token.

  latent_attention  sliding-window attention over a shared latent: per head an unrotated key and a value made from the latent, one
                    rotated key part for all heads, an output gate per head
  mamba2            state-space recurrence with a decay per token and head, a causal depthwise convolution with bias in front, a
                    gate and a norm over equal parts of the columns behind

  x <- x + norm1b(mixer(norm1(x)));  x <- x + norm2b(ff(norm2(x)))  (where the layer has a feed-forward: dense, or routed experts
  whose weight multiplies their input, beside a gated shared expert);  x <- x + rms(proj(gelu(gate x) * side[token, layer])) * w

The norms in front of and behind the sublayers are layer norms with a weight and no bias.  The residual stream, norms, scores,
router, step sizes, decays and states are fp32; projections and activations are bf16 (or everything fp32 with dtype float32).

Weights are packed for the kernels when they are loaded: every reader of a sublayer's input is one matrix (q | latent | key part |
gates; C | B | x | step sizes | z; router | shared gate | shared expert), the latent's key and value matrices another, the experts
two stacks.  Head widths are padded with zeros to what the kernels take, rows of every matrix to multiples of 8 columns.

``PotivikModel.forward_reference`` restates the packed model in PyTorch; ``PotivikRunner`` runs it on the sm_100a kernels
(`ops/mixers.py`), prompt portions and decoded tokens of several requests in one pass.
"""
from __future__ import annotations

from dataclasses import asdict, dataclass
from typing import Callable, Dict, List, Optional, Tuple, Union

import torch
import torch.nn.functional as F

from ..ops import core as ops
from ..ops import mixers as mx
from ..quant.formats import QuantLinear
from .packing import only_keys, pad_cols, pad_rows, pad_vec, up8
from .row_moe import RowExperts, RowExpertsScratch, run_experts
from .rows import RowRunner, RowRuns

BF = torch.bfloat16
GLU_ALPHA = 1.702
ABSORB_RUN = 8                  # runs of a mixed pass up to this length attend in the absorbed form, longer ones expanded


# ---------------------------------------------------------------------------------------------- configuration
@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int
    base: float
    rot: int                     # rotated columns (pairs of neighbours), from the first of the rotated part


@dataclass(frozen=True)
class StateSpaceSpec:
    heads: int
    groups: int
    vdim: int
    state: int
    taps: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class FeedForward:
    ff: int
    limit: float


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    expert: FeedForward
    shared: Optional[FeedForward]


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentSpec, StateSpaceSpec]
    mlp: Union[FeedForward, ExpertsSpec, None]


def _feed_forward(m: dict, what: str) -> FeedForward:
    only_keys(m, ("ff", "limit"), what)
    return FeedForward(int(m["ff"]), float(m["limit"]))


@dataclass
class PotivikConfig:
    width: int
    vocab: int
    plan: List[LayerSpec]
    eps: float
    side: int                    # columns of the per-layer token input
    softcap: float
    page: int = 64

    @staticmethod
    def from_dict(d: dict) -> "PotivikConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, kind, mlp = e["mixer"], e["type"], e.get("mlp")
            if kind == "latent_attention":
                only_keys(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask", "rot"), f"layer {i} mixer")
                only_keys(m["mask"], ("size",), f"layer {i} mask")
                only_keys(m["rot"], ("base", "dims"), f"layer {i} rotation")
                spec = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                                  int(m["mask"]["size"]), float(m["rot"]["base"]), int(m["rot"]["dims"]))
                if spec.rot % 2 or spec.rot > spec.rot_dim or spec.window < 1:
                    raise ValueError(f"layer {i}: {spec.rot} of {spec.rot_dim} columns rotated, window {spec.window}")
            elif kind == "mamba2":
                only_keys(m, ("heads", "groups", "vdim", "state", "conv", "norm_groups"), f"layer {i} mixer")
                spec = StateSpaceSpec(int(m["heads"]), int(m["groups"]), int(m["vdim"]), int(m["state"]), int(m["conv"]), int(m["norm_groups"]))
                if spec.heads % spec.groups or spec.inner % spec.norm_groups:
                    raise ValueError(f"layer {i}: {spec.heads} heads in {spec.groups} groups, {spec.inner} columns in {spec.norm_groups} parts")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            ff = None
            if mlp is not None and mlp.get("kind") == "dense":
                ff = _feed_forward({k: v for k, v in mlp.items() if k != "kind"}, f"layer {i} feed-forward")
            elif mlp is not None and mlp.get("kind") == "moe":
                only_keys(mlp, ("kind", "expert", "router"), f"layer {i} experts", ("shared",))
                only_keys(mlp["router"], ("experts", "top"), f"layer {i} router")
                shared = mlp.get("shared")
                ff = ExpertsSpec(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), _feed_forward(mlp["expert"], f"layer {i} expert"),
                                 None if shared is None else _feed_forward(shared, f"layer {i} shared expert"))
                if not 1 <= ff.top <= min(ff.experts, mx.MAX_TOP) or ff.experts > mx.MAX_EXPERTS:
                    raise ValueError(f"layer {i}: {ff.top} of {ff.experts} experts")
            elif mlp is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerSpec(spec, ff))
        only_keys(d["token_side"], ("dim",), "token_side")
        return PotivikConfig(int(d["width"]), int(d["vocab"]), layers, float(d["norm"]["eps"]), int(d["token_side"]["dim"]), float(d["logit_softcap"]))

    def to_dict(self) -> dict:
        out = []
        for L in self.plan:
            m = asdict(L.mixer)
            if isinstance(L.mixer, LatentSpec):
                m["mask"], m["rot"] = {"size": m.pop("window")}, {"base": m.pop("base"), "dims": m["rot"]}
                e = {"type": "latent_attention", "mixer": m}
            else:
                m["conv"] = m.pop("taps")
                e = {"type": "mamba2", "mixer": m}
            if L.mlp is None:
                e["mlp"] = None
            elif isinstance(L.mlp, FeedForward):
                e["mlp"] = {"kind": "dense", **asdict(L.mlp)}
            else:
                e["mlp"] = {"kind": "moe", "router": {"experts": L.mlp.experts, "top": L.mlp.top}, "expert": asdict(L.mlp.expert)}
                if L.mlp.shared is not None:
                    e["mlp"]["shared"] = asdict(L.mlp.shared)
            out.append(e)
        return {"architecture": "Potivik", "width": self.width, "vocab": self.vocab, "layers": out, "norm": {"eps": self.eps},
                "token_side": {"dim": self.side}, "logit_softcap": self.softcap}

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def layers(self) -> int:
        return len(self.plan)

    @staticmethod
    def uniform(layers: int, width: int, vocab: int, latent: LatentSpec, state: StateSpaceSpec, moe: Optional[ExpertsSpec], dense: FeedForward,
                side: int, every: int = 2, eps: float = 1e-5, softcap: float = 30.0) -> "PotivikConfig":
        """`layers` layers, every `every`-th (from the first) latent attention; the first one with a dense feed-forward, the others
        with experts (with `moe` None: all dense)."""
        return PotivikConfig(width, vocab, [LayerSpec(latent if i % every == 0 else state, dense if i == 0 or moe is None else moe)
                                            for i in range(layers)], eps, side, softcap)


def tensor_shapes(cfg: PotivikConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint of `cfg`."""
    H, S = cfg.width, cfg.side
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H), "side.embed": (cfg.vocab, cfg.layers * S)}

    def ff(p: str, f: FeedForward) -> None:
        out.update({p + "gate": (f.ff, H), p + "up": (f.ff, H), p + "down": (H, f.ff)})

    for i, L in enumerate(cfg.plan):
        p, m = f"l{i}.", L.mixer
        mp = p + "mix."
        out.update({p + "norm1": (H,), p + "norm1b": (H,)})
        if isinstance(m, LatentSpec):
            out.update({mp + "q": (m.heads * (m.dim + m.rot_dim), H), mp + "dkv": (m.kv_rank + m.rot_dim, H), mp + "dkv.norm": (m.kv_rank,),
                        mp + "uk": (m.heads * m.dim, m.kv_rank), mp + "uv": (m.heads * m.vdim, m.kv_rank), mp + "g": (m.heads, H),
                        mp + "o": (H, m.heads * m.vdim)})
        else:
            out.update({mp + "in": (m.inner + m.channels + m.heads, H), mp + "conv": (m.channels, m.taps), mp + "conv.b": (m.channels,),
                        mp + "dt_bias": (m.heads,), mp + "A_log": (m.heads,), mp + "D": (m.heads,), mp + "norm": (m.inner,), mp + "o": (H, m.inner)})
        if L.mlp is not None:
            out.update({p + "norm2": (H,), p + "norm2b": (H,)})
        if isinstance(L.mlp, FeedForward):
            ff(p + "mlp.", L.mlp)
        elif L.mlp is not None:
            for e in range(L.mlp.experts):
                ff(f"{p}mlp.e{e}.", L.mlp.expert)
            out[p + "mlp.router"] = (L.mlp.experts, H)
            if L.mlp.shared is not None:
                ff(p + "mlp.shared.", L.mlp.shared)
                out[p + "mlp.shared.sg"] = (1, H)
        out.update({p + "side.gate": (S, H), p + "side.proj": (H, S), p + "side.norm": (H,)})
    out.update({"final.norm": (H,), "head": (cfg.vocab, H)})
    return out


def random_tensors(cfg: PotivikConfig, seed: int = 0, std: Optional[float] = None, device="cpu") -> Dict[str, torch.Tensor]:
    """bf16 tensors of a random-init checkpoint: N(0, 1 / fan-in) matrices (or N(0, std^2)), norm weights around one, decays spread
    from short to long memories."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)
    uni = lambda n, lo, hi: lo + (hi - lo) * torch.rand(n, device=device, generator=g)
    out = {}
    for name, s in tensor_shapes(cfg).items():
        if name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 1 + 0.2 * rnd(*s)
        elif name.endswith("A_log"):
            t = uni(s[0], -1.0, 2.0)
        elif name.endswith("dt_bias"):
            t = uni(s[0], -5.0, -1.0)
        elif name.endswith(".D"):
            t = rnd(*s)
        elif name.endswith(".conv"):
            t = 0.6 * rnd(*s)
        elif name.endswith(".conv.b"):
            t = 0.1 * rnd(*s)
        elif name in ("embed", "side.embed"):
            t = rnd(*s)
        else:
            t = rnd(*s) * (std or s[1] ** -0.5)
        out[name] = t.to(BF)
    return out


# ---------------------------------------------------------------------------------------------- packed weights
@dataclass
class Packed:
    """Kernel-ready weights of one layer."""
    norm1: torch.Tensor                        # fp32 [Hp]
    norm1b: torch.Tensor
    w_in: QuantLinear                          # every projection of the mixer's input
    w_out: QuantLinear                         # [Hp, mixer outputs]
    side_gate: QuantLinear
    side_proj: QuantLinear
    side_norm: torch.Tensor
    latent: Optional[mx.LatentHeads] = None
    expand: Optional[QuantLinear] = None       # latent.w_up as a linear
    state: Optional[mx.StateHeads] = None
    z_off: int = 0                             # state space: the gate's columns of w_in
    part_norm: Optional[torch.Tensor] = None   # fp32 [inner]
    norm2: Optional[torch.Tensor] = None
    norm2b: Optional[torch.Tensor] = None
    gate_up: Optional[QuantLinear] = None      # dense feed-forward
    down: Optional[QuantLinear] = None
    moe: Optional[RowExperts] = None

    @property
    def n_out(self) -> int:
        return self.w_out.k

    def matrices(self) -> List[QuantLinear]:
        return [w for w in (self.w_in, self.w_out, self.expand, self.gate_up, self.down, self.side_gate, self.side_proj) if w is not None]


class PotivikModel:
    def __init__(self, cfg: PotivikConfig, embed: torch.Tensor, side: torch.Tensor, layers: List[Packed], final_norm: torch.Tensor, head: QuantLinear,
                 dtype: torch.dtype):
        self.cfg, self.embed, self.side, self.layers, self.final_norm, self.head, self.dtype = cfg, embed, side, layers, final_norm, head, dtype
        self.tp_size, self.tp_rank = 1, 0

    @property
    def hp(self) -> int:
        return self.embed.shape[1]

    @staticmethod
    def from_tensors(cfg: PotivikConfig, get: Callable[[str], torch.Tensor], device="cuda", dtype: torch.dtype = BF) -> "PotivikModel":
        """Packs the checkpoint tensors `get(name)` returns; shapes are checked against the configuration."""
        shapes = tensor_shapes(cfg)
        H, Hp, S, Sp = cfg.width, up8(cfg.width), cfg.side, up8(cfg.side)
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

        def latent(p: str, m: LatentSpec) -> dict:
            DN, DV, KC, RP = mx.latent_widths(m.dim, m.rot_dim, m.vdim, m.kv_rank)
            q = t(p + "q").view(m.heads, m.dim + m.rot_dim, H)
            q = torch.cat([F.pad(q[:, :m.dim], (0, 0, 0, DN - m.dim)), F.pad(q[:, m.dim:], (0, 0, 0, RP - m.rot_dim))], 1).reshape(-1, H)
            down = t(p + "dkv")
            w_in, off = stack([q, pad_rows(down[:m.kv_rank], 1, m.kv_rank, KC), pad_rows(down[m.kv_rank:], 1, m.rot_dim, RP),
                               pad_rows(t(p + "g"), 1, m.heads, up8(m.heads))])
            ups = torch.cat([pad_rows(t(p + "uk"), m.heads, m.dim, DN), pad_rows(t(p + "uv"), m.heads, m.vdim, DV)])
            expand = lin(pad_cols(ups, 1, m.kv_rank, KC))
            g = mx.LatentHeads(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window, m.scale, cfg.eps, m.base, m.rot, off[0], off[1], off[3],
                               t(p + "dkv.norm").contiguous(), expand.payload)
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(p + "o"), m.heads, m.vdim, DV))), latent=g, expand=expand)

        def state_space(p: str, m: StateSpaceSpec) -> dict:
            N, V = mx.pad_to(m.state, mx.STATE_WIDTHS), mx.pad_to(m.vdim, mx.STATE_WIDTHS)
            gn = m.groups * m.state

            def channels(w):                                        # published order x | B | C -> C | B | x, padded per head
                x, B, C = w.split([m.inner, gn, gn])
                return torch.cat([pad_rows(C, m.groups, m.state, N), pad_rows(B, m.groups, m.state, N), pad_rows(x, m.heads, m.vdim, V)])

            z, xbc, dt = t(p + "in").split([m.inner, m.channels, m.heads])
            w_in, off = stack([channels(xbc), pad_rows(dt, 1, m.heads, up8(m.heads)), pad_rows(z, 1, m.inner, up8(m.inner))])
            vec = lambda name: t(p + name).contiguous()
            s = mx.StateHeads(m.heads, m.groups, m.state, m.vdim, off[0], off[1], cfg.eps, channels(t(p + "conv")).T.contiguous(), vec("A_log"),
                              vec("dt_bias"), conv_b=channels(t(p + "conv.b")[:, None]).reshape(-1).contiguous(), skip=vec("D"))
            return dict(w_in=w_in, w_out=lin(hout(pad_cols(t(p + "o"), 1, m.inner, up8(m.inner)))), state=s, z_off=off[2], part_norm=vec("norm"))

        def gate_up(p: str, f: FeedForward) -> torch.Tensor:
            fp = up8(f.ff)
            return hid(torch.cat([pad_rows(t(p + "gate"), 1, f.ff, fp), pad_rows(t(p + "up"), 1, f.ff, fp)]))

        down = lambda p, f: hout(pad_cols(t(p + "down"), 1, f.ff, up8(f.ff)))

        def experts(p: str, m: ExpertsSpec) -> RowExperts:
            blocks = [hid(pad_rows(t(p + "router"), 1, m.experts, up8(m.experts)))]
            kw = {}
            if m.shared is not None:
                blocks += [hid(pad_rows(t(p + "shared.sg"), 1, 1, 8)), gate_up(p + "shared.", m.shared)]
                kw = dict(sg_col=up8(m.experts), shared_col=up8(m.experts) + 8, shared_ff=up8(m.shared.ff), shared_limit=m.shared.limit,
                          shared_down=lin(down(p + "shared.", m.shared)))
            cat = lambda f: torch.cat([f(f"{p}e{e}.", m.expert).to(dtype) for e in range(m.experts)]).contiguous()
            return RowExperts(m.experts, m.top, up8(m.expert.ff), m.expert.limit, lin(torch.cat(blocks)), cat(gate_up), cat(down), Hp, **kw)

        layers = []
        for i, L in enumerate(cfg.plan):
            p = f"l{i}."
            mixer = latent(p + "mix.", L.mixer) if isinstance(L.mixer, LatentSpec) else state_space(p + "mix.", L.mixer)
            w = Packed(hvec(p + "norm1"), hvec(p + "norm1b"), side_gate=lin(hid(pad_rows(t(p + "side.gate"), 1, S, Sp))),
                       side_proj=lin(hout(pad_cols(t(p + "side.proj"), 1, S, Sp))), side_norm=hvec(p + "side.norm"), **mixer)
            if L.mlp is not None:
                w.norm2, w.norm2b = hvec(p + "norm2"), hvec(p + "norm2b")
            if isinstance(L.mlp, FeedForward):
                w.gate_up, w.down = lin(gate_up(p + "mlp.", L.mlp)), lin(down(p + "mlp.", L.mlp))
            elif L.mlp is not None:
                w.moe = experts(p + "mlp.", L.mlp)
            layers.append(w)
        side = pad_cols(t("side.embed"), cfg.layers, S, Sp).to(dtype).contiguous()
        return PotivikModel(cfg, hid(t("embed")).to(dtype).contiguous(), side, layers, hvec("final.norm"), lin(hid(t("head"))), dtype)

    @staticmethod
    def random_init(cfg: PotivikConfig, device="cuda", seed: int = 0, std: Optional[float] = None, dtype: torch.dtype = BF) -> "PotivikModel":
        w = random_tensors(cfg, seed, std, device)
        return PotivikModel.from_tensors(cfg, w.__getitem__, device, dtype)

    def weight_bytes(self) -> int:
        return self.head.nbytes + sum(sum(w.nbytes for w in L.matrices()) + (L.moe.nbytes if L.moe is not None else 0) for L in self.layers)

    # ------------------------------------------------------------------ oracle
    @torch.no_grad()
    def forward_reference(self, tokens: torch.Tensor) -> torch.Tensor:
        """fp32 logits [T, V] of one request from position 0, on the packed weights (fp32 arithmetic, any device)."""
        c, n = self.cfg, self.cfg.width
        ids = tokens.to(self.embed.device).long()
        x = self.embed.float()[ids]
        rms = lambda v, w, n: v * torch.rsqrt(v.pow(2).sum(-1, keepdim=True) / n + c.eps) * w

        def norm(v, w):
            d = torch.cat([v[:, :n] - v[:, :n].mean(-1, keepdim=True), v[:, n:]], 1)
            return rms(d, w, n)

        mm = lambda v, w: v @ w.payload.float().T

        def glu(gu, limit):
            g, u = gu.chunk(2, -1)
            g = g.clamp(max=limit)
            return g * torch.sigmoid(GLU_ALPHA * g) * (u.clamp(-limit, limit) + 1)

        def experts(b: RowExperts, h):
            first = mm(h, b.w_first)
            score = torch.sigmoid(first[:, :b.experts])
            best = torch.argsort(-score, dim=-1, stable=True)[:, :b.top]
            gu, down = b.w_gu.float().view(b.experts, 2 * b.ff, -1), b.w_down.float().view(b.experts, b.hidden, -1)
            out = torch.zeros_like(h)
            for r in range(h.shape[0]):
                for e in best[r].tolist():
                    out[r] += glu((h[r] * score[r, e]) @ gu[e].T, b.limit) @ down[e].T
            if b.shared_ff:
                shared = mm(glu(first[:, b.shared_col:b.shared_col + 2 * b.shared_ff], b.shared_limit), b.shared_down)
                out = out + torch.sigmoid(first[:, b.sg_col:b.sg_col + 1]) * shared
            return out

        for i, (L, P) in enumerate(zip(c.plan, self.layers)):
            proj = mm(norm(x, P.norm1), P.w_in)
            mixed = self._latent_reference(P, proj, rms) if P.latent is not None else self._state_reference(L.mixer, P, proj, rms)
            x = x + norm(mm(mixed, P.w_out), P.norm1b)
            if L.mlp is not None:
                h = norm(x, P.norm2)
                x = x + norm(experts(P.moe, h) if P.moe is not None else mm(glu(mm(h, P.gate_up), L.mlp.limit), P.down), P.norm2b)
            Sp = P.side_gate.n
            g = F.gelu(mm(x, P.side_gate), approximate="tanh") * self.side.float()[ids, i * Sp:(i + 1) * Sp]
            x = x + rms(mm(g, P.side_proj), P.side_norm, n)
        logits = mm(norm(x, self.final_norm), self.head)
        return c.softcap * torch.tanh(logits / c.softcap)

    def _latent_reference(self, P: Packed, proj, rms):
        T, g = proj.shape[0], P.latent
        ang = torch.arange(T, device=proj.device)[:, None] * g.freq.double().sum(0)
        cos, sin = ang.cos().float(), ang.sin().float()

        def turn(v):                                                # [T, ..., RP]
            shape = (T,) + (1,) * (v.dim() - 2) + (-1,)
            c, s = cos.view(shape), sin.view(shape)
            a, b = v[..., 0:g.rot:2], v[..., 1:g.rot:2]
            return torch.cat([torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2), v[..., g.rot:]], -1)

        q = proj[:, g.q_off:g.kv_off].view(T, g.heads, g.DN + g.RP)
        lat = proj[:, g.kv_off:g.kv_off + g.KC]
        lat = rms(lat, F.pad(g.norm_w, (0, g.KC - g.rank)), g.rank)
        flat = lat @ g.w_up.float().T
        k = flat[:, :g.heads * g.DN].view(T, g.heads, g.DN)
        kr = turn(proj[:, g.kv_off + g.KC:g.kv_off + g.cache_cols])
        score = torch.einsum("ihd,jhd->hij", q[:, :, :g.DN], k) + torch.einsum("ihd,jd->hij", turn(q[:, :, g.DN:]), kr)
        i = torch.arange(T, device=proj.device)
        dist = i[:, None] - i[None, :]
        p = (score * g.scale).masked_fill((dist < 0) | (dist >= g.window), float("-inf")).softmax(-1)
        out = torch.einsum("hij,jhd->ihd", p, flat[:, g.heads * g.DN:].view(T, g.heads, g.DV))
        return (out * torch.sigmoid(proj[:, g.g_off:g.g_off + g.heads])[:, :, None]).reshape(T, -1)

    def _state_reference(self, m: StateSpaceSpec, P: Packed, proj, rms):
        T, s = proj.shape[0], P.state
        hist = F.pad(proj[:, s.c_off:s.c_off + s.channels], (0, 0, s.taps - 1, 0))
        act = F.silu(sum(hist[j:j + T] * s.conv_w[j] for j in range(s.taps)) + s.conv_b)
        nk, ratio = s.hk * s.DK, s.hv // s.hk
        C, B = (act[:, a:a + nk].view(T, s.hk, s.DK).repeat_interleave(ratio, 1) for a in (0, nk))
        v = act[:, 2 * nk:].view(T, s.hv, s.DV)
        dt = F.softplus(proj[:, s.b_off:s.b_off + s.hv] + s.dt_bias)
        a = torch.exp(-torch.exp(s.A_log) * dt)
        S, outs = proj.new_zeros(s.hv, s.DK, s.DV), []
        for t in range(T):
            S = S * a[t, :, None, None] + (dt[t, :, None] * B[t])[:, :, None] * v[t, :, None, :]
            outs.append(torch.einsum("hkv,hk->hv", S, C[t]) + s.skip[:, None] * v[t])
        y = torch.stack(outs)[:, :, :s.vdim].reshape(T, -1) * F.silu(proj[:, P.z_off:P.z_off + m.inner])
        n = m.inner // m.norm_groups
        y = rms(y.view(T, m.norm_groups, n), P.part_norm.view(m.norm_groups, n), n).reshape(T, -1)
        return F.pad(y, (0, P.n_out - m.inner))


# ---------------------------------------------------------------------------------------------- kernel runner
class PotivikRunner(RowRunner):
    """Executes the model on the sm_100a kernels.  A request holds pages of the shared latent pool (one table for all attention
    layers) and one slot of every state layer's fp32 memory; both are reused without clearing (a request's first token starts from
    zero states)."""

    mixed_runs = True

    def __init__(self, model: PotivikModel, max_rows: int, slots: int, max_seq_len: int, device, pool_tokens: int = 0):
        c = model.cfg
        self.m, self.model, self.c = model, model, c
        max_rows = max(max_rows, slots)
        T = model.dtype
        self.kv_index = {i: j for j, i in enumerate(i for i, P in enumerate(model.layers) if P.latent is not None)}
        heads = [model.layers[i].latent for i in self.kv_index]
        self._init_pool(slots, device, [(1, g.cache_cols, 0) for g in heads], T, c.page, max_seq_len, max_rows, pool_tokens)
        self.states = {i: P.state.new_state(slots, device) for i, P in enumerate(model.layers) if P.state is not None}
        e = lambda n, dt: torch.empty(n, dtype=dt, device=device)
        R, Hp = max_rows, model.hp
        big = lambda vals: max(list(vals) + [1])
        stream = lambda dt: e(R * Hp, dt).view(R, Hp)
        self.x, self.dx, self.xn = stream(torch.float32), stream(torch.float32), stream(T)
        self.proj = e(R * big(P.w_in.n for P in model.layers), T)
        self.mixed = e(R * big(P.n_out for P in model.layers), T)
        states = [P.state for P in model.layers if P.state is not None]
        self.o = e(R * big(s.hv * s.vdim for s in states), torch.float32)
        self.prep = e(big(s.prep_floats(R, slots) for s in states), torch.float32)
        self.gu = e(R * big(P.gate_up.n for P in model.layers if P.gate_up is not None), T)
        self.act = e(R * big(P.down.k for P in model.layers if P.down is not None), T)
        self.moe = RowExpertsScratch([P.moe for P in model.layers if P.moe is not None], R, T, device)
        self.sg = e(R * big(P.side_gate.n for P in model.layers), torch.float32)
        self.sv = e(R * big(P.side_gate.n for P in model.layers), T)
        # latent attention: absorbed queries and outputs of single rows, split partials, expanded keys and values of prompt runs
        self.tc_prefill = True
        self.max_span = self.kv.max_blocks * c.page
        self.max_splits = 16
        absorbed = [g for g in heads if not g.tc_runs(T)]
        rows_abs = R if absorbed else min(R, slots * ABSORB_RUN)
        self.q_abs = e(rows_abs * big(g.heads * g.cache_cols for g in heads), torch.float32)
        self.lat = e(rows_abs * big(g.heads * g.KC for g in heads), torch.float32)
        self.scratch = (e(slots * big(g.heads for g in heads) * self.max_splits * 2, torch.float32),
                        e(slots * big(g.heads * g.KC for g in heads) * self.max_splits, torch.float32))
        runs = [g for g in heads if g.tc_runs(T)]
        flat_rows = R + slots * (min(big(g.window for g in runs), self.max_span) + 2 * c.page)
        self.flat = e(flat_rows * max([g.flat_cols for g in runs] + [0]), T)
        self.gathered = e(flat_rows * max([g.cache_cols for g in runs] + [0]), T)
        self.capture: Optional[list] = None        # a list: receives the residual stream after every layer (tests, debugging)

    def _state_tensors(self):
        return [t for pair in self.states.values() for t in pair if t is not None]

    def _lin(self, x: torch.Tensor, w: QuantLinear, out: torch.Tensor) -> torch.Tensor:
        if w.fmt == "bf16" and out.dtype == torch.float32:
            return ops.gemm_tc(x, w, out32=out)
        return ops.linear(x, w, out=out)

    # ---- latent attention
    def _plan_runs(self, runs: RowRuns):
        """Splits a pass into runs that attend over expanded keys (per window: which pages, where) and single rows that attend in
        the absorbed form; one upload for all tables."""
        page = self.c.page
        short, long, start = runs.split(ABSORB_RUN)
        windows = sorted({P.latent.window for P in self.m.layers if P.latent is not None and P.latent.tc_runs(self.m.dtype)})
        host = short + [start[r] for r in long] + [runs.lens[r] for r in long]
        parts = []
        for w in windows if long else []:
            base, pages = [], []
            for r in long:
                first = max(0, runs.pos0[r] + 1 - w) // page
                last = (runs.pos0[r] + runs.lens[r] - 1) // page
                base.append((len(pages) - first) * page)
                pages += self.kv.req_blocks[runs.slots[r]][first:last + 1]
            parts.append((w, len(host), len(pages)))
            host += base + pages
        dev = torch.tensor(host, dtype=torch.int32).to(self.dev) if host else None
        n, k = len(short), len(long)
        tiles = sum(-(-runs.lens[r] // 128) for r in long)
        by_window = {w: mx.LatentRuns(dev[n:n + k], dev[n + k:n + 2 * k], dev[o:o + k], dev[o + k:o + k + np], tiles) for w, o, np in parts}
        return (dev[:n] if n else None), by_window

    def _absorbed(self, g: mx.LatentHeads, proj, mixed, positions, row_req, cache, rows: int, row_list, fused: bool) -> None:
        bt, page = self.kv.block_table, self.c.page
        mx.latent_absorb(g, proj, positions, row_req, bt, cache, page, self.q_abs, rows, row_list, fused)
        splits = mx.latent_splits(rows, g.heads, min(g.window, self.max_span), self.max_splits) if rows <= self.slots else 1
        mx.latent_attn(g, self.q_abs, cache, bt, row_req, positions, page, self.lat, rows, row_list, splits, self.scratch)
        mx.latent_up(g, self.lat, proj, mixed, rows, row_list)

    def _latent(self, i: int, P: Packed, proj, mixed, positions, row_req, runs: Optional[RowRuns], plan) -> None:
        g, cache, rows = P.latent, self.kv.layers[self.kv_index[i]].k, proj.shape[0]
        if runs is None:
            return self._absorbed(g, proj, mixed, positions, row_req, cache, rows, None, True)
        mx.latent_append(g, proj, positions, row_req, self.kv.block_table, cache, self.c.page)
        if not (self.tc_prefill and g.tc_runs(proj.dtype)):
            return self._absorbed(g, proj, mixed, positions, row_req, cache, rows, None, False)
        short, by_window = plan
        lr = by_window.get(g.window)
        if lr is not None:
            n = lr.pages.numel() * self.c.page
            gathered = mx.latent_gather(cache, lr.pages, self.gathered[:n * g.cache_cols].view(n, g.cache_cols), self.c.page)
            flat = self._lin(gathered[:, :g.KC], P.expand, self.flat[:n * g.flat_cols].view(n, g.flat_cols))
            mx.latent_prefill(g, proj, flat, gathered, row_req, positions, lr, mixed)
        if short is not None:
            self._absorbed(g, proj, mixed, positions, row_req, cache, short.numel(), short, False)

    # ---- state space
    def _state_space(self, i: int, P: Packed, proj, mixed, positions, row_req, runs: Optional[RowRuns]) -> None:
        m, rows = self.c.plan[i].mixer, proj.shape[0]
        o = self.o[:rows * m.inner].view(rows, m.inner)
        mx.linear_state(P.state, proj, *self.states[i], row_req, positions, runs=runs, prep=self.prep, o=o)
        mx.gated_part_norm(o, proj[:, P.z_off:], P.part_norm, mixed, m.norm_groups, self.c.eps)

    def _layers(self, tokens, positions, row_req, runs: Optional[RowRuns]) -> torch.Tensor:
        """-> the final norm's rows."""
        m, c, rows = self.m, self.c, tokens.shape[0]
        x, xn, dx = self.x[:rows], self.xn[:rows], self.dx[:rows]
        view = lambda buf, n: buf[:rows * n].view(rows, n)
        step = lambda delta, post, pre: mx.stream_norm(x, c.width, c.eps, xn, delta, post, pre)
        plan = self._plan_runs(runs) if runs is not None and self.kv_index else None
        mx.embed_rows(tokens, m.embed, x)
        step(None, (None, None), ("layer", m.layers[0].norm1 if m.layers else m.final_norm))
        for i, P in enumerate(m.layers):
            proj, mixed = self._lin(xn, P.w_in, view(self.proj, P.w_in.n)), view(self.mixed, P.n_out)
            if P.latent is not None:
                self._latent(i, P, proj, mixed, positions, row_req, runs, plan)
            else:
                self._state_space(i, P, proj, mixed, positions, row_req, runs)
            delta, post = self._lin(mixed, P.w_out, dx), ("layer", P.norm1b)
            if P.norm2 is not None:
                step(delta, post, ("layer", P.norm2))
                if P.moe is not None:
                    delta = run_experts(P.moe, self.moe, xn)
                else:
                    act = mx.clamped_glu(self._lin(xn, P.gate_up, view(self.gu, P.gate_up.n)), view(self.act, P.down.k), c.plan[i].mlp.limit, GLU_ALPHA)
                    delta = self._lin(act, P.down, dx)
                post = ("layer", P.norm2b)
            step(delta, post, (None, None))
            n = P.side_gate.n
            g = mx.token_gate(self._lin(xn, P.side_gate, view(self.sg, n)), tokens, m.side, i * n, view(self.sv, n))
            self._lin(g, P.side_proj, dx)
            step(dx, ("rms", P.side_norm), ("layer", m.layers[i + 1].norm1 if i + 1 < len(m.layers) else m.final_norm))
            if self.capture is not None:
                self.capture.append(x[:, :c.width].clone())
        return xn

    def _head(self, rows: torch.Tensor) -> torch.Tensor:
        logits = self._lin(rows, self.m.head, torch.empty(rows.shape[0], self.c.vocab, dtype=torch.float32, device=self.dev))
        return mx.softcap(logits, self.c.softcap)

    @torch.no_grad()
    def forward(self, tokens, positions, row_req, chunk_slot=None, all_logits=True, pos0=None, extra=None):
        """One new token per row (distinct requests) -> fp32 logits [rows, V]."""
        assert chunk_slot is None, "prompt portions go through forward_runs"
        return self._head(self._layers(tokens, positions, row_req, None))

    @torch.no_grad()
    def forward_runs(self, tokens, positions, row_req, runs: RowRuns, logit_rows: torch.Tensor):
        xn = self._layers(tokens, positions, row_req, runs)
        return self._head(xn.index_select(0, logit_rows)) if logit_rows.numel() else None
