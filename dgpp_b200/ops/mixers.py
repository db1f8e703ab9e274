"""Front ends of the kernels behind models with an fp32 residual stream, sliding-window attention (grouped heads, or a
shared latent), fp32 linear-attention, state-space and matrix memories, and experts of plain rows (``csrc/kernels/stream_ops.cu``,
``short_conv.cu``, ``window_attn.cuh``, ``window_attn_tc.cu``, ``latent_attn.cu``, ``mla_tc.cu``, ``linear_state.cu``, ``gated_delta.cu``,
``state_space.cu``, ``matrix_memory.cu``, ``moe_rows.cu``).  Every operator exists for bf16 and for true fp32 activations; the dtype of the tensors decides."""
from __future__ import annotations

import copy
import ctypes
import functools
from typing import Optional

import torch

from . import _lib
from ._lib import F, I, L, P, call, ptr, stream_ptr

_lib.declare("dgpp_embed_rows", [P, P, P, P, L, I, I, I, F, I, P])
_lib.declare("dgpp_resid_norm", [P, P, P, P, I, I, I, F, I, P])
_lib.declare("dgpp_gated_group_norm", [P, P, P, L, P, I, P, L, I, I, I, I, F, F, I, I, I, P])
_lib.declare("dgpp_geglu", [P, P, I, I, I, P])
_WINDOW = [P, L, I, I, I] + [P] * 11 + [I] * 12 + [F, F, P]
for _form in ("", "_ext"):
    _lib.declare("dgpp_qk_norm_append" + _form, _WINDOW + [I, P])
    _lib.declare("dgpp_window_attn" + _form, _WINDOW + [P, P, P, P, L, I, I, I, I, I, F, F, I, P])
_lib.declare("dgpp_diff_combine", [P, P, P, L, P, P, L, I, I, I, I, I, I, F, F, F, I, P])
_lib.declare("dgpp_state_space", [P, L, I, I, P, P, P, I, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, P])
_lib.declare("dgpp_gated_delta", [P, L, I, I, I, I, P, P, I, P, P, P, P, P, P, P, P, P, P, L, P, I, I, I, I, I, I, I, I, F, F, I, I, P])
_lib.declare("dgpp_linear_state", [P, L, I, I, P, L, P, P, I, P, P, P, P, P, P, P, P, P, P, P, L, P, I, I, I, I, I, I, I, I, F, F,
                                   I, I, I, P])


def _f32(t: torch.Tensor) -> int:
    if t.dtype == torch.float32:
        return 1
    if t.dtype != torch.bfloat16:
        raise TypeError(f"expected bf16 or fp32 activations, got {t.dtype}")
    return 0


def pad_to(n: int, options) -> int:
    """The smallest of `options` (ascending) that holds n columns."""
    for o in options:
        if n <= o:
            return o
    raise ValueError(f"head width {n} is larger than {options[-1]}")


ATTN_WIDTHS = (64, 128, 192, 256)      # padded head widths of the window attention kernels
STATE_WIDTHS = (32, 64, 128, 256)      # padded key / value widths of the linear-state kernels


def embed_rows(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor, scale: float = 1.0, copy: Optional[torch.Tensor] = None) -> torch.Tensor:
    """fp32 rows out[r] = scale * table[ids[r]] (table [vocab, cols] bf16 or fp32); copy [rows, cols] receives them in the table's type."""
    assert copy is None or copy.dtype == table.dtype
    call("dgpp_embed_rows", ptr(ids), ptr(table), ptr(out), ptr(copy), 0 if copy is None else copy.stride(0), ids.numel(), table.shape[1],
         table.shape[0], float(scale), _f32(table), stream_ptr())
    return out


def resid_norm(x: torch.Tensor, w: torch.Tensor, n: int, eps: float, out: torch.Tensor,
               delta: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [rows, cols] fp32 takes in `delta` (fp32) in place; out = rms norm of the sum over its n true columns, times w."""
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous()
    call("dgpp_resid_norm", ptr(x), ptr(delta), ptr(w), ptr(out), x.shape[0], x.shape[1], n, float(eps), _f32(out), stream_ptr())
    return out


def gated_group_norm(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, out: torch.Tensor, groups: int, n: int, eps: float,
                     scale: float = 1.0, silu: bool = False, den: Optional[torch.Tensor] = None) -> torch.Tensor:
    """o [rows, groups * gp] fp32 (divided by den [rows, groups] where it is given) -> rms norm per group (n true columns) * w ([gp], or
    [groups * gp]: a row per group) * sigmoid(gate) (or silu(gate)) * scale."""
    assert o.dtype == torch.float32 and o.is_contiguous() and o.shape[1] % groups == 0
    gp = o.shape[1] // groups
    assert w.numel() in (gp, groups * gp) and (den is None or (den.dtype == torch.float32 and den.numel() >= o.shape[0] * groups))
    call("dgpp_gated_group_norm", ptr(o), ptr(den), ptr(gate), gate.stride(0), ptr(w), gp if w.numel() > gp else 0, ptr(out), out.stride(0), o.shape[0], groups,
         o.shape[1] // groups, n, float(eps), float(scale), int(silu), _f32(out), _f32(gate), stream_ptr())
    return out


def geglu(gate_up: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """gate_up [rows, 2 I] -> gelu_tanh(gate) * up [rows, I]."""
    assert gate_up.is_contiguous() and out.is_contiguous()
    call("dgpp_geglu", ptr(gate_up), ptr(out), gate_up.shape[0], out.shape[1], _f32(out), stream_ptr())
    return out


NORMS = {None: 0, "rms": 1, "layer": 2, "parts": 3}
_lib.declare("dgpp_stream_norm", [P, P, P, P, I, P, P, L, P, P, P, P, P, P, P, F, P, F, I, P, P, I, P, P, I, P, L, I, I, I, F, I, P])
_lib.declare("dgpp_act_rows", [P, L, P, P, I, P, I, I, I, I, I, P])
ACTS = {"relu2": 0, "gelu": 1}         # square of relu; gelu in its erf form
_lib.declare("dgpp_gated_part_norm", [P, P, L, P, P, L, I, I, I, I, F, I, P])
_lib.declare("dgpp_clamped_glu", [P, L, P, P, I, P, I, I, F, F, F, I, I, I, P])
_lib.declare("dgpp_token_gate", [P, P, P, L, I, P, I, I, I, I, P])
_lib.declare("dgpp_softcap", [P, L, F, P])


class PairDelta:
    """The sum of two fp32 row blocks as ``stream_norm`` takes it in: factor * (rms(a + bias_a) * w_a + rms(b + bias_b) * w_b)."""

    def __init__(self, a, w_a, b, w_b, factor: float, bias_a=None, bias_b=None):
        assert a.shape == b.shape
        self.a, self.w_a, self.b, self.w_b, self.factor, self.bias_a, self.bias_b = a, w_a, b, w_b, factor, bias_a, bias_b


def stream_norm(x: torch.Tensor, n: int, eps: float, out: torch.Tensor, delta=None, post=(None, None), pre=(None, None), mult: float = 1.0,
                delta_b=None, vec=None, parts: int = 1) -> torch.Tensor:
    """x [rows, cols] fp32 takes in mult * post(delta + delta_b) + vec in place; out [rows, >= cols] = pre(x).  post / pre:
    (None | "rms" | "layer" | "parts", fp32 weight row[, fp32 bias row]) over the n true columns ("parts": each of `parts` equal runs of
    them on its own).  delta: an fp32 row block, a ``PairDelta``, a ``MoeDelta`` or None; delta_b, vec: fp32 rows or None."""
    assert x.dtype == torch.float32 and x.is_contiguous() and out.stride(1) == 1
    post, pre = (tuple(t) + (None,) * (3 - len(t)) for t in (post, pre))
    m = delta if isinstance(delta, MoeDelta) else None
    two = delta if isinstance(delta, PairDelta) else None
    d = None if m is not None else delta if two is None else two.a
    if two is not None:
        assert delta_b is None and two.b.dtype == torch.float32 and two.b.is_contiguous()
        delta_b = two.bias_a
    assert d is None or (d.dtype == torch.float32 and d.is_contiguous())
    call("dgpp_stream_norm", ptr(x), ptr(d), ptr(m and m.y), ptr(m and m.pair_row), m.top if m else 0, ptr(m and m.shared),
         ptr(m and m.gate), m.gate.stride(0) if m and m.gate is not None else 0, ptr(m and m.self_rows), ptr(m and m.wts), ptr(delta_b),
         ptr(two and two.b), ptr(two and two.bias_b), ptr(two and two.w_a), ptr(two and two.w_b), float(two.factor) if two else 1.0, ptr(vec), float(mult),
         NORMS[post[0]], ptr(post[1]), ptr(post[2]), NORMS[pre[0]], ptr(pre[1]), ptr(pre[2]), parts, ptr(out), out.stride(0), x.shape[0], x.shape[1], n,
         float(eps), _f32(out), stream_ptr())
    return out


def act_rows(x: torch.Tensor, out: torch.Tensor, act: str, row_w=None, tiles=None, bn: int = 1) -> torch.Tensor:
    """x [rows, >= I] -> row_w * act(x) [rows, I] (``ACTS``).  tiles [rows / bn]: rows of tiles with a negative entry are skipped."""
    assert out.is_contiguous() and x.shape[1] >= out.shape[1]
    call("dgpp_act_rows", ptr(x), x.stride(0), ptr(row_w), ptr(tiles), bn, ptr(out), out.shape[0], out.shape[1], ACTS[act], _f32(out), _f32(x), stream_ptr())
    return out


def gated_part_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, out: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """a = y * silu(z) (y [rows, n] fp32, z's first n columns); out = a / rms of each of `parts` equal runs of columns * w [n]; the
    columns of `out` behind n are cleared."""
    n = y.shape[1]
    assert y.dtype == torch.float32 and y.is_contiguous() and n % parts == 0 and w.numel() == n and out.shape[1] >= n
    call("dgpp_gated_part_norm", ptr(y), ptr(z), z.stride(0), ptr(w), ptr(out), out.stride(0), y.shape[0], parts, n // parts, out.shape[1],
         float(eps), _f32(out), stream_ptr())
    return out


def clamped_glu(gate_up: torch.Tensor, out: torch.Tensor, limit: float, alpha: float = 1.702, row_w=None, tiles=None, bn: int = 1,
                shift: float = 1.0, weigh_out: bool = False) -> torch.Tensor:
    """gate_up [rows, 2 I] -> min(s g, limit) sigmoid(alpha min(s g, limit)) (clamp(s u, +-limit) + shift) [rows, I]; s: `row_w` or one
    (weigh_out: the row's weight multiplies the result instead).  limit inf, alpha 1, shift 0: silu(g) u.  tiles [rows / bn]: rows of tiles with a negative entry are skipped."""
    assert out.is_contiguous() and gate_up.shape[1] >= 2 * out.shape[1]
    call("dgpp_clamped_glu", ptr(gate_up), gate_up.stride(0), ptr(row_w), ptr(tiles), bn, ptr(out), gate_up.shape[0], out.shape[1], float(limit),
         float(alpha), float(shift), int(weigh_out), _f32(out), _f32(gate_up), stream_ptr())
    return out


def token_gate(gate: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, col: int, out: torch.Tensor) -> torch.Tensor:
    """gelu_tanh(gate) * table[ids[r], col : col + dim] (gate [rows, dim] fp32)."""
    assert gate.dtype == torch.float32 and gate.is_contiguous() and out.is_contiguous() and table.dtype == out.dtype
    call("dgpp_token_gate", ptr(gate), ptr(ids), ptr(table), table.stride(0), col, ptr(out), gate.shape[0], out.shape[1], table.shape[0],
         _f32(out), stream_ptr())
    return out


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    """x (fp32, in place) = cap * tanh(x / cap)."""
    assert x.dtype == torch.float32 and x.is_contiguous()
    call("dgpp_softcap", ptr(x), x.numel(), float(cap), stream_ptr())
    return x


# ---------------------------------------------------------------------------------------------- experts over plain rows
_lib.declare("dgpp_moe_select", [P, L, P, P, P, P, I, I, I, I, I, F, P])
_lib.declare("dgpp_moe_route_small", [P, L, P, P, P, P, P, P, I, I, I, I, I, I, I, P])
_lib.declare("dgpp_moe_scatter_rows", [P, P, P, P, P, I, I, I, I, P])
_lib.declare("dgpp_gemm_tc_grouped", [I, P, L, I, I, P, I, P, P, I, I, I, I, P])
_lib.declare("dgpp_gemm_f32_grouped", [I, P, L, I, I, P, I, P, P, L, I, I, I, P])
SMALL_TOKENS = 16                      # rows up to which routing is one launch and every listed expert reads all rows
MAX_EXPERTS, MAX_TOP = 512, 16
SCORES = {"sigmoid": 0, "softmax": 1, "chosen": 2}      # of the logit; softmax over all experts; softmax over the chosen ones only


class MoeDelta:
    """The rows of a mixture of experts as ``stream_norm`` takes them in: sum over j of y[pair_row[r * top + j]] (negative
    entries: wts[r * top + j] * self_rows[r], or nothing), plus sigmoid(gate[r]) * shared[r] (no gate: shared[r])."""

    def __init__(self, y, pair_row, top: int, shared=None, gate=None, self_rows=None, wts=None):
        self.y, self.pair_row, self.top, self.shared, self.gate, self.self_rows, self.wts = y, pair_row, top, shared, gate, self_rows, wts


def moe_select(logits: torch.Tensor, experts: int, top: int, ids: torch.Tensor, weights: torch.Tensor, score: str = "sigmoid",
               norm_topk: bool = False, scaling: float = 1.0, bias=None, correction=None) -> None:
    """The `top` best of the first `experts` columns of fp32 logits (+ bias [experts] fp32) per row -> ids (ascending), weights.
    correction [experts] fp32: added to the scores for the choice alone."""
    call("dgpp_moe_select", ptr(logits), logits.stride(0), ptr(bias), ptr(correction), ptr(ids), ptr(weights), logits.shape[0], experts, top, SCORES[score], int(norm_topk),
         float(scaling), stream_ptr())


def moe_route_small(logits: torch.Tensor, experts: int, top: int, pair_row, tiles, row_w, score: str = "sigmoid", bias=None, correction=None,
                    norm_topk: bool = False, identity: int = 0, wts=None) -> None:
    """Up to 16 rows: tiles (experts in use), pair_row [rows * top] = tile * 16 + row, row_w [tiles * 16].  identity: that many outputs behind
    the first `experts` are identity experts, whose pairs get row -1; wts [rows * top] takes the pairs' weights."""
    call("dgpp_moe_route_small", ptr(logits), logits.stride(0), ptr(bias), ptr(correction), ptr(pair_row), ptr(tiles), ptr(row_w), ptr(wts), logits.shape[0],
         experts + identity, experts, top, tiles.numel(), SCORES[score], int(norm_topk), stream_ptr())


def moe_scatter_rows(x: torch.Tensor, pair_row, weights, xs, row_w, top: int) -> None:
    """xs[pair_row[p]] = x[p // top], row_w[pair_row[p]] = weights[p]."""
    assert x.is_contiguous() and xs.is_contiguous() and x.shape[1] == xs.shape[1]
    call("dgpp_moe_scatter_rows", ptr(x), ptr(pair_row), ptr(weights), ptr(xs), ptr(row_w), x.shape[0], x.shape[1], top, _f32(x), stream_ptr())


def grouped_linear(x: torch.Tensor, w: torch.Tensor, n: int, tiles: torch.Tensor, bn: int, out: torch.Tensor, shared_rows: bool = False) -> torch.Tensor:
    """Tile t of `out` [tiles * bn, n] = its rows of x times matrix tiles[t] of the stack w [experts * n, k] (negative: skipped).
    shared_rows: every tile reads the same x [<= bn, k]."""
    assert w.dtype == x.dtype == out.dtype and w.shape[0] % n == 0 and w.shape[1] == x.shape[1] and w.is_contiguous()
    call("dgpp_gemm_f32_grouped" if _f32(x) else "dgpp_gemm_tc_grouped", bn, ptr(x), x.stride(0), x.shape[0], int(not shared_rows), ptr(w),
         w.shape[0] // n, ptr(tiles), ptr(out), out.stride(0), tiles.numel(), n, w.shape[1], stream_ptr())
    return out


NO_WINDOW = 1 << 30                    # a window that nobody fills: every earlier key is visible


class WindowHeads:
    """Static description of one attention block inside a fused projection row.  `window` keys (chunked: the keys of the row's own
    chunk of `window` positions, counted from 0).  norm: "head" or "row" (over the whole projection) or None; biases fp32, padded as
    the heads are; freq: ``rotation_freqs`` of the first `rot` columns, paired (i, i + rot / 2); temp: (coef, every) of the query
    temperature; gate_off: column with one output gate per head.  maps 2: differential attention, query heads laid out
    [kv head][map][head of the group], `heads` counts output heads.  keep_first: the first tokens that every row sees; softcap: scores
    become cap * tanh(score / cap); sink: fp32 [heads], a number per head in the softmax's denominator.  conv_w: fp32 [taps, channels], a
    causal convolution over time on the channels q | k | v (behind the biases).  vnorm: values are divided by their root mean square;
    vfreq: ``value_freqs``, values are rotated by their position (halves of the padded width) and outputs turned back."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, window: int, scale: float, eps: float,
                 q_off: int, k_off: int, v_off: int, norm: Optional[str] = "head", bias=(None, None, None), freq=None, rot: int = 0,
                 temp=(0.0, 1), gate_off: int = -1, maps: int = 1, chunked: bool = False, keep_first: int = 0, softcap: float = 0.0,
                 sink=None, conv_w=None, vnorm: bool = False, vfreq=None):
        self.hq, self.hkv, self.dim, self.vdim, self.window, self.scale, self.eps = heads * maps, kv_heads, dim, vdim, window, scale, eps
        self.D, self.DV = pad_to(dim, ATTN_WIDTHS), pad_to(vdim, ATTN_WIDTHS)
        self.q_off, self.k_off, self.v_off = q_off, k_off, v_off
        self.norm, self.bias, self.freq, self.rot, self.temp, self.gate_off = norm, bias, freq, rot, temp, gate_off
        self.maps, self.chunked, self.group = maps, chunked, heads // kv_heads
        self.keep_first, self.softcap, self.sink, self.conv_w, self.vnorm, self.vfreq = keep_first, softcap, sink, conv_w, vnorm, vfreq

    @property
    def channels(self) -> int:
        return (self.hq + self.hkv * self.maps) * self.D + self.hkv * self.DV

    @property
    def taps(self) -> int:
        return 0 if self.conv_w is None else self.conv_w.shape[0]

    @property
    def ext(self) -> bool:
        """Whether these heads take the kernels' form with extras."""
        return bool(self.keep_first or self.softcap or self.sink is not None or self.conv_w is not None or self.vnorm or self.vfreq is not None)

    def new_ring(self, slots: int, device) -> Optional[torch.Tensor]:
        """History of the convolution [slots, taps, channels] fp32.  Needs no clearing between requests."""
        return torch.zeros(slots, self.taps, self.channels, dtype=torch.float32, device=device) if self.taps else None

    @functools.cached_property
    def after_conv(self) -> "WindowHeads":
        """The same heads over the rows that ``short_conv`` writes."""
        g = copy.copy(self)
        g.q_off, g.k_off, g.v_off = 0, self.hq * self.D, (self.hq + self.hkv * self.maps) * self.D
        g.bias, g.conv_w = (None, None, None), None
        return g

    @functools.cached_property
    def stacked_bias(self) -> Optional[torch.Tensor]:
        """The biases of q | k | v as one row."""
        return None if self.bias[0] is None else torch.cat([b.reshape(-1) for b in self.bias])

    @property
    def kv_shape(self):
        """(key heads, key width, value width, value heads) of the cache."""
        return self.hkv * self.maps, self.D, self.DV, self.hkv

    def splits(self, rows: int, max_span: int, most: int) -> int:
        """Splits of single rows' keys: at most one wave of CTAs (four per SM, three with two maps), at least 128 keys each (one more
        split for kept tokens, which lie in front of a window of whole rounds)."""
        chunks = -(-self.group // (8 // self.maps))
        return max(1, min(most, 148 * (5 - self.maps) // (self.hkv * chunks * rows), min(self.window, max_span) // 128 + (self.keep_first > 0)))


def value_freqs(base: float, vdim: int, width: int, device) -> torch.Tensor:
    """``rotation_freqs`` of values of vdim columns in heads of padded width `width`: pairs (m, m + width / 2), still beyond vdim / 2."""
    f = rotation_freqs(base, vdim, device)
    return torch.cat([f, f.new_zeros(2, width // 2 - vdim // 2)], 1).contiguous()


class _WindowExtras(ctypes.Structure):
    """``WindowExtras`` of csrc/kernels/window_attn.cuh."""
    _fields_ = [(n, ctypes.c_void_p) for n in ("vfreq", "turn", "conv_w", "ring", "sink")] + \
               [(n, ctypes.c_int) for n in ("vdim", "vnorm", "taps", "keep_first")] + [("softcap", ctypes.c_float)]


def _wa_common(g: WindowHeads, proj, wq, wk, cache, block_table, row_req, positions, rows: int, ring=None, turn=None):
    coef, every = g.temp
    norm = {None: 0, "head": 1, "row": 2}[g.norm]
    x = None
    if g.ext:
        x = _WindowExtras(ptr(g.vfreq), ptr(turn), ptr(g.conv_w) if ring is not None else None, ptr(ring), ptr(g.sink), g.vdim, int(g.vnorm), g.taps,
                          g.keep_first, float(g.softcap))
        x = ctypes.cast(ctypes.pointer(x), ctypes.c_void_p)
    return (ptr(proj), proj.stride(0), g.q_off, g.k_off, g.v_off, ptr(wq), ptr(wk), *(ptr(b) for b in g.bias), ptr(g.freq), ptr(cache.k), ptr(cache.v),
            ptr(block_table), ptr(row_req), ptr(positions), rows, g.hq, g.hkv, g.maps, g.D, g.DV, g.dim, cache.page, block_table.shape[1], norm,
            g.rot, int(every), float(coef), float(g.eps), x)


def qk_norm_append(g: WindowHeads, proj, wq, wk, cache, block_table, row_req, positions, turn=None) -> None:
    """Prepares the query heads of `proj` in place (bias, norm, rotation, temperature) and appends prepared keys and values to the
    paged cache.  A convolution comes before (``short_conv``; then g is ``WindowHeads.after_conv``).  turn: fp32 [rows, DV] takes the
    angles that ``window_prefill`` needs where values are rotated."""
    assert cache.k.dtype == proj.dtype and g.conv_w is None and (turn is None or turn.numel() >= proj.shape[0] * g.DV)
    call("dgpp_qk_norm_append" + ("_ext" if g.ext else ""), *_wa_common(g, proj, wq, wk, cache, block_table, row_req, positions, proj.shape[0], turn=turn), _f32(proj), stream_ptr())


def window_attn(g: WindowHeads, proj, wq, wk, cache, block_table, row_req, positions, out, out_scale: float = 1.0,
                fused: bool = False, splits: int = 1, scratch=None, row_list=None, ring=None) -> Optional[torch.Tensor]:
    """Every row attends to the positions of its request that it sees, its own included -> out [rows, >= hq * DV].
    fused: the rows are single new tokens; the kernel prepares and appends them itself (with a convolution: over `ring`, which it
    advances).  row_list: int32 subset of rows.
    scratch: (fp32 launch rows * hq * splits * 2, * DV) where splits > 1; with two maps always, and the result stays there for
    ``diff_combine`` (out unused)."""
    assert cache.k.dtype == proj.dtype and (g.maps == 2 or out.dtype == proj.dtype)
    assert g.conv_w is None or (fused and row_list is None and ring.dtype == torch.float32 and ring.shape[1:] == (g.taps, g.channels))
    rows = proj.shape[0] if row_list is None else row_list.numel()
    ml, acc = scratch if splits > 1 or g.maps == 2 else (None, None)
    assert ml is None or (ml.numel() >= rows * g.hq * splits * 2 and acc.numel() >= rows * g.hq * splits * g.DV)
    out = None if g.maps == 2 else out
    call("dgpp_window_attn" + ("_ext" if g.ext else ""), *_wa_common(g, proj, wq, wk, cache, block_table, row_req, positions, rows, ring), ptr(row_list), ptr(ml), ptr(acc),
         ptr(out), 0 if out is None else out.stride(0), splits, g.window, int(g.chunked), int(fused), g.gate_off, float(g.scale), float(out_scale),
         _f32(proj), stream_ptr())
    return out


_lib.declare("dgpp_short_conv", [P, L, P, P, P, P, P, P, P, P, I, I, I, I, I, P])


def short_conv(x: torch.Tensor, bias, w: torch.Tensor, ring: torch.Tensor, row_req, positions, runs, out: torch.Tensor) -> torch.Tensor:
    """out [rows, C] = causal convolution of the first C columns of x (+ bias) over the tokens of every request; w fp32 [taps, C] (last row:
    the current token), ring [slots, taps, C] fp32 carries the newest inputs from pass to pass."""
    taps, C = w.shape
    assert x.dtype == out.dtype and out.is_contiguous() and out.shape == (x.shape[0], C) and ring.shape[1:] == w.shape and ring.dtype == w.dtype == torch.float32
    call("dgpp_short_conv", ptr(x), x.stride(0), ptr(bias), ptr(w), ptr(ring), ptr(row_req), ptr(positions), ptr(runs.row_run0), ptr(runs.start), ptr(out),
         x.shape[0], len(runs.lens), C, taps, _f32(x), stream_ptr())
    return out


def diff_combine(g: WindowHeads, scratch, proj, gate_off: int, out, lam: float, factor: float, splits: int = 1, row_list=None,
                 finished: bool = False) -> torch.Tensor:
    """out [rows, >= heads * DV] = (a1 - lam * a2) / its root mean square per head * factor * sigmoid(gate columns of proj).  scratch as
    ``window_attn`` left it, or (finished) the fp32 outputs [rows, hq, DV] of ``window_prefill``."""
    ml, acc = (None, scratch) if finished else scratch
    rows = proj.shape[0] if row_list is None else row_list.numel()
    gate = proj[:, gate_off:]
    call("dgpp_diff_combine", ptr(ml), ptr(acc), ptr(gate), proj.stride(0), ptr(row_list), ptr(out), out.stride(0), rows, g.hq // 2, g.group, g.DV,
         g.vdim, splits, float(lam), float(factor), float(g.eps), _f32(out), stream_ptr())
    return out


class StateHeads:
    """Static description of one linear-attention block: widths (padded), offsets inside the fused projection row, and the
    constants of its rule (`decay` per head: lightning; `skip` per head with `A_log` / `dt_bias`: state space; a_off / gate_off, the
    columns of the raw decays and output gates: delta rule with a decay per head; `A_log` / `dt_bias` / low-rank rows: channel delta
    rule)."""

    def __init__(self, heads: int, key_heads: int, dim: int, vdim: int, c_off: int, b_off: int = 0, eps: float = 0.0,
                 conv_w=None, A_log=None, dt_bias=None, decay=None, norm_w=None, conv_b=None, skip=None, a_off: int = -1, gate_off: int = 0):
        self.hv, self.hk, self.dim, self.vdim = heads, key_heads, dim, vdim
        self.DK, self.DV = pad_to(dim, STATE_WIDTHS), pad_to(vdim, STATE_WIDTHS)
        self.c_off, self.b_off, self.eps = c_off, b_off, eps
        self.conv_w, self.A_log, self.dt_bias, self.decay, self.norm_w = conv_w, A_log, dt_bias, decay, norm_w
        self.conv_b, self.skip = conv_b, skip
        self.a_off, self.gate_off = a_off, gate_off
        self.delta = decay is None and skip is None
        self.taps = 0 if conv_w is None else conv_w.shape[0]

    @property
    def channels(self) -> int:
        return 2 * self.hk * self.DK + self.hv * self.DV

    def new_state(self, slots: int, device):
        """(state [slots, hv, DK, DV], ring [slots, taps, channels] or None), fp32.  Needs no clearing between requests."""
        state = torch.zeros(slots, self.hv, self.DK, self.DV, dtype=torch.float32, device=device)
        ring = torch.zeros(slots, self.taps, self.channels, dtype=torch.float32, device=device) if self.taps else None
        return state, ring

    def prep_floats(self, rows: int, runs: int) -> int:
        """Scratch of a pass over `rows` rows in at most `runs` runs."""
        blocks = rows // 16 + runs
        if self.skip is not None:
            return rows * (self.channels + 2 * self.hv) + blocks * self.hv * 288
        if self.a_off >= 0:
            return rows * (self.channels + 2 * self.hv) + blocks * self.hv * 576
        return rows * (self.channels + self.hv * (3 * self.DK + 1)) + blocks * self.hv * (self.DK + 512)


def linear_state(g: StateHeads, proj, state, ring, row_slot, positions, low=None, runs=None, prep=None, o=None, out=None) -> None:
    """Advances the states by the rows of `proj`.  runs None: one new token per row; the delta rule then writes its normed and
    gated read-outs to `out`, lightning its raw read-outs to `o` (fp32).  runs given: runs of consecutive rows, raw read-outs
    to `o`, `prep` is fp32 scratch (`StateHeads.prep_floats`)."""
    rows = proj.shape[0]
    blocks = 0 if runs is None else sum(-(-n // 16) for n in runs.lens)
    assert state.dtype == torch.float32 and (runs is None or prep.numel() >= g.prep_floats(rows, len(runs.lens)))
    if g.skip is not None:                       # raw read-outs [rows, heads * vdim] to `o` either way
        call("dgpp_state_space", ptr(proj), proj.stride(0), g.c_off, g.b_off, ptr(g.conv_w), ptr(g.conv_b), ptr(ring), g.taps, ptr(g.A_log),
             ptr(g.dt_bias), ptr(g.skip), ptr(state), ptr(row_slot), ptr(positions), None if runs is None else ptr(runs.start),
             None if runs is None else ptr(runs.row_run0), ptr(prep), ptr(o), rows, rows if runs is None else len(runs.lens), blocks, g.hk, g.hv,
             g.DK, g.DV, g.vdim, int(runs is None), _f32(proj), stream_ptr())
        return
    if g.a_off >= 0:
        call("dgpp_gated_delta", ptr(proj), proj.stride(0), g.c_off, g.b_off, g.a_off, g.gate_off, ptr(g.conv_w), ptr(ring), g.taps, ptr(g.A_log),
             ptr(g.dt_bias), ptr(state), ptr(row_slot), ptr(positions), None if runs is None else ptr(runs.start),
             None if runs is None else ptr(runs.row_run0), ptr(prep), ptr(o), ptr(out), 0 if out is None else out.stride(0), ptr(g.norm_w), rows,
             rows if runs is None else len(runs.lens), blocks, g.hk, g.hv, g.DK, g.DV, g.vdim, float(g.dim ** -0.5), float(g.eps),
             int(runs is None), _f32(proj), stream_ptr())
        return
    call("dgpp_linear_state", ptr(proj), proj.stride(0), g.c_off, g.b_off, ptr(low), 0 if low is None else low.stride(0),
         ptr(g.conv_w), ptr(ring), g.taps, ptr(g.A_log), ptr(g.dt_bias), ptr(g.decay), ptr(state), ptr(row_slot), ptr(positions),
         None if runs is None else ptr(runs.start), None if runs is None else ptr(runs.row_run0), ptr(prep), ptr(o), ptr(out),
         0 if out is None else out.stride(0), ptr(g.norm_w), rows, rows if runs is None else len(runs.lens), blocks, g.hk, g.hv, g.DK, g.DV,
         g.vdim, float(g.dim ** -0.5), float(g.eps), int(g.delta), int(runs is None), _f32(proj), stream_ptr())


_lib.declare("dgpp_matrix_memory", [P, L, I, I, I, I, P, P, F, P, P, P, P, P, P, P, P, P, P, L, P, I, I, I, I, I, I, I, F, F, I, I, P])


class MatrixHeads:
    """Static description of one matrix-memory block (mLSTM): widths (padded), offsets inside the fused projection row (q | k | v from
    c_off, raw input and forget gates, output gates), gate biases fp32 [heads], the gates' cap, norm_w fp32 [heads * DV]."""

    def __init__(self, heads: int, dim: int, vdim: int, c_off: int, i_off: int, f_off: int, gate_off: int, i_bias, f_bias, gate_cap: float, norm_w,
                 eps: float):
        self.heads, self.dim, self.vdim = heads, dim, vdim
        self.DK, self.DV = pad_to(dim, STATE_WIDTHS), pad_to(vdim, STATE_WIDTHS)
        self.c_off, self.i_off, self.f_off, self.gate_off = c_off, i_off, f_off, gate_off
        self.i_bias, self.f_bias, self.gate_cap, self.norm_w, self.eps = i_bias, f_bias, gate_cap, norm_w, eps

    def new_state(self, slots: int, device):
        """(S [slots, heads, DK, DV], n and the running maximum [slots, heads, DK + 4]), fp32.  Needs no clearing between requests."""
        z = lambda *s: torch.zeros(slots, self.heads, *s, dtype=torch.float32, device=device)
        return z(self.DK, self.DV), z(self.DK + 4)

    def prep_floats(self, rows: int, runs: int) -> int:
        """Scratch of a pass over `rows` rows in at most `runs` runs."""
        return self.heads * (rows * (2 * self.DK + self.DV + 3) + (rows // 16 + runs) * 288)


def matrix_memory(g: MatrixHeads, proj, state, nstate, row_slot, positions, runs=None, prep=None, o=None, den=None, out=None) -> None:
    """Advances the memories by the rows of `proj`.  runs None: one new token per row, normed and gated read-outs to `out`.  runs given:
    runs of consecutive rows, raw read-outs to `o` [rows, heads * DV] and their denominators to `den` [rows, heads] (fp32), for
    ``gated_group_norm``; `prep` is fp32 scratch (`prep_floats`)."""
    rows = proj.shape[0]
    blocks = 0 if runs is None else sum(-(-n // 16) for n in runs.lens)
    assert state.dtype == nstate.dtype == torch.float32 and (runs is None or prep.numel() >= g.prep_floats(rows, len(runs.lens)))
    call("dgpp_matrix_memory", ptr(proj), proj.stride(0), g.c_off, g.i_off, g.f_off, g.gate_off, ptr(g.i_bias), ptr(g.f_bias), float(g.gate_cap),
         ptr(state), ptr(nstate), ptr(row_slot), ptr(positions), None if runs is None else ptr(runs.start), None if runs is None else ptr(runs.row_run0),
         ptr(prep), ptr(o), ptr(den), ptr(out), 0 if out is None else out.stride(0), ptr(g.norm_w), rows, rows if runs is None else len(runs.lens), blocks,
         g.heads, g.DK, g.DV, g.vdim, float(g.dim ** -0.5), float(g.eps), int(runs is None), _f32(proj), stream_ptr())


_lib.declare("dgpp_window_attn_tc", [P, L, I] + [P] * 8 + [L, P] + [I] * 13 + [F, F, P, P, I, F, P])


def window_prefill_usable(g: WindowHeads, proj, page: int = 64) -> bool:
    """Whether the tensor-core kernel takes these rows (bf16, pages of 64 tokens, at most 128 query heads per key head)."""
    return proj.dtype == torch.bfloat16 and page == 64 and g.group <= 128


def window_tiles(g: WindowHeads, lens) -> int:
    """CTAs per key head of ``window_prefill`` over runs of these lengths."""
    per = 128 // g.group
    return sum(-(-n // per) for n in lens)


def window_prefill(g: WindowHeads, proj, cache, block_table, row_req, positions, runs, out, out_scale: float = 1.0, raw=None,
                   some=None, turn=None) -> torch.Tensor:
    """`window_attn` for runs of prompt rows on the tensor cores (tcgen05); `qk_norm_append` comes before it.  raw: fp32 [rows, hq, DV]
    takes the outputs instead of `out` (two maps: required).  some: (int32 first rows, int32 lengths, lengths on the host) of the runs
    to take, else all of them.  turn: as `qk_norm_append` filled it, where values are rotated."""
    assert g.conv_w is None and (g.vfreq is None or turn is not None)
    assert cache.k.dtype == proj.dtype == torch.bfloat16 and (raw is not None or out.dtype == torch.bfloat16)
    start, lens_dev, lens = (runs.start, None, runs.lens) if some is None else some
    call("dgpp_window_attn_tc", ptr(proj), proj.stride(0), g.q_off, ptr(cache.k), ptr(cache.v), ptr(block_table), ptr(row_req),
         ptr(positions), ptr(start), ptr(lens_dev), ptr(out), out.stride(0), ptr(raw), len(lens), window_tiles(g, lens), g.hq, g.hkv, g.maps, g.D, g.DV,
         cache.page, block_table.shape[1], cache.k.shape[0], g.window, int(g.chunked), g.gate_off, float(g.scale), float(out_scale), ptr(g.sink),
         ptr(turn) if g.vfreq is not None else None, g.keep_first, float(g.softcap), stream_ptr())
    return out


# ---------------------------------------------------------------------------------------------- latent attention
_LATENT = [P, L, I, I, P, P, P, P, P, P]
_lib.declare("dgpp_latent_append", _LATENT + [I] * 12 + [F, I, P])
_lib.declare("dgpp_latent_absorb", _LATENT + [P, P, P] + [I] * 13 + [F, I, P])
_lib.declare("dgpp_latent_rows", [P] * 7 + [I] * 7 + [F, I, P])
_lib.declare("dgpp_latent_decode_tc", [P] * 9 + [I] * 8 + [F, P])
_lib.declare("dgpp_latent_up", [P, P, P, L, P, P, L, I, I, I, I, I, P])
_lib.declare("dgpp_latent_gather", [P, P, P, I, I, I, P])
_lib.declare("dgpp_latent_prefill_tc", [P, L, I, I, P, P, I, I, P, P, P, P, P, P, L, I, I, I, I, I, I, I, I, F, P])


def rotation_freqs(base: float, dims: int, device) -> torch.Tensor:
    """[2, dims / 2] fp32: base^(-2 i / dims) as a leading and a residual term."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    hi = f.to(torch.float32)
    return torch.stack([hi, (f - hi.double()).to(torch.float32)]).contiguous().to(device)


class LatentHeads:
    """Static description of one latent-attention block inside a fused projection row: queries [heads, DN | RP] from q_off, the
    latent [KC | RP] from kv_off, one output gate per head from g_off.  w_up [heads * DN + heads * DV, KC]: key rows, then value
    rows, of every head."""

    def __init__(self, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, window: int, scale: float, eps: float, base: float, rot: int,
                 q_off: int, kv_off: int, g_off: int, norm_w: torch.Tensor, w_up: torch.Tensor):
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank = heads, dim, rot_dim, vdim, rank
        self.window, self.scale, self.eps, self.rot = window, scale, eps, rot
        self.DN, self.DV, self.KC, self.RP = latent_widths(dim, rot_dim, vdim, rank)
        self.q_off, self.kv_off, self.g_off, self.norm_w, self.w_up = q_off, kv_off, g_off, norm_w, w_up
        self.freq = rotation_freqs(base, rot, norm_w.device)

    @property
    def cache_cols(self) -> int:
        return self.KC + self.RP

    @property
    def flat_cols(self) -> int:
        return self.heads * (self.DN + self.DV)

    def tc_rows(self, dtype) -> bool:
        """Single rows run on the tensor cores."""
        return dtype == torch.bfloat16 and self.KC % 128 == 0 and self.KC <= 512 and self.RP == 64

    def tc_runs(self, dtype) -> bool:
        """Prompt runs run on the tensor cores, over keys and values expanded from the latents."""
        return dtype == torch.bfloat16 and self.DN + self.RP <= 256 and self.DV <= 256

    def _args(self, proj, positions, row_req, block_table, cache):
        assert cache.dtype == proj.dtype == self.w_up.dtype and cache.shape[-1] == self.cache_cols
        return (ptr(proj), proj.stride(0), self.q_off, self.kv_off, ptr(self.norm_w), ptr(self.freq), ptr(positions), ptr(row_req), ptr(block_table),
                ptr(cache))

    def _sizes(self, page: int, block_table):
        return (self.heads, self.DN, self.DV, self.dim, self.rank, self.KC, self.RP, self.rot_dim, self.rot, page, block_table.shape[1])


def latent_widths(dim: int, rot_dim: int, vdim: int, rank: int):
    """Padded widths (unrotated key part, value, latent, rotated part)."""
    up = lambda n, m: (n + m - 1) // m * m
    return up(dim, 64), up(vdim, 64), up(rank, 128) if rank <= 512 else up(rank, 64), max(64, up(rot_dim, 64))


def latent_append(g: LatentHeads, proj, positions, row_req, block_table, cache, page: int) -> None:
    """Appends the rows' latents and rotated key parts to the cache and rotates their queries in place."""
    call("dgpp_latent_append", *g._args(proj, positions, row_req, block_table, cache), proj.shape[0], *g._sizes(page, block_table), float(g.eps),
         _f32(proj), stream_ptr())


def latent_absorb(g: LatentHeads, proj, positions, row_req, block_table, cache, page: int, q_abs, rows: int, row_list=None, fused: bool = False):
    """q_abs [rows, heads, KC + RP] fp32 of the rows (`row_list`: of these pass rows).  fused: the rows are new tokens; their queries are
    rotated here and their latents appended."""
    assert q_abs.dtype == torch.float32 and q_abs.numel() >= rows * g.heads * g.cache_cols
    call("dgpp_latent_absorb", *g._args(proj, positions, row_req, block_table, cache), ptr(row_list), ptr(g.w_up), ptr(q_abs), rows,
         *g._sizes(page, block_table), int(fused), float(g.eps), _f32(proj), stream_ptr())
    return q_abs


def latent_splits(rows: int, heads: int, span: int, most: int, sms: int = 148) -> int:
    """Window splits of single rows: the fewest that finish soonest, counting 128-token tiles one after the other per CTA, one CTA
    per SM at a time, and a tile's time for the merge of the splits."""
    tiles, units = -(-(span + 127) // 128), rows * -(-heads // 16)
    cost = lambda s: -(-units * s // sms) * -(-tiles // s) + (s > 1)
    return min(range(1, max(1, min(most, tiles)) + 1), key=cost)


def latent_attn(g: LatentHeads, q_abs, cache, block_table, row_req, positions, page: int, lat, rows: int, row_list=None, splits: int = 1,
                scratch=None) -> torch.Tensor:
    """Windowed attention of absorbed rows -> lat [rows, heads, KC] fp32; on the tensor cores where the kernel takes the widths."""
    if g.tc_rows(cache.dtype):
        ml, acc = scratch if splits > 1 else (None, None)
        call("dgpp_latent_decode_tc", ptr(q_abs), ptr(cache), ptr(block_table), ptr(row_req), ptr(positions), ptr(row_list), ptr(ml), ptr(acc),
             ptr(lat), rows, g.heads, g.KC, page, block_table.shape[1], cache.shape[0], splits, g.window, float(g.scale), stream_ptr())
    else:
        call("dgpp_latent_rows", ptr(q_abs), ptr(cache), ptr(block_table), ptr(row_req), ptr(positions), ptr(row_list), ptr(lat), rows, g.heads,
             g.KC, g.RP, page, block_table.shape[1], g.window, float(g.scale), _f32(cache), stream_ptr())
    return lat


def latent_up(g: LatentHeads, lat, proj, out, rows: int, row_list=None) -> torch.Tensor:
    """out[row, h * DV + v] = (W_uv lat)[v] * sigmoid(gate of head h)."""
    w = g.w_up[g.heads * g.DN:]
    gate = proj[:, g.g_off:]
    call("dgpp_latent_up", ptr(lat), ptr(w), ptr(gate), proj.stride(0), ptr(row_list), ptr(out), out.stride(0), rows, g.heads, g.DV, g.KC,
         _f32(out), stream_ptr())
    return out


def latent_gather(cache, pages, out, page: int) -> torch.Tensor:
    """out [n * page, cols] bf16 = the cache's pages pages[0 .. n - 1]."""
    assert cache.dtype == torch.bfloat16 and out.is_contiguous()
    call("dgpp_latent_gather", ptr(cache), ptr(pages), ptr(out), pages.numel(), page, cache.shape[-1], stream_ptr())
    return out


class LatentRuns:
    """The longer runs of a pass for ``latent_prefill`` with one window: int32 device arrays first row, length, flat row of position 0
    per run; physical ids of the pages to expand; 128-row tiles."""

    def __init__(self, start, lens, base, pages, tiles: int):
        self.start, self.lens, self.base, self.pages, self.tiles = start, lens, base, pages, tiles


def latent_prefill(g: LatentHeads, proj, flat, gathered, row_req, positions, runs: LatentRuns, out) -> torch.Tensor:
    """Windowed attention of prompt runs over expanded keys and values (flat [n, flat_cols], gathered [n, KC + RP]), gate included.
    `latent_append` comes before it."""
    assert proj.dtype == flat.dtype == gathered.dtype == out.dtype == torch.bfloat16 and flat.is_contiguous() and gathered.is_contiguous()
    call("dgpp_latent_prefill_tc", ptr(proj), proj.stride(0), g.q_off, g.g_off, ptr(flat), ptr(gathered), gathered.shape[1], g.KC, ptr(row_req),
         ptr(positions), ptr(runs.start), ptr(runs.lens), ptr(runs.base), ptr(out), out.stride(0), runs.lens.numel(), runs.tiles, flat.shape[0],
         g.heads, g.DN, g.RP, g.DV, g.window, float(g.scale), stream_ptr())
    return out
