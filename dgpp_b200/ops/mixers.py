"""Front ends of the kernels behind models with an fp32 residual stream, sliding-window attention without rotation and
fp32 linear-attention states (``csrc/kernels/stream_ops.cu``, ``window_attn.cu``, ``window_attn_tc.cu``,
``linear_state.cu``).  Every operator exists for bf16 and for true fp32 activations; the dtype of the tensors decides."""
from __future__ import annotations

from typing import Optional

import torch

from . import _lib
from ._lib import F, I, L, P, call, ptr, stream_ptr

_lib.declare("dgpp_embed_rows", [P, P, P, I, I, I, I, P])
_lib.declare("dgpp_resid_norm", [P, P, P, P, I, I, I, F, I, P])
_lib.declare("dgpp_gated_group_norm", [P, P, L, P, P, L, I, I, I, I, F, F, I, I, P])
_lib.declare("dgpp_geglu", [P, P, I, I, I, P])
_lib.declare("dgpp_qk_norm_append", [P, L, I, I, I, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, P])
_lib.declare("dgpp_window_attn", [P, L, I, I, I, P, P, P, P, P, P, P, P, P, P, P, L, I, I, I, I, I, I, I, I, I, I, I, F, F, F, I, P])
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


def embed_rows(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """fp32 rows out[r] = table[ids[r]] (table [vocab, cols] bf16 or fp32)."""
    call("dgpp_embed_rows", ptr(ids), ptr(table), ptr(out), ids.numel(), table.shape[1], table.shape[0], _f32(table), stream_ptr())
    return out


def resid_norm(x: torch.Tensor, w: torch.Tensor, n: int, eps: float, out: torch.Tensor,
               delta: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [rows, cols] fp32 takes in `delta` (fp32) in place; out = rms norm of the sum over its n true columns, times w."""
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous()
    call("dgpp_resid_norm", ptr(x), ptr(delta), ptr(w), ptr(out), x.shape[0], x.shape[1], n, float(eps), _f32(out), stream_ptr())
    return out


def gated_group_norm(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, out: torch.Tensor, groups: int, n: int, eps: float,
                     scale: float = 1.0) -> torch.Tensor:
    """o [rows, groups * gp] fp32 -> rms norm per group (n true columns) * w [gp] * sigmoid(gate) * scale."""
    assert o.dtype == torch.float32 and o.is_contiguous() and o.shape[1] % groups == 0
    call("dgpp_gated_group_norm", ptr(o), ptr(gate), gate.stride(0), ptr(w), ptr(out), out.stride(0), o.shape[0], groups,
         o.shape[1] // groups, n, float(eps), float(scale), _f32(out), _f32(gate), stream_ptr())
    return out


def geglu(gate_up: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """gate_up [rows, 2 I] -> gelu_tanh(gate) * up [rows, I]."""
    assert gate_up.is_contiguous() and out.is_contiguous()
    call("dgpp_geglu", ptr(gate_up), ptr(out), gate_up.shape[0], out.shape[1], _f32(out), stream_ptr())
    return out


class WindowHeads:
    """Static description of one window-attention block inside a fused projection row."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, window: int, scale: float, eps: float,
                 q_off: int, k_off: int, v_off: int):
        self.hq, self.hkv, self.dim, self.window, self.scale, self.eps = heads, kv_heads, dim, window, scale, eps
        self.D, self.DV = pad_to(dim, ATTN_WIDTHS), pad_to(vdim, ATTN_WIDTHS)
        self.q_off, self.k_off, self.v_off = q_off, k_off, v_off


def _wa_common(g: WindowHeads, proj, wq, wk, cache, block_table, row_req, positions):
    return (ptr(proj), proj.stride(0), g.q_off, g.k_off, g.v_off, ptr(wq), ptr(wk), ptr(cache.k), ptr(cache.v),
            ptr(block_table), ptr(row_req), ptr(positions))


def qk_norm_append(g: WindowHeads, proj, wq, wk, cache, block_table, row_req, positions) -> None:
    """Norms the query heads of `proj` in place and appends normed keys and values to the paged cache."""
    assert cache.k.dtype == proj.dtype
    call("dgpp_qk_norm_append", *_wa_common(g, proj, wq, wk, cache, block_table, row_req, positions), proj.shape[0], g.hq, g.hkv,
         g.D, g.DV, g.dim, cache.page, block_table.shape[1], float(g.eps), _f32(proj), stream_ptr())


def window_attn(g: WindowHeads, proj, wq, wk, cache, block_table, row_req, positions, out, out_scale: float = 1.0,
                fused: bool = False, splits: int = 1, scratch=None, row_list=None) -> torch.Tensor:
    """Every row attends to the last `window` positions of its request, its own included -> out [rows, >= hq * DV].
    fused: the rows are single new tokens; the kernel norms and appends them itself.  row_list: int32 subset of rows."""
    assert cache.k.dtype == proj.dtype and out.dtype == proj.dtype
    ml, acc = scratch if splits > 1 else (None, None)
    rows = proj.shape[0] if row_list is None else row_list.numel()
    call("dgpp_window_attn", *_wa_common(g, proj, wq, wk, cache, block_table, row_req, positions), ptr(row_list), ptr(ml), ptr(acc),
         ptr(out), out.stride(0), rows, g.hq, g.hkv, g.D, g.DV, g.dim, cache.page, block_table.shape[1], splits, g.window,
         int(fused), float(g.scale), float(g.eps), float(out_scale), _f32(proj), stream_ptr())
    return out


class StateHeads:
    """Static description of one linear-attention block: widths (padded), offsets inside the fused projection row, and the
    constants of its rule (`decay` per head: lightning; `A_log` / `dt_bias` / low-rank rows: channel delta rule)."""

    def __init__(self, heads: int, key_heads: int, dim: int, vdim: int, c_off: int, b_off: int = 0, eps: float = 0.0,
                 conv_w=None, A_log=None, dt_bias=None, decay=None, norm_w=None):
        self.hv, self.hk, self.dim, self.vdim = heads, key_heads, dim, vdim
        self.DK, self.DV = pad_to(dim, STATE_WIDTHS), pad_to(vdim, STATE_WIDTHS)
        self.c_off, self.b_off, self.eps = c_off, b_off, eps
        self.conv_w, self.A_log, self.dt_bias, self.decay, self.norm_w = conv_w, A_log, dt_bias, decay, norm_w
        self.delta = decay is None
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
        return rows * (self.channels + self.hv * (3 * self.DK + 1)) + blocks * self.hv * (self.DK + 512)


def linear_state(g: StateHeads, proj, state, ring, row_slot, positions, low=None, runs=None, prep=None, o=None, out=None) -> None:
    """Advances the states by the rows of `proj`.  runs None: one new token per row; the delta rule then writes its normed and
    gated read-outs to `out`, lightning its raw read-outs to `o` (fp32).  runs given: runs of consecutive rows, raw read-outs
    to `o`, `prep` is fp32 scratch (`StateHeads.prep_floats`)."""
    rows = proj.shape[0]
    blocks = 0 if runs is None else sum(-(-n // 16) for n in runs.lens)
    assert state.dtype == torch.float32 and (runs is None or prep.numel() >= g.prep_floats(rows, len(runs.lens)))
    call("dgpp_linear_state", ptr(proj), proj.stride(0), g.c_off, g.b_off, ptr(low), 0 if low is None else low.stride(0),
         ptr(g.conv_w), ptr(ring), g.taps, ptr(g.A_log), ptr(g.dt_bias), ptr(g.decay), ptr(state), ptr(row_slot), ptr(positions),
         None if runs is None else ptr(runs.start), None if runs is None else ptr(runs.row_run0), ptr(prep), ptr(o), ptr(out),
         0 if out is None else out.stride(0), ptr(g.norm_w), rows, rows if runs is None else len(runs.lens), blocks, g.hk, g.hv, g.DK, g.DV,
         g.vdim, float(g.dim ** -0.5), float(g.eps), int(g.delta), int(runs is None), _f32(proj), stream_ptr())


_lib.declare("dgpp_window_attn_tc", [P, L, I, P, P, P, P, P, P, P, L, I, I, I, I, I, I, I, I, I, I, F, F, P])


def window_prefill_usable(g: WindowHeads, proj, page: int = 64) -> bool:
    """Whether the tensor-core kernel takes these rows (bf16, pages of 64 tokens, at most 128 query heads per key head)."""
    return proj.dtype == torch.bfloat16 and page == 64 and g.hq // g.hkv <= 128


def window_prefill(g: WindowHeads, proj, cache, block_table, row_req, positions, runs, out, out_scale: float = 1.0) -> torch.Tensor:
    """`window_attn` for runs of prompt rows on the tensor cores (tcgen05); `qk_norm_append` comes before it."""
    assert cache.k.dtype == proj.dtype == out.dtype == torch.bfloat16
    per = 128 // (g.hq // g.hkv)
    tiles = sum(-(-n // per) for n in runs.lens)
    call("dgpp_window_attn_tc", ptr(proj), proj.stride(0), g.q_off, ptr(cache.k), ptr(cache.v), ptr(block_table), ptr(row_req),
         ptr(positions), ptr(runs.start), ptr(out), out.stride(0), len(runs.lens), tiles, g.hq, g.hkv, g.D, g.DV, cache.page,
         block_table.shape[1], cache.k.shape[0], g.window, float(g.scale), float(out_scale), stream_ptr())
    return out
