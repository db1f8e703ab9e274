"""Padding helpers for packed weights: head widths go up to what the kernels take, rows of matrices to multiples of 8 columns,
always with zeros, so padded columns stay exact zeros through a layer."""
from __future__ import annotations

import torch
import torch.nn.functional as F


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


def up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def pad_rows(w: torch.Tensor, groups: int, n: int, npad: int) -> torch.Tensor:
    """[groups * n, K] -> [groups * npad, K] with zero rows behind every group."""
    if n == npad:
        return w
    return F.pad(w.reshape(groups, n, -1), (0, 0, 0, npad - n)).reshape(groups * npad, -1)


def pad_cols(w: torch.Tensor, groups: int, n: int, npad: int) -> torch.Tensor:
    return pad_rows(w.T, groups, n, npad).T


def pad_vec(v: torch.Tensor, groups: int, n: int, npad: int) -> torch.Tensor:
    return pad_rows(v.reshape(-1, 1), groups, n, npad).reshape(-1)


def only_keys(d: dict, keys, what: str, optional=()) -> None:
    """A configuration section has exactly these keys (and perhaps optional ones): an unknown one would be silently ignored."""
    if not set(keys) <= set(d) or not set(d) <= set(keys) | set(optional):
        raise ValueError(f"{what}: expected the keys {sorted(keys)}, got {sorted(d)}")
