"""Zero padding of weights to the sizes the kernels work in."""
from __future__ import annotations

from typing import Optional

import torch

HEAD_ALIGN = 16
ROW_ALIGN = 8


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


def pad_rows(w: torch.Tensor, rows: int, cols: Optional[int] = None) -> torch.Tensor:
    """w [r, c] with zero rows (and columns) added."""
    cols = w.shape[1] if cols is None else cols
    if tuple(w.shape) == (rows, cols):
        return w
    out = w.new_zeros(rows, cols)
    out[: w.shape[0], : w.shape[1]] = w
    return out


def pad_heads(w: torch.Tensor, heads: int, padded: int) -> torch.Tensor:
    """w [heads * size, c] with every head's rows padded to `padded`."""
    size = w.shape[0] // heads
    if size == padded:
        return w
    out = w.new_zeros(heads, padded, w.shape[1])
    out[:, :size] = w.view(heads, size, -1)
    return out.view(heads * padded, -1)


def pad_vector(w: torch.Tensor, n: int) -> torch.Tensor:
    return pad_rows(w.reshape(1, -1), 1, n).reshape(-1)
