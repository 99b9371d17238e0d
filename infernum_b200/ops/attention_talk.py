"""The tensor-core kernel for attention whose heads exchange their scores."""

from __future__ import annotations

import torch

PLAIN_SMEM = 220 * 1024  # what the plain kernel may hold of a row, in bytes


def plain_floats(heads: int, dim: int, vdim: int) -> int:
    """Floats of shared memory the plain kernel needs for a row."""
    return heads * (dim + vdim) + heads * 2 * 33 + 3 * heads


def run(q, k_pool, v_pool, out, ctx, tables, n_heads, scale, talk, temp, gate, chunk, window, rt) -> bool:
    return False
