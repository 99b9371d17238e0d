"""The tensor-core kernel for attention whose heads exchange their scores before
the softmax (``attention_talk_mma.cu``), one compiled module per (query heads,
key/value heads, key size, value size), built when a model first needs it.

``run`` returns False when the sizes have no variant (bfloat16; key and value
sizes multiples of 16, at most 256; all heads of eight queries and one tile of keys
in an SM's shared memory) or ``rt.options["attention"] == "plain"``; the caller
then takes the plain 32-bit kernel (``core.attention_talk``).

A CTA takes eight rows of an entry with all heads.  A step of few rows would
leave SMs idle: ``choose_splits`` then cuts the keys in slices over several CTAs.
The plan and the scratch buffer are worked out once per step and kept in
``ctx.scratch``.
"""

from __future__ import annotations

import ctypes
import math
from typing import Dict, Tuple

import torch

from ..csrc.build import load_module
from ..errors import KernelError
from . import core

_c_int, _c_float, _c_void_p, _c_ll = ctypes.c_int, ctypes.c_float, ctypes.c_void_p, ctypes.c_longlong
_libs: Dict[Tuple[int, int, int, int], ctypes.CDLL] = {}

PLAIN_SMEM = 220 * 1024  # what the plain kernel may hold of a row, in bytes
SMEM_MAX = 227 * 1024
SM_COUNT_FALLBACK = 148
ROW_TILE, MAX_SPLITS = 8, 64


def plain_floats(heads: int, dim: int, vdim: int) -> int:
    """Floats of shared memory the plain kernel needs for a row."""
    return heads * (dim + vdim) + heads * 2 * 33 + 3 * heads


def layout(heads: int, kv_heads: int, dim: int, vdim: int) -> Tuple[int, int, int]:
    """(keys of a tile, blocks of the values, bytes of shared memory) of the kernel compiled for
    these sizes; restates the constants at the head of ``attention_talk_mma.cu``."""
    warps = 8 if heads >= 8 else 4
    per_warp = -(-heads // warps)
    padded = -(-heads // 16) * 16
    block = next((e for e in range(vdim, 15, -16) if vdim % e == 0 and per_warp * e <= 512), 16)

    def smem(bn: int) -> int:
        plane, mix = bn * (padded + 8) * 2, heads * (bn + 8) * 4
        alias = bn // 8 * (padded // 16) * 6 <= 48
        region = (max(3 * plane, mix) if alias else 3 * plane + mix)
        region = -(-region // 128) * 128 + 32
        total = 8 * heads * (dim + 8) * 2 + kv_heads * bn * (dim + 8) * 2 + 2 * kv_heads * bn * (block + 8) * 2 \
            + 8 * region + padded * (padded + 8) * 2 + -(-heads // 4) * 16 + 3 * bn * 4
        return max(total, warps * 8 * (block + 8) * 2)

    bn = 32 if smem(32) <= SMEM_MAX else 16
    return bn, vdim // block, smem(bn)


def supported(heads: int, kv_heads: int, dim: int, vdim: int) -> bool:
    if dim % 16 or vdim % 16 or not 16 <= dim <= 256 or not 16 <= vdim <= 256 or heads % kv_heads:
        return False
    bn, blocks, smem = layout(heads, kv_heads, dim, vdim)
    per_warp = -(-heads // (8 if heads >= 8 else 4))
    # the exchange keeps a query's planes of one piece of heads after the other in registers
    return smem <= SMEM_MAX and per_warp * (vdim // blocks) <= 512 and heads <= 96


def lib_for(heads: int, kv_heads: int, dim: int, vdim: int) -> ctypes.CDLL:
    key = (heads, kv_heads, dim, vdim)
    lib = _libs.get(key)
    if lib is None:
        lib = load_module(f"attn_talk_h{heads}_g{kv_heads}_d{dim}_e{vdim}", ["attention_talk_mma.cu"],
                          [f"-DTALK_H={heads}", f"-DTALK_G={kv_heads}", f"-DTALK_D={dim}", f"-DTALK_E={vdim}"])
        lib.ib_attention_talk_mma.argtypes = [
            _c_void_p, _c_int, _c_void_p, _c_void_p, _c_void_p, _c_int, _c_void_p, _c_void_p, _c_void_p, _c_int,
            _c_void_p, _c_void_p, _c_void_p, _c_int, _c_int, _c_int, _c_int, _c_int, _c_float, _c_int, _c_int, _c_void_p,
            _c_int, _c_int, _c_int, _c_void_p, _c_ll, _c_void_p]
        lib.ib_attention_talk_mma.restype = _c_int
        lib.ib_attention_talk_mma_scratch_bytes.argtypes = [_c_int, _c_int]
        lib.ib_attention_talk_mma_scratch_bytes.restype = _c_ll
        lib.ib_attention_talk_mma_info.argtypes = [_c_int]
        lib.ib_attention_talk_mma_info.restype = _c_int
        built = tuple(lib.ib_attention_talk_mma_info(i) for i in range(8))
        bn, blocks, smem = layout(*key)
        if built != (*key, bn, blocks, 1, smem):
            raise KernelError(f"the module for heads and sizes {key} was built as {built}")
        _libs[key] = lib
    return lib


def key_span(max_kv_len: int, max_rows: int, chunk: int, window: int, bn: int) -> int:
    """The most keys between the first that a row tile reads, rounded down to a key tile, and its last row."""
    span, behind = max_kv_len, min(max_rows, ROW_TILE) - 1
    if chunk > 0:
        span = min(span, chunk + behind)
    if window > 0:
        span = min(span, window + behind)
    return span + bn - 1


def choose_splits(max_rows: int, n_entries: int, blocks: int, span: int, bn: int, slots: int) -> Tuple[int, int]:
    """(slices of the keys, keys per slice): one when the row tiles fill the SMs' ``slots`` for CTAs or there
    are few keys, else as many as fill them about twice, each of at least two tiles of keys."""
    ctas = max(1, -(-max_rows // ROW_TILE) * n_entries * blocks)
    want = min(-(-2 * slots // ctas), span // (2 * bn), MAX_SPLITS, 65535 // blocks)
    if ctas >= slots or want < 2:
        return 1, 0
    slice_len = -(-(-(-span // want)) // bn) * bn
    return -(-span // slice_len), slice_len


def run(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, out: torch.Tensor, ctx, tables: torch.Tensor,
        n_heads: int, scale: float, talk, temp, gate, chunk: int, window: int, rt) -> bool:
    """Arguments as ``core.attention_talk``; entries and their rows come from ``ctx.cu_rows`` and
    ``ctx.positions`` (an entry's rows are consecutive positions)."""
    num_pages, nkv, page_size, dim = k_pool.shape
    vdim = v_pool.shape[3]
    if q.dtype != torch.bfloat16 or rt.options.get("attention", "auto") == "plain" \
            or not supported(n_heads, nkv, dim, vdim) or q.stride(0) % 8 or out.stride(0) % 8 \
            or q.data_ptr() % 16 or out.data_ptr() % 16:
        return False
    core.require_cuda(q, k_pool, v_pool, out, talk, temp, gate, tables)
    core.check_talk_arguments(q, k_pool, v_pool, out, tables, n_heads, talk, temp, gate)
    lib = lib_for(n_heads, nkv, dim, vdim)
    key = ("talk_plan", n_heads, nkv, dim, vdim, chunk, window)
    plan = ctx.scratch.get(key) if hasattr(ctx, "scratch") else None
    if plan is None:
        bn, blocks, smem = layout(n_heads, nkv, dim, vdim)
        sms = rt.options.get("sm_count") or SM_COUNT_FALLBACK
        forced = rt.options.get("talk_splits")
        span = key_span(ctx.max_kv_len, ctx.max_rows_per_entry, chunk, window, bn)
        if forced:
            slice_len = -(-math.ceil(span / forced) // bn) * bn
            plan = (-(-span // slice_len), slice_len)
        else:
            plan = choose_splits(ctx.max_rows_per_entry, ctx.n_entries, blocks, span, bn,
                                 sms * max(1, min(2, SMEM_MAX // smem)))
        if hasattr(ctx, "scratch"):
            ctx.scratch[key] = plan
    splits, slice_len = plan
    N = q.shape[0]
    scratch_ptr, scratch_bytes = None, 0
    if splits > 1:
        need = lib.ib_attention_talk_mma_scratch_bytes(N, splits)
        buf = ctx.scratch.get("talk_split") if hasattr(ctx, "scratch") else None
        if buf is None or buf.numel() * 4 < need:
            buf = torch.empty((need + 3) // 4, dtype=torch.float32, device=q.device)
            if hasattr(ctx, "scratch"):
                ctx.scratch["talk_split"] = buf
        scratch_ptr, scratch_bytes = buf.data_ptr(), buf.numel() * 4
    code = lib.ib_attention_talk_mma(
        q.data_ptr(), q.stride(0), k_pool.data_ptr(), v_pool.data_ptr(), out.data_ptr(), out.stride(0),
        core._ptr(talk), core._ptr(temp), core._ptr(gate), gate.stride(0) if gate is not None else 0,
        ctx.cu_rows.data_ptr(), ctx.positions.data_ptr(), tables.data_ptr(), tables.shape[1], ctx.n_entries,
        ctx.max_rows_per_entry, page_size, num_pages, float(scale), int(chunk), int(window), rt.err.data_ptr(), N, splits,
        slice_len, scratch_ptr, scratch_bytes, core.stream_ptr(q))
    core.check(code, "attention_talk_mma")
    return True
