"""The tensor-core kernel for attention whose heads exchange their scores before
the softmax (``attention_talk_mma.cu``), one compiled module per (query heads,
key/value heads, key size, value size), built when a model first needs it.

``run`` returns False when the sizes have no variant (bfloat16; key and value
sizes multiples of 16, at most 256; all heads of eight queries and one tile of keys
in an SM's shared memory) or ``rt.options["attention"] == "plain"``; the caller
then takes the plain 32-bit kernel (``core.attention_talk``).

A CTA takes eight rows of an entry with all heads, or - when no entry has more
rows than fill eight (row, head) columns of a key/value head, decoded tokens - those.
A step of few rows would leave SMs idle: ``choose_splits`` then cuts the keys in slices over several CTAs.
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

_c_int, _c_void_p, _c_ll = ctypes.c_int, ctypes.c_void_p, ctypes.c_longlong
_libs: Dict[Tuple[int, int, int, int], ctypes.CDLL] = {}

PLAIN_SMEM = 220 * 1024  # what the plain kernel may hold of a row, in bytes
SMEM_MAX = 227 * 1024
SM_COUNT_FALLBACK = 148
MAX_SPLITS = 64


def plain_floats(heads: int, dim: int, vdim: int) -> int:
    """Floats of shared memory the plain kernel needs for a row."""
    return heads * (dim + vdim) + heads * 2 * 33 + 3 * heads


def queries_of_few(heads: int, kv_heads: int) -> int:
    """Queries of a CTA in the variant for few rows: as many as fill eight columns of a key/value head."""
    return max(1, 8 // (heads // kv_heads))


def layout(heads: int, kv_heads: int, dim: int, vdim: int, queries: int) -> Tuple[int, int, int, bool]:
    """(keys of a tile, blocks of the values, bytes of shared memory, whether it can run) of the kernel
    for these sizes with this many queries a CTA; restates ``Cfg`` in ``attention_talk_mma.cu``."""
    per_kv = heads // kv_heads
    units_of_kv = -(-queries * per_kv // 8)
    units = kv_heads * units_of_kv
    warps = 16 if units >= 16 and queries == 8 else (8 if units >= 8 else 4)
    mine = -(-units // warps)
    most = 256 if warps == 16 else 512
    padded = -(-heads // 16) * 16
    block = next((e for e in range(vdim, 15, -16) if vdim % e == 0 and mine * e <= most), 16)

    def smem(bn: int, stages: int = 1) -> int:
        region = -(-(3 * bn * (padded + 8) * 2 + heads * (bn + 8) * 4) // 128) * 128 + 32
        total = units * 8 * (dim + 8) * 2 + kv_heads * bn * (stages * (dim + 8) + (block + 8)) * 2 + queries * region \
            + padded * (padded + 8) * 2 + 3 * bn * 4
        return max(total, warps * 8 * (block + 8) * 2)

    bn = 32 if smem(32) <= SMEM_MAX else 16
    if queries != 8 or queries_of_few(heads, kv_heads) == 8:
        # few rows: as many keys as leave room for a second CTA on the SM, if any do
        half = SMEM_MAX // 2 - 1024
        bn = 32 if smem(32) <= half else (16 if smem(16) <= half else bn)
    stages = 2 if queries == 8 and smem(bn, 2) <= SMEM_MAX else 1
    total = smem(bn, stages)
    return bn, vdim // block, total, total <= SMEM_MAX and mine * block <= most


def supported(heads: int, kv_heads: int, dim: int, vdim: int) -> bool:
    if dim % 16 or vdim % 16 or not 16 <= dim <= 256 or not 16 <= vdim <= 256 or heads % kv_heads or heads > 96:
        return False
    return all(layout(heads, kv_heads, dim, vdim, n)[3] for n in (8, queries_of_few(heads, kv_heads)))


def lib_for(heads: int, kv_heads: int, dim: int, vdim: int) -> ctypes.CDLL:
    key = (heads, kv_heads, dim, vdim)
    lib = _libs.get(key)
    if lib is None:
        lib = load_module(f"attn_talk_h{heads}_g{kv_heads}_d{dim}_e{vdim}", ["attention_talk_mma.cu"],
                          [f"-DTALK_H={heads}", f"-DTALK_G={kv_heads}", f"-DTALK_D={dim}", f"-DTALK_E={vdim}"])
        lib.ib_attention_talk_mma.argtypes = [
            _c_void_p, _c_int, _c_void_p, _c_void_p, _c_void_p, _c_int, _c_void_p, _c_void_p, _c_int, _c_void_p, _c_void_p,
            _c_void_p, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_void_p,
            _c_int, _c_int, _c_int, _c_int, _c_void_p, _c_ll, _c_void_p]
        lib.ib_attention_talk_mma.restype = _c_int
        lib.ib_attention_talk_mma_scratch_bytes.argtypes = [_c_int, _c_int]
        lib.ib_attention_talk_mma_scratch_bytes.restype = _c_ll
        lib.ib_attention_talk_mma_info.argtypes = [_c_int, _c_int]
        lib.ib_attention_talk_mma_info.restype = _c_int
        for few, queries in ((0, 8), (1, queries_of_few(heads, kv_heads))):
            built = [lib.ib_attention_talk_mma_info(i, few) for i in range(9)]
            if built != [*key, queries, *(int(v) for v in layout(*key, queries))]:
                raise KernelError(f"the module for heads and sizes {key} was built as {built}")
        _libs[key] = lib
    return lib


def key_span(max_kv_len: int, max_rows: int, chunk: int, window: int, bn: int, queries: int = 8) -> int:
    """The most keys between the first that a row tile reads, rounded down to a key tile, and its last row."""
    span, behind = max_kv_len, min(max_rows, queries) - 1
    if chunk > 0:
        span = min(span, chunk + behind)
    if window > 0:
        span = min(span, window + behind)
    return span + bn - 1


def choose_splits(max_rows: int, n_entries: int, blocks: int, span: int, bn: int, slots: int,
                  queries: int = 8) -> Tuple[int, int]:
    """(slices of the keys, keys per slice): as many slices as the SMs' ``slots`` for CTAs hold at once,
    each of at least 32 keys; one when the row tiles alone fill more than half of the slots."""
    ctas = max(1, -(-max_rows // queries) * n_entries * blocks)
    want = min(slots // ctas, span // 32, MAX_SPLITS, 65535 // blocks)
    if want < 2:
        return 1, 0
    slice_len = -(-(-(-span // want)) // bn) * bn
    return -(-span // slice_len), slice_len


def run(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, out: torch.Tensor, ctx, tables: torch.Tensor,
        n_heads: int, talk, gate, chunk: int, window: int, rt) -> bool:
    """Arguments as ``core.attention_talk``; entries and their rows come from ``ctx.cu_rows`` and
    ``ctx.positions`` (an entry's rows are consecutive positions)."""
    num_pages, nkv, page_size, dim = k_pool.shape
    vdim = v_pool.shape[3]
    if q.dtype != torch.bfloat16 or rt.options.get("attention", "auto") == "plain" \
            or not supported(n_heads, nkv, dim, vdim) or q.stride(0) % 8 or out.stride(0) % 8 \
            or q.data_ptr() % 16 or out.data_ptr() % 16:
        return False
    core.require_cuda(q, k_pool, v_pool, out, talk, gate, tables)
    core.check_talk_arguments(q, k_pool, v_pool, out, tables, n_heads, talk, gate)
    lib = lib_for(n_heads, nkv, dim, vdim)
    key = ("talk_plan", n_heads, nkv, dim, vdim, chunk, window)
    plan = ctx.scratch.get(key) if hasattr(ctx, "scratch") else None
    if plan is None:
        # entries whose (row, head) pairs fill no more than eight columns of a key/value head
        few = int(ctx.max_rows_per_entry <= queries_of_few(n_heads, nkv))
        if rt.options.get("talk_few") is not None:
            few = int(rt.options["talk_few"])
        queries = queries_of_few(n_heads, nkv) if few else 8
        bn, blocks, smem, _ = layout(n_heads, nkv, dim, vdim, queries)
        sms = rt.options.get("sm_count") or SM_COUNT_FALLBACK
        forced = rt.options.get("talk_splits")
        span = key_span(ctx.max_kv_len, ctx.max_rows_per_entry, chunk, window, bn, queries)
        if forced:
            slice_len = -(-math.ceil(span / forced) // bn) * bn
            plan = (-(-span // slice_len), slice_len, few)
        else:
            plan = (*choose_splits(ctx.max_rows_per_entry, ctx.n_entries, blocks, span, bn,
                                   sms * (2 if 2 * (smem + 1024) <= SMEM_MAX else 1), queries), few)
        if hasattr(ctx, "scratch"):
            ctx.scratch[key] = plan
    splits, slice_len, few = plan
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
        core._ptr(talk), core._ptr(gate), gate.stride(0) if gate is not None else 0,
        ctx.cu_rows.data_ptr(), ctx.positions.data_ptr(), tables.data_ptr(), tables.shape[1], ctx.n_entries,
        ctx.max_rows_per_entry, page_size, num_pages, int(chunk), int(window), rt.err.data_ptr(), N, few,
        splits, slice_len, scratch_ptr, scratch_bytes, core.stream_ptr(q))
    core.check(code, "attention_talk_mma")
    return True
