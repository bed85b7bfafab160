"""Grouped-query attention over per-layer caches, with normed queries and keys, a query temperature that grows with the position
and a linear distance bias per head.

A layer's ``KVCache`` has one K and one V row of all key / value heads per token (``[sequence * max_seq_len, kv_heads * dim]``,
V rows ``v_head_dim`` wide per head).  Several layers may read one such cache, each with queries of its own.  Single rows
(decoding, short portions) go to ``gqa_decode``, prompt portions to ``gqa_prefill``; both read the cache in place, after
``gqa_append`` has written the step's rows.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _native
from .batch import batch_op_begin, dev_status_ptr, reference_op
from .kv_cache import dtype_code
from .latent import PromptPlan, RowPlaces
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext, KVCache


@dataclass
class GqaShape:
    """Sizes and constants of one grouped-query attention layer."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 0  # tokens per step of the query temperature; 0: none


def geometric_slopes(heads: int) -> torch.Tensor:
    """Slopes of a distance bias that fall geometrically over the heads, down to 2^-8 at the last one."""
    return torch.exp2(-8.0 * torch.arange(1, heads + 1, dtype=torch.float64) / heads).float()


def _caches(cache: KVCache, s: GqaShape):
    if (cache.head_dim, cache.v_head_dim or cache.head_dim, cache.n_heads) != (s.dim, s.vdim, s.kv_heads) or cache.layout != "bthd":
        raise ValueError("the cache does not hold keys and values of this layer's sizes")
    layer = cache.layers[0]
    return layer.k_cache.buffer.data_ptr(), layer.v_cache.buffer.data_ptr()


@reference_op("gqa_append")
def gqa_append(ctx: GPUContext, y: GPUBuffer2D, shape: GqaShape, places: RowPlaces, cache: KVCache, own: bool,
               q_norm: Optional[GPUBuffer1D], k_norm: Optional[GPUBuffer1D], eps: float) -> None:
    """Norms and scales the queries in ``y`` (``[rows, >= heads * dim (+ kv_heads * (dim + vdim))]``) in place and, with ``own``,
    writes every row's normed key and value to its place in ``cache``.  Lengths are not advanced."""
    k, v = _caches(cache, shape)
    ptr = lambda b: None if b is None else b.buffer.data_ptr()  # noqa: E731
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_gqa_append(
        y.buffer.data_ptr(), y.buffer.stride(0), shape.heads, shape.kv_heads, shape.dim, shape.vdim, ptr(q_norm), ptr(k_norm), eps,
        shape.temp_coef, shape.temp_every, k if own else None, v if own else None, places.slot_ptr(), places.pos.data_ptr(),
        cache.batch_size, cache.max_seq_len, y.shape[0], dtype_code(y.buffer.dtype), dev_status_ptr(ctx), stream))


@reference_op("gqa_decode")
def gqa_decode(ctx: GPUContext, q: GPUBuffer2D, shape: GqaShape, slopes: Optional[GPUBuffer1D], places: RowPlaces, cache: KVCache,
               out: GPUBuffer2D, span: int, path: int = 0) -> None:
    """Attention of single rows: ``q`` as ``gqa_append`` leaves it, ``out`` ``[rows, >= heads * vdim]``.  ``span`` bounds the tokens
    any row sees.  ``path`` forces a kernel (1 CUDA cores, 2 tensor cores)."""
    k, v = _caches(cache, shape)
    rows, dt = q.shape[0], dtype_code(q.buffer.dtype)
    nbytes = _native.lib.b2kv_gqa_decode_workspace_bytes(rows, shape.heads, shape.kv_heads, shape.vdim, span, dt) if path != 1 else 0
    if nbytes and (cache.workspace is None or cache.workspace.numel() < nbytes):
        cache.workspace = torch.empty(nbytes, dtype=torch.uint8, device=ctx.device)
    ws = cache.workspace if nbytes else None
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_gqa_decode(
        q.buffer.data_ptr(), q.buffer.stride(0), k, v, out.buffer.data_ptr(), out.buffer.stride(0),
        None if slopes is None else slopes.buffer.data_ptr(), places.slot_ptr(), places.pos.data_ptr(), cache.batch_size,
        cache.max_seq_len, rows, shape.heads, shape.kv_heads, shape.dim, shape.vdim, span, shape.scale, dt, path,
        None if ws is None else ws.data_ptr(), 0 if ws is None else ws.numel(), dev_status_ptr(ctx), stream))


def prefill_supported(shape: GqaShape, dtype: torch.dtype) -> bool:
    return shape.scale > 0 and bool(_native.lib.b2kv_gqa_prefill_supported(shape.dim, shape.vdim, dtype_code(dtype)))


@reference_op("gqa_prefill")
def gqa_prefill(ctx: GPUContext, q: GPUBuffer2D, shape: GqaShape, slopes: Optional[GPUBuffer1D], plan: PromptPlan, cache: KVCache,
                out: GPUBuffer2D) -> None:
    """Attention of prompt portions: ``q`` and ``out`` are the step's rows, ``plan`` was built ``in_place`` without a window."""
    k, v = _caches(cache, shape)
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_gqa_prefill(
        q.buffer.data_ptr(), q.buffer.stride(0), k, v, cache.batch_size * cache.max_seq_len, out.buffer.data_ptr(),
        out.buffer.stride(0), None if slopes is None else slopes.buffer.data_ptr(), plan.table.data_ptr(), len(plan.portions),
        plan.n_blocks, q.shape[0], shape.heads, shape.kv_heads, shape.dim, shape.vdim, shape.scale, dtype_code(q.buffer.dtype),
        dev_status_ptr(ctx), stream))
