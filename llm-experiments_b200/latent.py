"""Latent attention: the operations on a cache that keeps one latent row and one rotated key part per token.

A latent layer's ``KVCache`` has one head: ``k_cache`` rows are the rotated key part all heads share (``head_dim`` = its
width), ``v_cache`` rows the latent (``v_head_dim`` = its width), from which every head makes its own unrotated keys and its
values.  Several layers may read one such cache, each with matrices of its own.

Two forms of the attention, chosen by the caller:

* single query rows (decoding, short portions) stay in the latent space: the head's unrotated query is carried through its
  key matrix (a per-head ``linear``), ``latent_decode`` attends over the cached rows once for all heads, and the head's value
  matrix is applied to the result (another per-head ``linear``);
* prompt portions expand the visible rows into per-head keys and values with one matrix product and run ``latent_prefill``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _native
from .batch import batch_op_begin, dev_status_ptr, reference_op
from .kv_cache import dtype_code
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext, KVCache


@dataclass
class RowPlaces:
    """Where the rows of a step belong: sequence (``None``: row i is sequence i) and position, int32 on the device."""

    slot: Optional[torch.Tensor]
    pos: torch.Tensor

    def slot_ptr(self):
        return None if self.slot is None else self.slot.data_ptr()


@dataclass
class LatentShape:
    """Sizes and constants of one latent attention layer."""

    heads: int
    dim: int       # unrotated query / key elements per head
    rot: int       # rotated ones
    rot_dims: int  # how many of them are turned (the rest pass)
    vdim: int
    kv_rank: int
    window: int    # visible tokens, the row's own included; 0 = all earlier ones
    scale: float


def _latent_cache(cache: KVCache, shape: LatentShape):
    if (cache.head_dim, cache.v_head_dim or cache.head_dim, cache.n_heads) != (shape.rot, shape.kv_rank, 1):
        raise ValueError("the cache does not hold latent rows of this layer's sizes")
    layer = cache.layers[0]
    return layer.k_cache.buffer.data_ptr(), layer.v_cache.buffer.data_ptr()


@reference_op("latent_append")
def latent_append(ctx: GPUContext, y: GPUBuffer2D, shape: LatentShape, inv_freq: GPUBuffer1D, places: RowPlaces,
                  cache: KVCache, norm_weight: Optional[GPUBuffer1D], eps: float) -> None:
    """Rotates the queries in ``y`` (``[rows, heads * (dim + rot) (+ kv_rank + rot)]``) in place and, with ``norm_weight``,
    writes every row's latent and rotated key part to its place in ``cache``.  Lengths are not advanced."""
    key, lat = _latent_cache(cache, shape)
    own = norm_weight is not None
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_latent_append(
        y.buffer.data_ptr(), y.buffer.stride(0), shape.heads, shape.dim, shape.rot, shape.rot_dims, inv_freq.buffer.data_ptr(),
        shape.heads * (shape.dim + shape.rot) if own else 0, shape.kv_rank, norm_weight.buffer.data_ptr() if own else None, eps,
        key if own else None, lat if own else None, places.slot_ptr(), places.pos.data_ptr(), cache.batch_size,
        cache.max_seq_len, y.shape[0], dtype_code(y.buffer.dtype), dev_status_ptr(ctx), stream))


@reference_op("latent_decode")
def latent_decode(ctx: GPUContext, q_latent: GPUBuffer2D, y: GPUBuffer2D, shape: LatentShape, places: RowPlaces,
                  cache: KVCache, out: GPUBuffer2D, span: int, path: int = 0) -> None:
    """Attention of single rows over the cached latent rows: ``q_latent`` and ``out`` are ``[rows, heads * kv_rank]``, ``y`` the
    rotated query rows.  ``span`` bounds the tokens any row sees.  ``path`` forces a kernel (1 CUDA cores, 2 tensor cores)."""
    key, lat = _latent_cache(cache, shape)
    rows, dt = q_latent.shape[0], dtype_code(q_latent.buffer.dtype)
    span = min(span, shape.window) if shape.window > 0 else span
    nbytes = _native.lib.b2kv_latent_decode_workspace_bytes(rows, shape.heads, shape.kv_rank, span, dt) if path != 1 else 0
    if nbytes and (cache.workspace is None or cache.workspace.numel() < nbytes):
        cache.workspace = torch.empty(nbytes, dtype=torch.uint8, device=ctx.device)
    ws = cache.workspace if nbytes else None
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_latent_decode(
        q_latent.buffer.data_ptr(), y.buffer.data_ptr(), y.buffer.stride(0), shape.dim, key, lat, out.buffer.data_ptr(),
        places.slot_ptr(), places.pos.data_ptr(), cache.batch_size, cache.max_seq_len, rows, shape.heads, shape.kv_rank,
        shape.rot, shape.window, span, shape.scale, dt, path, None if ws is None else ws.data_ptr(),
        0 if ws is None else ws.numel(), dev_status_ptr(ctx), stream))


@dataclass
class PromptPlan:
    """Prompt portions of one step for layers with one window: per portion its rows of the step, the visible part of its
    sequence's cache and where that part is expanded to, and the device table ``latent_prefill`` reads."""

    portions: list          # (row0, n, first cache row, visible rows, first expanded row)
    table: Optional[torch.Tensor]  # int32 [portions, 6] on the device
    n_blocks: int
    kv_rows: int

    BLOCK = 256  # query rows of one block of the kernel

    @staticmethod
    def build(spans, window: int, max_seq_len: int, in_place: bool = False) -> "PromptPlan":
        """``spans``: (row0, n, sequence, start position); the table is filled in by ``rows()`` + an upload.  ``in_place``: keys
        and values are read from the cache itself, nothing is expanded."""
        portions, at, blocks = [], 0, 0
        for row0, n, slot, start in spans:
            lo = max(0, start - window + 1) if window > 0 else 0
            portions.append((row0, n, slot * max_seq_len + lo, start + n - lo, slot * max_seq_len + lo if in_place else at))
            at += start + n - lo
            blocks += (n + PromptPlan.BLOCK - 1) // PromptPlan.BLOCK
        return PromptPlan(portions=portions, table=None, n_blocks=blocks, kv_rows=at)

    def rows(self) -> list:
        """The table as a flat list of integers (``b2kv_prompt_segment``)."""
        out, first = [], 0
        for row0, n, cache_row, visible, kv_row in self.portions:
            out += [row0, n, kv_row, cache_row, visible - n, first]
            first += (n + PromptPlan.BLOCK - 1) // PromptPlan.BLOCK
        return out


def prefill_supported(shape: LatentShape, dtype: torch.dtype) -> bool:
    return shape.scale > 0 and bool(_native.lib.b2kv_latent_prefill_supported(shape.dim, shape.rot, shape.vdim, shape.kv_rank,
                                                                             dtype_code(dtype)))


@reference_op("latent_prefill")
def latent_prefill(ctx: GPUContext, y: GPUBuffer2D, keys: GPUBuffer2D, values: GPUBuffer2D, shape: LatentShape,
                   plan: PromptPlan, cache: KVCache, out: GPUBuffer2D) -> None:
    """Attention of prompt portions: ``y`` and ``out`` are the step's rows, ``keys`` ``[kv_rows, heads * dim]`` and ``values``
    ``[kv_rows, heads * vdim]`` (views of one buffer) the expanded visible rows of the plan's portions."""
    key, _ = _latent_cache(cache, shape)
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_latent_prefill(
        y.buffer.data_ptr(), y.buffer.stride(0), keys.buffer.data_ptr(), values.buffer.data_ptr(), keys.buffer.stride(0), key,
        cache.batch_size * cache.max_seq_len, out.buffer.data_ptr(), out.buffer.stride(0), plan.table.data_ptr(),
        len(plan.portions), plan.n_blocks, y.shape[0], plan.kv_rows, shape.heads, shape.dim, shape.rot, shape.vdim, shape.window,
        shape.scale, dtype_code(y.buffer.dtype), dev_status_ptr(ctx), stream))
