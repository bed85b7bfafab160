"""Recurrent layers: states that are carried from token to token instead of a cache of all tokens.

Gated linear attention keeps one matrix per sequence and head, ``[dim, vdim]`` in fp32, whose rows fade per key channel.  A
layer's states are one tensor ``[sequences, heads, dim, vdim]``; a run of rows that begins at position 0 starts from zero, so a
place that is given back needs no clearing.  Decoding and short portions take token after token; prompt portions take sixteen
tokens at a time on the tensor cores (bfloat16), with the state in registers.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Tuple

import torch

from . import _native
from .batch import batch_op_begin, dev_status_ptr, reference_op
from .kv_cache import dtype_code
from .serving import RowSegments
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext


@dataclass
class GlaShape:
    """Sizes and constants of one gated linear attention layer."""

    heads: int
    dim: int
    vdim: int
    tau: float  # the decay is the tau-th root of a sigmoid


def gla_state_create(ctx: GPUContext, shape: GlaShape, batch_size: int) -> torch.Tensor:
    return torch.zeros((batch_size, shape.heads, shape.dim, shape.vdim), dtype=torch.float32, device=ctx.device)


@reference_op("gated_linear_attention")
def gated_linear_attention(ctx: GPUContext, y: GPUBuffer2D, cols: Tuple[int, int, int, int], alpha: GPUBuffer2D, shape: GlaShape,
                           norm: GPUBuffer1D, eps: float, segments: RowSegments, pos: torch.Tensor, state: torch.Tensor,
                           out: GPUBuffer2D, path: int = 0) -> None:
    """The recurrence over the rows of ``segments``, with the heads' norm and gate behind it.  ``y`` holds queries, keys, values
    and gates from the columns ``cols`` on, ``alpha`` (fp32) the decays, ``pos`` every row's position.  ``path`` forces a
    kernel (1 token after token, 2 chunks on the tensor cores)."""
    if state.dtype != torch.float32 or tuple(state.shape[1:]) != (shape.heads, shape.dim, shape.vdim) or not state.is_contiguous():
        raise ValueError("the state does not have this layer's sizes")
    if alpha.buffer.dtype != torch.float32 or out.buffer.dtype != y.buffer.dtype or norm.buffer.dtype != torch.float32:
        raise ValueError("gated_linear_attention: alpha and norm are float32, out has the type of y")
    dt = dtype_code(y.buffer.dtype)
    nbytes = _native.lib.b2kv_gla_workspace_bytes(shape.heads, shape.dim, shape.vdim, segments.count, segments.max_n, dt, path)
    if nbytes and (ctx.recurrent_workspace is None or ctx.recurrent_workspace.numel() < nbytes):
        ctx.recurrent_workspace = torch.empty(nbytes, dtype=torch.uint8, device=ctx.device)
    a = _native.GlaArgs(
        y=y.buffer.data_ptr(), alpha=alpha.buffer.data_ptr(), norm=norm.buffer.data_ptr(), state=state.data_ptr(), out=out.buffer.data_ptr(),
        segments=None if segments.table is None else segments.table.data_ptr(), row_pos=pos.data_ptr(),
        workspace=ctx.recurrent_workspace.data_ptr() if nbytes else None, workspace_bytes=nbytes, ld_y=y.buffer.stride(0),
        ld_alpha=alpha.buffer.stride(0), ld_out=out.buffer.stride(0), q_col=cols[0], k_col=cols[1], v_col=cols[2], g_col=cols[3],
        H=shape.heads, dim=shape.dim, vdim=shape.vdim, n_segments=segments.count, max_n=segments.max_n, rows=y.shape[0],
        n_slots=state.shape[0], dtype=dt, path=path, q_scale=shape.dim ** -0.5, eps=eps)
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_gla(ctypes.byref(a), dev_status_ptr(ctx), stream))
