"""Mixture-of-experts feed-forward: expert choice, the experts' grouped products and their weighted sum.

``moe_feed_forward`` runs one layer's experts for the rows of a step from the router's scores: softmax and grouped top-k
(32-bit), the chosen rows sorted by expert, two grouped ``linear`` calls (gate / up with the gated activation in the
epilogue, then down), and the sum weighted by the scores onto the fp32 residual stream.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import _native
from .batch import batch_op_begin, reference_op
from .kv_cache import dtype_code
from .projection import SEG_GLU_SILU, SEG_STORE, OutputSegment, linear
from .types import GPUBuffer2D, GPUContext


@dataclass
class RouterShape:
    experts: int
    top: int
    groups: int = 1  # equal groups of neighbouring experts
    keep: int = 1    # groups whose experts may be chosen


@dataclass
class ExpertWeights:
    """``[in, out]`` matrices of all experts, one after the other: gate and up in neighbouring columns, and down."""

    gate_up: GPUBuffer2D  # [experts * width, 2 * ff]
    down: GPUBuffer2D     # [experts * ff, width]
    ff: int


@dataclass
class MoeScratch:
    idx: torch.Tensor      # int32 [rows, top]
    score: torch.Tensor    # fp32 [rows, top]
    slot: torch.Tensor     # int32 [rows, top]
    counts: torch.Tensor   # int32 [2 * experts]
    offsets: torch.Tensor  # int32 [experts + 1]
    sorted_h: GPUBuffer2D  # [rows * top, width]
    m: GPUBuffer2D         # [rows * top, ff]
    y: GPUBuffer2D         # [rows * top, width]


@reference_op("moe_route")
def route(ctx: GPUContext, logits: GPUBuffer2D, rows: int, shape: RouterShape, s: MoeScratch) -> None:
    """Expert ids, scores and per-expert row counts of ``rows`` rows of router scores (fp32)."""
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_route(logits.buffer.data_ptr(), logits.buffer.stride(0), rows, shape.experts, shape.groups,
                                         shape.keep, shape.top, s.idx.data_ptr(), s.score.data_ptr(), s.counts.data_ptr(),
                                         stream))


@reference_op("moe_plan")
def plan(ctx: GPUContext, h: GPUBuffer2D, shape: RouterShape, s: MoeScratch) -> None:
    """Sorts the chosen rows of ``h`` by expert into ``s.sorted_h``."""
    rows, width = h.shape
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_moe_plan(s.idx.data_ptr(), s.counts.data_ptr(), rows, shape.experts, shape.top,
                                            s.offsets.data_ptr(), s.slot.data_ptr(), h.buffer.data_ptr(), h.buffer.stride(0),
                                            s.sorted_h.buffer.data_ptr(), s.sorted_h.buffer.stride(0), width,
                                            dtype_code(h.buffer.dtype), stream))


@reference_op("moe_combine")
def combine(ctx: GPUContext, x: GPUBuffer2D, shape: RouterShape, s: MoeScratch) -> None:
    """``x[i] += sum_k score[i, k] * y[slot[i, k]]``."""
    rows, width = x.shape
    stream = batch_op_begin(ctx)
    _native.check(_native.lib.b2kv_moe_combine(x.buffer.data_ptr(), x.buffer.stride(0), s.y.buffer.data_ptr(),
                                               s.y.buffer.stride(0), s.slot.data_ptr(), s.score.data_ptr(), rows, shape.top,
                                               width, dtype_code(s.y.buffer.dtype), stream))


def moe_feed_forward(ctx: GPUContext, h: GPUBuffer2D, logits: GPUBuffer2D, w: ExpertWeights, shape: RouterShape,
                     s: MoeScratch, x: GPUBuffer2D, path: int = 0) -> None:
    """Adds the chosen experts' weighted outputs for the rows ``h`` to ``x``."""
    rows, width = h.shape
    route(ctx, logits, rows, shape, s)
    plan(ctx, h, shape, s)
    grouped = dict(groups=shape.experts, group_rows=s.offsets, max_group_rows=rows, path=path)
    n = rows * shape.top
    view = lambda b: GPUBuffer2D(buffer=b.buffer[:n], shape=(n, b.shape[1]), size=n * b.shape[1])  # noqa: E731
    linear(ctx, view(s.sorted_h), w.gate_up, width, [OutputSegment(2 * w.ff, SEG_GLU_SILU, s.m)],
           group_w=width * w.gate_up.buffer.stride(0), **grouped)
    linear(ctx, view(s.m), w.down, w.ff, [OutputSegment(width, SEG_STORE, s.y)], group_w=w.ff * w.down.buffer.stride(0),
           **grouped)
    combine(ctx, x, shape, s)
