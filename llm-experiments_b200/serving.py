"""What the served decoders share: sequences of unequal length in numbered places, steps over any mix of them and of portions
of their tokens, and the model object that the registry hands out.

A design brings a ``SequenceState`` of its own: ``run`` (its layers over the rows of a step) and ``prompt_plans`` (the tables
its attention kernels want for prompt portions).  Everything else is here: the caches and lengths, the scratch rows, the order
of a step's rows (short entries first), the single upload of a step, decoding one token per sequence in a form that a CUDA graph
can hold, and giving places back.  Nothing beyond a sequence's length is ever read, and a recurrent state counts as zero at
position 0, so a place that is used again needs no clearing.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from ._native import check as _check
from ._native import lib as _lib
from .batch import batch_begin, batch_commit, batch_op_begin
from .latent import PromptPlan, RowPlaces
from .step_tail import argmax
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext, KVCache

# Entries of at most this many tokens go row by row through the kernels of a decode step; longer ones are prompt portions.
SHORT_ENTRY = 16


def buffer1(t: torch.Tensor) -> GPUBuffer1D:
    return GPUBuffer1D(buffer=t, shape=tuple(t.shape), size=t.numel())


def buffer2(t: torch.Tensor) -> GPUBuffer2D:
    return GPUBuffer2D(buffer=t, shape=tuple(t.shape), size=t.numel())


def sub(b: GPUBuffer2D, r0: int, n: int, c0: int = 0, cols: Optional[int] = None) -> GPUBuffer2D:
    """Rows ``r0 .. r0 + n - 1`` and ``cols`` columns from ``c0`` on, as a view."""
    cols = b.shape[1] - c0 if cols is None else cols
    return GPUBuffer2D(buffer=b.buffer[r0:r0 + n, c0:c0 + cols], shape=(n, cols), size=n * cols)


def pad_to(n: int, to: int) -> int:
    return (n + to - 1) // to * to


@dataclass
class RowSegments:
    """Runs of rows that belong to one sequence each, in order (``b2kv_row_segment``).  ``table`` int32 ``[count, 3]`` on the
    device; ``None``: row i is the only one of sequence i."""

    table: Optional[torch.Tensor]
    count: int
    max_n: int


@dataclass
class Step:
    """The rows of one step.  The first ``n_single`` belong to short entries, the rest to prompt portions."""

    ids: torch.Tensor
    places: RowPlaces
    rows: int
    n_single: int
    span: int                        # bounds the tokens that a row of a short entry sees
    plans: Dict[int, PromptPlan]     # prompt portions, by the key the state's prompt_plans chose
    short: Optional[RowSegments]     # the short entries and
    long: Optional[RowSegments]      # the prompt portions, as runs of rows
    row_index: Optional[torch.Tensor]  # rows whose logits are wanted (None: all)
    n_out: int

    def single_places(self) -> RowPlaces:
        p = self.places
        return RowPlaces(None if p.slot is None else p.slot[:self.n_single], p.pos[:self.n_single])


@dataclass
class SequenceState:
    """Caches (by the layer that owns them), recurrent states, lengths and scratch rows of ``batch_size`` sequences."""

    batch_size: int
    max_seq_len: int
    dtype: torch.dtype
    owned: Dict[int, KVCache]
    seq_lens: torch.Tensor           # int32 [batch_size] on the device, shared by all caches
    lengths: List[int]               # the same on the host
    recurrent: Dict[int, torch.Tensor] = field(default_factory=dict)  # by layer, fp32, first dimension = sequence
    scratch: Dict[str, torch.Tensor] = field(default_factory=dict)
    prompt_form: bool = False        # every layer's sizes have a form for prompt portions
    logits: Optional[GPUBuffer2D] = None  # fp32 rows of the last step
    layer_tap: Optional[list] = None      # debugging: receives a copy of the residual rows after every layer

    def __post_init__(self):
        # a model without any attention still has lengths and a capacity
        self._bare = None if self.owned else KVCache(layers=[], batch_size=self.batch_size, max_seq_len=self.max_seq_len,
                                                     current_len=0, n_heads=0, head_dim=0, seq_lens=self.seq_lens)

    # ---- what a design defines
    def run(self, ctx: GPUContext, step: Step) -> None:
        """Embedding, all layers and, for the wanted rows, the logits (into ``self.logits``)."""
        raise NotImplementedError

    def prompt_plans(self, spans) -> Dict[int, PromptPlan]:
        """Plans for prompt portions ``(row0, n, sequence, start position)``; their tables are uploaded with the step."""
        return {}

    # ---- caches and scratch
    @property
    def caches(self) -> List[KVCache]:
        return list(self.owned.values()) or [self._bare]

    def rows(self, name: str, rows: int, cols: int, dtype: torch.dtype) -> GPUBuffer2D:
        """The first ``rows`` rows of a scratch buffer that grows on demand.  It starts at zero: padding columns that nothing
        writes are multiplied with zero weights and must be numbers."""
        t = self.scratch.get(name)
        if t is None or t.shape[0] < rows or t.shape[1] != cols:
            t = torch.zeros((rows, cols), dtype=dtype, device=self.seq_lens.device)
            self.scratch[name] = t
        return GPUBuffer2D(buffer=t[:rows], shape=(rows, cols), size=rows * cols)

    def advance_host(self, n: int = 1) -> None:
        """Host-side part of advancing every sequence by ``n`` tokens."""
        self.lengths = [v + n for v in self.lengths]
        self._sync_upper_bound()

    def _sync_upper_bound(self) -> None:
        for c in self.caches:
            c.current_len = max(self.lengths)


def state_set_lengths(state: SequenceState, lens: Sequence[int]) -> None:
    if len(lens) != state.batch_size or min(lens) < 0 or max(lens) > state.max_seq_len:
        raise ValueError(f"lengths must be {state.batch_size} values in [0, {state.max_seq_len}]")
    state.lengths = [int(v) for v in lens]
    state.seq_lens.copy_(torch.tensor(state.lengths, dtype=torch.int32), non_blocking=False)
    state._sync_upper_bound()


def state_reset(state: SequenceState) -> None:
    state_set_lengths(state, [0] * state.batch_size)


def state_release(state: SequenceState, slot: int) -> None:
    """Gives a finished sequence's place back: its cache rows and recurrent state are free for the next sequence."""
    lens = list(state.lengths)
    lens[slot] = 0
    state_set_lengths(state, lens)


def decode_step(ctx: GPUContext, state: SequenceState, token_ids: GPUBuffer1D, next_ids: Optional[GPUBuffer1D] = None) -> None:
    """One new token for every sequence (``token_ids`` int32 ``[batch_size]``): positions come from the lengths on the device,
    which advance behind the step, so the call can be captured into a graph (``model.GraphedDecodeStep``).  Logits (fp32) are
    left in ``state.logits``, the greedy tokens in ``next_ids``.  Between ``batch_begin`` and ``batch_commit``."""
    upper = state.caches[0].current_len
    if upper >= state.max_seq_len:
        raise ValueError(f"Cache is full: current_len={upper}, max_seq_len={state.max_seq_len}")
    B = state.batch_size
    state.run(ctx, Step(ids=token_ids.buffer, places=RowPlaces(None, state.seq_lens), rows=B, n_single=B, span=upper + 1, plans={},
                        short=RowSegments(None, B, 1), long=None, row_index=None, n_out=B))
    if next_ids is not None:
        argmax(ctx, state.logits, next_ids)
    _check(_lib.b2kv_advance_lengths(state.seq_lens.data_ptr(), B, 1, batch_op_begin(ctx)))
    state.lengths = [v + 1 for v in state.lengths]
    for c in state.caches:
        c.current_len += 1


def forward(ctx: GPUContext, state: SequenceState, entries: Sequence[Tuple[int, Sequence[int], Sequence[int]]]) -> Optional[torch.Tensor]:
    """One step over ``entries`` = (sequence, its next tokens, the places among them whose logits are wanted): appends the
    tokens to their sequences and returns the wanted logits, fp32 ``[wanted, vocab]`` in the order asked for (None if none).
    Opens and commits a batch of its own."""
    seen = set()
    for slot, tokens, _ in entries:
        if not 0 <= slot < state.batch_size or slot in seen:
            raise ValueError(f"sequence {slot} is out of range or appears twice in a step")
        seen.add(slot)
        if len(tokens) == 0:
            raise ValueError("an entry needs at least one token")
        if state.lengths[slot] + len(tokens) > state.max_seq_len:
            raise ValueError(f"Cache is full: current_len={state.lengths[slot]} + {len(tokens)}, max_seq_len={state.max_seq_len}")
    short = [len(t) <= SHORT_ENTRY or not state.prompt_form for _, t, _ in entries]
    order = sorted(range(len(entries)), key=lambda j: not short[j])  # stable: short entries first
    ids, slots, pos, first_row, spans, lens = [], [], [], {}, [], list(state.lengths)
    runs = {True: [], False: []}  # (first row, rows, sequence) of the short entries and of the prompt portions
    T, n_single, span = 0, 0, 1
    for j in order:
        slot, tokens, _ = entries[j]
        first_row[j] = T
        start, n = lens[slot], len(tokens)
        if short[j]:
            n_single += n
            span = max(span, start + n)
        else:
            spans.append((T, n, slot, start))
        runs[short[j]].append((T, n, slot))
        ids.append(np.asarray(tokens, dtype=np.int32))
        slots.append(np.full(n, slot, dtype=np.int32))
        pos.append(np.arange(start, start + n, dtype=np.int32))
        T += n
        lens[slot] = start + n
    want = [first_row[j] + int(p) for j in range(len(entries)) for p in entries[j][2]]
    n_out = len(want)
    plans = state.prompt_plans(spans) if spans else {}
    # one upload per step: ids, sequences, positions, wanted rows, lengths behind the step, runs of rows, prompt tables
    parts = [np.concatenate(ids), np.concatenate(slots), np.concatenate(pos), want, lens, np.ravel(runs[True]), np.ravel(runs[False])]
    parts += [plan.rows() for plan in plans.values()]
    host = torch.from_numpy(np.concatenate([np.asarray(part, dtype=np.int32) for part in parts])).pin_memory()
    pieces = list(host.to(ctx.device, non_blocking=True).split([len(part) for part in parts]))
    for plan, table in zip(plans.values(), pieces[7:]):
        plan.table = table
    segments = [RowSegments(table, len(r), max(n for _, n, _ in r)) if r else None
                for table, r in ((pieces[5], runs[True]), (pieces[6], runs[False]))]
    batch_begin(ctx)
    state.run(ctx, Step(ids=pieces[0], places=RowPlaces(pieces[1], pieces[2]), rows=T, n_single=n_single, span=span, plans=plans,
                        short=segments[0], long=segments[1], row_index=pieces[3], n_out=n_out))
    batch_commit(ctx)
    state.seq_lens.copy_(pieces[4])
    state.lengths = lens
    state._sync_upper_bound()
    return state.logits.buffer if n_out else None


class _Lengths:
    """What ``generate_text`` resets before a generation: every sequence at once."""

    seq_lens = None

    def __init__(self, state: SequenceState):
        self.state = state

    @property
    def current_len(self) -> int:
        return max(self.state.lengths)

    @current_len.setter
    def current_len(self, value: int) -> None:
        state_set_lengths(self.state, [value] * self.state.batch_size)


class ServedModel:
    """The registry's face of a design: the interface ``generate_text`` drives (on sequence 0), and steps over any mix of
    sequences and portions."""

    def __init__(self, ctx: GPUContext, state: SequenceState, vocab_size: int):
        self.ctx, self.state, self.vocab_size = ctx, state, vocab_size
        self.context = state.max_seq_len
        self.cache = _Lengths(state)

    def forward(self, entries) -> Optional[torch.Tensor]:
        return forward(self.ctx, self.state, entries)

    def release(self, slot: int) -> None:
        state_release(self.state, slot)

    def prefill(self, tokens: Sequence[int]) -> torch.Tensor:
        return self.forward([(0, list(tokens), [len(tokens) - 1])])

    def decode_step(self, token: int) -> torch.Tensor:
        return self.forward([(0, [int(token)], [0])])
