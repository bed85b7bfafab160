"""Gigezen: a decoder whose layers run latent attention and a gated feed-forward (dense, or a mixture of experts) in
parallel on one zero-centred RMS norm of a 32-bit residual stream.

    x = table[token]                                                                    embedding_rows
    per layer:
        h = rms_norm(x)                                                                 rms_norm
        [q | latent | key part], [router scores], [gated hidden rows] = h @ w_in        linear, one product for both sublayers
        rotate q; norm the latent, rotate the key part, both into the cache             latent_append
        attention over the cached latents -> a                                          latent_decode or latent_prefill
        x += [a | hidden rows] @ w_out                                                  linear, one product for both sublayers
        x += the chosen experts' weighted outputs (mixture layers)                      moe_feed_forward
    logits = rms_norm(x) @ head                                                         rms_norm, linear

The concatenations are free: the two sublayers of a layer read the same rows and add to the same rows, so their first
matrices stand side by side and their last ones on top of each other, and a layer is two weight-streaming launches beside its
attention.  A layer may read another layer's cached latents (``kv_from``) with matrices of its own.

A step runs any mix of sequences and portions: rows of (sequence, position), short entries first.  Every layer that owns
latents has a ``KVCache`` of one layer; all share one tensor of lengths on the device.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from . import latent, moe
from ._native import lib as _lib
from ._native import check as _check
from .batch import batch_begin, batch_commit, batch_op_begin
from .kv_cache import kv_cache_create
from .latent import LatentShape, PromptPlan, RowPlaces
from .moe import ExpertWeights, MoeScratch, RouterShape
from .projection import SEG_F32, SEG_GLU_CLAMP, SEG_STORE, OutputSegment, linear
from .registry import register_model
from .step_tail import argmax, embedding_rows, rms_norm
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext, KVCache, KVCacheConfig

# Entries of at most this many tokens are attended row by row in the latent space; longer ones expand the visible latents
# into keys and values first, which pays once several rows share them.
SHORT_ENTRY = 16


# ---------------------------------------------------------------------------------------------------------------
# configuration
# ---------------------------------------------------------------------------------------------------------------

@dataclass
class LayerConfig:
    attention: LatentShape
    rot_base: float
    kv_from: Optional[int]         # layer whose latents this one reads; None: its own
    dense_ff: int = 0              # width of the dense feed-forward, 0: none
    limit: float = 0.0
    router: Optional[RouterShape] = None
    expert_ff: int = 0


@dataclass
class GigezenConfig:
    vocab_size: int
    width: int
    eps: float
    layers: List[LayerConfig]

    @staticmethod
    def from_json(c: dict) -> "GigezenConfig":
        layers = []
        for i, entry in enumerate(c["layers"]):
            if entry["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            m, mlp = entry["mixer"], entry.get("mlp")
            mask = m.get("mask") or {}
            shape = LatentShape(heads=m["heads"], dim=m["dim"], rot=m["rot_dim"], rot_dims=m["rot"]["dims"], vdim=m["vdim"],
                                kv_rank=m["kv_rank"], window=int(mask.get("size") or 0), scale=float(m["scale"]))
            layer = LayerConfig(attention=shape, rot_base=float(m["rot"]["base"]), kv_from=m.get("kv_from"))
            if layer.kv_from is not None and not (0 <= layer.kv_from < i and layers[layer.kv_from].kv_from is None):
                raise ValueError(f"layer {i}: kv_from {layer.kv_from} is not an earlier layer with latents of its own")
            if mlp is None:
                pass
            elif mlp["kind"] == "dense":
                layer.dense_ff, layer.limit = mlp["ff"], float(mlp["limit"])
            elif mlp["kind"] == "moe":
                r = mlp["router"]
                groups = r.get("groups") or {"count": 1, "keep": 1}
                layer.router = RouterShape(experts=r["experts"], top=r["top"], groups=groups["count"], keep=groups["keep"])
                layer.expert_ff = mlp["expert"]["ff"]
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(layer)
        return GigezenConfig(vocab_size=c["vocab"], width=c["width"], eps=float(c["norm"]["eps"]), layers=layers)


# ---------------------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------------------

def _pad(n: int, to: int) -> int:
    return (n + to - 1) // to * to


def _b2(t: torch.Tensor) -> GPUBuffer2D:
    return GPUBuffer2D(buffer=t, shape=tuple(t.shape), size=t.numel())


def _b1(t: torch.Tensor) -> GPUBuffer1D:
    return GPUBuffer1D(buffer=t, shape=tuple(t.shape), size=t.numel())


@dataclass
class LayerWeights:
    """Matrices ``[in, out]``; ``w_in`` and ``w_out`` hold both sublayers' first and last matrices (see the module text).
    Column counts are padded with zero columns so that the segments of a product start on 32-column boundaries."""

    norm: GPUBuffer1D
    w_in: GPUBuffer2D         # [width, y_cols + router_cols + 2 * ff_cols]
    w_out: GPUBuffer2D        # [a_cols + ff_cols, width]
    key_absorb: GPUBuffer2D   # [heads * dim, kv_rank]: per head [dim, kv_rank]
    expand: GPUBuffer2D       # [kv_rank, k_cols + heads * vdim]: all heads' keys, then values
    inv_freq: GPUBuffer1D
    latent_norm: Optional[GPUBuffer1D]  # None: the layer reads another layer's latents
    y_cols: int
    router_cols: int
    a_cols: int
    ff_cols: int
    k_cols: int
    experts: Optional[ExpertWeights] = None


@dataclass
class GigezenWeights:
    embedding: GPUBuffer2D  # [vocab, width]
    layers: List[LayerWeights]
    final_norm: GPUBuffer1D
    head: GPUBuffer2D       # [width, vocab]


def _interleave(gate: torch.Tensor, up: torch.Tensor, cols: int) -> torch.Tensor:
    """``[ff, width]`` matrices -> ``[width, 2 * cols]`` with (gate, up) in neighbouring columns, zero columns behind."""
    out = torch.zeros(gate.shape[1], 2 * cols, dtype=gate.dtype, device=gate.device)
    out[:, 0:2 * gate.shape[0]:2] = gate.t()
    out[:, 1:2 * gate.shape[0]:2] = up.t()
    return out


def prepare_weights(ctx: GPUContext, cfg: GigezenConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype) -> GigezenWeights:
    """Checkpoint tensors (``[out, in]`` matrices) -> the layouts the kernels read."""
    dev, width = ctx.device, cfg.width

    def get(name, *shape):
        if name not in tensors:
            raise ValueError(f"the checkpoint has no tensor {name!r}")
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name}: expected shape {shape}, got {tuple(t.shape)}")
        return t.to(dev)

    mat = lambda name, *shape: get(name, *shape).to(dtype)  # noqa: E731
    vec = lambda name, n: _b1(get(name, n).float().contiguous())  # noqa: E731
    layers = []
    for i, lc in enumerate(cfg.layers):
        p, a = f"l{i}.", lc.attention
        q_cols, down_cols = a.heads * (a.dim + a.rot), 0 if lc.kv_from is not None else a.kv_rank + a.rot
        y_cols, a_cols, k_cols = _pad(q_cols + down_cols, 32), _pad(a.heads * a.vdim, 16), _pad(a.heads * a.dim, 8)
        router_cols = _pad(lc.router.experts, 32) if lc.router else 0
        ff_cols = _pad(lc.dense_ff, 16)
        w_in = torch.zeros(width, y_cols + router_cols + 2 * ff_cols, dtype=dtype, device=dev)
        w_in[:, :q_cols] = mat(p + "mix.q", q_cols, width).t()
        if down_cols:
            w_in[:, q_cols:q_cols + down_cols] = mat(p + "mix.dkv", down_cols, width).t()
        w_out = torch.zeros(a_cols + ff_cols, width, dtype=dtype, device=dev)
        w_out[:a.heads * a.vdim] = mat(p + "mix.o", width, a.heads * a.vdim).t()
        experts = None
        if lc.dense_ff:
            ff = lc.dense_ff
            w_in[:, y_cols:] = _interleave(mat(p + "mlp.gate", ff, width), mat(p + "mlp.up", ff, width), ff_cols)
            w_out[a_cols:a_cols + ff] = mat(p + "mlp.down", width, ff).t()
        elif lc.router:
            n_e, ff = lc.router.experts, lc.expert_ff
            e_cols = _pad(ff, 16)
            w_in[:, y_cols:y_cols + n_e] = mat(p + "mlp.router", n_e, width).t()
            gate_up = torch.zeros(n_e, width, 2 * e_cols, dtype=dtype, device=dev)
            down = torch.zeros(n_e, e_cols, width, dtype=dtype, device=dev)
            for e in range(n_e):
                pe = f"{p}mlp.e{e}."
                gate_up[e] = _interleave(mat(pe + "gate", ff, width), mat(pe + "up", ff, width), e_cols)
                down[e, :ff] = mat(pe + "down", width, ff).t()
            experts = ExpertWeights(gate_up=_b2(gate_up.view(n_e * width, 2 * e_cols)), down=_b2(down.view(n_e * e_cols, width)),
                                    ff=e_cols)
        uk = mat(p + "mix.uk", a.heads * a.dim, a.kv_rank).contiguous()
        expand = torch.zeros(a.kv_rank, k_cols + a.heads * a.vdim, dtype=dtype, device=dev)
        expand[:, :a.heads * a.dim] = uk.t()
        expand[:, k_cols:] = mat(p + "mix.uv", a.heads * a.vdim, a.kv_rank).t()
        pair = torch.arange(a.rot_dims // 2, dtype=torch.float64)
        inv_freq = (lc.rot_base ** (-2.0 * pair / a.rot_dims)).float().to(dev)
        layers.append(LayerWeights(
            norm=vec(p + "norm1", width), w_in=_b2(w_in), w_out=_b2(w_out), key_absorb=_b2(uk), expand=_b2(expand),
            inv_freq=_b1(inv_freq), latent_norm=vec(p + "mix.dkv.norm", a.kv_rank) if down_cols else None, y_cols=y_cols,
            router_cols=router_cols, a_cols=a_cols, ff_cols=ff_cols, k_cols=k_cols, experts=experts))
    head = torch.zeros(width, _pad(cfg.vocab_size, 8), dtype=dtype, device=dev)
    head[:, :cfg.vocab_size] = mat("head", cfg.vocab_size, width).t()
    return GigezenWeights(embedding=_b2(mat("embed", cfg.vocab_size, width).contiguous()), layers=layers,
                          final_norm=vec("final.norm", width), head=_b2(head))


def random_tensors(ctx: GPUContext, config: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors of a configuration drawn on the device (benchmarks): matrices N(0, 1 / fan_in), norms near identity."""
    gen = torch.Generator(device=ctx.device).manual_seed(seed)
    rnd = lambda shape, s: (torch.randn(shape, generator=gen, device=ctx.device) * s).to(torch.bfloat16)  # noqa: E731
    mat = lambda out, inp: rnd((out, inp), inp ** -0.5)  # noqa: E731
    width, t = config["width"], {}
    t["embed"], t["head"], t["final.norm"] = rnd((config["vocab"], width), 1.0), mat(config["vocab"], width), rnd((width,), 0.1)
    for i, entry in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry.get("mlp")
        t[p + "norm1"] = rnd((width,), 0.1)
        t[p + "mix.q"] = mat(m["heads"] * (m["dim"] + m["rot_dim"]), width)
        if m.get("kv_from") is None:
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], width), rnd((m["kv_rank"],), 0.1) + 1
        t[p + "mix.uk"], t[p + "mix.uv"] = mat(m["heads"] * m["dim"], m["kv_rank"]), mat(m["heads"] * m["vdim"], m["kv_rank"])
        t[p + "mix.o"] = mat(width, m["heads"] * m["vdim"])
        blocks = [] if mlp is None else [(p + "mlp.", mlp["ff"])] if mlp["kind"] == "dense" else \
            [(f"{p}mlp.e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        for name, ff in blocks:
            t[name + "gate"], t[name + "up"], t[name + "down"] = mat(ff, width), mat(ff, width), mat(width, ff)
        if mlp is not None and mlp["kind"] == "moe":
            t[p + "mlp.router"] = mat(mlp["router"]["experts"], width)
    return t


# ---------------------------------------------------------------------------------------------------------------
# state
# ---------------------------------------------------------------------------------------------------------------

@dataclass
class GigezenState:
    """Caches (one per layer that owns latents), lengths and scratch rows of ``batch_size`` sequences."""

    cfg: GigezenConfig
    weights: GigezenWeights
    batch_size: int
    max_seq_len: int
    dtype: torch.dtype
    owned: Dict[int, KVCache]
    seq_lens: torch.Tensor           # int32 [batch_size] on the device, shared by all caches
    lengths: List[int]               # the same on the host
    scratch: Dict[str, torch.Tensor] = field(default_factory=dict)
    prompt_form: bool = False        # every layer's sizes have a tensor-core form for prompt portions
    logits: Optional[GPUBuffer2D] = None  # fp32 rows of the last step
    layer_tap: Optional[list] = None      # debugging: receives a copy of the residual rows after every layer

    @property
    def caches(self) -> List[KVCache]:
        return list(self.owned.values())

    def cache_of(self, layer: int) -> KVCache:
        src = self.cfg.layers[layer].kv_from
        return self.owned[layer if src is None else src]

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
        for c in self.owned.values():
            c.current_len = max(self.lengths)


def state_create(ctx: GPUContext, cfg: GigezenConfig, weights: GigezenWeights, batch_size: int, max_seq_len: int,
                 dtype: torch.dtype = torch.bfloat16) -> GigezenState:
    owned: Dict[int, KVCache] = {}
    seq_lens = torch.zeros(batch_size, dtype=torch.int32, device=ctx.device)
    for i, lc in enumerate(cfg.layers):
        if lc.kv_from is None:
            a = lc.attention
            owned[i] = kv_cache_create(ctx, KVCacheConfig(batch_size=batch_size, max_seq_len=max_seq_len, n_layers=1, n_heads=1,
                                                          head_dim=a.rot, v_head_dim=a.kv_rank, dtype=dtype, ragged=True))
            owned[i].seq_lens = seq_lens
    return GigezenState(cfg=cfg, weights=weights, batch_size=batch_size, max_seq_len=max_seq_len, dtype=dtype, owned=owned,
                        seq_lens=seq_lens, lengths=[0] * batch_size,
                        prompt_form=all(latent.prefill_supported(lc.attention, dtype) for lc in cfg.layers))


def state_set_lengths(state: GigezenState, lens: Sequence[int]) -> None:
    if len(lens) != state.batch_size or min(lens) < 0 or max(lens) > state.max_seq_len:
        raise ValueError(f"lengths must be {state.batch_size} values in [0, {state.max_seq_len}]")
    state.lengths = [int(v) for v in lens]
    state.seq_lens.copy_(torch.tensor(state.lengths, dtype=torch.int32), non_blocking=False)
    state._sync_upper_bound()


def state_reset(state: GigezenState) -> None:
    state_set_lengths(state, [0] * state.batch_size)


def state_release(state: GigezenState, slot: int) -> None:
    """Gives a finished sequence's place back: its cache rows are free for the next sequence."""
    lens = list(state.lengths)
    lens[slot] = 0
    state_set_lengths(state, lens)


# ---------------------------------------------------------------------------------------------------------------
# the step
# ---------------------------------------------------------------------------------------------------------------

def _sub(b: GPUBuffer2D, r0: int, n: int, c0: int = 0, cols: Optional[int] = None) -> GPUBuffer2D:
    cols = b.shape[1] - c0 if cols is None else cols
    return GPUBuffer2D(buffer=b.buffer[r0:r0 + n, c0:c0 + cols], shape=(n, cols), size=n * cols)


def _attend_rows(ctx, state: GigezenState, i: int, y: GPUBuffer2D, z: GPUBuffer2D, places: RowPlaces, span: int) -> None:
    """Attention of single rows in the latent space: per-head key matrix, latent attention, per-head value matrix."""
    a, w, n = state.cfg.layers[i].attention, state.weights.layers[i], y.shape[0]
    ql = state.rows("q_latent", n, a.heads * a.kv_rank, state.dtype)
    ol = state.rows("o_latent", n, a.heads * a.kv_rank, state.dtype)
    linear(ctx, y, w.key_absorb, a.dim, [OutputSegment(a.kv_rank, SEG_STORE, ql, group=a.kv_rank)], groups=a.heads,
           group_x=a.dim + a.rot, group_w=a.dim * a.kv_rank)
    latent.latent_decode(ctx, ql, y, a, places, state.cache_of(i), ol, span)
    linear(ctx, ol, _sub(w.expand, 0, a.kv_rank, w.k_cols), a.kv_rank, [OutputSegment(a.vdim, SEG_STORE, z, group=a.vdim)],
           groups=a.heads, group_x=a.kv_rank, group_w=a.vdim)


def _layer(ctx, state: GigezenState, i: int, x: GPUBuffer2D, places: RowPlaces, n_single: int, span: int,
           plans: Dict[int, PromptPlan]) -> None:
    lc, w, T = state.cfg.layers[i], state.weights.layers[i], x.shape[0]
    a, cfg, dt = lc.attention, state.cfg, state.dtype
    cache = state.cache_of(i)
    h = state.rows("h", T, cfg.width, dt)
    rms_norm(ctx, x, w.norm, h, cfg.eps, weight_offset=1.0)
    y = state.rows(f"y{w.y_cols}", T, w.y_cols, dt)
    z = state.rows(f"z{w.a_cols + w.ff_cols}", T, w.a_cols + w.ff_cols, dt)
    segments = [OutputSegment(w.y_cols, SEG_STORE, y)]
    logits = None
    if lc.router:
        logits = state.rows("router", T, w.router_cols, torch.float32)
        segments.append(OutputSegment(w.y_cols + w.router_cols, SEG_F32, logits))
    if lc.dense_ff:
        segments.append(OutputSegment(w.y_cols + 2 * w.ff_cols, SEG_GLU_CLAMP, _sub(z, 0, T, w.a_cols)))
    linear(ctx, h, w.w_in, cfg.width, segments, limit=lc.limit)
    latent.latent_append(ctx, y, a, w.inv_freq, places, cache, w.latent_norm, cfg.eps)
    if n_single:
        head_places = RowPlaces(None if places.slot is None else places.slot[:n_single], places.pos[:n_single])
        _attend_rows(ctx, state, i, _sub(y, 0, n_single), _sub(z, 0, n_single, 0, a.heads * a.vdim), head_places, span)
    if plans:
        _attend_prompts(ctx, state, i, y, _sub(z, 0, T, 0, a.heads * a.vdim), plans[a.window])
    linear(ctx, z, w.w_out, w.a_cols + w.ff_cols, [OutputSegment(cfg.width, SEG_F32, x)], residual=x)
    if lc.router:
        moe.moe_feed_forward(ctx, h, logits, w.experts, lc.router, _moe_scratch(state, lc, w, T), x)
    if state.layer_tap is not None:
        state.layer_tap.append(x.buffer.clone())


def _moe_scratch(state: GigezenState, lc: LayerConfig, w: LayerWeights, T: int) -> MoeScratch:
    r, width, dt = lc.router, state.cfg.width, state.dtype
    ints = lambda name, n: state.rows(name, n, 1, torch.int32).buffer  # noqa: E731
    n = T * r.top
    return MoeScratch(idx=ints("moe_idx", n), score=state.rows("moe_score", n, 1, torch.float32).buffer,
                      slot=ints("moe_slot", n), counts=ints("moe_counts", 2 * r.experts),
                      offsets=ints("moe_offsets", r.experts + 1), sorted_h=state.rows("moe_h", n, width, dt),
                      m=state.rows(f"moe_m{w.experts.ff}", n, w.experts.ff, dt), y=state.rows("moe_y", n, width, dt))


def _attend_prompts(ctx, state: GigezenState, i: int, y: GPUBuffer2D, z: GPUBuffer2D, plan: PromptPlan) -> None:
    """Attention of prompt portions: their visible latents become keys and values of all heads in one product."""
    a, w, cache = state.cfg.layers[i].attention, state.weights.layers[i], state.cache_of(i)
    cols = w.k_cols + a.heads * a.vdim
    kv = state.rows(f"kv{cols}", plan.kv_rows, cols, state.dtype)
    latents = cache.layers[0].v_cache.buffer.view(-1, a.kv_rank)
    for _, _, cache_row, visible, kv_row in plan.portions:
        linear(ctx, _b2(latents[cache_row:cache_row + visible]), w.expand, a.kv_rank,
               [OutputSegment(cols, SEG_STORE, _sub(kv, kv_row, visible))])
    latent.latent_prefill(ctx, y, _sub(kv, 0, plan.kv_rows, 0, a.heads * a.dim), _sub(kv, 0, plan.kv_rows, w.k_cols), a, plan,
                          cache, z)


def _run(ctx, state: GigezenState, ids: torch.Tensor, places: RowPlaces, rows: int, n_single: int, span: int,
         plans: Dict[int, PromptPlan], row_index: Optional[torch.Tensor], n_out: int) -> None:
    """Embedding, all layers and, for the ``n_out`` rows of ``row_index`` (None: all), the logits."""
    cfg, w = state.cfg, state.weights
    x = state.rows("x", rows, cfg.width, torch.float32)
    embedding_rows(ctx, w.embedding, ids, x)
    for i in range(len(cfg.layers)):
        _layer(ctx, state, i, x, places, n_single, span, plans)
    if n_out == 0:
        return
    hl = state.rows("h_out", n_out, cfg.width, state.dtype)
    rms_norm(ctx, x, w.final_norm, hl, cfg.eps, weight_offset=1.0, row_index=row_index)
    out = state.rows("logits", n_out, cfg.vocab_size, torch.float32)
    linear(ctx, hl, w.head, cfg.width, [OutputSegment(cfg.vocab_size, SEG_F32, out)])
    state.logits = out


def decode_step(ctx: GPUContext, state: GigezenState, token_ids: GPUBuffer1D, next_ids: Optional[GPUBuffer1D] = None) -> None:
    """One new token for every sequence (``token_ids`` int32 ``[batch_size]``): positions come from the lengths on the device,
    which advance behind the step, so the call can be captured into a graph (``model.GraphedDecodeStep``).  Logits (fp32) are
    left in ``state.logits``, the greedy tokens in ``next_ids``.  Between ``batch_begin`` and ``batch_commit``."""
    upper = state.caches[0].current_len
    if upper >= state.max_seq_len:
        raise ValueError(f"Cache is full: current_len={upper}, max_seq_len={state.max_seq_len}")
    B = state.batch_size
    _run(ctx, state, token_ids.buffer, RowPlaces(None, state.seq_lens), B, B, upper + 1, {}, None, B)
    if next_ids is not None:
        argmax(ctx, state.logits, next_ids)
    _check(_lib.b2kv_advance_lengths(state.seq_lens.data_ptr(), B, 1, batch_op_begin(ctx)))
    state.lengths = [v + 1 for v in state.lengths]
    for c in state.owned.values():
        c.current_len += 1


def forward(ctx: GPUContext, state: GigezenState, entries: Sequence[Tuple[int, Sequence[int], Sequence[int]]]) -> Optional[torch.Tensor]:
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
        ids.append(np.asarray(tokens, dtype=np.int32))
        slots.append(np.full(n, slot, dtype=np.int32))
        pos.append(np.arange(start, start + n, dtype=np.int32))
        T += n
        lens[slot] = start + n
    want = [first_row[j] + int(p) for j in range(len(entries)) for p in entries[j][2]]
    n_out = len(want)
    windows = sorted({lc.attention.window for lc in state.cfg.layers}) if spans else []
    plans = {win: PromptPlan.build(spans, win, state.max_seq_len) for win in windows}
    # one upload per step: ids, sequences, positions, wanted rows, lengths behind the step, prompt tables
    parts = [np.concatenate(ids), np.concatenate(slots), np.concatenate(pos), want, lens] + [plans[win].rows() for win in windows]
    host = torch.from_numpy(np.concatenate([np.asarray(part, dtype=np.int32) for part in parts])).pin_memory()
    pieces = list(host.to(ctx.device, non_blocking=True).split([len(part) for part in parts]))
    for win, table in zip(windows, pieces[5:]):
        plans[win].table = table
    batch_begin(ctx)
    _run(ctx, state, pieces[0], RowPlaces(pieces[1], pieces[2]), T, n_single, span, plans, pieces[3], n_out)
    batch_commit(ctx)
    state.seq_lens.copy_(pieces[4])
    state.lengths = lens
    state._sync_upper_bound()
    return state.logits.buffer if n_out else None


# ---------------------------------------------------------------------------------------------------------------
# the served model
# ---------------------------------------------------------------------------------------------------------------

class _Lengths:
    """What ``generate_text`` resets before a generation: every sequence at once."""

    seq_lens = None

    def __init__(self, state: GigezenState):
        self.state = state

    @property
    def current_len(self) -> int:
        return max(self.state.lengths)

    @current_len.setter
    def current_len(self, value: int) -> None:
        state_set_lengths(self.state, [value] * self.state.batch_size)


class GigezenModel:
    """The registry's face of the design: the interface ``generate_text`` drives (on sequence 0), and steps over any mix of
    sequences and portions."""

    def __init__(self, ctx: GPUContext, cfg: GigezenConfig, weights: GigezenWeights, dtype: torch.dtype, batch_size: int,
                 max_tokens: int):
        self.ctx, self.cfg = ctx, cfg
        self.state = state_create(ctx, cfg, weights, batch_size, max_tokens, dtype)
        self.context, self.vocab_size = max_tokens, cfg.vocab_size
        self.cache = _Lengths(self.state)

    def forward(self, entries) -> Optional[torch.Tensor]:
        return forward(self.ctx, self.state, entries)

    def release(self, slot: int) -> None:
        state_release(self.state, slot)

    def prefill(self, tokens: Sequence[int]) -> torch.Tensor:
        return self.forward([(0, list(tokens), [len(tokens) - 1])])

    def decode_step(self, token: int) -> torch.Tensor:
        return self.forward([(0, [int(token)], [0])])


@register_model("Gigezen")
def _build(ctx: GPUContext, config: dict, weights: Dict[str, torch.Tensor], dtype: torch.dtype, batch_size: int,
           max_tokens: int) -> GigezenModel:
    cfg = GigezenConfig.from_json(config)
    return GigezenModel(ctx, cfg, prepare_weights(ctx, cfg, weights, dtype), dtype, batch_size, max_tokens)
