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

Steps, places and lengths are those of ``serving``.  Every layer that owns latents has a ``KVCache`` of one layer; all share one
tensor of lengths on the device.  Short entries are attended row by row in the latent space; prompt portions expand the visible
latents into keys and values first, which pays once several rows share them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from . import latent, moe
from .kv_cache import kv_cache_create
from .latent import LatentShape, PromptPlan, RowPlaces
from .moe import ExpertWeights, MoeScratch, RouterShape
from .projection import SEG_F32, SEG_GLU_CLAMP, SEG_STORE, OutputSegment, linear
from .registry import register_model
from .serving import SequenceState, ServedModel, Step, decode_step, forward, state_release, state_reset, state_set_lengths  # noqa: F401
from .serving import buffer1 as _b1
from .serving import buffer2 as _b2
from .serving import pad_to as _pad
from .serving import sub as _sub
from .step_tail import embedding_rows, rms_norm
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext, KVCache, KVCacheConfig


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
class GigezenState(SequenceState):
    """One cache per layer that owns latents."""

    cfg: Optional[GigezenConfig] = None
    weights: Optional[GigezenWeights] = None

    def cache_of(self, layer: int) -> KVCache:
        src = self.cfg.layers[layer].kv_from
        return self.owned[layer if src is None else src]

    def prompt_plans(self, spans) -> Dict[int, PromptPlan]:
        windows = sorted({lc.attention.window for lc in self.cfg.layers})
        return {win: PromptPlan.build(spans, win, self.max_seq_len) for win in windows}

    def run(self, ctx: GPUContext, step: Step) -> None:
        cfg, w = self.cfg, self.weights
        x = self.rows("x", step.rows, cfg.width, torch.float32)
        embedding_rows(ctx, w.embedding, step.ids, x)
        for i in range(len(cfg.layers)):
            _layer(ctx, self, i, x, step)
        if step.n_out == 0:
            return
        hl = self.rows("h_out", step.n_out, cfg.width, self.dtype)
        rms_norm(ctx, x, w.final_norm, hl, cfg.eps, weight_offset=1.0, row_index=step.row_index)
        out = self.rows("logits", step.n_out, cfg.vocab_size, torch.float32)
        linear(ctx, hl, w.head, cfg.width, [OutputSegment(cfg.vocab_size, SEG_F32, out)])
        self.logits = out


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


# ---------------------------------------------------------------------------------------------------------------
# the step
# ---------------------------------------------------------------------------------------------------------------

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


def _layer(ctx, state: GigezenState, i: int, x: GPUBuffer2D, step: Step) -> None:
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
    latent.latent_append(ctx, y, a, w.inv_freq, step.places, cache, w.latent_norm, cfg.eps)
    n_single = step.n_single
    if n_single:
        _attend_rows(ctx, state, i, _sub(y, 0, n_single), _sub(z, 0, n_single, 0, a.heads * a.vdim), step.single_places(), step.span)
    if step.plans:
        _attend_prompts(ctx, state, i, y, _sub(z, 0, T, 0, a.heads * a.vdim), step.plans[a.window])
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


# ---------------------------------------------------------------------------------------------------------------
# the served model
# ---------------------------------------------------------------------------------------------------------------

@register_model("Gigezen")
def _build(ctx: GPUContext, config: dict, weights: Dict[str, torch.Tensor], dtype: torch.dtype, batch_size: int,
           max_tokens: int) -> ServedModel:
    cfg = GigezenConfig.from_json(config)
    return ServedModel(ctx, state_create(ctx, cfg, prepare_weights(ctx, cfg, weights, dtype), batch_size, max_tokens, dtype),
                       cfg.vocab_size)
