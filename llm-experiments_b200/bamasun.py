"""Bamasun: a decoder whose layers mix tokens by grouped-query attention with a distance bias or by gated linear attention, with
the layer norms behind the sublayers and a 32-bit residual stream.

    x = table[token] * scale                                                            embedding_rows
    per layer:
        attention: [q | k | v] = x @ w_in + bias                                        linear
                   norm q over all heads, times a temperature; norm k; k, v -> cache    gqa_append
                   softmax(q k scale - slope distance) v                                gqa_decode or gqa_prefill
        gla:       [q | k | v | gate | decay rows] = x @ w_in                           linear
                   decays = sigmoid(decay rows @ w_a2 + bias)^(1 / tau)                 linear (fp32 out)
                   recurrence, norm per head, gate                                      gated_linear_attention
        x += layer_norm(mixed @ w_o)                                                    linear (fp32 out), layernorm_rows
        x += layer_norm(relu(x @ w_up)^2 @ w_down)                                      linear, linear (fp32 out), layernorm_rows
    logits = cap tanh(layer_norm(x) @ head / cap)                                       layernorm_rows, linear

The norm that writes the residual rows also leaves them in the storage type for the next product.  An attention layer may read an
earlier one's cached keys and values (``kv_from``).  Steps, places and lengths are those of ``serving``; every attention layer that
owns keys has a ``KVCache`` of one layer, every recurrent layer one fp32 state per sequence.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from . import gqa, recurrent
from .gqa import GqaShape
from .kv_cache import kv_cache_create
from .latent import PromptPlan
from .projection import SEG_DECAY, SEG_F32, SEG_RELU2, SEG_SOFTCAP, SEG_STORE, OutputSegment, linear
from .recurrent import GlaShape
from .registry import register_model
from .serving import SequenceState, ServedModel, Step, buffer1, buffer2, pad_to, sub
from .step_tail import embedding_rows, layernorm_rows
from .types import GPUBuffer1D, GPUBuffer2D, GPUContext, KVCache, KVCacheConfig


# ---------------------------------------------------------------------------------------------------------------
# configuration
# ---------------------------------------------------------------------------------------------------------------

@dataclass
class LayerConfig:
    attention: Optional[GqaShape] = None
    gla: Optional[GlaShape] = None
    kv_from: Optional[int] = None  # layer whose keys and values an attention layer reads; None: its own
    ff: int = 0                    # width of the feed-forward, 0: none


@dataclass
class BamasunConfig:
    vocab_size: int
    width: int
    eps: float
    embedding_scale: float
    softcap: float
    layers: List[LayerConfig]

    @staticmethod
    def from_json(c: dict) -> "BamasunConfig":
        layers: List[LayerConfig] = []
        for i, entry in enumerate(c["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry["type"] == "attention":
                temp = m.get("q_temp") or {"coef": 0.0, "every": 0}
                if int(temp["every"]) != temp["every"]:
                    raise ValueError(f"layer {i}: q_temp.every must be a whole number of tokens")
                shape = GqaShape(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                                 temp_coef=float(temp["coef"]), temp_every=int(temp["every"]))
                if shape.heads % shape.kv_heads:
                    raise ValueError(f"layer {i}: {shape.heads} heads do not share {shape.kv_heads} key / value heads evenly")
                layer = LayerConfig(attention=shape, kv_from=m.get("kv_from"))
                if layer.kv_from is not None:
                    src = layers[layer.kv_from] if 0 <= layer.kv_from < i else None
                    if src is None or src.attention is None or src.kv_from is not None:
                        raise ValueError(f"layer {i}: kv_from {layer.kv_from} is not an earlier attention layer with keys of its own")
                    if (src.attention.kv_heads, src.attention.dim, src.attention.vdim) != (shape.kv_heads, shape.dim, shape.vdim):
                        raise ValueError(f"layer {i}: the keys and values of layer {layer.kv_from} have other sizes")
            elif entry["type"] == "gla":
                layer = LayerConfig(gla=GlaShape(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=float(m["tau"])))
            else:
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            if mlp is not None:
                if mlp["kind"] != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
                layer.ff = mlp["ff"]
            layers.append(layer)
        return BamasunConfig(vocab_size=c["vocab"], width=c["width"], eps=float(c["norm"]["eps"]),
                             embedding_scale=float(c["embedding"]["scale"]), softcap=float(c["logit_softcap"]), layers=layers)


# ---------------------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------------------

@dataclass
class NormWeights:
    w: GPUBuffer1D
    b: GPUBuffer1D


@dataclass
class LayerWeights:
    """Matrices ``[in, out]``, column counts padded with zero columns to multiples of 32 (16 for inner dimensions)."""

    w_in: GPUBuffer2D                  # attention [q | k | v] or [q]; gla [q | k | v | gate | decay rows]
    w_o: GPUBuffer2D
    norm1: NormWeights
    bias: Optional[GPUBuffer1D] = None     # of w_in (attention)
    q_norm: Optional[GPUBuffer1D] = None
    k_norm: Optional[GPUBuffer1D] = None
    slopes: Optional[GPUBuffer1D] = None
    cols: Tuple[int, ...] = ()             # gla: first columns of q, k, v, gate, decay rows
    w_a2: Optional[GPUBuffer2D] = None     # gla: decay rows -> logits of the decays
    a2_bias: Optional[GPUBuffer1D] = None
    head_norm: Optional[GPUBuffer1D] = None
    w_up: Optional[GPUBuffer2D] = None
    w_down: Optional[GPUBuffer2D] = None
    norm2: Optional[NormWeights] = None


@dataclass
class BamasunWeights:
    embedding: GPUBuffer2D  # [vocab, width]
    layers: List[LayerWeights]
    final_norm: NormWeights
    head: GPUBuffer2D       # [width, vocab]


def prepare_weights(ctx: GPUContext, cfg: BamasunConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype) -> BamasunWeights:
    """Checkpoint tensors (``[out, in]`` matrices) -> the layouts the kernels read."""
    dev, width = ctx.device, cfg.width

    def get(name, *shape):
        if name not in tensors:
            raise ValueError(f"the checkpoint has no tensor {name!r}")
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name}: expected shape {shape}, got {tuple(t.shape)}")
        return t.to(dev)

    def stack(pieces, rows, to=32):
        """Matrices ``[out, in]`` side by side as ``[rows, columns]`` (zero rows below, zero columns between and behind):
        ``pieces`` = (first column, name, outputs, inputs)."""
        end = max(c + n for c, _, n, _ in pieces)
        out = torch.zeros(rows, pad_to(end, to), dtype=dtype, device=dev)
        for c, name, n, k in pieces:
            out[:k, c:c + n] = get(name, n, k).to(dtype).t()
        return buffer2(out)

    def vector(name, n, padded=None):
        out = torch.zeros(padded or n, dtype=torch.float32, device=dev)
        out[:n] = get(name, n).float()
        return buffer1(out)

    norm = lambda name: NormWeights(w=vector(name, width), b=vector(name + ".b", width))  # noqa: E731
    layers = []
    for i, lc in enumerate(cfg.layers):
        p = f"l{i}."
        if lc.attention is not None:
            a = lc.attention
            nq, nk, nv = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
            parts = [(0, p + "mix.q", nq, width)]
            if lc.kv_from is None:
                parts += [(nq, p + "mix.k", nk, width), (nq + nk, p + "mix.v", nv, width)]
            w_in = stack(parts, width)
            bias = torch.zeros(w_in.shape[1], dtype=torch.float32, device=dev)
            for c, name, n, _ in parts:
                bias[c:c + n] = get(name + ".b", n).float()
            mixed = a.heads * a.vdim
            lw = LayerWeights(w_in=w_in, bias=buffer1(bias), w_o=stack([(0, p + "mix.o", width, mixed)], pad_to(mixed, 16)),
                              norm1=norm(p + "norm1"), q_norm=vector(p + "mix.q.norm", nq),
                              k_norm=vector(p + "mix.k.norm", nk) if lc.kv_from is None else None,
                              slopes=buffer1(gqa.geometric_slopes(a.heads).to(dev)))
        else:
            g = lc.gla
            nk, nv = g.heads * g.dim, g.heads * g.vdim
            if p + "mix.a1" not in tensors:
                raise ValueError(f"the checkpoint has no tensor {p + 'mix.a1'!r}")
            rank = tensors[p + "mix.a1"].shape[0]
            cols = [0]
            for n in (nk, nk, nv, nv):  # every part starts on a 16-byte boundary
                cols.append(pad_to(cols[-1] + n, 8))
            w_in = stack([(c, p + "mix." + name, n, width)
                          for c, name, n in zip(cols, ("q", "k", "v", "g", "a1"), (nk, nk, nv, nv, rank))], width)
            w_a2 = stack([(0, p + "mix.a2", nk, rank)], pad_to(rank, 8))
            lw = LayerWeights(w_in=w_in, w_o=stack([(0, p + "mix.o", width, nv)], pad_to(nv, 16)), norm1=norm(p + "norm1"),
                              cols=tuple(cols), w_a2=w_a2, a2_bias=vector(p + "mix.a2.b", nk, w_a2.shape[1]),
                              head_norm=vector(p + "mix.norm", g.vdim))
        if lc.ff:
            ff = pad_to(lc.ff, 32)
            lw.w_up, lw.w_down = stack([(0, p + "mlp.up", lc.ff, width)], width), stack([(0, p + "mlp.down", width, lc.ff)], ff)
            lw.norm2 = norm(p + "norm2")
        layers.append(lw)
    return BamasunWeights(embedding=buffer2(get("embed", cfg.vocab_size, width).to(dtype).contiguous()), layers=layers,
                          final_norm=norm("final.norm"), head=stack([(0, "head", cfg.vocab_size, width)], width, 8))


def random_tensors(ctx: GPUContext, config: dict, rank: int = 16, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors of a configuration drawn on the device (benchmarks): matrices N(0, 1 / fan_in), norms near identity."""
    gen = torch.Generator(device=ctx.device).manual_seed(seed)
    rnd = lambda shape, s: (torch.randn(shape, generator=gen, device=ctx.device) * s).to(torch.bfloat16)  # noqa: E731
    width, t = config["width"], {}

    def mat(name, out, inp, bias=False):
        t[name] = rnd((out, inp), inp ** -0.5)
        if bias:
            t[name + ".b"] = rnd((out,), 0.1)

    def norm(name):
        t[name], t[name + ".b"] = rnd((width,), 0.1) + 1, rnd((width,), 0.1)

    t["embed"] = rnd((config["vocab"], width), 1.0)
    mat("head", config["vocab"], width)
    norm("final.norm")
    for i, entry in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry.get("mlp")
        norm(p + "norm1")
        if entry["type"] == "attention":
            mat(p + "mix.q", m["heads"] * m["dim"], width, True)
            t[p + "mix.q.norm"] = rnd((m["heads"] * m["dim"],), 0.1) + 1
            if m.get("kv_from") is None:
                mat(p + "mix.k", m["kv_heads"] * m["dim"], width, True)
                mat(p + "mix.v", m["kv_heads"] * m["vdim"], width, True)
                t[p + "mix.k.norm"] = rnd((m["kv_heads"] * m["dim"],), 0.1) + 1
        else:
            nk = m["heads"] * m["dim"]
            for name, n in (("q", nk), ("k", nk), ("v", m["heads"] * m["vdim"]), ("g", m["heads"] * m["vdim"]), ("a1", rank)):
                mat(p + "mix." + name, n, width)
            mat(p + "mix.a2", nk, rank, True)
            t[p + "mix.a2.b"] = t[p + "mix.a2.b"] + 2
            t[p + "mix.norm"] = rnd((m["vdim"],), 0.1) + 1
        mat(p + "mix.o", width, m["heads"] * m["vdim"])
        if mlp is not None:
            norm(p + "norm2")
            mat(p + "mlp.up", mlp["ff"], width)
            mat(p + "mlp.down", width, mlp["ff"])
    return t


# ---------------------------------------------------------------------------------------------------------------
# state and step
# ---------------------------------------------------------------------------------------------------------------

@dataclass
class BamasunState(SequenceState):
    """One cache per attention layer that owns keys, one recurrent state per gla layer."""

    cfg: Optional[BamasunConfig] = None
    weights: Optional[BamasunWeights] = None

    def cache_of(self, layer: int) -> KVCache:
        src = self.cfg.layers[layer].kv_from
        return self.owned[layer if src is None else src]

    def prompt_plans(self, spans) -> Dict[int, PromptPlan]:
        return {0: PromptPlan.build(spans, 0, self.max_seq_len, in_place=True)} if self.owned else {}

    def run(self, ctx: GPUContext, step: Step) -> None:
        cfg, w, T = self.cfg, self.weights, step.rows
        x = self.rows("x", T, cfg.width, torch.float32)
        # the residual rows in the storage type, which the products read
        xs = x if self.dtype == torch.float32 else self.rows("x_storage", T, cfg.width, self.dtype)
        copy = None if xs is x else xs
        embedding_rows(ctx, w.embedding, step.ids, x, scale=cfg.embedding_scale, copy=copy)
        for i, (lc, lw) in enumerate(zip(cfg.layers, w.layers)):
            mixed = _attend(ctx, self, i, xs, step) if lc.attention is not None else _recur(ctx, self, i, xs, step)
            y = self.rows("y", T, lw.w_o.shape[1], torch.float32)
            linear(ctx, mixed, lw.w_o, mixed.shape[1], [OutputSegment(cfg.width, SEG_F32, y)])
            _add_normed(ctx, y, cfg, lw.norm1, x, copy)
            if lc.ff:
                ff = lw.w_up.shape[1]
                hidden = self.rows(f"hidden{ff}", T, ff, self.dtype)
                linear(ctx, xs, lw.w_up, cfg.width, [OutputSegment(ff, SEG_RELU2, hidden)])
                linear(ctx, hidden, lw.w_down, ff, [OutputSegment(cfg.width, SEG_F32, y)])
                _add_normed(ctx, y, cfg, lw.norm2, x, copy)
            if self.layer_tap is not None:
                self.layer_tap.append(x.buffer.clone())
        if step.n_out == 0:
            return
        hl = self.rows("h_out", step.n_out, cfg.width, self.dtype)
        layernorm_rows(ctx, x, w.final_norm.w, w.final_norm.b, cfg.eps, output=hl, row_index=step.row_index)
        out = self.rows("logits", step.n_out, cfg.vocab_size, torch.float32)
        linear(ctx, hl, w.head, cfg.width, [OutputSegment(cfg.vocab_size, SEG_SOFTCAP, out)], limit=cfg.softcap)
        self.logits = out


def state_create(ctx: GPUContext, cfg: BamasunConfig, weights: BamasunWeights, batch_size: int, max_seq_len: int,
                 dtype: torch.dtype = torch.bfloat16) -> BamasunState:
    owned: Dict[int, KVCache] = {}
    states: Dict[int, torch.Tensor] = {}
    seq_lens = torch.zeros(batch_size, dtype=torch.int32, device=ctx.device)
    for i, lc in enumerate(cfg.layers):
        if lc.gla is not None:
            states[i] = recurrent.gla_state_create(ctx, lc.gla, batch_size)
        elif lc.kv_from is None:
            a = lc.attention
            owned[i] = kv_cache_create(ctx, KVCacheConfig(batch_size=batch_size, max_seq_len=max_seq_len, n_layers=1,
                                                          n_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim, dtype=dtype,
                                                          ragged=True))
            owned[i].seq_lens = seq_lens
    return BamasunState(cfg=cfg, weights=weights, batch_size=batch_size, max_seq_len=max_seq_len, dtype=dtype, owned=owned,
                        recurrent=states, seq_lens=seq_lens, lengths=[0] * batch_size,
                        prompt_form=all(gqa.prefill_supported(lc.attention, dtype) for lc in cfg.layers if lc.attention))


def _add_normed(ctx, y: GPUBuffer2D, cfg: BamasunConfig, norm: NormWeights, x: GPUBuffer2D, copy: Optional[GPUBuffer2D]) -> None:
    layernorm_rows(ctx, sub(y, 0, y.shape[0], 0, cfg.width), norm.w, norm.b, cfg.eps, x=x, output=copy)


def _attend(ctx, state: BamasunState, i: int, xs: GPUBuffer2D, step: Step) -> GPUBuffer2D:
    lc, w, T, width = state.cfg.layers[i], state.weights.layers[i], step.rows, state.cfg.width
    a, cache = lc.attention, state.cache_of(i)
    y = state.rows(f"in{w.w_in.shape[1]}", T, w.w_in.shape[1], state.dtype)
    out = state.rows(f"mixed{w.w_o.shape[0]}", T, w.w_o.shape[0], state.dtype)
    linear(ctx, xs, w.w_in, width, [OutputSegment(y.shape[1], SEG_STORE, y)], bias=w.bias)
    gqa.gqa_append(ctx, y, a, step.places, cache, lc.kv_from is None, w.q_norm, w.k_norm, state.cfg.eps)
    if step.n_single:
        gqa.gqa_decode(ctx, sub(y, 0, step.n_single), a, w.slopes, step.single_places(), cache, sub(out, 0, step.n_single), step.span)
    if step.plans:
        gqa.gqa_prefill(ctx, y, a, w.slopes, step.plans[0], cache, out)
    return out


def _recur(ctx, state: BamasunState, i: int, xs: GPUBuffer2D, step: Step) -> GPUBuffer2D:
    g, w, T, width = state.cfg.layers[i].gla, state.weights.layers[i], step.rows, state.cfg.width
    y = state.rows(f"in{w.w_in.shape[1]}", T, w.w_in.shape[1], state.dtype)
    alpha = state.rows(f"decay{w.w_a2.shape[1]}", T, w.w_a2.shape[1], torch.float32)
    out = state.rows(f"mixed{w.w_o.shape[0]}", T, w.w_o.shape[0], state.dtype)
    linear(ctx, xs, w.w_in, width, [OutputSegment(y.shape[1], SEG_STORE, y)])
    linear(ctx, sub(y, 0, T, w.cols[4]), w.w_a2, w.w_a2.shape[0], [OutputSegment(alpha.shape[1], SEG_DECAY, alpha)],
           limit=g.tau, bias=w.a2_bias)
    for segments in (step.short, step.long):
        if segments is not None:
            recurrent.gated_linear_attention(ctx, y, w.cols[:4], alpha, g, w.head_norm, state.cfg.eps, segments, step.places.pos,
                                             state.recurrent[i], out)
    return out


# ---------------------------------------------------------------------------------------------------------------
# the served model
# ---------------------------------------------------------------------------------------------------------------

@register_model("Bamasun")
def _build(ctx: GPUContext, config: dict, weights: Dict[str, torch.Tensor], dtype: torch.dtype, batch_size: int,
           max_tokens: int) -> ServedModel:
    cfg = BamasunConfig.from_json(config)
    return ServedModel(ctx, state_create(ctx, cfg, prepare_weights(ctx, cfg, weights, dtype), batch_size, max_tokens, dtype),
                       cfg.vocab_size)
