"""CPU restatement of the Bamasun decoder (numpy, float64 by default).  TEST INFRASTRUCTURE ONLY.

One function per mechanism, each written from the equations and none of it shared with the product code.  Everything is
computed for a whole sequence at once, without a cache; the recurrence runs token by token, without chunks.  Weights are a flat
dict of arrays under the names of the checkpoint (``l<i>.mix.q`` and so on, matrices [out, in]); the configuration is the parsed
config.json.
"""
from __future__ import annotations

import numpy as np


def layer_norm(x, w, b, eps):
    """Mean taken off, divided by the root of variance + eps, then an affine map; over the last axis."""
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def query_temperature(positions, coef, every):
    """Factor of the queries, which grows with the logarithm of the position in steps of ``every`` tokens."""
    return 1.0 + coef * np.log(np.floor((np.asarray(positions) + 1) / every) + 1.0)


def head_slopes(heads):
    """Slope of the distance bias per head: a geometric series that ends at 2^-8."""
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def keys_and_values(h, w, prefix, m, eps):
    """What a layer keeps of every token: normed keys [n, kv_heads, dim] and values [n, kv_heads, vdim]."""
    k = rms_norm(h @ w[prefix + "k"].T + w[prefix + "k.b"], w[prefix + "k.norm"], eps)
    v = h @ w[prefix + "v"].T + w[prefix + "v.b"]
    return k.reshape(len(h), m["kv_heads"], m["dim"]), v.reshape(len(h), m["kv_heads"], m["vdim"])


def attention(h, k, v, w, prefix, m, eps):
    """Causal softmax attention with grouped keys and values, normed queries with a temperature, and a linear distance bias."""
    n, heads = len(h), m["heads"]
    q = rms_norm(h @ w[prefix + "q"].T + w[prefix + "q.b"], w[prefix + "q.norm"], eps)
    if m.get("q_temp"):
        q = q * query_temperature(np.arange(n), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
    q = q.reshape(n, heads, m["dim"])
    per = heads // m["kv_heads"]
    dist = np.arange(n)[:, None] - np.arange(n)[None, :]
    out = np.zeros((n, heads, m["vdim"]), dtype=h.dtype)
    slopes = head_slopes(heads)
    for head in range(heads):
        s = q[:, head] @ k[:, head // per].T * m["scale"] - slopes[head] * dist
        out[:, head] = softmax(np.where(dist >= 0, s, -np.inf)) @ v[:, head // per]
    return out.reshape(n, -1) @ w[prefix + "o"].T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def key_decay(h, w, prefix, m):
    """Per token, head and key channel: the factor the state's rows are multiplied with, [n, heads, dim]."""
    z = (h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "a2.b"]
    return (sigmoid(z) ** (1.0 / m["tau"])).reshape(len(h), m["heads"], m["dim"])


def recurrence(q, k, v, alpha, state=None):
    """S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t for one head; q, k, alpha [n, dim], v [n, vdim].  Returns (o, last S)."""
    s = np.zeros((k.shape[1], v.shape[1]), dtype=v.dtype) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(len(k)):
        s = alpha[t][:, None] * s + k[t][:, None] * v[t][None, :]
        o[t] = q[t] @ s
    return o, s


def gated_linear_attention(h, w, prefix, m, eps):
    n, heads, dim, vdim = len(h), m["heads"], m["dim"], m["vdim"]
    q = (h @ w[prefix + "q"].T).reshape(n, heads, dim) * dim ** -0.5
    k = (h @ w[prefix + "k"].T).reshape(n, heads, dim)
    v = (h @ w[prefix + "v"].T).reshape(n, heads, vdim)
    alpha = key_decay(h, w, prefix, m)
    o = np.stack([recurrence(q[:, i], k[:, i], v[:, i], alpha[:, i])[0] for i in range(heads)], axis=1)
    o = rms_norm(o, w[prefix + "norm"], eps).reshape(n, heads * vdim)
    g = h @ w[prefix + "g"].T
    return (o * g * sigmoid(g)) @ w[prefix + "o"].T


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def dense_ff(h, w, prefix):
    return squared_relu(h @ w[prefix + "up"].T) @ w[prefix + "down"].T


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def forward(config, weights, tokens, layers_out=None, dtype=np.float64):
    """Logits [n, vocab] of a whole sequence; appends the residual rows after every layer to layers_out."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = keys_and_values(x, w, p + "mix.", m, eps)
            y = attention(x, *kept[i if src is None else src], w, p + "mix.", m, eps)
        else:
            y = gated_linear_attention(x, w, p + "mix.", m, eps)
        x = x + layer_norm(y, w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer.get("mlp") is not None:
            x = x + layer_norm(dense_ff(x, w, p + "mlp."), w[p + "norm2"], w[p + "norm2.b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return soft_cap(layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T, config["logit_softcap"])
