"""CPU restatement of the Gigezen decoder (numpy, float64 by default).  TEST INFRASTRUCTURE ONLY.

One function per mechanism, each written from the equations and none of it shared with the product code.
Everything is computed for a whole sequence at once, without a cache, so a comparison with the cached product path
also checks the cache.  Weights are a flat dict of arrays under the names of the checkpoint
(``l<i>.mix.q`` and so on, matrices [out, in]); the configuration is the parsed config.json.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def zero_centred_norm(x, w, eps):
    """RMS norm whose stored weight w means a factor of 1 + w."""
    return rms_norm(x, eps) * (1.0 + w)


def plain_norm(x, w, eps):
    """RMS norm whose stored weight is the factor itself."""
    return rms_norm(x, eps) * w


def rotate_half(x, positions, base):
    """Rotary positions on the last axis of x [tokens, ..., dims]: element i is paired with element i + dims / 2 and
    the pair is turned by position * base^(-2 i / dims)."""
    dims = x.shape[-1]
    half = dims // 2
    freq = base ** (-2.0 * np.arange(half) / dims)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (half,)
    cos, sin = np.cos(angle).reshape(shape), np.sin(angle).reshape(shape)
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin], axis=-1)


def window_mask(n, size):
    """[n, n] bool: query i sees key j when 0 <= i - j < size (every earlier key when size is None)."""
    dist = np.arange(n)[:, None] - np.arange(n)[None, :]
    seen = dist >= 0
    return seen if size is None else seen & (dist < size)


def masked_softmax(scores, seen):
    s = np.where(seen, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_rows(h, w, prefix, mixer, eps):
    """What a layer keeps of every token: (latent [n, kv_rank], rotated key part [n, rot_dim])."""
    r = mixer["kv_rank"]
    down = h @ w[prefix + "mix.dkv"].T
    latent = plain_norm(down[:, :r], w[prefix + "mix.dkv.norm"], eps)
    return latent, rotate_half(down[:, r:], np.arange(len(h)), mixer["rot"]["base"])


def latent_attention(h, latent, key_rot, w, prefix, mixer):
    """Multi-head attention whose keys and values are expanded from the latent rows of every token."""
    n, heads, dim, rot, vdim = len(h), mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"]
    q = (h @ w[prefix + "mix.q"].T).reshape(n, heads, dim + rot)
    q_rot = rotate_half(q[..., dim:], np.arange(n), mixer["rot"]["base"])
    k = (latent @ w[prefix + "mix.uk"].T).reshape(n, heads, dim)
    v = (latent @ w[prefix + "mix.uv"].T).reshape(n, heads, vdim)
    scores = np.einsum("ihd,jhd->hij", q[..., :dim], k) + np.einsum("ihd,jd->hij", q_rot, key_rot)
    mask = mixer.get("mask")
    weights = masked_softmax(scores * mixer["scale"], window_mask(n, None if mask is None else mask["size"])[None])
    out = np.einsum("hij,jhd->ihd", weights, v).reshape(n, heads * vdim)
    return out @ w[prefix + "mix.o"].T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def clamped_glu(gate, up, limit):
    """g sigmoid(1.702 g) (u + 1) with g cut from above at limit and u cut to [-limit, limit]."""
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def silu_glu(gate, up):
    return gate * sigmoid(gate) * up


def dense_ff(h, w, prefix, mlp):
    m = clamped_glu(h @ w[prefix + "mlp.gate"].T, h @ w[prefix + "mlp.up"].T, mlp["limit"])
    return m @ w[prefix + "mlp.down"].T


def route(h, w_router, router):
    """Expert choice: (indices [n, top], weights [n, top]); softmax scores, the best groups by their largest score,
    then the best experts of those groups; the weights are the scores themselves."""
    z = h @ w_router.T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    n, experts = s.shape
    groups = router.get("groups")
    allowed = np.ones_like(s, dtype=bool)
    if groups is not None:
        per = experts // groups["count"]
        best = s.reshape(n, groups["count"], per).max(axis=-1)
        order = np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]]
        allowed[:] = False
        for i in range(n):
            for g in order[i]:
                allowed[i, g * per:(g + 1) * per] = True
    idx = np.argsort(np.where(allowed, -s, np.inf), axis=-1, kind="stable")[:, :router["top"]]
    return idx, np.take_along_axis(s, idx, axis=-1)


def moe_ff(h, w, prefix, mlp):
    idx, weights = route(h, w[prefix + "mlp.router"], mlp["router"])
    out = np.zeros((len(h), h.shape[1]), dtype=h.dtype)
    for i in range(len(h)):
        for e, s in zip(idx[i], weights[i]):
            p = f"{prefix}mlp.e{e}."
            m = silu_glu(h[i] @ w[p + "gate"].T, h[i] @ w[p + "up"].T)
            out[i] += s * (m @ w[p + "down"].T)
    return out


def forward(config, weights, tokens, layers_out=None, dtype=np.float64):
    """Logits [n, vocab] of a whole sequence; appends the residual rows after every layer to layers_out."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    kept = {}
    for i, layer in enumerate(config["layers"]):
        prefix, mixer, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        h = zero_centred_norm(x, w[prefix + "norm1"], eps)
        src = mixer.get("kv_from")
        if src is None:
            kept[i] = latent_rows(h, w, prefix, mixer, eps)
        latent, key_rot = kept[i if src is None else src]
        y = latent_attention(h, latent, key_rot, w, prefix, mixer)
        if mlp is not None:
            y = y + (dense_ff if mlp["kind"] == "dense" else moe_ff)(h, w, prefix, mlp)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T
