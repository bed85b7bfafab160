"""Small Bamasun models for the tests (not a test module): configurations with sizes of their own, seeded weights that are exact
in bfloat16."""
import numpy as np
import torch

from tests.gigezen_util import check_rows, numpy_weights, row_errors, tokens  # noqa: F401


def attention(heads, kv_heads, dim, vdim, scale=None, temp=None, kv_from=None, ff=None):
    mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5)
    if temp is not None:
        mixer["q_temp"] = dict(coef=temp[0], every=temp[1])
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return dict(type="attention", mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))


def gla(heads, dim, vdim, tau, rank, ff=None):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau), mlp=None if ff is None else dict(kind="dense", ff=ff), rank=rank)


def config(layers, vocab, width, scale=1.0, cap=30.0, eps=1e-5):
    """The ranks of the decays' bottlenecks are not part of a configuration: they are read off the tensors."""
    return dict(architecture="Bamasun", layers=[{k: v for k, v in layer.items() if k != "rank"} for layer in layers], vocab=vocab, width=width,
                embedding=dict(scale=scale), logit_softcap=cap, norm=dict(eps=eps)), [layer.get("rank") for layer in layers]


# sizes that fill no tile and no 16-byte row: every operation on CUDA cores
ODD = config([gla(3, 5, 7, 4.0, 3, 17), attention(3, 1, 6, 5, 0.5, (0.4, 7), ff=19), attention(4, 2, 9, 3, None, None), gla(1, 9, 33, 1.0, 11),
              attention(6, 1, 6, 5, 0.3, (0.2, 1), kv_from=1, ff=8)], vocab=37, width=26, scale=2.5, cap=4.0)
# sizes of the tensor-core kernels, none of them the width of a tile
TC = config([attention(6, 2, 40, 72, 0.3, (0.3, 50), ff=208), gla(3, 24, 40, 8.0, 5, 136), attention(6, 3, 104, 56, 0.1, (0.5, 33), ff=None),
             attention(9, 2 + 1, 104, 56, 0.15, None, kv_from=2, ff=96), gla(2, 72, 88, 2.0, 24, None),
             attention(4, 2, 40, 72, 0.25, (0.1, 20), kv_from=0, ff=72)], vocab=336, width=264, scale=0.7, cap=20.0)
# head shapes of full-size models
WIDE = config([attention(8, 2, 128, 128, None, (0.2, 64), ff=640), gla(2, 128, 256, 16.0, 16, 512), attention(4, 2, 128, 128, None, (0.2, 64), kv_from=0)],
              vocab=512, width=384, scale=3.0, cap=15.0)
# nothing but recurrence
ONLY_GLA = config([gla(2, 16, 24, 4.0, 8, 64), gla(3, 40, 16, 1.0, 8, None)], vocab=96, width=64)
# every element of a kind equal to one, or as small as it goes
TINY = config([attention(1, 1, 1, 1, 1.0, (1.0, 1), ff=1), gla(1, 1, 1, 1.0, 1, 2)], vocab=5, width=2, scale=1.0, cap=1.0)


def weights(cfg_ranks, seed=0, qk_gain=1.5, decay_mean=2.0):
    cfg, ranks = cfg_ranks
    rs = np.random.RandomState(seed)

    def mat(out, inp, gain=1.0):
        return torch.from_numpy((rs.randn(out, inp) * gain * inp ** -0.5).astype(np.float32)).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.2):
        return torch.from_numpy((rs.randn(n) * std + mean).astype(np.float32)).to(torch.bfloat16)

    W, V, w = cfg["width"], cfg["vocab"], {}

    def norm(name):
        w[name], w[name + ".b"] = vec(W, 1.0), vec(W)

    w["embed"] = mat(V, W, W ** 0.5)
    for i, (lc, rank) in enumerate(zip(cfg["layers"], ranks)):
        p, m, mlp = f"l{i}.", lc["mixer"], lc["mlp"]
        H = m["heads"]
        norm(p + "norm1")
        if lc["type"] == "attention":
            G = m["kv_heads"]
            w[p + "mix.q"], w[p + "mix.q.b"], w[p + "mix.q.norm"] = mat(H * m["dim"], W), vec(H * m["dim"]), vec(H * m["dim"], qk_gain)
            if "kv_from" not in m:
                w[p + "mix.k"], w[p + "mix.k.b"], w[p + "mix.k.norm"] = mat(G * m["dim"], W), vec(G * m["dim"]), vec(G * m["dim"], qk_gain)
                w[p + "mix.v"], w[p + "mix.v.b"] = mat(G * m["vdim"], W), vec(G * m["vdim"])
        else:
            for name, n in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", H * m["vdim"]), ("g", H * m["vdim"]), ("a1", rank)):
                w[p + "mix." + name] = mat(n, W)
            w[p + "mix.a2"], w[p + "mix.a2.b"] = mat(H * m["dim"], rank, 2.0), vec(H * m["dim"], decay_mean, 1.5)
            w[p + "mix.norm"] = vec(m["vdim"], 1.0)
        w[p + "mix.o"] = mat(W, H * m["vdim"])
        if mlp is not None:
            norm(p + "norm2")
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(mlp["ff"], W, 1.5), mat(W, mlp["ff"])
    norm("final.norm")
    w["head"] = mat(V, W, 3.0)
    return w
