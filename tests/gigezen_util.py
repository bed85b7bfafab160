"""Small Gigezen models for the tests (not a test module): configurations with sizes of their own, seeded weights that are
exact in bfloat16."""
import numpy as np
import torch


def layer(heads, dim, rot, vdim, rank, window, mlp, kv_from=None, base=10000.0, scale=None):
    mixer = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=scale or (dim + rot) ** -0.5,
                 rot=dict(base=base, dims=rot))
    if window is not None:
        mixer["mask"] = dict(size=window)
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=mixer, mlp=mlp)


def dense(ff, limit=1.5):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts, top, ff, groups=None):
    router = dict(experts=experts, top=top)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff), router=router)


def config(layers, vocab, width, eps=1e-5):
    return dict(architecture="Gigezen", layers=layers, vocab=vocab, width=width, norm=dict(eps=eps))


# sizes that fill no tile and no 16-byte row: every operation on CUDA cores
ODD = config([layer(3, 6, 4, 5, 10, 7, dense(17), base=700.0), layer(2, 9, 4, 7, 10, 20, moe(6, 2, 11, (3, 2)), kv_from=0, base=700.0, scale=0.4),
              layer(3, 5, 2, 6, 12, 1, None), layer(1, 4, 4, 3, 7, None, moe(5, 5, 6))], vocab=37, width=26)
# sizes of the tensor-core kernels, none of them a power of two; the last layer reads layer 1's latents with a wider window
TC = config([layer(5, 48, 16, 40, 72, 33, dense(208)), layer(3, 96, 24, 104, 136, 17, moe(12, 3, 56, (4, 2)), base=3000.0),
             layer(4, 64, 24, 48, 136, 150, moe(10, 4, 24, (2, 1)), kv_from=1, base=3000.0), layer(5, 48, 16, 40, 72, 40, None, kv_from=0)],
            vocab=336, width=264)
# a head shape of full-size models
WIDE = config([layer(2, 128, 64, 128, 512, 130, dense(384, 3.0)), layer(2, 128, 64, 128, 512, 64, moe(8, 2, 128, (4, 2)), kv_from=0)],
              vocab=512, width=384)


def weights(cfg, seed=0, router_scale=3.0):
    rs = np.random.RandomState(seed)

    def mat(out, inp, gain=1.0):
        return torch.from_numpy((rs.randn(out, inp) * gain * inp ** -0.5).astype(np.float32)).to(torch.bfloat16)

    def vec(n, mean=0.0):
        return torch.from_numpy((rs.randn(n) * 0.2 + mean).astype(np.float32)).to(torch.bfloat16)

    W, V, w = cfg["width"], cfg["vocab"], {}
    w["embed"] = mat(V, W, W ** 0.5)
    for i, lc in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lc["mixer"], lc["mlp"]
        H, R = m["heads"], m["kv_rank"]
        w[p + "norm1"] = vec(W)
        w[p + "mix.q"] = mat(H * (m["dim"] + m["rot_dim"]), W, 1.5)
        if "kv_from" not in m:
            w[p + "mix.dkv"] = mat(R + m["rot_dim"], W, 1.5)
            w[p + "mix.dkv.norm"] = vec(R, 1.0)
        w[p + "mix.uk"] = mat(H * m["dim"], R, 1.5)
        w[p + "mix.uv"] = mat(H * m["vdim"], R)
        w[p + "mix.o"] = mat(W, H * m["vdim"])
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(mlp["ff"], W, 1.5), mat(mlp["ff"], W, 1.5), mat(W, mlp["ff"])
        else:
            w[p + "mlp.router"] = mat(mlp["router"]["experts"], W, router_scale)
            for e in range(mlp["router"]["experts"]):
                pe, ff = f"{p}mlp.e{e}.", mlp["expert"]["ff"]
                w[pe + "gate"], w[pe + "up"], w[pe + "down"] = mat(ff, W), mat(ff, W), mat(W, ff)
    w["final.norm"] = vec(W)
    w["head"] = mat(V, W)
    return w


def numpy_weights(w):
    return {k: v.float().numpy() for k, v in w.items()}


def tokens(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], size=n)]


def row_errors(got, want):
    """Root mean square error of every row (mean taken off), relative to the spread of the wanted logits."""
    d = got.double().cpu().numpy() - want
    d -= d.mean(axis=1, keepdims=True)
    return np.sqrt((d * d).mean(axis=1)) / want.std()


def check_rows(got, want, dtype, what):
    """fp32: every row.  bf16: nearly every row (rounding may tip the choice of an expert now and then)."""
    err = row_errors(got, want)
    assert np.isfinite(err).all(), what
    if dtype == torch.float32:
        assert err.max() < 1e-4, (what, err.max(), int(err.argmax()))
    else:
        assert np.quantile(err, 0.9) < 0.04, (what, float(np.quantile(err, 0.9)))
        assert np.median(err) < 0.03, (what, float(np.median(err)))
