"""Latent attention, one operation at a time, against the oracle's equations: the cache append (norm of the latent, rotation of
the key part and of the queries), attention of single rows in the latent space on both kernels, and attention of prompt
portions; windows, keys just inside and just outside, several sequences, sizes that fill no tile, garbage beyond the lengths."""
import numpy as np
import pytest
import torch

from oracle import gigezen_oracle as go
from tests.kv_util import make_ctx, to_f32

pytestmark = pytest.mark.gpu

BF, F32 = torch.bfloat16, torch.float32


def wrap(pkg, t):
    return pkg.gpu.GPUBuffer2D(buffer=t, shape=tuple(t.shape), size=t.numel())


def rnd(shape, dtype, seed, scale=1.0):
    gen = torch.Generator(device="cuda").manual_seed(seed)
    return (torch.randn(shape, generator=gen, device="cuda") * scale).to(dtype)


def ints(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


def make_cache(pkg, ctx, slots, T, rot, rank, dtype):
    cache = pkg.gpu.kv_cache_create(ctx, pkg.gpu.KVCacheConfig(batch_size=slots, max_seq_len=T, n_layers=1, n_heads=1, head_dim=rot,
                                                               v_head_dim=rank, dtype=dtype, ragged=True))
    return cache, cache.layers[0].k_cache.buffer.view(slots, T, rot), cache.layers[0].v_cache.buffer.view(slots, T, rank)


def run(pkg, ctx, fn, *a, **kw):
    ctx.config.check_device_status = True
    pkg.gpu.batch_begin(ctx)
    fn(ctx, *a, **kw)
    pkg.gpu.batch_commit(ctx)
    torch.cuda.synchronize()


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,dim,rot,rank,base", [(3, 8, 4, 10, 500.0), (6, 48, 24, 72, 10000.0), (2, 128, 64, 512, 1e6), (5, 48, 16, 72, 1e4)])
def test_append_norms_rotates_and_stores(pkg, dtype, H, dim, rot, rank, base):
    """Rows of several sequences at scattered positions; every other cache row keeps its value."""
    from llm_experiments_b200 import latent

    ctx = make_ctx(pkg)
    slot, pos = [2, 0, 2, 1, 2], [0, 7, 1, 4000, 4095]
    cache, key, lat = make_cache(pkg, ctx, 3, 4096, rot, rank, dtype)
    key.fill_(3.0), lat.fill_(3.0)
    q_cols = H * (dim + rot)
    y = rnd((5, q_cols + rank + rot + (7 if dim == 8 else 8)), dtype, 1)
    before = to_f32(y).astype(np.float64)
    w = torch.randn(rank, device="cuda") + 1
    inv = torch.tensor([base ** (-2.0 * j / rot) for j in range(rot // 2)], dtype=F32, device="cuda")
    shape = latent.LatentShape(H, dim, rot, rot, 8, rank, 0, 1.0)
    b1 = lambda t: pkg.gpu.GPUBuffer1D(buffer=t, shape=tuple(t.shape), size=t.numel())  # noqa: E731
    run(pkg, ctx, latent.latent_append, wrap(pkg, y), shape, b1(inv), latent.RowPlaces(ints(slot), ints(pos)), cache, b1(w), 1e-5)
    tol = dict(rtol=1e-4, atol=2e-3) if dtype == F32 else dict(rtol=1e-2, atol=2e-2)
    down = before[:, q_cols:q_cols + rank + rot]
    want_lat = go.plain_norm(down[:, :rank], to_f32(w).astype(np.float64), 1e-5)
    want_key = go.rotate_half(down[:, rank:], pos, base)
    for i in range(5):
        np.testing.assert_allclose(to_f32(lat[slot[i], pos[i]]), want_lat[i], **tol)
        np.testing.assert_allclose(to_f32(key[slot[i], pos[i]]), want_key[i], **tol)
    q = before[:, :q_cols].reshape(5, H, dim + rot)
    want_q = np.concatenate([q[..., :dim], go.rotate_half(q[..., dim:], pos, base)], axis=-1).reshape(5, q_cols)
    np.testing.assert_allclose(to_f32(y[:, :q_cols]), want_q, **tol)
    assert np.array_equal(to_f32(y[:, q_cols:]), before[:, q_cols:].astype(np.float32))
    touched = torch.zeros(3, 4096, dtype=torch.bool)
    touched[slot, pos] = True
    assert (key.cpu()[~touched] == 3).all() and (lat.cpu()[~touched] == 3).all()


def test_append_outside_the_cache_is_reported_and_skipped(pkg):
    from llm_experiments_b200 import latent

    ctx = make_ctx(pkg)
    cache, key, lat = make_cache(pkg, ctx, 1, 8, 4, 8, F32)
    y = torch.ones((1, 16 + 12), device="cuda")
    b1 = lambda t: pkg.gpu.GPUBuffer1D(buffer=t, shape=tuple(t.shape), size=t.numel())  # noqa: E731
    shape = latent.LatentShape(2, 4, 4, 4, 4, 8, 0, 1.0)
    with pytest.raises(RuntimeError, match="position"):
        run(pkg, ctx, latent.latent_append, wrap(pkg, y), shape, b1(torch.ones(2, device="cuda")),
            latent.RowPlaces(None, ints([8])), cache, b1(torch.ones(8, device="cuda")), 1e-5)
    assert (key == 0).all() and (lat == 0).all()


def single_rows(q_lat, q, lat, key, slot, pos, shape):
    """Float64 attention of single rows in the latent space."""
    rows, H, R = len(pos), shape.heads, shape.kv_rank
    ql, out = q_lat.view(rows, H, R).double().cpu(), torch.empty(rows, H, R, dtype=torch.float64)
    qr = q[:, :H * (shape.dim + shape.rot)].reshape(rows, H, -1)[..., shape.dim:].double().cpu()
    for i in range(rows):
        lo = max(0, pos[i] - shape.window + 1) if shape.window else 0
        L, K = lat[slot[i], lo:pos[i] + 1].double().cpu(), key[slot[i], lo:pos[i] + 1].double().cpu()
        out[i] = torch.softmax((ql[i] @ L.T + qr[i] @ K.T) * shape.scale, -1) @ L
    return out.view(rows, H * R)


CASES = [  # heads, dim, rot, kv_rank, window, positions
    (7, 8, 16, 56, 45, (0, 1, 43, 44, 45, 46, 300)), (3, 24, 8, 40, 1, (0, 5, 127, 128, 129)),
    (16, 16, 64, 512, 129, (0, 127, 128, 129, 900)), (32, 8, 32, 256, 0, (500, 3)), (50, 8, 64, 512, 200, (700, 10)),
    (70, 8, 24, 136, 0, (383, 384)), (5, 8, 16, 128, 0, (1000,)), (16, 8, 64, 512, 0, tuple(range(250, 250 + 40)))]


@pytest.mark.parametrize("path", [1, 2])
@pytest.mark.parametrize("H,dim,rot,rank,window,pos", CASES)
def test_single_rows_in_the_latent_space(pkg, path, H, dim, rot, rank, window, pos):
    """Both kernels; what lies outside a row's window is made so large that touching it would show, what lies beyond its
    length is not a number of this sequence at all."""
    from llm_experiments_b200 import latent

    ctx = make_ctx(pkg)
    rows = len(pos)
    T = max(pos) + 130
    shape = latent.LatentShape(H, dim, rot, rot, 8, rank, window, (rank + rot) ** -0.5)
    cache, key, lat = make_cache(pkg, ctx, rows, T, rot, rank, BF)
    key.copy_(rnd(key.shape, BF, 2)), lat.copy_(rnd(lat.shape, BF, 3))
    slot = list(range(rows))[::-1]
    for i, p in enumerate(pos):
        lat[slot[i], p + 1:] = 1e4
        if window and p - window >= 0:
            lat[slot[i], :p - window + 1] = -1e4
    q, ql = rnd((rows, H * (dim + rot) + 8), BF, 4), rnd((rows, H * rank), BF, 5)
    out = torch.empty((rows, H * rank), dtype=BF, device="cuda")
    run(pkg, ctx, latent.latent_decode, wrap(pkg, ql), wrap(pkg, q), shape, latent.RowPlaces(ints(slot), ints(pos)), cache,
        wrap(pkg, out), max(pos) + 1, path=path)
    torch.testing.assert_close(out.double().cpu(), single_rows(ql, q, lat, key, slot, pos, shape), rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("path", [1, 2])
def test_growing_scores_and_one_score_that_stands_out(pkg, path):
    """Scores that rise from tile to tile (the reference maximum has to follow), and one key among a thousand that takes all
    the weight: at the far end of the window, and one token further, where it must not be seen."""
    from llm_experiments_b200 import latent

    ctx = make_ctx(pkg)
    H, dim, rot, rank, W = 8, 8, 16, 128, 1000
    shape = latent.LatentShape(H, dim, rot, rot, 8, rank, W, 1.0)
    pos = [1400, 1400, 1400]
    cache, key, lat = make_cache(pkg, ctx, 3, 1500, rot, rank, BF)
    key.zero_(), lat.copy_(rnd(lat.shape, BF, 6, 0.1))
    lat[0, :, 0] = torch.arange(1500, device="cuda") * 0.25  # slot 0: rising scores
    q = torch.zeros((3, H * (dim + rot)), dtype=BF, device="cuda")
    ql = torch.zeros((3, H, rank), dtype=BF, device="cuda")
    ql[0, :, 0] = 1.0
    ql[1:, :, 1] = 8.0
    lat[1, 1400 - W + 1, 1] = 8.0  # slot 1: the first visible key
    lat[2, 1400 - W, 1] = 8.0      # slot 2: one before it
    ql = ql.view(3, H * rank)
    out = torch.empty((3, H * rank), dtype=BF, device="cuda")
    run(pkg, ctx, latent.latent_decode, wrap(pkg, ql), wrap(pkg, q), shape, latent.RowPlaces(None, ints(pos)), cache,
        wrap(pkg, out), 1401, path=path)
    want = single_rows(ql, q, lat, key, [0, 1, 2], pos, shape)
    torch.testing.assert_close(out.double().cpu(), want, rtol=2e-2, atol=2e-2)
    got = out.view(3, H, rank)
    assert (got[1, :, 1] > 7.9).all() and (got[2, :, 1] < 1.0).all()


def test_fp32_single_rows(pkg):
    from llm_experiments_b200 import latent

    ctx = make_ctx(pkg)
    H, dim, rot, rank = 5, 7, 6, 33
    shape = latent.LatentShape(H, dim, rot, rot, 8, rank, 37, 0.2)
    pos, slot = [0, 36, 37, 200], [3, 1, 0, 2]
    cache, key, lat = make_cache(pkg, ctx, 4, 256, rot, rank, F32)
    key.copy_(rnd(key.shape, F32, 2)), lat.copy_(rnd(lat.shape, F32, 3))
    q, ql = rnd((4, H * (dim + rot)), F32, 4), rnd((4, H * rank), F32, 5)
    out = torch.empty((4, H * rank), dtype=F32, device="cuda")
    run(pkg, ctx, latent.latent_decode, wrap(pkg, ql), wrap(pkg, q), shape, latent.RowPlaces(ints(slot), ints(pos)), cache,
        wrap(pkg, out), 201)
    torch.testing.assert_close(out.double().cpu(), single_rows(ql, q, lat, key, slot, pos, shape), rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("H,dim,rot,vdim", [(3, 128, 64, 128), (2, 64, 40, 56), (3, 128, 64, 64), (2, 64, 16, 128), (3, 48, 24, 40),
                                            (2, 96, 64, 80)])
@pytest.mark.parametrize("window", [0, 1, 17, 128, 300])
def test_prompt_portions(pkg, H, dim, rot, vdim, window):
    """Portions of three sequences in one launch: a first one, a short one behind 130 tokens, one of 513 behind 77.  The score of
    one key is raised so that it dominates every query that sees it."""
    from llm_experiments_b200 import latent

    ctx = make_ctx(pkg)
    T, slots = 700, 3
    spans = [(0, 300, 0, 0), (300, 20, 1, 130), (320, 513, 2, 77)]
    rows = sum(n for _, n, _, _ in spans)
    shape = latent.LatentShape(H, dim, rot, rot, vdim, 64, window, (dim + rot) ** -0.5)
    cache, key, _ = make_cache(pkg, ctx, slots, T, rot, 64, BF)
    key.copy_(rnd(key.shape, BF, 1))
    plan = latent.PromptPlan.build(spans, window, T)
    plan.table = ints(plan.rows())
    q, kv = rnd((rows, H * (dim + rot)), BF, 2), rnd((plan.kv_rows, H * (dim + vdim)), BF, 3)
    q.view(rows, H, dim + rot)[:, :, 0] = 4.0
    for (_, n, _, _), (_, _, _, visible, kv0) in zip(spans, plan.portions):
        kv[kv0 + visible - n // 2, :H * dim].view(H, dim)[:, 0] = 30.0  # one far key per sequence
    out = torch.full((rows + 1, H * vdim), 7.0, dtype=BF, device="cuda")
    run(pkg, ctx, latent.latent_prefill, wrap(pkg, q), wrap(pkg, kv[:, :H * dim]), wrap(pkg, kv[:, H * dim:]), shape, plan, cache,
        wrap(pkg, out[:rows]))
    for (row0, n, slot, start), (_, _, _, visible, kv0) in zip(spans, plan.portions):
        qq = q[row0:row0 + n].double().view(n, H, dim + rot)
        k = kv[kv0:kv0 + visible, :H * dim].double().view(visible, H, dim)
        v = kv[kv0:kv0 + visible, H * dim:].double().view(visible, H, vdim)
        kr = key[slot, start + n - visible:start + n].double()
        s = (torch.einsum("ihd,jhd->hij", qq[..., :dim], k) + torch.einsum("ihd,jd->hij", qq[..., dim:], kr)) * shape.scale
        dist = (torch.arange(n, device="cuda") + visible - n)[:, None] - torch.arange(visible, device="cuda")[None]
        seen = (dist >= 0) & ((dist < window) if window else True)
        want = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, -1e300), -1), v).reshape(n, H * vdim)
        torch.testing.assert_close(out[row0:row0 + n].double(), want, rtol=2e-2, atol=2e-2)
    assert (out[rows] == 7).all()
