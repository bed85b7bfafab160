"""Grouped-query attention against float64: norms, temperature and cache append, single rows on CUDA cores and tensor cores, prompt
portions; distance bias, unequal positions, shares of long rows, keys that stand out far away and at tile borders."""
import numpy as np
import pytest
import torch

from oracle import bamasun_oracle as bo
from tests.kv_util import make_ctx

pytestmark = pytest.mark.gpu

F32, BF = torch.float32, torch.bfloat16
SIMT, TC = 1, 2


def wrap(pkg, t):
    return pkg.gpu.GPUBuffer2D(buffer=t, shape=tuple(t.shape), size=t.numel())


def wrap1(pkg, t):
    return pkg.gpu.GPUBuffer1D(buffer=t, shape=tuple(t.shape), size=t.numel())


def rnd(shape, dtype, seed, scale=1.0):
    gen = torch.Generator(device="cuda").manual_seed(seed)
    return (torch.randn(shape, generator=gen, device="cuda") * scale).to(dtype)


def make_cache(pkg, ctx, shape, slots, T, dtype, fill=True, seed=1):
    cache = pkg.gpu.kv_cache_create(ctx, pkg.gpu.KVCacheConfig(batch_size=slots, max_seq_len=T, n_layers=1, n_heads=shape.kv_heads,
                                                               head_dim=shape.dim, v_head_dim=shape.vdim, dtype=dtype, ragged=True))
    if fill:
        for j, b in enumerate((cache.layers[0].k_cache, cache.layers[0].v_cache)):
            b.buffer.copy_(rnd(b.buffer.shape, dtype, seed + j))
    return cache


def cache_views(cache, shape):
    lay = cache.layers[0]
    T = cache.max_seq_len
    return (lay.k_cache.buffer.view(cache.batch_size, T, shape.kv_heads, shape.dim),
            lay.v_cache.buffer.view(cache.batch_size, T, shape.kv_heads, shape.vdim))


def reference(q, k, v, slots, pos, shape, slopes):
    """q [rows, heads, dim], k / v [slots, T, kv_heads, *] as float64 arrays."""
    out = np.zeros((len(q), shape.heads, shape.vdim))
    per = shape.heads // shape.kv_heads
    for i, (s, p) in enumerate(zip(slots, pos)):
        dist = p - np.arange(p + 1)
        for h in range(shape.heads):
            sc = k[s, :p + 1, h // per] @ q[i, h] * shape.scale - (slopes[h] * dist if slopes is not None else 0)
            out[i, h] = bo.softmax(sc) @ v[s, :p + 1, h // per]
    return out.reshape(len(q), -1)


def np64(t):
    return t.double().cpu().numpy()


def in_batch(pkg, ctx, fn):
    ctx.config.check_device_status = True
    pkg.gpu.batch_begin(ctx)
    fn()
    pkg.gpu.batch_commit(ctx)
    torch.cuda.synchronize()


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim,own", [(F32, 3, 1, 5, 7, True), (BF, 3, 3, 5, 7, True), (F32, 8, 2, 24, 40, True),
                                                        (BF, 6, 3, 40, 24, True), (BF, 32, 8, 128, 128, True), (BF, 4, 2, 72, 64, False)])
@pytest.mark.parametrize("every,coef", [(0, 0.0), (1, 0.7), (37, 0.25)])
def test_append_norms_scales_and_stores(pkg, dtype, heads, kv, dim, vdim, own, every, coef):
    from llm_experiments_b200 import gqa
    from llm_experiments_b200.latent import RowPlaces

    ctx = make_ctx(pkg)
    shape = gqa.GqaShape(heads, kv, dim, vdim, 1.0, coef, every)
    cache = make_cache(pkg, ctx, shape, 3, 200, dtype, fill=False)
    pos = [0, 36, 37, 199, 73, 74]  # either side of a step of the temperature
    slots = [0, 1, 1, 2, 2, 2]
    nq, nk, nv = heads * dim, kv * dim, kv * vdim
    pad = 8
    y = rnd((len(pos), nq + (nk + nv if own else 0) + pad), dtype, 3, 2.0)
    before = np64(y)
    wq, wk = rnd((nq,), F32, 4), rnd((nk,), F32, 5)
    places = RowPlaces(torch.tensor(slots, dtype=torch.int32, device="cuda"), torch.tensor(pos, dtype=torch.int32, device="cuda"))
    in_batch(pkg, ctx, lambda: gqa.gqa_append(ctx, wrap(pkg, y), shape, places, cache, own, wrap1(pkg, wq),
                                              wrap1(pkg, wk) if own else None, 1e-3))
    temp = bo.query_temperature(np.array(pos), coef, every) if every else np.ones(len(pos))
    want_q = bo.rms_norm(before[:, :nq], np64(wq), 1e-3) * temp[:, None]
    tol = 1e-5 if dtype == F32 else 8e-3
    np.testing.assert_allclose(np64(y)[:, :nq], want_q, rtol=tol, atol=tol)
    assert np.array_equal(np64(y)[:, nq:], before[:, nq:])
    k, v = (np64(t) for t in cache_views(cache, shape))
    if not own:
        assert not k.any() and not v.any()
        return
    want_k = bo.rms_norm(before[:, nq:nq + nk], np64(wk), 1e-3).reshape(-1, kv, dim)
    seen = np.zeros(k.shape[:2], dtype=bool)
    for i, (s, p) in enumerate(zip(slots, pos)):
        np.testing.assert_allclose(k[s, p], want_k[i], rtol=tol, atol=tol)
        assert np.array_equal(v[s, p], before[i, nq + nk:nq + nk + nv].reshape(kv, vdim))
        seen[s, p] = True
    assert not k[~seen].any() and not v[~seen].any()


def test_append_refuses_positions_outside_the_cache(pkg):
    from llm_experiments_b200 import gqa
    from llm_experiments_b200.latent import RowPlaces

    ctx = make_ctx(pkg)
    shape = gqa.GqaShape(2, 1, 16, 16, 1.0)
    cache = make_cache(pkg, ctx, shape, 2, 8, BF, fill=False)
    y = rnd((1, 64), BF, 1)
    places = RowPlaces(torch.tensor([1], dtype=torch.int32, device="cuda"), torch.tensor([8], dtype=torch.int32, device="cuda"))
    with pytest.raises(RuntimeError, match="position"):
        in_batch(pkg, ctx, lambda: gqa.gqa_append(ctx, wrap(pkg, y), shape, places, cache, True, None, None, 1e-5))
    assert not cache.layers[0].k_cache.buffer.any()


SHAPES = [(SIMT, F32, 3, 1, 5, 7), (SIMT, BF, 4, 4, 9, 6), (SIMT, F32, 6, 2, 72, 130), (SIMT, F32, 2, 1, 300, 20),
          (TC, BF, 7, 1, 56, 40), (TC, BF, 4, 4, 8, 128), (TC, BF, 10, 2, 128, 128), (TC, BF, 6, 1, 72, 40), (TC, BF, 40, 2, 64, 72),
          (TC, BF, 17, 1, 128, 64), (TC, BF, 70, 2, 24, 24)]


@pytest.mark.parametrize("path,dtype,heads,kv,dim,vdim", SHAPES)
@pytest.mark.parametrize("bias", [False, True])
def test_single_rows(pkg, path, dtype, heads, kv, dim, vdim, bias):
    """Rows at positions either side of every tile border, several of one sequence, against all earlier tokens."""
    from llm_experiments_b200 import gqa
    from llm_experiments_b200.latent import RowPlaces

    ctx = make_ctx(pkg)
    shape = gqa.GqaShape(heads, kv, dim, vdim, 1.3 * dim ** -0.5)
    T = 700
    cache = make_cache(pkg, ctx, shape, 3, T, dtype)
    pos = [0, 1, 63, 64, 127, 128, 129, 255, 256, 383, 384, 500, 640, 699]
    slots = [i % 3 for i in range(len(pos))]
    y = rnd((len(pos), heads * dim + 16), dtype, 7)
    out = torch.full((len(pos) + 1, heads * vdim + 8), 7.0, dtype=dtype, device="cuda")
    slopes = gqa.geometric_slopes(heads).cuda() if bias else None
    places = RowPlaces(torch.tensor(slots, dtype=torch.int32, device="cuda"), torch.tensor(pos, dtype=torch.int32, device="cuda"))
    in_batch(pkg, ctx, lambda: gqa.gqa_decode(ctx, wrap(pkg, y), shape, wrap1(pkg, slopes) if bias else None, places, cache,
                                              wrap(pkg, out[:len(pos)]), T, path=path))
    k, v = (np64(t) for t in cache_views(cache, shape))
    want = reference(np64(y)[:, :heads * dim].reshape(len(pos), heads, dim), k, v, slots, pos, shape, bo.head_slopes(heads) if bias else None)
    tol = 2e-5 if dtype == F32 else 2e-2
    np.testing.assert_allclose(np64(out)[:len(pos), :heads * vdim], want, rtol=tol, atol=tol)
    assert (out[len(pos)] == 7).all() and (out[:, heads * vdim:] == 7).all()


@pytest.mark.parametrize("share", [1, 2, 3, 5, 16])
def test_single_rows_in_shares(pkg, share):
    """However a row's tokens are cut into shares the result is the same; rows of one share sit beside rows of many."""
    from llm_experiments_b200 import gqa
    from llm_experiments_b200.latent import RowPlaces

    ctx = make_ctx(pkg)
    shape = gqa.GqaShape(12, 3, 64, 96, 0.2)
    cache = make_cache(pkg, ctx, shape, 4, 1500, BF, seed=11)
    pos = [1499, 3, 700, 128 * 5 - 1]
    y = rnd((4, 12 * 64), BF, 13)
    out = torch.empty((4, 12 * 96), dtype=BF, device="cuda")
    slopes = gqa.geometric_slopes(12).cuda()
    places = RowPlaces(None, torch.tensor(pos, dtype=torch.int32, device="cuda"))
    pkg._native.tune("gqa_decode_share", share)
    try:
        in_batch(pkg, ctx, lambda: gqa.gqa_decode(ctx, wrap(pkg, y), shape, wrap1(pkg, slopes), places, cache, wrap(pkg, out), 1500, path=TC))
    finally:
        pkg._native.tune("gqa_decode_share", 0)
    k, v = (np64(t) for t in cache_views(cache, shape))
    want = reference(np64(y).reshape(4, 12, 64), k, v, range(4), pos, shape, bo.head_slopes(12))
    np.testing.assert_allclose(np64(out), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("path,dtype", [(SIMT, F32), (TC, BF)])
def test_a_single_key_among_hundreds_is_found(pkg, path, dtype):
    """One key per place in turn - first, last, either side of tile borders - scores far above the others: the output is its value."""
    from llm_experiments_b200 import gqa
    from llm_experiments_b200.latent import RowPlaces

    ctx = make_ctx(pkg)
    shape = gqa.GqaShape(4, 2, 64, 64, 1.0)
    T = 900
    cache = make_cache(pkg, ctx, shape, 1, T, dtype, seed=21)
    k, v = cache_views(cache, shape)
    k.mul_(0.05)
    targets = [0, 1, 127, 128, 255, 256, 383, 511, 512, 767, 768, 897, 898]
    pos = 898
    q = torch.zeros((len(targets), 4, 64), dtype=dtype, device="cuda")
    for r, t in enumerate(targets):  # query r meets only key t: unit vectors of their own
        q[r, :, r] = 40.0
        k[0, t, :, :] = 0
        k[0, t, :, r] = 1.0
    out = torch.empty((len(targets), 4 * 64), dtype=dtype, device="cuda")
    places = RowPlaces(torch.zeros(len(targets), dtype=torch.int32, device="cuda"), torch.full((len(targets),), pos, dtype=torch.int32, device="cuda"))
    in_batch(pkg, ctx, lambda: gqa.gqa_decode(ctx, wrap(pkg, q.view(len(targets), -1)), shape, None, places, cache, wrap(pkg, out), T, path=path))
    for r, t in enumerate(targets):
        want = v[0, t].repeat_interleave(2, 0).reshape(-1).double()
        torch.testing.assert_close(out[r].double(), want, rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("heads,kv,dim,vdim", [(7, 1, 56, 40), (6, 3, 128, 128), (4, 4, 72, 40), (5, 1, 64, 104), (2, 2, 8, 8)])
@pytest.mark.parametrize("bias", [False, True])
def test_prompt_portions(pkg, heads, kv, dim, vdim, bias):
    """Several sequences' portions in one launch: from the start, behind a cached part, across tile borders, of two rows."""
    from llm_experiments_b200 import gqa
    from llm_experiments_b200.latent import PromptPlan

    ctx = make_ctx(pkg)
    shape = gqa.GqaShape(heads, kv, dim, vdim, 1.2 * dim ** -0.5)
    T = 640
    cache = make_cache(pkg, ctx, shape, 5, T, BF, seed=31)
    portions = [(0, 300, 0), (2, 17, 111), (4, 257, 383), (1, 2, 127), (3, 130, 0)]  # (sequence, rows, start)
    spans, row = [], 0
    for slot, n, start in portions:
        spans.append((row, n, slot, start))
        row += n
    plan = PromptPlan.build(spans, 0, T, in_place=True)
    plan.table = torch.tensor(plan.rows(), dtype=torch.int32, device="cuda")
    y = rnd((row, heads * dim + 24), BF, 33)
    out = torch.full((row + 1, heads * vdim + 8), 7.0, dtype=BF, device="cuda")
    slopes = gqa.geometric_slopes(heads).cuda() if bias else None
    in_batch(pkg, ctx, lambda: gqa.gqa_prefill(ctx, wrap(pkg, y), shape, wrap1(pkg, slopes) if bias else None, plan, cache,
                                               wrap(pkg, out[:row])))
    k, v = (np64(t) for t in cache_views(cache, shape))
    slots = np.concatenate([[s] * n for s, n, _ in portions])
    pos = np.concatenate([np.arange(n) + start for _, n, start in portions])
    want = reference(np64(y)[:, :heads * dim].reshape(row, heads, dim), k, v, slots, pos, shape, bo.head_slopes(heads) if bias else None)
    np.testing.assert_allclose(np64(out)[:row, :heads * vdim], want, rtol=2e-2, atol=2e-2)
    assert (out[row] == 7).all() and (out[:, heads * vdim:] == 7).all()
