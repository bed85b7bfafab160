"""b2kv_linear against float64 products: every kernel behind it, every kind of segment, per-head and per-expert groups, sizes
that fill no tile, empty experts, and guards around what may be written."""
import numpy as np
import pytest
import torch

from tests.kv_util import make_ctx

pytestmark = pytest.mark.gpu

SIMT, ROWS, TILED, THIN = 1, 2, 3, 4


def glu(kind, g, u, limit, proj):
    if kind == proj.SEG_GLU_SILU:
        return g * torch.sigmoid(g) * u
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def wrap(pkg, t):
    return pkg.gpu.GPUBuffer2D(buffer=t, shape=tuple(t.shape), size=t.numel())


def rnd(shape, dtype, seed, scale=1.0):
    gen = torch.Generator(device="cuda").manual_seed(seed)
    return (torch.randn(shape, generator=gen, device="cuda") * scale).to(dtype)


def close(got, want, dtype):
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.6e-2, atol=1.6e-2)
    assert torch.isfinite(got).all()
    torch.testing.assert_close(got.double(), want, **tol)


def run(pkg, ctx, *a, **kw):
    from llm_experiments_b200 import projection

    ctx.config.check_device_status = True
    pkg.gpu.batch_begin(ctx)
    projection.linear(ctx, *a, **kw)
    pkg.gpu.batch_commit(ctx)
    torch.cuda.synchronize()


@pytest.mark.parametrize("path,dtype,rows,K,cols", [
    (SIMT, torch.float32, 5, 37, (30, 7)), (SIMT, torch.bfloat16, 70, 100, (64, 33)),
    (ROWS, torch.bfloat16, 1, 176, (64, 24)), (ROWS, torch.bfloat16, 3, 72, (32, 40)),
    (ROWS, torch.bfloat16, 64, 1000, (96, 200)), (ROWS, torch.bfloat16, 128, 4096, (256, 256)),
    (TILED, torch.bfloat16, 129, 64, (32, 16)), (TILED, torch.bfloat16, 300, 200, (320, 72)),
    (TILED, torch.bfloat16, 1000, 520, (64, 704))])
def test_store_and_fp32_segments(pkg, path, dtype, rows, K, cols):
    """A strided x, a bf16 segment into some columns of a wider buffer, an fp32 segment added to a residual in place."""
    from llm_experiments_b200 import projection as proj

    ctx = make_ctx(pkg)
    a, b = cols
    pad = 0 if path == SIMT else 8
    x = rnd((rows, K + 2 * pad), dtype, 1)[:, pad:pad + K]
    w = rnd((K, (a + b + 7) // 8 * 8), dtype, 2, K ** -0.5)
    wide = torch.full((rows + 1, a + 16), 7.0, dtype=dtype, device="cuda")
    res = rnd((rows, (b + 3) // 4 * 4), torch.float32, 3)
    keep = res.clone()
    run(pkg, ctx, wrap(pkg, x), wrap(pkg, w), K,
        [proj.OutputSegment(a, proj.SEG_STORE, wrap(pkg, wide[:, 8:8 + a])), proj.OutputSegment(a + b, proj.SEG_F32, wrap(pkg, res))],
        residual=wrap(pkg, res), path=path)
    want = x.double() @ w.double()
    close(wide[:rows, 8:8 + a], want[:, :a], dtype)
    close(res[:, :b], want[:, a:a + b] + keep[:, :b].double(), torch.float32)
    assert (wide[rows] == 7).all() and (wide[:, :8] == 7).all() and (wide[:, 8 + a:] == 7).all()
    assert torch.equal(res[:, b:], keep[:, b:])


@pytest.mark.parametrize("kind", ["SEG_GLU_SILU", "SEG_GLU_CLAMP"])
@pytest.mark.parametrize("path,dtype,rows,K,ff", [
    (SIMT, torch.float32, 9, 40, 21), (ROWS, torch.bfloat16, 2, 96, 48), (ROWS, torch.bfloat16, 33, 2048, 64),
    (ROWS, torch.bfloat16, 100, 256, 400), (TILED, torch.bfloat16, 200, 256, 208), (TILED, torch.bfloat16, 600, 208, 352)])
def test_gated_segments(pkg, kind, path, dtype, rows, K, ff):
    from llm_experiments_b200 import projection as proj

    ctx, kind = make_ctx(pkg), getattr(proj, kind)
    x, w = rnd((rows, K), dtype, 4), rnd((K, 32 + 2 * ff), dtype, 5, 2 * K ** -0.5)
    plain = torch.empty((rows, 32), dtype=dtype, device="cuda")
    out = torch.full((rows + 1, ff + 8), 7.0, dtype=dtype, device="cuda")
    run(pkg, ctx, wrap(pkg, x), wrap(pkg, w), K,
        [proj.OutputSegment(32, proj.SEG_STORE, wrap(pkg, plain)),
         proj.OutputSegment(32 + 2 * ff, kind, wrap(pkg, out[:, :ff]))], limit=1.5, path=path)
    prod = x.double() @ w.double()
    close(plain, prod[:, :32], dtype)
    close(out[:rows, :ff], glu(kind, prod[:, 32::2], prod[:, 33::2], 1.5, proj), dtype)
    assert (out[rows] == 7).all() and (out[:, ff:] == 7).all()


@pytest.mark.parametrize("path,dtype,rows,heads,k,n,gap", [
    (SIMT, torch.float32, 3, 5, 12, 20, 7), (ROWS, torch.bfloat16, 4, 7, 56, 72, 40), (ROWS, torch.bfloat16, 17, 3, 40, 136, 24),
    (ROWS, torch.bfloat16, 64, 16, 128, 512, 64), (0, torch.bfloat16, 300, 4, 64, 96, 16)])
def test_per_head_products(pkg, path, dtype, rows, heads, k, n, gap):
    """Head h multiplies its own columns of x with its own matrix; what lies between the heads' columns is not touched, even
    when it is not a number."""
    from llm_experiments_b200 import projection as proj

    ctx = make_ctx(pkg)
    x, w = rnd((rows, heads * (k + gap)), dtype, 6), rnd((heads * k, n), dtype, 7, k ** -0.5)
    x.view(rows, heads, k + gap)[:, :, k:] = float("nan")
    out = torch.empty((rows, heads * n), dtype=dtype, device="cuda")
    run(pkg, ctx, wrap(pkg, x), wrap(pkg, w), k, [proj.OutputSegment(n, proj.SEG_STORE, wrap(pkg, out), group=n)], groups=heads,
        group_x=k + gap, group_w=k * n, path=path)
    want = torch.einsum("rhk,hkn->rhn", x.view(rows, heads, k + gap)[:, :, :k].double(), w.view(heads, k, n).double())
    close(out.view(rows, heads, n), want, dtype)


def test_per_head_columns_of_one_matrix(pkg):
    """The heads' matrices may be column ranges of one wide matrix (a group step smaller than its row pitch)."""
    from llm_experiments_b200 import projection as proj

    ctx = make_ctx(pkg)
    rows, heads, k, n, c0 = 10, 5, 96, 48, 40
    x, w = rnd((rows, heads * k), torch.bfloat16, 8), rnd((k, c0 + heads * n), torch.bfloat16, 9, k ** -0.5)
    out = torch.empty((rows, heads * n), dtype=torch.bfloat16, device="cuda")
    run(pkg, ctx, wrap(pkg, x), wrap(pkg, w[:, c0:]), k, [proj.OutputSegment(n, proj.SEG_STORE, wrap(pkg, out), group=n)],
        groups=heads, group_x=k, group_w=n, path=ROWS)
    want = torch.einsum("rhk,khn->rhn", x.view(rows, heads, k).double(), w[:, c0:].reshape(k, heads, n).double())
    close(out.view(rows, heads, n), want, torch.bfloat16)


@pytest.mark.parametrize("path,dtype,counts,K,n,glu_kind", [
    (SIMT, torch.float32, (3, 0, 5, 1), 20, 24, False), (ROWS, torch.bfloat16, (3, 0, 17, 1, 0), 176, 96, True),
    (ROWS, torch.bfloat16, (0, 128, 1), 1408, 264, False), (TILED, torch.bfloat16, (0, 300, 1, 128, 0, 257, 129), 64, 328, False),
    (TILED, torch.bfloat16, (700, 513, 0), 256, 272, True)])
def test_rows_grouped_by_expert(pkg, path, dtype, counts, K, n, glu_kind):
    from llm_experiments_b200 import projection as proj

    ctx = make_ctx(pkg)
    E, R = len(counts), sum(counts)
    offs = np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)
    x, w = rnd((R, K), dtype, 10), rnd((E * K, n), dtype, 11, K ** -0.5)
    cols = n // 2 if glu_kind else n
    out = torch.full((R + 1, cols), 7.0, dtype=dtype, device="cuda")
    kind = proj.SEG_GLU_SILU if glu_kind else proj.SEG_STORE
    run(pkg, ctx, wrap(pkg, x), wrap(pkg, w), K, [proj.OutputSegment(n, kind, wrap(pkg, out))], groups=E, group_w=K * n,
        group_rows=torch.from_numpy(offs).cuda(), max_group_rows=max(counts), path=path)
    for e in range(E):
        prod = x[offs[e]:offs[e + 1]].double() @ w[e * K:(e + 1) * K].double()
        close(out[offs[e]:offs[e + 1]], glu(kind, prod[:, 0::2], prod[:, 1::2], 0, proj) if glu_kind else prod, dtype)
    assert (out[R] == 7).all()


def activated(kind, z, limit, proj):
    if kind == proj.SEG_RELU2:
        return z.clamp(min=0) ** 2
    if kind == proj.SEG_SOFTCAP:
        return limit * torch.tanh(z / limit)
    return torch.exp(torch.nn.functional.logsigmoid(z) / limit) if kind == proj.SEG_DECAY else z


@pytest.mark.parametrize("kind", ["SEG_STORE", "SEG_F32", "SEG_RELU2", "SEG_SOFTCAP", "SEG_DECAY"])
@pytest.mark.parametrize("path,dtype,rows,K,n", [
    (SIMT, torch.float32, 9, 40, 21), (SIMT, torch.bfloat16, 70, 100, 33), (ROWS, torch.bfloat16, 3, 72, 40), (ROWS, torch.bfloat16, 100, 2048, 104),
    (ROWS, torch.bfloat16, 64, 4096, 128), (TILED, torch.bfloat16, 200, 256, 208), (TILED, torch.bfloat16, 700, 136, 72),
    (THIN, torch.bfloat16, 5, 16, 34), (THIN, torch.bfloat16, 1100, 24, 300), (THIN, torch.bfloat16, 65, 32, 256), (0, torch.bfloat16, 40, 8, 64)])
def test_bias_and_single_column_forms(pkg, kind, path, dtype, rows, K, n):
    """A bias added ahead of the square of the positive part, a soft cap, the root of a sigmoid, or nothing."""
    from llm_experiments_b200 import projection as proj

    ctx, kind = make_ctx(pkg), getattr(proj, kind)
    pad = (n + 7) // 8 * 8
    x, w = rnd((rows, K), dtype, 20), rnd((K, pad), dtype, 21, 2 * K ** -0.5)
    bias = rnd((n,), torch.float32, 22, 2.0)
    fp32 = kind in (proj.SEG_F32, proj.SEG_SOFTCAP, proj.SEG_DECAY)
    out = torch.full((rows + 1, pad), 7.0, dtype=torch.float32 if fp32 else dtype, device="cuda")
    run(pkg, ctx, wrap(pkg, x), wrap(pkg, w), K, [proj.OutputSegment(n, kind, wrap(pkg, out))], limit=2.5, path=path,
        bias=pkg.gpu.GPUBuffer1D(buffer=bias, shape=(n,), size=n))
    want = activated(kind, x.double() @ w.double()[:, :n] + bias.double(), 2.5, proj)
    close(out[:rows, :n], want, torch.float32 if fp32 else dtype)
    assert (out[rows] == 7).all() and (out[:, n:] == 7).all()


@pytest.mark.parametrize("path,rows", [(SIMT, 6), (ROWS, 6), (TILED, 160), (THIN, 6)])
def test_decays_close_to_one_keep_what_they_take_away(pkg, path, rows):
    """For large logits the decay is one minus something tiny; far below zero it is a tiny number of its own."""
    from llm_experiments_b200 import projection as proj

    ctx = make_ctx(pkg)
    z = torch.tensor([-120.0, -60.0, -20.0, -3.0, -0.5, 0.0, 0.5, 3.0, 8.0, 12.0, 14.0, 20.0, 40.0, 90.0, 1.0, -1.0], device="cuda")
    x, w = torch.zeros((rows, 16), dtype=torch.bfloat16, device="cuda"), torch.zeros((16, 16), dtype=torch.bfloat16, device="cuda")
    out = torch.empty((rows, 16), device="cuda")
    for tau in (1.0, 16.0):
        run(pkg, ctx, wrap(pkg, x), wrap(pkg, w), 16, [proj.OutputSegment(16, proj.SEG_DECAY, wrap(pkg, out))], limit=tau, path=path,
            bias=pkg.gpu.GPUBuffer1D(buffer=z, shape=(16,), size=16))
        want = torch.exp(torch.nn.functional.logsigmoid(z.double()) / tau)
        torch.testing.assert_close(out[rows - 1].double(), want, rtol=2e-6 if tau == 16 else 2e-5, atol=1e-12)
        torch.testing.assert_close(1 - out[0].double(), 1 - want, rtol=2e-3, atol=3e-7)
