"""Gated linear attention against float64: token after token and sixteen tokens at a time, any cut of a sequence, strong and
vanishing decays, states carried from call to call, places used again, sizes that fill no tile."""
import numpy as np
import pytest
import torch

from oracle import bamasun_oracle as bo
from tests.kv_util import make_ctx

pytestmark = pytest.mark.gpu

F32, BF = torch.float32, torch.bfloat16
STEP, CHUNK = 1, 2


def wrap(pkg, t):
    return pkg.gpu.GPUBuffer2D(buffer=t, shape=tuple(t.shape), size=t.numel())


class Layer:
    """Rows of random queries, keys, values, gates and decays, and what the equations make of them."""

    def __init__(self, pkg, heads, dim, vdim, tau, dtype, z_mean=3.0, z_std=2.0, seed=0):
        from llm_experiments_b200 import recurrent

        self.pkg, self.ctx, self.dtype = pkg, make_ctx(pkg), dtype
        self.ctx.config.check_device_status = True
        self.shape = recurrent.GlaShape(heads, dim, vdim, tau)
        self.gen = torch.Generator(device="cuda").manual_seed(seed)
        pad = lambda n: (n + 7) // 8 * 8  # noqa: E731
        nk, nv = heads * dim, heads * vdim
        self.cols = (0, pad(nk), 2 * pad(nk), 2 * pad(nk) + pad(nv))
        self.width = 2 * pad(nk) + 2 * pad(nv)
        self.norm = torch.randn(vdim, generator=self.gen, device="cuda") * 0.3 + 1
        self.z_mean, self.z_std = z_mean, z_std

    def rows(self, n):
        y = torch.randn((n, self.width), generator=self.gen, device="cuda").to(self.dtype)
        z = torch.randn((n, self.shape.heads * self.shape.dim), generator=self.gen, device="cuda") * self.z_std + self.z_mean
        return y, (torch.sigmoid(z.double()) ** (1 / self.shape.tau)).float()

    def states(self, slots):
        from llm_experiments_b200 import recurrent

        s = recurrent.gla_state_create(self.ctx, self.shape, slots)
        s.fill_(float("nan"))  # a run that starts at position 0 takes nothing over
        return s

    def run(self, y, al, segments, pos, state, path, eps=1e-4):
        """``segments``: (row0, n, slot)."""
        from llm_experiments_b200 import recurrent
        from llm_experiments_b200.serving import RowSegments

        pkg, sh = self.pkg, self.shape
        out = torch.full((len(y) + 1, sh.heads * sh.vdim + 8), 7.0, dtype=self.dtype, device="cuda")
        seg = RowSegments(torch.tensor(segments, dtype=torch.int32, device="cuda"), len(segments), max(n for _, n, _ in segments))
        pkg.gpu.batch_begin(self.ctx)
        recurrent.gated_linear_attention(self.ctx, wrap(pkg, y), self.cols, wrap(pkg, al), sh,
                                         pkg.gpu.GPUBuffer1D(buffer=self.norm, shape=(sh.vdim,), size=sh.vdim), eps, seg,
                                         torch.tensor(pos, dtype=torch.int32, device="cuda"), state, wrap(pkg, out[:len(y)]), path=path)
        pkg.gpu.batch_commit(self.ctx)
        torch.cuda.synchronize()
        assert (out[len(y)] == 7).all() and (out[:, sh.heads * sh.vdim:] == 7).all()
        return out[:len(y), :sh.heads * sh.vdim].double().cpu().numpy()

    def want(self, y, al, state=None, eps=1e-4):
        """Output and last state of one sequence, float64."""
        sh = self.shape
        n = len(y)
        y, alpha = y.double().cpu().numpy(), al.double().cpu().numpy().reshape(n, sh.heads, sh.dim)
        part = lambda c, d: y[:, c:c + sh.heads * d].reshape(n, sh.heads, d)  # noqa: E731
        q, k = part(self.cols[0], sh.dim) * sh.dim ** -0.5, part(self.cols[1], sh.dim)
        v, g = part(self.cols[2], sh.vdim), part(self.cols[3], sh.vdim)
        outs, states = [], []
        for h in range(sh.heads):
            o, s = bo.recurrence(q[:, h], k[:, h], v[:, h], alpha[:, h], None if state is None else state[h])
            outs.append(bo.rms_norm(o, self.norm.double().cpu().numpy(), eps))
            states.append(s)
        return (np.stack(outs, 1) * g * bo.sigmoid(g)).reshape(n, -1), np.stack(states)


def close(got, want, dtype, what=""):
    """The state and the output before rounding are fp32 whatever the storage type."""
    assert np.isfinite(got).all(), what
    tol = 3e-5 if dtype == F32 else 8e-3
    np.testing.assert_allclose(got, want, rtol=tol, atol=tol * max(1.0, np.abs(want).std()), err_msg=str(what))


def state_close(state, want, rtol=1e-4):
    got = state.double().cpu().numpy()
    assert np.abs(got - want).max() <= rtol * np.abs(want).max()


CASES = [(STEP, F32, 3, 5, 7), (STEP, BF, 2, 9, 33), (STEP, F32, 2, 48, 300), (STEP, BF, 4, 128, 256),
         (CHUNK, BF, 5, 40, 24), (CHUNK, BF, 1, 8, 8), (CHUNK, BF, 3, 24, 72), (CHUNK, BF, 2, 64, 160), (CHUNK, BF, 2, 128, 256),
         (CHUNK, BF, 2, 104, 104), (CHUNK, BF, 3, 128, 64)]


@pytest.mark.parametrize("path,dtype,heads,dim,vdim", CASES)
@pytest.mark.parametrize("n", [1, 2, 15, 16, 17, 33, 100])
def test_whole_sequences(pkg, path, dtype, heads, dim, vdim, n):
    layer = Layer(pkg, heads, dim, vdim, 4.0, dtype, seed=n)
    y, al = layer.rows(n)
    state = layer.states(2)
    got = layer.run(y, al, [(0, n, 1)], range(n), state, path)
    want, last = layer.want(y, al)
    close(got, want, dtype, n)
    state_close(state[1], last)
    assert torch.isnan(state[0]).all()


@pytest.mark.parametrize("path,dtype,heads,dim,vdim", [(STEP, F32, 3, 5, 7), (CHUNK, BF, 5, 56, 40), (0, BF, 2, 128, 128), (0, BF, 2, 64, 64)])
def test_portions_carry_the_state(pkg, path, dtype, heads, dim, vdim):
    """Any cut gives the outputs of the whole, with two sequences in unequal portions per call and the rows of a call in any
    order; both kernels take turns when the choice is left open."""
    layer = Layer(pkg, heads, dim, vdim, 8.0, dtype, seed=3)
    (ya, ala), (yb, alb) = layer.rows(143), layer.rows(90)
    wa, sa = layer.want(ya, ala)
    wb, sb = layer.want(yb, alb)
    state = layer.states(3)
    at = [0, 0]
    for na, nb in [(2, 40), (30, 1), (1, 2), (64, 16), (17, 31), (29, 0)]:
        ra, rb = slice(at[0], at[0] + na), slice(at[1], at[1] + nb)
        y, al = torch.cat([yb[rb], ya[ra]]), torch.cat([alb[rb], ala[ra]])
        segs = ([(0, nb, 2)] if nb else []) + [(nb, na, 0)]
        pos = list(range(rb.start, rb.stop)) + list(range(ra.start, ra.stop))
        got = layer.run(y, al, segs, pos, state, path)
        if nb:
            close(got[:nb], wb[rb], dtype, (na, nb))
        close(got[nb:], wa[ra], dtype, (na, nb))
        at = [ra.stop, rb.stop]
    assert at == [143, 90]
    state_close(state[0], sa)
    state_close(state[2], sb)


@pytest.mark.parametrize("path,dtype", [(STEP, F32), (STEP, BF), (CHUNK, BF)])
@pytest.mark.parametrize("z_mean,z_std,tau", [(-30.0, 5.0, 1.0), (-3.0, 30.0, 0.5), (60.0, 1.0, 16.0), (0.0, 200.0, 1.0), (-100.0, 1.0, 16.0)])
def test_strong_and_vanishing_decays(pkg, path, dtype, z_mean, z_std, tau):
    """Channels that forget everything at once, that forget nothing, and both in turn: nothing overflows and nothing is lost."""
    layer = Layer(pkg, 2, 40, 48, tau, dtype, z_mean, z_std, seed=5)
    y, al = layer.rows(75)
    state = layer.states(1)
    got = layer.run(y, al, [(0, 75, 0)], range(75), state, path)
    want, last = layer.want(y, al)
    close(got, want, dtype)
    state_close(state[0], last)


@pytest.mark.parametrize("path,dtype", [(STEP, F32), (CHUNK, BF)])
def test_a_far_token_is_remembered_for_hundreds_of_tokens(pkg, path, dtype):
    """Without decay the value written at token 3 is read back by the only query that matches its key, 500 tokens later."""
    layer = Layer(pkg, 1, 16, 32, 1.0, dtype, z_mean=80.0, z_std=0.0, seed=7)
    y, al = layer.rows(520)
    c = layer.cols
    y[:, c[0]:c[0] + 16], y[:, c[1]:c[1] + 16] = 0, 0
    y[:, c[1] + 1] = 1.0         # every key is unit vector 1 ...
    y[3, c[1]:c[1] + 16] = 0
    y[3, c[1] + 9] = 1.0         # ... but token 3's is unit vector 9
    y[503, c[0] + 9] = 4.0
    got = layer.run(y, al, [(0, 520, 0)], range(520), layer.states(1), path)
    v, g = (y[r, k:k + 32].double().cpu().numpy() for r, k in ((3, c[2]), (503, c[3])))
    close(got[503], bo.rms_norm(v, layer.norm.double().cpu().numpy(), 1e-4) * g * bo.sigmoid(g), dtype)
    assert np.abs(got[502]).max() == 0  # (a query of zeros)


def test_a_decode_step_takes_one_row_per_sequence(pkg):
    """Without a table row i is the next token of sequence i, at positions of their own."""
    from llm_experiments_b200 import recurrent
    from llm_experiments_b200.serving import RowSegments

    layer = Layer(pkg, 4, 64, 96, 16.0, BF, seed=9)
    state = torch.randn((3, 4, 64, 96), generator=layer.gen, device="cuda")
    before = state.double().cpu().numpy()
    y, al = layer.rows(3)
    out = torch.empty((3, 4 * 96), dtype=BF, device="cuda")
    pos = torch.tensor([12, 0, 1], dtype=torch.int32, device="cuda")
    pkg.gpu.batch_begin(layer.ctx)
    recurrent.gated_linear_attention(layer.ctx, wrap(pkg, y), layer.cols, wrap(pkg, al), layer.shape,
                                     pkg.gpu.GPUBuffer1D(buffer=layer.norm, shape=(96,), size=96), 1e-4, RowSegments(None, 3, 1), pos, state,
                                     wrap(pkg, out))
    pkg.gpu.batch_commit(layer.ctx)
    for i in range(3):
        want, last = layer.want(y[i:i + 1], al[i:i + 1], None if i == 1 else before[i])
        close(out[i:i + 1].double().cpu().numpy(), want, BF, i)
        state_close(state[i], last)


def test_segments_outside_the_buffers_are_refused(pkg):
    layer = Layer(pkg, 2, 16, 16, 2.0, BF)
    y, al = layer.rows(20)
    for path in (STEP, CHUNK):
        for seg in ((0, 21, 0), (5, 16, 0), (0, 20, 1), (-1, 4, 0)):
            with pytest.raises(RuntimeError, match="position"):
                layer.run(y, al, [seg], range(20), layer.states(1), path)
