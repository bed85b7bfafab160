"""The Bamasun oracle, one mechanism at a time, against worked values; the reader of its configuration; the argument checks of the
C entry points.  No GPU."""
import copy
import ctypes
import json

import numpy as np
import pytest

from oracle import bamasun_oracle as bo
from tests import bamasun_util as U


def test_norms():
    x = np.array([[1.0, 3.0, 5.0, 7.0]])
    np.testing.assert_allclose(bo.layer_norm(x, np.ones(4), np.zeros(4), 4.0), [[-1.0, -1 / 3, 1 / 3, 1.0]])  # deviations over sqrt(5 + 4)
    np.testing.assert_allclose(bo.layer_norm(x, np.array([2.0, 1, 1, 1]), np.array([5.0, 0, 0, 0]), 4.0)[0, 0], 3.0)
    np.testing.assert_allclose(bo.layer_norm(np.full((1, 3), 9.0), np.ones(3), np.arange(3.0), 1e-5), [[0, 1, 2]])
    np.testing.assert_allclose(bo.rms_norm(np.array([[3.0, 4.0]]), np.array([2.0, 1.0]), 0.0), [[6 / 12.5 ** 0.5, 4 / 12.5 ** 0.5]])
    np.testing.assert_allclose(bo.rms_norm(np.ones((1, 3)), np.ones(3), 3.0), 0.5)  # eps inside the root


def test_query_temperature_steps_up_with_the_position():
    t = bo.query_temperature([0, 2, 3, 6, 7], 0.5, 4)
    np.testing.assert_allclose(t, 1 + 0.5 * np.log([1, 1, 2, 2, 3]))
    np.testing.assert_allclose(bo.query_temperature([0, 1], 1.0, 1), 1 + np.log([2, 3]))


def test_slopes_end_at_two_to_the_minus_eight():
    np.testing.assert_allclose(bo.head_slopes(8), 2.0 ** -np.arange(1, 9))
    np.testing.assert_allclose(bo.head_slopes(1), [2.0 ** -8])
    np.testing.assert_allclose(bo.head_slopes(3), 2.0 ** (-8 * np.array([1, 2, 3]) / 3))


def test_attention_takes_the_distance_off_and_shares_keys():
    """Zero queries: what is left is the distance bias; query heads 0 and 1 read key / value head 0."""
    m = dict(heads=2, kv_heads=1, dim=2, vdim=1, scale=1.0)
    w = {"q": np.zeros((4, 3)), "q.b": np.zeros(4), "q.norm": np.ones(4), "o": np.eye(2)}
    v = np.array([1.0, 10.0, 100.0]).reshape(3, 1, 1)
    out = bo.attention(np.zeros((3, 3)), np.ones((3, 1, 2)), v, w, "", m, 1e-5)
    for head, slope in enumerate(bo.head_slopes(2)):
        e = np.exp(-slope * np.array([2.0, 1.0, 0.0]))
        np.testing.assert_allclose(out[2, head], (e / e.sum()) @ v[:, 0, 0])
    np.testing.assert_allclose(out[0], 1.0)


def test_recurrence_is_the_sum_over_decayed_outer_products():
    rs = np.random.RandomState(0)
    q, k, v, a = rs.randn(6, 3), rs.randn(6, 3), rs.randn(6, 2), rs.uniform(0.2, 1, (6, 3))
    o, s = bo.recurrence(q, k, v, a)
    for t in range(6):
        want = sum((q[t] * k[j] * np.prod(a[j + 1:t + 1], axis=0)).sum() * v[j] for j in range(t + 1))
        np.testing.assert_allclose(o[t], want)
    o2, s2 = bo.recurrence(q[4:], k[4:], v[4:], a[4:], bo.recurrence(q[:4], k[:4], v[:4], a[:4])[1])
    np.testing.assert_allclose(o2, o[4:])
    np.testing.assert_allclose(s2, s)


def test_decay_is_the_root_of_a_sigmoid():
    w = {"a1": np.array([[2.0]]), "a2": np.array([[1.0], [0.0]]), "a2.b": np.array([0.0, 3.0])}
    a = bo.key_decay(np.array([[0.5]]), w, "", dict(heads=1, dim=2, tau=4.0))
    np.testing.assert_allclose(a[0, 0], [bo.sigmoid(1.0) ** 0.25, bo.sigmoid(3.0) ** 0.25])


def test_small_forms():
    np.testing.assert_allclose(bo.squared_relu(np.array([-2.0, 3.0])), [0, 9])
    np.testing.assert_allclose(bo.soft_cap(np.array([0.0, 1e9, -1e9]), 5.0), [0, 5, -5])


def test_readers_use_the_keys_of_their_source_with_queries_of_their_own():
    cfg, _ = U.ODD
    w = U.numpy_weights(U.weights(U.ODD, seed=1))
    seq = U.tokens(cfg, 12, 3)
    taps, taps2 = [], []
    bo.forward(cfg, w, seq, taps)
    bo.forward(cfg, dict(w, **{"l1.mix.k": w["l1.mix.k"] * -1}), seq, taps2)
    assert np.array_equal(taps[0], taps2[0]) and np.abs(taps[1] - taps2[1]).max() > 1e-3
    bo.forward(cfg, dict(w, **{"l4.mix.q": w["l4.mix.q"] * -1}), seq, taps2 := [])
    assert np.array_equal(taps[3], taps2[3]) and np.abs(taps[4] - taps2[4]).max() > 1e-3


def test_configuration_is_read_in_full(pkg):
    from llm_experiments_b200.bamasun import BamasunConfig

    c = BamasunConfig.from_json(json.loads(json.dumps(U.ODD[0])))
    assert (c.vocab_size, c.width, c.eps, c.embedding_scale, c.softcap) == (37, 26, 1e-5, 2.5, 4.0)
    g, a, b, last = c.layers[0], c.layers[1], c.layers[2], c.layers[4]
    assert (g.gla.heads, g.gla.dim, g.gla.vdim, g.gla.tau, g.ff) == (3, 5, 7, 4.0, 17) and g.attention is None
    s = a.attention
    assert (s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.temp_coef, s.temp_every) == (3, 1, 6, 5, 0.5, 0.4, 7) and a.kv_from is None
    assert b.attention.temp_every == 0 and b.ff == 0 and (last.kv_from, last.attention.heads) == (1, 6)


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown mixer"), (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "feed-forward"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=0), "kv_from"), (lambda c: c["layers"][4]["mixer"].update(kv_from=4), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "other sizes"), (lambda c: c["layers"][1]["mixer"].update(heads=5, kv_heads=2), "share"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=2.5), "whole number")])
def test_configurations_that_do_not_fit_are_refused(pkg, change, match):
    from llm_experiments_b200.bamasun import BamasunConfig

    c = copy.deepcopy(U.ODD[0])
    change(c)
    with pytest.raises(ValueError, match=match):
        BamasunConfig.from_json(c)


def test_slopes_of_the_product(pkg):
    from llm_experiments_b200 import gqa

    for heads in (1, 3, 8, 40):
        np.testing.assert_allclose(gqa.geometric_slopes(heads).numpy(), bo.head_slopes(heads), rtol=1e-7)


def test_prompt_plan_in_place_points_into_the_cache(pkg):
    from llm_experiments_b200.latent import PromptPlan

    plan = PromptPlan.build([(0, 300, 0, 0), (300, 20, 2, 130)], 0, 1000, in_place=True)
    assert plan.rows() == [0, 300, 0, 0, 0, 0, 300, 20, 2000, 2000, 130, 2]


def test_argument_checks_of_the_entry_points(pkg):
    native = pkg._native
    lib, A = native.lib, 0x1000
    row = lambda H, G, **k: lib.b2kv_gqa_append(A, 256, H, G, 16, 16, A, A, 1e-5, 0.0, 0, k.get("kc", A), k.get("vc", A), None, A, 2, 8, 4,  # noqa: E731
                                                k.get("dt", 1), None, None)
    assert row(3, 2) == -1                      # heads that do not share evenly
    assert row(4, 2, vc=None) == -1             # keys without values
    assert row(16, 8) == -1                     # rows narrower than q, k and v
    assert row(4, 2, dt=9) == -3
    dec = lambda H, G, dim, path, dt: lib.b2kv_gqa_decode(A, 4096, A, A, A, 4096, None, None, A, 2, 8, 4, H, G, dim, 16, 8, 1.0, dt, path, None, 0,  # noqa: E731
                                                          None, None)
    assert dec(3, 2, 16, 0, 1) == -1 and dec(4, 2, 16, 3, 1) == -1 and dec(4, 2, 0, 0, 1) == -1
    assert dec(4, 2, 16, 2, 0) == -3            # no tensor-core form in fp32
    assert dec(4, 2, 12, 2, 1) == -3            # rows that are not whole 16-byte pieces
    assert dec(2, 1, 600, 1, 0) == -3           # wider than the CUDA-core kernel
    assert lib.b2kv_gqa_prefill_supported(128, 64, 1) == 1 and lib.b2kv_gqa_prefill_supported(136, 64, 1) == 0
    assert lib.b2kv_gqa_prefill_supported(64, 64, 0) == 0 and lib.b2kv_gqa_prefill_supported(12, 64, 1) == 0
    assert lib.b2kv_layernorm_rows(A, 8, None, A, A, None, 0, None, 0, 4, 8, 1e-5, 1, None) == -1  # nothing to write
    assert lib.b2kv_embed_rows(A, A, A, None, 1.0, 0, 8, 8, 1, None, None) == -1

    def gla(**k):
        a = native.GlaArgs(y=A, alpha=A, norm=A, state=A, out=A, segments=A, row_pos=A, ld_y=64, ld_alpha=16, ld_out=16, q_col=0, k_col=16, v_col=32,
                           g_col=48, H=2, dim=8, vdim=8, n_segments=1, max_n=4, rows=4, n_slots=1, dtype=1, path=0, q_scale=1.0, eps=1e-5)
        for name, v in k.items():
            setattr(a, name, v)
        return lib.b2kv_gla(ctypes.byref(a), None, None)

    assert gla(g_col=56) == -1 and gla(ld_alpha=8) == -1 and gla(state=None) == -1 and gla(path=3) == -1
    assert gla(segments=None, n_segments=2, n_slots=1) == -1
    assert gla(path=2, dtype=0) == -3 and gla(path=2, dim=136, ld_y=4096, ld_alpha=4096) == -3

    seg = native.Segment(out=A, ld=8, group=0, end=8, kind=native.SEG_SOFTCAP)
    lin = native.LinearArgs(x=A, w=A, ld_x=8, ld_w=8, rows=1, K=8, N=8, groups=1, n_seg=1, dtype=1, path=0, limit=0.0)
    lin.seg[0] = seg
    assert lib.b2kv_linear(ctypes.byref(lin), None, None) == -1  # a cap of zero
    lin.limit, lin.bias, lin.groups = 1.0, A, 2
    assert lib.b2kv_linear(ctypes.byref(lin), None, None) == -1  # a bias with groups
