"""The Gigezen oracle, one mechanism at a time, against worked values; the reader of its configuration, the checkpoint files and
the registry; the argument checks of the C entry points.  No GPU."""
import ctypes
import json

import numpy as np
import pytest
import torch

from oracle import gigezen_oracle as go
from tests import gigezen_util as U


def test_norms():
    x = np.array([[3.0, 4.0]])
    np.testing.assert_allclose(go.plain_norm(x, np.array([2.0, 1.0]), 0.0), [[6 / 12.5 ** 0.5, 4 / 12.5 ** 0.5]])
    np.testing.assert_allclose(go.zero_centred_norm(x, np.array([1.0, 0.0]), 0.0), [[6 / 12.5 ** 0.5, 4 / 12.5 ** 0.5]])
    np.testing.assert_allclose(go.rms_norm(np.zeros((1, 3)), 4.0), 0)
    np.testing.assert_allclose(go.rms_norm(np.ones((1, 3)), 3.0), 0.5)  # eps inside the root


def test_rotation_pairs_halves_and_depends_on_distance_only():
    x = np.zeros((2, 4))
    x[:, 0] = 1.0
    r = go.rotate_half(x, [0, 2], 100.0)
    np.testing.assert_allclose(r[0], [1, 0, 0, 0])
    np.testing.assert_allclose(r[1], [np.cos(2), 0, np.sin(2), 0], atol=1e-15)
    y = np.zeros((1, 4))
    y[0, 1] = 1.0
    np.testing.assert_allclose(go.rotate_half(y, [3], 100.0)[0], [0, np.cos(0.3), 0, np.sin(0.3)], atol=1e-15)  # 100^(-2/4) = 0.1
    rs = np.random.RandomState(0)
    a, b = rs.randn(1, 8), rs.randn(1, 8)
    dots = [float(go.rotate_half(a, [p + 5], 50.0)[0] @ go.rotate_half(b, [p], 50.0)[0]) for p in (0, 3, 100)]
    np.testing.assert_allclose(dots, dots[0])


def test_window_keeps_the_token_itself_and_size_minus_one_before():
    m = go.window_mask(5, 2)
    assert [list(np.flatnonzero(r)) for r in m] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    assert (go.window_mask(4, 1) == np.eye(4, dtype=bool)).all() and go.window_mask(3, None).sum() == 6


def test_gated_activations():
    s = lambda z: 1 / (1 + np.exp(-z))  # noqa: E731
    np.testing.assert_allclose(go.clamped_glu(np.array([5.0, -5.0]), np.array([9.0, -9.0]), 2.0),
                               [2 * s(3.404) * 3.0, -5 * s(-8.51) * -1.0])
    np.testing.assert_allclose(go.silu_glu(np.array([2.0]), np.array([3.0])), [6 * s(2.0)])


def test_router_drops_experts_of_groups_that_are_not_kept():
    w = np.eye(6)
    h = np.array([[0.0, 5.0, 4.9, 4.8, 1.0, 5.1]])  # groups (0 1) (2 3) (4 5): best members 5.0, 4.9, 5.1
    idx, s = go.route(h, w, dict(experts=6, top=3, groups=dict(count=3, keep=2)))
    assert list(idx[0]) == [5, 1, 4]  # experts 2 and 3 score higher than 4 but their group is not kept
    soft = np.exp(h[0]) / np.exp(h[0]).sum()
    np.testing.assert_allclose(s[0], soft[[5, 1, 4]])  # not renormalised
    idx, _ = go.route(h, w, dict(experts=6, top=3))
    assert list(idx[0]) == [5, 1, 2]


def test_shared_latents_use_the_readers_own_matrices_and_window():
    cfg = U.config([U.layer(2, 4, 2, 3, 5, 3, None), U.layer(1, 6, 2, 4, 5, 6, None, kv_from=0)], vocab=11, width=8)
    w = U.numpy_weights(U.weights(cfg, seed=1))
    seq = U.tokens(cfg, 12, 3)
    taps = []
    go.forward(cfg, w, seq, taps)
    other = dict(w)
    other["l1.mix.uk"] = w["l1.mix.uk"] * 1.5
    taps2 = []
    go.forward(cfg, other, seq, taps2)
    assert np.array_equal(taps[0], taps2[0]) and np.abs(taps[1] - taps2[1]).max() > 1e-3


def test_configuration_is_read_in_full(pkg):
    from llm_experiments_b200.gigezen import GigezenConfig

    c = GigezenConfig.from_json(json.loads(json.dumps(U.ODD)))
    assert (c.vocab_size, c.width, c.eps) == (37, 26, 1e-5)
    a = c.layers[1].attention
    assert (a.heads, a.dim, a.rot, a.rot_dims, a.vdim, a.kv_rank, a.window, a.scale) == (2, 9, 4, 4, 7, 10, 20, 0.4)
    assert (c.layers[1].kv_from, c.layers[1].rot_base, c.layers[1].expert_ff) == (0, 700.0, 11)
    assert (c.layers[1].router.experts, c.layers[1].router.top, c.layers[1].router.groups, c.layers[1].router.keep) == (6, 2, 3, 2)
    assert (c.layers[0].dense_ff, c.layers[0].limit, c.layers[0].router) == (17, 1.5, None)
    assert (c.layers[2].dense_ff, c.layers[2].router, c.layers[3].attention.window, c.layers[3].router.groups) == (0, None, 0, 1)
    bad = json.loads(json.dumps(U.ODD))
    bad["layers"][0]["mixer"]["kv_from"] = 2
    with pytest.raises(ValueError, match="kv_from"):
        GigezenConfig.from_json(bad)
    bad = json.loads(json.dumps(U.ODD))
    bad["layers"][0]["type"] = "something"
    with pytest.raises(ValueError, match="mixer"):
        GigezenConfig.from_json(bad)


def test_safetensors_round_trip_and_damage(pkg, tmp_path):
    from llm_experiments_b200 import checkpoint

    t = {"a": torch.arange(6, dtype=torch.int32).reshape(2, 3), "b.c": torch.randn(5).to(torch.bfloat16), "e": torch.empty(0, 3),
         "odd": torch.tensor([1, 2, 3], dtype=torch.uint8), "f": torch.randn(2, 2)}
    checkpoint.write_safetensors(tmp_path / "m", t)
    back = checkpoint.read_safetensors(tmp_path / "m")
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) and back[k].dtype == t[k].dtype for k in t)
    raw = (tmp_path / "m").read_bytes()
    (tmp_path / "short").write_bytes(raw[:-4])
    with pytest.raises(ValueError, match="data_offsets"):
        checkpoint.read_safetensors(tmp_path / "short")
    (tmp_path / "no").write_bytes(b"\xff" * 20)
    with pytest.raises(ValueError, match="safetensors"):
        checkpoint.read_safetensors(tmp_path / "no")


def test_registry_knows_the_models_and_says_so(pkg):
    from llm_experiments_b200 import registry

    assert registry.architectures() == ["Bamasun", "GPTDecoder", "Gigezen"]
    with pytest.raises(ValueError, match="Bamasun, GPTDecoder, Gigezen"):
        registry.build_model(None, {"architecture": "none"}, {})


def test_prompt_plan_counts_blocks_and_visible_rows(pkg):
    from llm_experiments_b200.latent import PromptPlan

    plan = PromptPlan.build([(0, 300, 0, 0), (300, 20, 2, 130)], 100, 1000)
    assert plan.n_blocks == 3 and plan.kv_rows == 300 + 119
    assert plan.portions == [(0, 300, 0, 300, 0), (300, 20, 2031, 119, 300)]
    assert plan.rows() == [0, 300, 0, 0, 0, 0, 300, 20, 300, 2031, 99, 2]


def test_entry_points_check_their_arguments_before_any_launch(pkg):
    native = pkg._native
    lib, A = native.lib, 0x1000
    assert lib.b2kv_embed_rows(None, A, A, None, 1.0, 1, 8, 8, 0, None, None) == -1
    assert lib.b2kv_rmsnorm(A, 8, None, A, 1.0, A, 4, 1, 8, 1e-6, 0, None) == -1  # output pitch below the row
    args = native.LinearArgs(x=A, w=A, ld_x=8, ld_w=8, rows=1, K=8, N=8, groups=1, n_seg=1, dtype=1)
    args.seg[0] = native.Segment(out=A, ld=8, end=6, kind=0)
    assert lib.b2kv_linear(ctypes.byref(args), None, None) == -1  # the segments do not cover the columns
    args.seg[0] = native.Segment(out=A, ld=8, end=8, kind=9)
    assert lib.b2kv_linear(ctypes.byref(args), None, None) == -1
    args.seg[0], args.path, args.dtype = native.Segment(out=A, ld=8, end=8, kind=0), 2, 0
    assert lib.b2kv_linear(ctypes.byref(args), None, None) == -3  # fp32 has no tensor-core form
    assert lib.b2kv_latent_append(A, 8, 1, 4, 4, 3, A, 0, 4, A, 1e-6, None, None, None, A, 1, 8, 1, 0, None, None) == -1
    assert lib.b2kv_latent_decode(A, A, 4, 4, A, A, A, None, A, 1, 8, 1, 1, 8, 4, 0, 8, 1.0, 0, 0, None, 0, None, None) == -1
    assert lib.b2kv_latent_decode(A, A, 8, 4, A, A, A, None, A, 1, 8, 1, 1, 8, 4, 0, 8, 1.0, 0, 2, None, 0, None, None) == -3
    assert lib.b2kv_latent_prefill_supported(128, 64, 128, 512, 1) == 1 and lib.b2kv_latent_prefill_supported(132, 64, 128, 512, 1) == 0
    assert lib.b2kv_latent_prefill_supported(64, 32, 64, 64, 0) == 0
    assert lib.b2kv_route(A, 4, 1, 4, 3, 1, 1, A, A, A, None) == -1  # groups do not divide the experts
    assert lib.b2kv_route(A, 8, 1, 8, 4, 1, 3, A, A, A, None) == -1  # more choices than the kept groups have experts
    assert lib.b2kv_moe_plan(A, A, 0, 8, 1, A, A, A, 8, A, 8, 8, 1, None) == -1
    assert lib.b2kv_moe_combine(A, 8, A, 4, A, A, 1, 1, 8, 1, None) == -1
