"""The Bamasun decoder end to end against the oracle (whole sequences, no cache, float64): prompts, portions, token-by-token
decoding, batches of unequal sequences, places used again, keys read from another layer, generation through the package's own
loop, the graphed step and the command line; and the row operations around its sublayers."""
import json
import pathlib
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import bamasun_oracle as bo
from tests import bamasun_util as U
from tests.kv_util import make_ctx

pytestmark = pytest.mark.gpu

ROOT = pathlib.Path(__file__).resolve().parent.parent
F32, BF = torch.float32, torch.bfloat16
CASES = [("ODD", F32), ("ODD", BF), ("TC", F32), ("TC", BF), ("WIDE", F32), ("WIDE", BF), ("ONLY_GLA", F32), ("ONLY_GLA", BF)]
_cache = {}


def oracle(name, seq):
    key = (name, tuple(seq))
    if key not in _cache:
        if name not in _cache:
            _cache[name] = U.numpy_weights(U.weights(getattr(U, name)))
        _cache[key] = bo.forward(getattr(U, name)[0], _cache[name], list(seq))
    return _cache[key]


def build_from(pkg, cfg, w, dtype, batch=1, max_tokens=512):
    from llm_experiments_b200 import registry

    ctx = make_ctx(pkg)
    ctx.config.check_device_status = True
    return registry.build_model(ctx, cfg, w, dtype, batch, max_tokens)


def build(pkg, name, dtype, batch=1, max_tokens=512):
    pair = getattr(U, name)
    return build_from(pkg, pair[0], U.weights(pair), dtype, batch, max_tokens), pair[0]


def feed(model, slot, seq, cuts):
    """Feeds seq in portions and returns the logits of every token."""
    out, at = [], 0
    for n in cuts:
        if at >= len(seq):
            break
        part = seq[at:at + n]
        out.append(model.forward([(slot, part, list(range(len(part))))]).clone())
        at += len(part)
    assert at == len(seq)
    return torch.cat(out)


@pytest.mark.parametrize("name,dtype", CASES + [("TINY", F32)])
def test_whole_prompt_and_every_layer(pkg, name, dtype):
    model, cfg = build(pkg, name, dtype)
    seq = U.tokens(cfg, 300, 1)
    taps, model.state.layer_tap = [], []
    got = feed(model, 0, seq, [300])
    want_logits = bo.forward(cfg, U.numpy_weights(U.weights(getattr(U, name))), seq, taps)
    for i, want in enumerate(taps):
        err = np.abs(model.state.layer_tap[i].double().cpu().numpy() - want).max(axis=1) / want.std()
        assert (err.max() < 2e-4) if dtype == F32 else (np.quantile(err, 0.9) < 0.15), f"layer {i}: {err.max()}"
    U.check_rows(got, want_logits, dtype, name)


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("cuts", [[1] * 200, [2, 3] * 40, [17] * 12, [40, 1, 129, 2, 28], [150] + [1] * 50, [15, 16, 17, 100, 52], [128, 72]])
def test_portions_and_decoding(pkg, name, dtype, cuts):
    """However a sequence is cut, its logits are those of the whole."""
    model, cfg = build(pkg, name, dtype)
    seq = U.tokens(cfg, 200, 2)
    U.check_rows(feed(model, 0, seq, cuts), oracle(name, seq), dtype, (name, cuts[:4]))


@pytest.mark.parametrize("name", ["TC", "WIDE"])
def test_cuts_agree_with_each_other_to_rounding(pkg, name):
    """In fp32 the logits of a position do not depend on the cut, on its neighbours in the batch or on its place."""
    model, cfg = build(pkg, name, F32, batch=3)
    seq, other = U.tokens(cfg, 150, 3), U.tokens(cfg, 90, 4)
    whole = feed(model, 0, seq, [150])
    model.forward([(1, other, [])])
    parts, at = [], 0
    for n in (2, 61, 1, 40, 46):  # in another place, beside another sequence
        got = model.forward([(1, [int(seq[at])], []), (2, seq[at:at + n], list(range(n)))])
        parts.append(got.clone())
        at += n
    assert (torch.cat(parts) - whole).abs().max() < 2e-4 * whole.abs().max()


@pytest.mark.parametrize("name,dtype", CASES)
def test_mixed_batches_match_each_sequence_alone(pkg, name, dtype):
    """Prompts, portions and single tokens of four sequences in the same steps; one ends and its place is used again."""
    model, cfg = build(pkg, name, dtype, batch=4, max_tokens=256)
    seqs = [U.tokens(cfg, n, 50 + n) for n in (230, 60, 35, 120, 77)]
    out = [[] for _ in seqs]
    at = [0] * len(seqs)
    place = {0: 3, 1: 0, 2: 2, 3: 1}
    steps = [{0: 100, 1: 1, 2: 35}, {0: 1, 1: 30, 3: 1}, {3: 90, 0: 2, 1: 1}, {0: 17, 3: 1, 1: 28}, {4: 20, 0: 109, 3: 3}, {4: 1, 0: 1, 3: 25},
             {4: 56}]
    for step in steps:
        if 4 in step and 4 not in place:  # sequence 2 ended: its place goes to the newcomer
            model.release(place[2])
            place[4] = place[2]
        entries = []
        for s, n in step.items():
            part = seqs[s][at[s]:at[s] + n]
            entries.append((place[s], part, list(range(len(part)))))
            at[s] += n
        got = model.forward(entries)
        r = 0
        for s, n in step.items():
            out[s].append(got[r:r + n].clone())
            r += n
    assert at == [len(s) for s in seqs]
    for s, seq in enumerate(seqs):
        U.check_rows(torch.cat(out[s]), oracle(name, seq), dtype, (name, s))


@pytest.mark.parametrize("name", ["TC", "WIDE", "ONLY_GLA"])
def test_a_place_used_again_carries_nothing_over(pkg, name):
    model, cfg = build(pkg, name, BF)
    a, b = U.tokens(cfg, 180, 21), U.tokens(cfg, 90, 22)
    for cuts in ([90], [1] * 90, [20, 70]):
        model.release(0)
        first = feed(model, 0, b, cuts)
        model.release(0)
        feed(model, 0, a, [50] * 4)
        model.release(0)
        assert torch.equal(feed(model, 0, b, cuts), first)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("cuts", [[420], [1] * 420, [200, 2] + [1] * 218, [130, 290]])
def test_a_far_token_is_recalled_through_attention_and_through_the_state(pkg, dtype, cuts):
    """The last token's query matches the key of one token far back (and nothing else does), or the state forgets nothing: the answer
    depends on what stood there hundreds of positions earlier, and by as much as the oracle says."""
    att = U.config([U.attention(8, 1, 16, 16, 2.0)], vocab=64, width=32)
    rec = U.config([U.gla(2, 16, 16, 16.0, 4)], vocab=64, width=32)
    for pair in (att, rec):
        cfg = pair[0]
        w = U.weights(pair, seed=5, decay_mean=12.0)
        if pair is att:  # token 61's query is token 62's key, and the opposite of its own
            w["l0.mix.k.b"] = torch.zeros_like(w["l0.mix.k.b"])
            for end in ("", ".b", ".norm"):
                k = w["l0.mix.k" + end]
                w["l0.mix.q" + end] = (k if end == ".norm" else -k).repeat(8, *[1] * (k.dim() - 1))
            w["embed"][61] = -w["embed"][62]
        model = build_from(pkg, cfg, w, dtype)
        a = [t % 60 for t in U.tokens(cfg, 420, 6)]
        a[3], a[419] = 62, 61
        b = list(a)
        b[3] = 63
        wn = U.numpy_weights(w)
        rows, want = [], []
        for seq in (a, b):
            model.release(0)
            rows.append(feed(model, 0, seq, cuts))
            want.append(bo.forward(cfg, wn, seq))
        assert torch.equal(rows[0][:3], rows[1][:3])  # nothing sees what comes later
        U.check_rows(rows[0], want[0], dtype, cfg["layers"][0]["type"])
        U.check_rows(rows[1], want[1], dtype, cfg["layers"][0]["type"])
        if dtype == F32:
            moved, expected = (rows[0] - rows[1])[3:].double().cpu().numpy(), (want[0] - want[1])[3:]
            assert np.abs(moved - expected).max() < 1e-4 * np.abs(want[0]).max()
            assert np.abs(expected[-1]).max() > 5e-3 * np.abs(want[0]).max()


@pytest.mark.parametrize("name", ["TC", "ONLY_GLA"])
def test_long_decoding_with_the_graphed_step(pkg, name):
    """Three sequences of unequal length decode 150 tokens as replayed graphs: the logits are the oracle's."""
    from llm_experiments_b200 import serving
    from llm_experiments_b200.model import GraphedDecodeStep

    model, cfg = build(pkg, name, BF, batch=3, max_tokens=400)
    model.ctx.config.check_device_status = False
    seqs = [U.tokens(cfg, n + 150, 30 + n) for n in (5, 120, 64)]
    model.forward([(s, seq[:len(seq) - 150], []) for s, seq in enumerate(seqs)])
    graphed = GraphedDecodeStep(model.ctx, model.state, step_fn=serving.decode_step)
    out = [[] for _ in seqs]
    for t in range(150):
        graphed.token_ids.buffer.copy_(torch.tensor([seq[len(seq) - 150 + t] for seq in seqs], dtype=torch.int32))
        graphed.step()
        rows = model.state.logits.buffer.clone()
        assert torch.equal(graphed.next_ids.buffer.long(), rows.argmax(dim=1))
        for s in range(3):
            out[s].append(rows[s:s + 1])
    assert model.state.lengths == [len(s) for s in seqs] and model.state.seq_lens.tolist() == model.state.lengths
    for s, seq in enumerate(seqs):
        U.check_rows(torch.cat(out[s]), oracle(name, seq)[-150:], BF, s)


@pytest.mark.parametrize("name", ["ODD", "TC", "ONLY_GLA"])
def test_greedy_generation_matches_the_oracle(pkg, name):
    """generate_text over the registry's model, fp32: the oracle's greedy tokens."""
    from llm_experiments_b200 import generate

    model, cfg = build(pkg, name, F32, max_tokens=128)
    prompt = U.tokens(cfg, 45, 40)
    w = U.numpy_weights(U.weights(getattr(U, name)))
    want = list(prompt)
    for _ in range(12):
        want.append(int(bo.forward(cfg, w, want)[-1].argmax()))
    assert generate.generate_text(model, prompt, max_tokens=12, temperature=0.0) == want
    assert generate.generate_text(model, prompt, max_tokens=12, temperature=0.0) == want  # from used caches and states
    sampled = generate.generate_text(model, prompt, max_tokens=5, temperature=0.8, top_k=5, top_p=0.9)
    assert len(sampled) == 50


def test_limits_are_refused(pkg):
    model, cfg = build(pkg, "ONLY_GLA", BF, batch=2, max_tokens=32)
    with pytest.raises(ValueError, match="full"):
        model.forward([(0, U.tokens(cfg, 33, 1), [])])
    with pytest.raises(RuntimeError, match="token id"):
        model.forward([(0, [cfg["vocab"]], [0])])
    with pytest.raises(ValueError, match="mix.a1"):
        w = U.weights(U.ONLY_GLA)
        build_from(pkg, cfg, {k: v for k, v in w.items() if k != "l0.mix.a1"}, BF)


def test_folder_trace_runner_and_command_line(pkg, tmp_path):
    """A folder written by the package, replayed step by step and used for generation by the programs in bin/."""
    from llm_experiments_b200 import checkpoint, generate, registry

    cfg = U.TC[0]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(tmp_path / "model.safetensors", U.weights(U.TC))
    seqs = {"a": U.tokens(cfg, 40, 1), "b": U.tokens(cfg, 25, 2)}
    steps = [dict(step=0, entries=[dict(id="a", tokens=seqs["a"][:30], want=[0, 29])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=seqs["a"][30:], want=[])], end=["a"]),
             dict(step=2, entries=[dict(id="b", tokens=seqs["b"], want=[24])], end=["b"])]
    for dtype in (F32, BF):
        res = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", str(dtype).split(".")[1], "--out", str(tmp_path),
                              "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=600)
        assert res.returncode == 0, res.stderr
        assert [x for x in res.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert not (tmp_path / "1.f32").exists()
        U.check_rows(torch.from_numpy(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1)), oracle("TC", seqs["a"])[[0, 29]], dtype, "a")
        U.check_rows(torch.from_numpy(np.fromfile(tmp_path / "2.f32", "<f4").reshape(1, -1)), oracle("TC", seqs["b"])[[24]], dtype, "b")
    res = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), "--model", str(tmp_path), "--dtype", "float32", "--tokens", "3,5,8",
                          "--max-new", "4"], text=True, capture_output=True, timeout=600)
    assert res.returncode == 0, res.stderr
    model = registry.load_model(make_ctx(pkg), tmp_path, F32, max_tokens=7)
    assert res.stdout.split() == [",".join(map(str, generate.generate_text(model, [3, 5, 8], 4, temperature=0.0)))]


# ---- row operations

def wrap(pkg, t):
    return (pkg.gpu.GPUBuffer1D if t.dim() == 1 else pkg.gpu.GPUBuffer2D)(buffer=t, shape=tuple(t.shape), size=t.numel())


@pytest.mark.parametrize("out_dtype", [None, F32, BF])
@pytest.mark.parametrize("rows,size,pad", [(1, 1, 0), (5, 26, 3), (70, 264, 8), (3, 4096, 0), (2, 6000, 0), (2, 20000, 0)])
@pytest.mark.parametrize("add", [True, False])
def test_layer_norm_of_fp32_rows(pkg, out_dtype, rows, size, pad, add):
    """Onto a residual or not, stored in the storage type or not, picked by index, rows far from zero."""
    if not add and out_dtype is None:
        return
    ctx = make_ctx(pkg)
    gen = torch.Generator(device="cuda").manual_seed(size)
    rnd = lambda *s: torch.randn(s, generator=gen, device="cuda")  # noqa: E731
    y, w, b = rnd(rows + 2, size + pad)[:, :size] * 3 + 50, rnd(size), rnd(size)
    x = rnd(rows, size) if add else None
    out = torch.full((rows + 1, size + pad), 7.0, dtype=out_dtype, device="cuda") if out_dtype else None
    index = torch.randperm(rows + 2, generator=torch.Generator().manual_seed(1))[:rows].int().cuda()
    want = torch.from_numpy(bo.layer_norm(y[index.long()].double().cpu().numpy(), w.double().cpu().numpy(), b.double().cpu().numpy(), 1e-3)).cuda()
    if add:
        want = want + x.double()
    pkg.gpu.batch_begin(ctx)
    pkg.gpu.layernorm_rows(ctx, wrap(pkg, y), wrap(pkg, w), wrap(pkg, b), 1e-3, x=wrap(pkg, x) if add else None,
                           output=wrap(pkg, out[:rows, :size]) if out_dtype else None, row_index=index)
    pkg.gpu.batch_commit(ctx)
    if add:
        torch.testing.assert_close(x.double(), want, rtol=2e-5, atol=2e-5)
    if out_dtype:
        tol = 2e-5 if out_dtype == F32 else 1e-2
        torch.testing.assert_close(out[:rows, :size].double(), want, rtol=tol, atol=tol)
        assert (out[rows] == 7).all() and (out[:, size:] == 7).all()


@pytest.mark.parametrize("dtype", [F32, BF])
def test_embedding_rows_are_scaled_and_copied(pkg, dtype):
    ctx = make_ctx(pkg)
    table = torch.randn((11, 34), device="cuda").to(dtype)
    ids = torch.tensor([3, 10, 0, 3], dtype=torch.int32, device="cuda")
    out, copy = torch.empty((4, 34), device="cuda"), torch.empty((4, 34), dtype=dtype, device="cuda")
    pkg.gpu.batch_begin(ctx)
    pkg.gpu.embedding_rows(ctx, wrap(pkg, table), ids, wrap(pkg, out), scale=1.7, copy=wrap(pkg, copy))
    pkg.gpu.batch_commit(ctx)
    want = table[ids.long()].float() * np.float32(1.7)
    assert torch.equal(out, want) and torch.equal(copy, want.to(dtype))
