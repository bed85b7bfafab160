"""The Gigezen decoder end to end against the oracle (whole sequences, no cache, float64): prompts, portions, token-by-token
decoding, batches of unequal sequences, places used again, shared latents with a wider window, generation through the
package's own loop, the graphed step and the command line."""
import json
import pathlib
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import gigezen_oracle as go
from tests import gigezen_util as U
from tests.kv_util import make_ctx

pytestmark = pytest.mark.gpu

ROOT = pathlib.Path(__file__).resolve().parent.parent
F32, BF = torch.float32, torch.bfloat16
CASES = [("ODD", F32), ("ODD", BF), ("TC", F32), ("TC", BF), ("WIDE", BF)]
_cache = {}


def oracle(name, seq):
    key = (name, tuple(seq))
    if key not in _cache:
        cfg = getattr(U, name)
        if name not in _cache:
            _cache[name] = U.numpy_weights(U.weights(cfg))
        _cache[key] = go.forward(cfg, _cache[name], list(seq))
    return _cache[key]


def build(pkg, name, dtype, batch=1, max_tokens=512):
    from llm_experiments_b200 import registry

    ctx = make_ctx(pkg)
    ctx.config.check_device_status = True
    cfg = getattr(U, name)
    return registry.build_model(ctx, cfg, U.weights(cfg), dtype, batch, max_tokens), cfg


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


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompt_and_every_layer(pkg, name, dtype):
    model, cfg = build(pkg, name, dtype)
    seq = U.tokens(cfg, 300, 1)
    taps, model.state.layer_tap = [], []
    got = feed(model, 0, seq, [300])
    go_logits = go.forward(cfg, U.numpy_weights(U.weights(cfg)), seq, taps)
    for i, want in enumerate(taps):
        err = np.abs(model.state.layer_tap[i].double().cpu().numpy() - want).max(axis=1) / want.std()
        assert (err.max() < 1e-4) if dtype == F32 else (np.quantile(err, 0.9) < 0.15), f"layer {i}"
    U.check_rows(got, go_logits, dtype, name)


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("cuts", [[1] * 200, [2, 3] * 40, [17] * 12, [40, 1, 129, 2, 28], [150] + [1] * 50, [15, 16, 17, 100, 52]])
def test_portions_and_decoding(pkg, name, dtype, cuts):
    """However a sequence is cut, its logits are those of the whole."""
    model, cfg = build(pkg, name, dtype)
    seq = U.tokens(cfg, 200, 2)
    U.check_rows(feed(model, 0, seq, cuts), oracle(name, seq), dtype, (name, cuts[:4]))


@pytest.mark.parametrize("name", ["ODD", "TC"])
def test_window_edges_in_prompts_and_in_decoding(pkg, name):
    """Two sequences that differ in one token: rows that cannot reach it (stacked windows taken into account) agree to the bit
    pattern of rounding, the first row that can does not; the changed token is met by a prompt, by a portion and by decoding."""
    cfg = getattr(U, name)
    one = dict(cfg, layers=[cfg["layers"][0]])  # a single layer: its window is the reach
    W = one["layers"][0]["mixer"]["mask"]["size"]
    from llm_experiments_b200 import registry

    ctx = make_ctx(pkg)
    w = U.weights(one, seed=4)
    w["l0.mix.uv"] = w["l0.mix.uv"] * 8
    model = registry.build_model(ctx, one, w, F32, 1, 256)
    a = U.tokens(one, 3 * W + 20, 5)
    b = list(a)
    b[10] = (a[10] + 1) % one["vocab"]
    for cuts in ([len(a)], [11 + W // 2] + [1] * len(a), [9, 2] + [W] * len(a), [1] * len(a)):
        rows = []
        for seq in (a, b):
            model.release(0)
            rows.append(feed(model, 0, seq, cuts))
        diff = (rows[0] - rows[1]).abs().amax(dim=1).cpu()
        assert (diff[:10] == 0).all() and diff[10 + W - 1] > 1e-4, cuts
        assert diff[10 + W:].max() < 1e-4 * rows[0].abs().max().item(), cuts


@pytest.mark.parametrize("name,dtype", CASES)
def test_mixed_batches_match_each_sequence_alone(pkg, name, dtype):
    """Prompts, portions and single tokens of four sequences in the same steps; one ends and its place is used again."""
    model, cfg = build(pkg, name, dtype, batch=4, max_tokens=256)
    seqs = [U.tokens(cfg, n, 10 + n) for n in (230, 60, 35, 120, 77)]
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


def test_a_place_used_again_carries_nothing_over(pkg):
    model, cfg = build(pkg, "TC", BF)
    a, b = U.tokens(cfg, 180, 21), U.tokens(cfg, 90, 22)
    first = feed(model, 0, b, [90])
    model.release(0)
    feed(model, 0, a, [50] * 4)
    model.release(0)
    assert torch.equal(feed(model, 0, b, [90]), first)


def test_long_decoding_with_the_graphed_step(pkg):
    """Three sequences of unequal length decode 150 tokens as replayed graphs: the logits are the oracle's."""
    from llm_experiments_b200 import gigezen
    from llm_experiments_b200.model import GraphedDecodeStep

    model, cfg = build(pkg, "TC", BF, batch=3, max_tokens=400)
    model.ctx.config.check_device_status = False
    seqs = [U.tokens(cfg, n + 150, 30 + n) for n in (5, 120, 64)]
    model.forward([(s, seq[:len(seq) - 150], []) for s, seq in enumerate(seqs)])
    graphed = GraphedDecodeStep(model.ctx, model.state, step_fn=gigezen.decode_step)
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
        U.check_rows(torch.cat(out[s]), oracle("TC", seq)[-150:], BF, s)


@pytest.mark.parametrize("name", ["ODD", "TC"])
def test_greedy_generation_matches_the_oracle(pkg, name):
    """generate_text over the registry's model, fp32: the oracle's greedy tokens."""
    from llm_experiments_b200 import generate

    model, cfg = build(pkg, name, F32, max_tokens=128)
    prompt = U.tokens(cfg, 45, 40)
    w = U.numpy_weights(U.weights(cfg))
    want = list(prompt)
    for _ in range(12):
        want.append(int(go.forward(cfg, w, want)[-1].argmax()))
    assert generate.generate_text(model, prompt, max_tokens=12, temperature=0.0) == want
    assert generate.generate_text(model, prompt, max_tokens=12, temperature=0.0) == want  # from a used cache
    sampled = generate.generate_text(model, prompt, max_tokens=5, temperature=0.8, top_k=5, top_p=0.9)
    assert len(sampled) == 50


def test_limits_are_refused(pkg):
    model, cfg = build(pkg, "TC", BF, batch=2, max_tokens=32)
    with pytest.raises(ValueError, match="full"):
        model.forward([(0, U.tokens(cfg, 33, 1), [])])
    with pytest.raises(ValueError, match="twice"):
        model.forward([(0, [1], []), (0, [2], [])])
    model.ctx.config.check_device_status = True
    with pytest.raises(RuntimeError, match="token id"):
        model.forward([(0, [cfg["vocab"]], [0])])


def test_folder_trace_runner_and_command_line(pkg, tmp_path):
    """A folder written by the package, replayed step by step and used for generation by the programs in bin/."""
    from llm_experiments_b200 import checkpoint, generate, registry

    cfg = U.ODD
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(tmp_path / "model.safetensors", U.weights(cfg))
    seqs = {"a": U.tokens(cfg, 40, 1), "b": U.tokens(cfg, 25, 2)}
    steps = [dict(step=0, entries=[dict(id="a", tokens=seqs["a"][:30], want=[0, 29])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=seqs["a"][30:], want=[])], end=["a"]),
             dict(step=2, entries=[dict(id="b", tokens=seqs["b"], want=[24])], end=["b"])]
    res = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=600)
    assert res.returncode == 0, res.stderr
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "1.f32").exists()
    U.check_rows(torch.from_numpy(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1)), oracle("ODD", seqs["a"])[[0, 29]], F32, "a")
    U.check_rows(torch.from_numpy(np.fromfile(tmp_path / "2.f32", "<f4").reshape(1, -1)), oracle("ODD", seqs["b"])[[24]], F32, "b")
    res = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), "--model", str(tmp_path), "--dtype", "float32", "--tokens", "3,5,8",
                          "--max-new", "4"], text=True, capture_output=True, timeout=600)
    assert res.returncode == 0, res.stderr
    model = registry.load_model(make_ctx(pkg), tmp_path, F32, max_tokens=7)
    assert res.stdout.split() == [",".join(map(str, generate.generate_text(model, [3, 5, 8], 4, temperature=0.0)))]
