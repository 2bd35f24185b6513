"""Whole Tobovik models of several sizes through the registry's model, session and engine against the plain
restatement: prompts, portions, single tokens, sequences one after another, greedy generation, the trace
runner as a process."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle.tobovik_oracle import TobovikOracle
from petotar_util import Tensors, row_errors, write_folder
from tobovik_util import CONFIGS, weights

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 5e-5, "bfloat16": 0.1}                 # worst row
MEDIAN = {"float32": 1e-5, "bfloat16": 2.5e-2}
_cache = {}


def reference(name, length=150, seed=3):
    """(config, weights, tokens, logits of the whole sequence), computed once per configuration."""
    key = (name, length, seed)
    if key not in _cache:
        cfg, rank = CONFIGS[name]
        w = weights(cfg, rank, seed=1)
        tokens = np.random.default_rng(seed).integers(0, cfg["vocab"], length)
        _cache[key] = (cfg, w, tokens, TobovikOracle(cfg, w).step(tokens))
    return _cache[key]


def model(name, dtype, **kw):
    from meganeura_b200.registry import model_class
    cfg, w, _, _ = reference(name)
    args = dict(dtype=dtype, max_rows=64, max_picked=32, max_tokens=400)
    args.update(kw)
    return model_class(cfg).from_tensors(cfg, Tensors(w), **args)


def engine(name, dtype, greedy=False, **kw):
    from meganeura_b200.engine import Engine
    return Engine(model(name, dtype, **kw), greedy=greedy)


def feed_cut(e, tokens, sizes):
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[i % len(sizes)], len(tokens) - at)
        out.append(e.feed(tokens[at:at + n], range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_logits_do_not_depend_on_the_cut(name, dtype):
    """One step per prompt, single tokens, portions down to two tokens; all in one session, one sequence after
    another (the cache of the one before is still in memory)."""
    _, _, tokens, want = reference(name)
    e = engine(name, dtype, max_rows=150, max_picked=150)
    worst = {}
    for label, sizes in (("whole", [150]), ("single", [1]), ("two", [2]), ("cuts", [37, 2, 3, 64, 1, 16, 9, 8]), ("mostly", [118] + [1] * 32)):
        got = feed_cut(e, tokens, sizes)
        e.end()
        errors = row_errors(got, want)
        worst[label] = errors.max()
        assert np.median(errors) <= MEDIAN[dtype], label
    assert max(worst.values()) <= TOL[dtype], worst


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_longer_than_a_step_and_few_picks(dtype):
    _, _, tokens, want = reference("shared")
    e = engine("shared", dtype, max_rows=70, max_picked=5)
    places = [149, 0, 69, 70, 69, 139, 140, 3, 2, 1, 4, 5, 6, 100]
    got = e.feed(tokens, places)
    assert row_errors(got, want[places]).max() <= TOL[dtype]
    assert (got[2] == got[4]).all()


@pytest.mark.parametrize("name", ["odd", "shared"])
def test_unfused_session_gives_the_same_logits(name):
    from meganeura_b200 import ops
    _, _, tokens, want = reference(name)
    ops.set_option("session.fuse_mixer", 0)
    try:
        e = engine(name, "float32")
    finally:
        ops.set_option("session.fuse_mixer", 1)
    assert row_errors(feed_cut(e, tokens[:70], [40, 1, 1, 28]), want[:70]).max() <= TOL["float32"]


@pytest.mark.parametrize("name", ["odd", "shared"])
def test_layer_outputs(name):
    """The residual stream after every layer; layers without weights of their own have no tensors."""
    from meganeura_b200.engine import Engine
    cfg, w, tokens, _ = reference(name)
    m = model(name, "float32", max_rows=50, max_tokens=60, tap_layers=True)
    assert sorted(n for n, _, _ in m.parameters()) == sorted(w)
    Engine(m, greedy=False).feed(tokens[:50], [49])
    o = TobovikOracle(cfg, w)
    o.step(tokens[:50])
    for i, res in enumerate(o.residuals):
        got = m.session.read_output_by_index(1 + i, res.size).reshape(res.shape)
        assert np.abs(got - res).max() <= 5e-5 * np.abs(res).max(), f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sequences_after_one_another_equal_each_alone(dtype):
    e = engine("shared", dtype)
    cfg, w, _, _ = reference("shared")
    rng = np.random.default_rng(9)            # the first tokens' outputs turn around where q . k is near zero: not with these
    for length in (1, 33, 2, 130, 64):
        tokens = rng.integers(0, cfg["vocab"], length)
        got = feed_cut(e, tokens, [29, 1, 2])
        e.end()
        assert row_errors(got[-8:], TobovikOracle(cfg, w).step(tokens)[-8:]).max() <= TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decode_to_the_last_position(dtype):
    """Single tokens (captured graph) up to the session's limit."""
    cfg, w, tokens, want = reference("shared", length=330, seed=12)
    e = engine("shared", dtype, max_rows=16, max_tokens=330)
    got = [e.feed(tokens[:16], range(16))] + [e.feed([t], [0]) for t in tokens[16:]]
    assert e._captured
    assert row_errors(np.concatenate(got), want).max() <= TOL[dtype]
    with pytest.raises(ValueError):
        e.feed([0], [])


@pytest.mark.parametrize("name", ["odd", "wide", "shared"])
def test_greedy_generation(name):
    """generate(): prompt in portions, then the device picks and feeds its own tokens.  The oracle follows the picked
    tokens; every pick must be its maximum up to rounding, twice in one engine."""
    cfg, w, tokens, _ = reference(name)
    e = engine(name, "float32", greedy=True, max_rows=20)
    for prompt in (tokens[:47], tokens[50:53]):
        new = e.generate(prompt, 40)
        e.end()
        logits = TobovikOracle(cfg, w).step(np.concatenate([prompt, new[:-1]]))[len(prompt) - 1:]
        gap = logits.max(axis=1) - logits[np.arange(40), new]
        assert (gap <= 1e-4 * logits.std()).all()
    assert len(set(new.tolist())) > 1


def test_wrong_tensor_shape_is_refused():
    from meganeura_b200.registry import model_class
    cfg, w, _, _ = reference("odd")
    for name in ("l1.mix.a2", "l0.mix.left.k.b", "head"):
        with pytest.raises(ValueError):
            model_class(cfg).from_tensors(cfg, Tensors({**w, name: w[name][:-1]}), max_rows=8, max_tokens=16)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_process(tmp_path, dtype):
    cfg, w, tokens, want = reference("shared")
    write_folder(str(tmp_path), cfg, w)
    out = tmp_path / "out"
    out.mkdir()
    steps, expect, n = [], {}, 0
    for rid in ("a", "b"):
        at = 0
        for size in (70, 2, 1, 1, 30):
            places = [0, size - 1] if size > 1 else [0]
            if size == 30:
                places = []
            steps.append({"step": n, "entries": [{"id": rid, "tokens": tokens[at:at + size].tolist(), "want": places}], "end": [rid] if size == 30 else []})
            if places:
                expect[n] = want[[at + p for p in places]]
            at, n = at + size, n + 1
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "110"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=120)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(n)]
    assert sorted(os.listdir(out)) == sorted(f"{i}.f32" for i in expect)
    for i, rows in expect.items():
        got = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(rows.shape)
        assert row_errors(got, rows).max() <= TOL[dtype]


def test_command_line_generates(tmp_path):
    cfg, w, tokens, _ = reference("odd")
    write_folder(str(tmp_path), cfg, w)
    p = subprocess.run([sys.executable, "-m", "meganeura_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, tokens[:9])),
                        "--max-new", "5", "--dtype", "float32"], capture_output=True, text=True, cwd=ROOT, timeout=120)
    assert p.returncode == 0, p.stderr
    logits = TobovikOracle(cfg, w).step(tokens[:9])[-1]
    assert int(p.stdout.split(",")[0]) == int(logits.argmax())
