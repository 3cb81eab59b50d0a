"""Somipel models through the framework's own decoder — prompts, portions, decoding, batches, generation, commands — against
the plain implementation in tests/somipel_ref.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import somipel_models as sm
import somipel_ref as ref
from deepj_b200 import registry
from deepj_b200.hybrid import HybridDecoder
from test_punilix_gpu import check, run

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# root mean square of the difference over the vocabulary relative to the spread of the logits: every position, nine in ten
TOL = {"f32": (4e-5, 2e-5), "bf16": (6e-2, 2.5e-2)}
SHARP = {"f32": 3.0, "bf16": 1.5}
_cache = {}


def weights(name, dtype):
    if ("w", name, dtype) not in _cache:
        _cache[("w", name, dtype)] = sm.random_weights(name, len(name), SHARP[dtype])
    return _cache[("w", name, dtype)]


def reference(name, tokens, dtype):
    key = (name, dtype, tuple(int(t) for t in tokens))
    if key not in _cache:
        _cache[key] = ref.Model(sm.CONFIGS[name], weights(name, dtype)).forward(np.asarray(tokens))
    return _cache[key]


def prompt(name, n, seed=0):
    return np.random.default_rng(seed + n).integers(0, sm.CONFIGS[name]["vocab"], size=n)


@pytest.fixture()
def decoder():
    made = []

    def make(name, dtype, max_seq=600, batch=1):
        w = weights(name, dtype)
        d = HybridDecoder(sm.parse(name, max_seq), batch=batch, dtype=dtype)
        made.append(d)
        d.load_weights(lambda n: w[n])
        return d
    yield make
    for d in made:
        assert d.stats()["device_error"] == 0
        d.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(sm.CONFIGS))
def test_portions_of_every_size(decoder, name, dtype):
    """Whole, token by token, pairs, mixtures around every path's borders; a shorter request and the same one again on the same
    buffers afterwards."""
    dec = decoder(name, dtype)
    long, short = prompt(name, 170), prompt(name, 5)
    for cuts in ([170], [1], [2], [3, 1, 2, 17, 4, 1, 64, 5], [48, 1, 47, 2, 16], [130, 1]):
        check(reference(name, long, dtype), run(dec, long, cuts), TOL[dtype])
        check(reference(name, short, dtype), run(dec, short, cuts), TOL[dtype])


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(decoder, dtype):
    dec = decoder("mixed", dtype)
    t = prompt("mixed", 420)
    check(reference("mixed", t, dtype), run(dec, t, [40] + [1] * 380), TOL[dtype])


def test_several_chunks_of_a_long_prompt(decoder):
    """More tokens than one pass carries: the chunk limit is lowered so that a prompt takes several."""
    dec = decoder("mixed", "bf16")
    dec.PREFILL_CHUNK = 64
    t, places = prompt("mixed", 300), [0, 63, 64, 65, 127, 128, 200, 299, 64]
    dec.reset()
    check(reference("mixed", t, "bf16")[places], dec.feed(t, places), TOL["bf16"])


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_a_batch_against_each_sequence_alone(decoder, dtype):
    B, n = 3, 60
    dec = decoder("mixed", dtype, batch=B)
    prompts = np.stack([prompt("mixed", n, seed=100 * b) for b in range(B)])
    dec.reset()
    dec.prefill(prompts)
    rows = [dec.logits()]
    fed = np.stack([prompt("mixed", 12, seed=7 + b) for b in range(B)])
    for t in range(12):
        dec.step(fed[:, t])
        rows.append(dec.logits())
    rows = np.stack(rows, axis=1)
    for b in range(B):
        check(reference("mixed", np.concatenate([prompts[b], fed[b]]), dtype)[n - 1:], rows[b], TOL[dtype])


def test_a_batch_beyond_the_gemv(decoder):
    """Twenty sequences: token steps go through the many-row kernels."""
    B = 20
    dec = decoder("odd", "bf16", max_seq=40, batch=B)
    prompts = np.stack([prompt("odd", 9, seed=b) for b in range(B)])
    dec.reset()
    for t in range(9):
        dec.step(prompts[:, t])
    got = dec.logits()
    check(np.stack([reference("odd", prompts[b], "bf16")[-1] for b in range(B)]), got, TOL["bf16"])


def test_greedy_and_sampled_generation(decoder):
    dec = decoder("mixed", "f32")
    p = prompt("mixed", 33)
    toks, logits = dec.generate_greedy(p, 25, keep_logits=True)
    want = reference("mixed", np.concatenate([p, toks[:-1]]), "f32")[len(p) - 1:]
    check(want, logits, TOL["f32"])
    gap = np.sort(want, axis=1)[:, -1] - np.sort(want, axis=1)[:, -2]
    assert np.all((want.argmax(1) == toks) | (gap < 1e-3))
    assert np.array_equal(dec.generate_greedy(p, 25), toks)
    a, b = dec.generate(p, 20, temperature=0.7, top_k=5, seed=3), dec.generate(p, 20, temperature=0.7, top_k=5, seed=3)
    assert np.array_equal(a, b)
    order = np.argsort(-reference("mixed", np.concatenate([p, a]), "f32")[len(p) - 1:-1], axis=1)[:, :6]
    assert all(t in row for t, row in zip(a, order))            # every draw is one of the top five (or ties with the fifth)


def test_device_feedback_equals_host_steps(decoder):
    dec = decoder("wide", "bf16")
    p = prompt("wide", 50)
    dec.reset()
    nxt = dec.prefill(p.reshape(1, -1))
    want = [int(nxt[0])]
    for _ in range(9):
        want.append(int(dec.step([want[-1]])[0]))
    dec.reset()
    dec.set_tokens(dec.prefill(p.reshape(1, -1)))
    got = []
    for _ in range(9):
        dec.step_device(1)
        got.append(int(dec.next_tokens()[0]))
    assert got == want[1:]


def test_limits_are_errors(decoder):
    dec = decoder("odd", "f32", max_seq=20)
    dec.reset()
    dec.feed(prompt("odd", 20), [])
    with pytest.raises(ValueError, match="exceeds maxSeqLen"):
        dec.feed([1], [])
    with pytest.raises(ValueError, match="recurrent state"):
        dec.set_position(5)
    dec.set_position(0)
    with pytest.raises(ValueError, match="out of range"):
        dec.feed([1, sm.CONFIGS["odd"]["vocab"]], [])


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    path = str(tmp_path_factory.mktemp("somipel"))
    sm.write_folder(path, sm.CONFIGS["mixed"], weights("mixed", "bf16"))
    return path


def test_registry_and_generate_command(folder):
    dec = registry.load_model(folder, "float32", 100)
    p = prompt("mixed", 20)
    want = dec.generate_greedy(p, 10)
    dec.close()
    out = subprocess.run([sys.executable, "-m", "deepj_b200.generate", "--model", folder, "--dtype", "f32", "--prompt", ",".join(map(str, p)), "--max-new-tokens", "10"],
                         cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert json.loads(out.stdout)["tokens"] == [int(t) for t in want]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_command(folder, tmp_path, dtype):
    """Two requests one after the other, cut differently."""
    a, b = prompt("mixed", 90), prompt("mixed", 9, seed=4)
    steps, want, lo = [], {}, 0
    for n in (50, 2, 1, 30, 7):
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": a[lo:lo + n].tolist(), "want": [0, n - 1]}], "end": ["a"] if lo + n == 90 else []})
        want[len(steps) - 1] = reference("mixed", a, "bf16")[[lo, lo + n - 1]]
        lo += n
    for i, n in ((0, 8), (8, 1)):
        steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": b[i:i + n].tolist(), "want": [n - 1]}], "end": ["b"] if i else []})
        want[len(steps) - 1] = reference("mixed", b, "bf16")[[i + n - 1]]
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "90"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert out.stdout.split("\n")[:-1] == [f"done {s['step']}" for s in steps]
    for s, w in want.items():
        check(w, np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(w.shape), TOL["f32" if dtype == "float32" else "bf16"])
