"""Punilix models through the framework's own decoder — prompts, portions, decoding, generation, commands — against the
plain implementation in tests/punilix_ref.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import punilix_models as pm
import punilix_ref as ref
from deepj_b200 import registry
from deepj_b200.decoder import DecoderConfig, Q8Decoder
from deepj_b200.hybrid import HybridConfig, HybridDecoder

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# logits: root mean square of the difference over the vocabulary, relative to the spread of the logits — every position, and
# nine positions in ten.  Rounding every activation of the plain implementation to bf16 gives about the bf16 bounds (its
# queries are less sharp for that reason: a near tie of two scores costs per cents); a key, a state or an expert that is
# wrong moves a position by tens of per cents.
TOL = {"f32": (4e-5, 2e-5), "bf16": (4e-2, 1.5e-2)}
SHARP = {"f32": 5.0, "bf16": 1.5}
_cache = {}


def reference(name, tokens, dtype):
    """Reference logits [T, vocab] (computed once per prompt)."""
    key = (name, dtype, tuple(int(t) for t in tokens))
    if key not in _cache:
        _cache[key] = ref.Model(pm.CONFIGS[name], weights(name, dtype)).forward(np.asarray(tokens))
    return _cache[key]


def weights(name, dtype):
    if ("w", name, dtype) not in _cache:
        _cache[("w", name, dtype)] = pm.random_weights(pm.CONFIGS[name], len(name), SHARP[dtype])
    return _cache[("w", name, dtype)]


@pytest.fixture()
def decoder():
    made = []

    def make(name, dtype, max_seq=600, batch=1):
        w = weights(name, dtype)
        d = HybridDecoder(HybridConfig.parse(pm.CONFIGS[name], max_seq, lambda n: w[n].shape[0] if n in w else None), batch=batch, dtype=dtype)
        made.append(d)
        d.load_weights(lambda n: w[n])
        return d
    yield make
    for d in made:
        assert d.stats()["device_error"] == 0
        d.close()


def prompt(name, n, seed=0):
    return np.random.default_rng(seed + n).integers(0, pm.CONFIGS[name]["vocab"], size=n)


def check(want, got, tol):
    assert np.all(np.isfinite(got))
    d = got - want
    err = np.sqrt((d - d.mean(-1, keepdims=True)).__pow__(2).mean(-1)) / want.std()
    assert err.max() <= tol[0], (float(err.max()), int(err.argmax()))
    assert np.sort(err)[max(0, int(0.9 * len(err)) - 1)] <= tol[1], np.sort(err)[::-1][:20]


def run(dec, tokens, cuts):
    """Feed `tokens` in portions of the sizes `cuts` (cycled), all logits."""
    dec.reset()
    rows, lo, i = [], 0, 0
    while lo < len(tokens):
        n = min(cuts[i % len(cuts)], len(tokens) - lo)
        rows.append(dec.feed(tokens[lo:lo + n], list(range(n))))
        lo, i = lo + n, i + 1
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_portions_of_every_size(decoder, name, dtype):
    """Whole, token by token, pairs, and mixtures around every path's borders (one token, GEMV passes, many-row kernels,
    expanded attention); a shorter request and the same one again on the same buffers afterwards."""
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
    t = prompt("mixed", 300)
    dec.reset()
    got = dec.feed(t, [0, 63, 64, 65, 127, 128, 200, 299, 64])
    check(reference("mixed", t, "bf16")[[0, 63, 64, 65, 127, 128, 200, 299, 64]], got, TOL["bf16"])


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
    dec = decoder("mixed", "bf16")
    p = prompt("mixed", 50)
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
    p = prompt("odd", 20)
    dec.reset()
    dec.feed(p, [])
    with pytest.raises(ValueError, match="exceeds maxSeqLen"):
        dec.feed([1], [])
    with pytest.raises(ValueError, match="recurrent state"):
        dec.set_position(5)
    dec.set_position(0)
    with pytest.raises(ValueError, match="out of range"):
        dec.feed([1, pm.CONFIGS["odd"]["vocab"]], [])
    with pytest.raises(ValueError, match="outside the tokens"):
        dec.feed([1, 2], [2])
    with pytest.raises(ValueError, match="dtype"):
        HybridDecoder(dec.cfg, dtype="f16", id_base=3 << 24)


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    path = str(tmp_path_factory.mktemp("punilix"))
    pm.write_folder(path, pm.CONFIGS["mixed"], weights("mixed", "bf16"))
    return path


def test_registry_generate_command(folder):
    dec = registry.load_model(folder, "float32", 100)
    p = prompt("mixed", 20)
    want = dec.generate_greedy(p, 10)
    dec.close()
    out = subprocess.run([sys.executable, "-m", "deepj_b200.generate", "--model", folder, "--dtype", "f32", "--prompt", ",".join(map(str, p)), "--max-new-tokens", "10"],
                         cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert json.loads(out.stdout)["tokens"] == [int(t) for t in want]
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(folder, "q8")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_command(folder, tmp_path, dtype):
    """Two requests one after the other, cut differently; files appear exactly where logits are wanted."""
    a, b = prompt("mixed", 90), prompt("mixed", 9, seed=4)
    steps, want, lo = [], {}, 0
    for n in (50, 2, 1, 30, 7):
        places = [0, n - 1] if n > 2 else []
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": a[lo:lo + n].tolist(), "want": places}], "end": ["a"] if lo + n == 90 else []})
        want[len(steps) - 1] = [reference("mixed", a, "bf16")[lo + i] for i in places]
        lo += n
    for i, n in ((0, 8), (8, 1)):
        steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": b[i:i + n].tolist(), "want": [n - 1]}], "end": ["b"] if i else []})
        want[len(steps) - 1] = [reference("mixed", b, "bf16")[i + n - 1]]
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "90"]
    p = subprocess.Popen(cmd, stdin=subprocess.PIPE, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True)
    for s in steps:
        p.stdin.write(json.dumps(s) + "\n")
        p.stdin.flush()
        line = p.stdout.readline()
        assert line.strip() == f"done {s['step']}", (line, p.poll(), p.stderr.read() if p.poll() is not None else "")
        path = tmp_path / f"{s['step']}.f32"
        assert path.exists() == bool(want[s["step"]])
        if want[s["step"]]:
            got = np.fromfile(path, dtype="<f4").reshape(len(want[s["step"]]), -1)
            check(np.stack(want[s["step"]]), got, TOL["f32" if dtype == "float32" else "bf16"])
    p.stdin.close()
    assert p.wait(timeout=60) == 0


def test_feed_drives_the_q8_families_too():
    """The same entry point on a Llama-shaped model: a chunked prompt with wanted places equals token-by-token steps."""
    d = Q8Decoder(DecoderConfig("llama", 96, 80, 64, 2, 2, 96), id_base=4 << 24)
    d.load_synthetic(3, 0.1)
    t = np.random.default_rng(0).integers(0, 96, size=50)
    d.reset()
    steps = np.concatenate([d.feed([x], [0]) for x in t])
    d.reset()
    chunk = d.feed(t, [0, 20, 49])
    assert np.abs(steps[[0, 20, 49]] - chunk).max() <= 2e-3 * (steps.max() - steps.min())
    d.close()
