"""Host side of the layer-list models — configuration, checkpoint, registry, trace replay — and the reference itself."""
import json
import os

import numpy as np
import pytest

import punilix_models as pm
import punilix_ref as ref
from deepj_b200 import build, checkpoint, compute_graph as cg, registry, trace
from deepj_b200.decoder import scaled_rope_tables
from deepj_b200.hybrid import HybridConfig, pad8

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_reference_is_the_same_however_a_prompt_is_cut(name):
    c = pm.CONFIGS[name]
    m = ref.Model(c, pm.random_weights(c, 1))
    t = np.random.default_rng(2).integers(0, c["vocab"], size=23)
    whole = m.forward(t)
    m.reset()
    cut = np.concatenate([m.forward(t[lo:hi]) for lo, hi in ((0, 1), (1, 3), (3, 20), (20, 23))])
    assert np.allclose(whole, cut, atol=1e-10)
    m.reset()
    changed = t.copy()
    changed[15] = (t[15] + 1) % c["vocab"]
    other = m.forward(changed)
    assert np.allclose(whole[:15], other[:15]) and np.abs(whole[16:] - other[16:]).max() > 1e-3      # causal, and it remembers


def test_delta_rule_against_its_matrix_form():
    """S ← (diag(w) − (a ⊙ u) uᵀ) S + k vᵀ."""
    rng = np.random.default_rng(0)
    S, r, k, v = rng.standard_normal((5, 5)), *(rng.standard_normal(5) for _ in range(3))
    w, a = rng.random(5), rng.random(5)
    u = k / np.sqrt(k @ k + 1e-6)
    S2, o = ref.delta_step(S, r, k, v, w, a)
    assert np.allclose(S2, (np.diag(w) - np.outer(a * u, u)) @ S + np.outer(k, v)) and np.allclose(o, r @ S2)


@pytest.mark.parametrize("dims,base,scaling", [(16, 10000.0, None), (64, 1e6, pm.YARN2), (8, 500.0, pm.YARN), (2, 100.0, pm.YARN)])
def test_rotary_tables(dims, base, scaling):
    x = np.random.default_rng(dims).standard_normal((40, 3, dims))
    want = ref.rotate_interleaved(x, np.arange(40), dims, base, scaling)
    cos, sin = scaled_rope_tables(dims, 40, base, scaling)
    u, v = x[..., 0::2], x[..., 1::2]
    assert np.allclose(want[..., 0::2], u * cos[:, None] - v * sin[:, None], atol=1e-5)
    assert np.allclose(want[..., 1::2], v * cos[:, None] + u * sin[:, None], atol=1e-5)
    if scaling is not None:              # rotations keep lengths up to the gain
        assert np.allclose(np.linalg.norm(want, axis=-1) / np.linalg.norm(x, axis=-1), 0.1 * np.log(scaling["factor"]) + 1)


def test_yarn_blends_between_the_two_frequencies():
    f0, _ = ref.rotary_frequencies(64, 1e6)
    f, _ = ref.rotary_frequencies(64, 1e6, pm.YARN2)
    assert f[0] == f0[0] and np.isclose(f[-1], f0[-1] / pm.YARN2["factor"]) and np.all(np.diff(f / f0) <= 1e-12)


def test_configuration_rules():
    good = pm.CONFIGS["mixed"]
    cfg = HybridConfig.parse(good, 64, lambda n: 11)
    assert len(cfg.layers) == 5 and cfg.logit_softcap == 12.0 and HybridConfig.parse(pm.CONFIGS["odd"], 64, lambda n: 3).logit_softcap == 0.0
    assert cfg.tensors()["l2.mix.w1"] == (11, 144) and cfg.tensors()["l3.mlp.table"] == (211, 1) and "l1.mlp.gate" not in cfg.tensors()

    def broken(change):
        c = json.loads(json.dumps(good))
        change(c)
        with pytest.raises((ValueError, KeyError)):
            HybridConfig.parse(c, 64, lambda n: 11)
    broken(lambda c: c["layers"][0].update(type="mystery"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="mystery"))
    broken(lambda c: c["norm"].update(groups=5))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4))
    broken(lambda c: c["layers"][1]["mixer"].update(heads=0))
    broken(lambda c: c["layers"][2]["mlp"]["router"].update(top=9))
    broken(lambda c: c.pop("width"))
    with pytest.raises(ValueError):
        HybridConfig.parse(good, 0, lambda n: 11)
    with pytest.raises(ValueError):
        HybridConfig.parse(good, 64, lambda n: None)            # no weights to take the decay rank from


def test_safetensors_round_trip_and_damage(tmp_path):
    rng = np.random.default_rng(0)
    tensors = {"a.w": pm.bf16(rng.standard_normal((3, 5))), "t": rng.integers(0, 9, size=(4, 2)).astype(np.int32), "v": pm.bf16(rng.standard_normal(7))}
    path = str(tmp_path / "m.safetensors")
    checkpoint.write_safetensors(path, tensors)
    f = checkpoint.SafetensorsFile(path)
    for n, a in tensors.items():
        assert f.shape(n) == a.shape and np.array_equal(f.get(n), a)
    assert f.get("t").dtype == np.int32
    with pytest.raises(IOError):
        f.get("missing")
    blob = open(path, "rb").read()
    for bad in (b"", blob[:5], blob[:20], blob[:-3]):
        p = str(tmp_path / "bad")
        open(p, "wb").write(bad)
        with pytest.raises((IOError, ValueError)):
            g = checkpoint.SafetensorsFile(p)
            for n in tensors:
                g.get(n)


def test_registry_knows_its_architectures(tmp_path):
    def write(rec):
        with open(tmp_path / "config.json", "w") as f:
            json.dump(rec, f)
        return str(tmp_path)
    assert registry.read_config(write(pm.CONFIGS["odd"]))["architecture"] == "Punilix"
    assert registry.dtypes_of("Punilix") == ("bf16", "f32") and registry.dtypes_of("llama") == ("q8",)
    with pytest.raises(ValueError):
        registry.read_config(write({"architecture": "unheard-of"}))
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(write({"architecture": "gpt"}), "float32")
    # a number format that no kernel of the family has ends the trace command with code 3, before anything is loaded
    assert trace.main(["--model", write({"architecture": "llama"}), "--dtype", "float32", "--out", str(tmp_path)]) == 3


class FakeDecoder:
    def __init__(self):
        self.calls = []

    def reset(self):
        self.calls.append("reset")

    def feed(self, tokens, want):
        self.calls.append(list(tokens))
        return np.array([[float(tokens[i]), 0.5] for i in want], dtype=np.float32).reshape(len(want), 2)


def test_trace_replay_order_and_files(tmp_path):
    lines = [json.dumps(s) for s in (
        {"step": 0, "entries": [{"id": "x", "tokens": [4, 5], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "x", "tokens": [6], "want": []}], "end": ["x"]},
        {"step": 2, "entries": [{"id": "y", "tokens": [7, 8, 9], "want": [2, 0]}], "end": ["y"]})]
    dec, done = FakeDecoder(), []
    trace.replay(dec, lines, str(tmp_path), done.append)
    assert done == [0, 1, 2] and sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32"]
    assert np.fromfile(tmp_path / "2.f32", dtype="<f4").tolist() == [9.0, 0.5, 7.0, 0.5]
    assert [c for c in dec.calls if c != "reset"] == [[4, 5], [6], [7, 8, 9]] and dec.calls[0] == "reset" and dec.calls[dec.calls.index([7, 8, 9]) - 1] == "reset"
    with pytest.raises(ValueError):
        trace.replay(FakeDecoder(), [lines[0], lines[2]], str(tmp_path), done.append)


def test_partial_library_holds_what_the_family_needs():
    """A library with only the bf16 parts loads, exports the core, and leaves the other parts out."""
    import ctypes
    lib = ctypes.CDLL(build.build_cuda(parts=("bf16",)))
    for name in ("deepj_cuda_flush_ops", "deepj_cuda_bf16_alloc", "deepj_cuda_bf16_store", "deepj_cuda_latent_alloc"):
        assert hasattr(lib, name)
    assert not hasattr(lib, "deepj_cuda_tp_create")


def test_op_strides_of_the_bf16_ops():
    for code in (cg.OP_BF16_LINEAR, cg.OP_BF16_BLOCK_LINEAR, cg.OP_DELTA_RULE, cg.OP_ATTN_LATENT, cg.OP_TABLE_EXPERTS, cg.OP_ATTN_LATENT_CHUNK):
        stride, slots = cg.OP_METADATA[code]
        assert max(slots) < stride
    src = open(os.path.join(ROOT, "deepj_b200", "csrc", "runtime.cu")).read()
    for name, code in (("BF16_LINEAR", 77), ("BF16_BLOCK_LINEAR", 78), ("DELTA_RULE", 79), ("ATTN_LATENT", 80), ("TABLE_EXPERTS", 81), ("ATTN_LATENT_CHUNK", 82)):
        assert f"case DEEPJ_OP_{name}: return {cg.OP_METADATA[code][0]};" in src
    assert [pad8(n) for n in (1, 8, 9)] == [8, 8, 16]
