"""Host side of the Somipel models — configuration, tables, registry — and the reference itself."""
import json
import math
import os

import numpy as np
import pytest

import somipel_models as sm
import somipel_ref as ref
from deepj_b200 import build, compute_graph as cg, registry
from deepj_b200.hybrid import DESIGNS, GroupedAttention, HybridConfig, MatrixLstm, distance_buckets

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", sorted(sm.CONFIGS))
def test_reference_is_the_same_however_a_prompt_is_cut(name):
    m = ref.Model(sm.CONFIGS[name], sm.random_weights(name, 1))
    t = np.random.default_rng(2).integers(0, sm.CONFIGS[name]["vocab"], size=23)
    whole = m.forward(t)
    m.reset()
    cut = np.concatenate([m.forward(t[lo:hi]) for lo, hi in ((0, 1), (1, 3), (3, 20), (20, 23))])
    assert np.allclose(whole, cut, atol=1e-9)
    m.reset()
    changed = t.copy()
    changed[15] = (t[15] + 1) % sm.CONFIGS[name]["vocab"]
    other = m.forward(changed)
    assert np.allclose(whole[:15], other[:15]) and np.abs(whole[16:] - other[16:]).max() > 1e-3      # causal, and it remembers


def test_recurrence_against_its_closed_form():
    """Without the running maximum: S_t = Σ_s exp(f_{s+1} + … + f_t + i_s) k_s v_sᵀ, and the denominator's floor is 1."""
    rng = np.random.default_rng(0)
    T, dim, vdim = 9, 5, 3
    q, k, v = rng.standard_normal((T, dim)), rng.standard_normal((T, dim)), rng.standard_normal((T, vdim))
    i, f = rng.standard_normal(T) * 2, -rng.random(T)
    state = (np.zeros((dim, vdim)), np.zeros(dim), 0.0)
    for t in range(T):
        state, o = ref.mlstm_step(state, q[t], k[t], v[t], i[t], f[t])
        w = np.array([math.exp(f[s + 1:t + 1].sum() + i[s]) for s in range(t + 1)])
        p = w * (k[:t + 1] @ q[t])
        # the small constant is added after scaling by the running maximum
        assert np.allclose(o, p @ v[:t + 1] / (max(abs(p.sum()), 1.0) + 1e-6 * math.exp(state[2])))
    assert state[2] >= f.sum() - 1e-12                  # the maximum starts at zero, which decays like everything else


def test_distance_rows():
    got = [ref.distance_bucket(n, 8, 32) for n in (0, 3, 4, 5, 6, 8, 11, 16, 31, 32, 1000)]
    assert got == [0, 3, 4, 4, 4, 5, 5, 6, 7, 7, 7]      # 4 + floor(4 · log2(n/4) / 3), whole numbers reached exactly
    for rows, far in ((8, 32), (12, 37), (32, 128), (32, 100), (2, 5), (24, 96), (6, 400), (64, 33)):
        table = distance_buckets(rows, far, 5000)
        assert table[-1] == rows - 1 and (len(table) < 2 or table[-2] < rows - 1)
        want = [ref.distance_bucket(n, rows, far) for n in range(len(table) + 50)]
        assert want[:len(table)] == table.tolist() and set(want[len(table):]) == {rows - 1}
    assert len(distance_buckets(32, 4096, 100)) == 100   # no longer than the positions there can be
    with pytest.raises(ValueError):
        distance_buckets(32, 16, 100)


def test_sink_and_temperature():
    s = np.array([[0.5, -2.0, 3.0]])
    assert np.allclose(ref.softmax_with_sink(s), np.exp(s) / (1.0 + np.exp(s).sum()))
    assert ref.softmax_with_sink(np.array([[-800.0]]))[0, 0] == 0.0 and np.allclose(ref.softmax_with_sink(np.array([[800.0]])), 1.0)
    assert [ref.temperature(p, 0.5, 4) for p in (0, 2)] == [1.0, 1.0] and np.isclose(ref.temperature(3, 0.5, 4), 1 + 0.5 * math.log(2))


def test_configuration_rules():
    cfg = sm.parse("mixed", 64)
    assert cfg.block == "post_norm" and cfg.residual_mult == 0.37 and cfg.norm_groups == 1
    t = cfg.tensors()
    assert t["l1.mix.rel"] == (12, 6) and t["l1.mix.k.b"] == (80,) and t["l0.mix.i"] == (3, 144) and "l2.norm2" not in t and "l2.mix.v" not in t
    assert not any(n.startswith(("l3.mix.k", "l3.mix.v")) for n in t) and t["l3.mix.rel"] == (12, 4) and "l2.mix.g" not in t and "l2.mix.q.b" not in t
    kinds = [type(m) for m, _ in cfg.layers]
    assert kinds.count(MatrixLstm) == 2 and kinds.count(GroupedAttention) == 4 and set(DESIGNS) == set(registry.HYBRID)

    def broken(change):
        c = json.loads(json.dumps(sm.CONFIGS["mixed"]))
        change(c)
        with pytest.raises((ValueError, KeyError)):
            HybridConfig.parse(c, 64, lambda n: 12 if n.endswith(".rel") else None)
    broken(lambda c: c["layers"][0].update(type="general_delta"))            # another design's
    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))             # does not divide the heads
    broken(lambda c: c["layers"][1]["mixer"].update(bias_max=6))             # not beyond the table's first half
    broken(lambda c: c["layers"][2]["mixer"].update(vdim=24))
    broken(lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=0))
    for j in (0, 2, 3, 4, -1, 99):                                           # no keys, other sizes, itself, later, nowhere
        broken(lambda c, j=j: c["layers"][3]["mixer"].update(kv_from=j))
    broken(lambda c: c["layers"][0]["mixer"].update(gate_cap=0))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    broken(lambda c: c.pop("residual_mult"))


def test_registry_and_ops(tmp_path):
    with open(tmp_path / "config.json", "w") as f:
        json.dump(sm.CONFIGS["odd"], f)
    assert registry.read_config(str(tmp_path))["architecture"] == "Somipel" and registry.dtypes_of("Somipel") == ("bf16", "f32")
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(str(tmp_path), "q8")
    src = open(os.path.join(ROOT, "deepj_b200", "csrc", "runtime.cu")).read()
    for name in ("BF16_LINEAR_SUM", "NORM_ADD", "ATTN_GROUPED", "MLSTM"):
        stride, slots = cg.OP_METADATA[getattr(cg, "OP_" + name)]
        assert max(slots) < stride and f"case DEEPJ_OP_{name}: return {stride};" in src
    assert {"attn_grouped.cu", "attn_grouped_mma.cu", "mlstm.cu", "mlstm_mma.cu"} <= set(build.PARTS["bf16"])
