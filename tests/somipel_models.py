"""Small Somipel configurations and random weights for the tests."""
import numpy as np

from deepj_b200.hybrid import HybridConfig
from punilix_models import bf16, write_folder  # noqa: F401  (the same folder layout)


def _attention(heads, kv_heads, dim, vdim, scale, far, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": far}
    return {"type": "attention", "mixer": m if kv_from is None else dict(m, kv_from=kv_from)}


def _keys(heads, kv_heads, dim, scale, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    return {"type": "attention_2", "mixer": m if temp is None else dict(m, q_temp={"coef": temp[0], "every": temp[1]})}


def _lstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _config(vocab, width, eps, mult, layers):
    return {"architecture": "Somipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": [dict(L, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for L, ff in layers]}


# "mixed": sizes in multiples of eight, a layer without feed-forward, a recurrence first and last, a layer that reads another's
# keys across a layer of another kind; "odd": nothing a multiple of eight, one head, unequal key and value sizes; "wide": head
# sizes of real models, more query heads per group than an operand has rows
CONFIGS = {
    "mixed": _config(211, 144, 3e-4, 0.37, [
        (_lstm(3, 24, 40, 5.0), 88), (_attention(6, 2, 40, 24, 0.2, 37), 136), (_keys(4, 2, 32, 0.3, (0.4, 7)), None), (_attention(4, 2, 40, 24, 0.25, 90, 1), 72),
        (_keys(3, 3, 48, 0.15), 64), (_lstm(2, 72, 16, 11.0), None)]),
    "odd": _config(83, 90, 1e-5, 1.0, [
        (_attention(3, 1, 13, 7, 0.4, 21), 50), (_attention(1, 1, 13, 7, 0.3, 400, 0), None), (_lstm(2, 21, 10, 3.0), 35), (_keys(5, 1, 11, 0.5, (1.5, 3)), 19)]),
    "wide": _config(300, 256, 1e-6, 0.6, [
        (_attention(20, 1, 128, 64, 0.09, 128), 264), (_keys(2, 1, 200, 0.07, (0.2, 50)), 72), (_lstm(1, 160, 96, 15.0), 40), (_attention(2, 2, 64, 136, 0.12, 60), None)]),
}
REL_ROWS = {"mixed": 12, "odd": 6, "wide": 32}       # of the distance table: only the weights' shapes tell them


def parse(name, max_seq=8):
    return HybridConfig.parse(CONFIGS[name], max_seq, lambda n: REL_ROWS[name] if n.endswith(".rel") else None)


def random_weights(name, seed, sharp=3.0):
    """Weights whose queries are sharp (a key that is missed or moved shows), whose distance biases differ from row to row, and
    whose gates forget and remember."""
    rng = np.random.default_rng(seed)
    config, out = CONFIGS[name], {}
    for n, shape in parse(name).tensors().items():
        leaf = n.split(".", 1)[-1]
        if len(shape) == 1:
            a = rng.standard_normal(shape) * 0.3 + (1.0 if "norm" in leaf else 0.0)
            if leaf == "mix.q.norm":
                a *= sharp
            if leaf == "mix.f.b":
                a = rng.standard_normal(shape) + 2.0
        elif leaf == "mix.rel":
            a = rng.standard_normal(shape) * 1.5
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
            if leaf in ("mix.i", "mix.f"):
                a *= 2.0
        if leaf == "mix.k" and config["layers"][int(n.split(".")[0][1:])]["type"] == "mlstm":
            # keys that resemble the queries: where a head's sums cancel, its norm blows rounding up
            a = 0.7 * out[n[:-1] + "q"] + 0.7 * a
        out[n] = bf16(a)
    return out
