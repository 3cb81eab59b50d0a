"""Small Punilix configurations and random weights for the tests."""
import json
import os

import numpy as np

from deepj_b200.checkpoint import write_safetensors
from deepj_b200.hybrid import HybridConfig

RANK = 11        # of the decay's low-rank projection: only the weights' shapes tell it


def _latent(heads, dim, rot, vdim, q_rank, kv_rank, scale, scaling, base=10000.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": {"base": base, "dims": rot, "scaling": scaling}}}


def _delta(heads, dim):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


YARN = {"factor": 3.0, "original": 48, "fast": 8.0, "slow": 1.0}
YARN2 = {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def _config(vocab, width, groups, eps, cap, layers):
    return {"architecture": "Punilix", "vocab": vocab, "width": width, "norm": {"groups": groups, "eps": eps}, "logit_softcap": cap,
            "layers": [dict(L, mlp=f) for L, f in layers]}


# "mixed": every branch, sizes in multiples of eight (tensor-core kernels), attention first; "odd": nothing a multiple of
# eight, no YaRN, one norm group, no cap; "wide": head sizes of real models, one attention head, an expert table row with
# every expert
CONFIGS = {
    "mixed": _config(211, 144, 3, 3e-4, 12.0, [
        (_latent(5, 24, 8, 40, 72, 56, 0.21, YARN), _dense(136, 0.9)), (_delta(3, 40), None), (_delta(2, 72), _moe(5, 2, 56, 0.6)),
        (_latent(3, 48, 16, 16, 40, 136, 0.15, YARN2, 500.0), _moe(4, 1, 24, 2.5)), (_latent(2, 32, 16, 24, 64, 64, 0.2, None), None)]),
    "odd": _config(83, 90, 1, 1e-5, None, [
        (_delta(2, 21), _dense(50, 1.5)), (_latent(3, 13, 6, 10, 30, 22, 0.3, None), _moe(3, 3, 19, 0.7)), (_delta(1, 35), _moe(6, 1, 30, 1.0)),
        (_latent(1, 20, 2, 33, 17, 9, 0.4, YARN), None)]),
    "wide": _config(300, 256, 2, 1e-6, 25.0, [
        (_delta(2, 128), _dense(264, 3.0)), (_latent(1, 128, 64, 128, 96, 512, 0.1, YARN2, 1e6), _dense(72, 0.5)), (_delta(1, 160), _moe(2, 2, 40, 1.1))]),
}


def tensor_shapes(config):
    return HybridConfig.parse(config, 8, lambda _n: RANK).tensors()


def bf16(a):
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def random_weights(config, seed, sharp=5.0):
    """Weights whose queries are sharp (a key that is missed or moved shows) and whose clamps and gates are exercised."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".", 1)[-1]
        if leaf == "mlp.table":
            layer = config["layers"][int(name.split(".")[0][1:])]
            out[name] = np.argsort(rng.random((shape[0], layer["mlp"]["router"]["experts"])), axis=1)[:, :shape[1]].astype(np.int32)
            continue
        if len(shape) == 1:
            a = rng.standard_normal(shape) * 0.3 + (1.0 if "norm" in leaf else 0.0)
            if leaf == "mix.w0":
                a = rng.standard_normal(shape) * 3.0
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
            if leaf == "mix.uq":
                a *= sharp
            if leaf in ("mix.o", "mlp.down") or leaf.endswith(".down"):
                a *= 0.5
        out[name] = bf16(a)
    return out


def write_folder(path, config, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(path, "model.safetensors"), weights)
