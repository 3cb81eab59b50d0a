"""Prefill and decode throughput of a few layers at the widths of real models, and every kind of op against its roofline:

    python bench.py --layers [--layers-case NAME] [--steps K --warmup W]

Each case holds layer-list stacks (Punilix, Somipel) with random weights and the Q8 model of this package that is closest to
them, at equal width, feed-forward, heads, depth, vocabulary and context.  Times are CUDA events on the library's stream: a whole prompt chunk,
K decode steps behind it (token fed back on the device), and per op code the ops of a step or of a chunk back to back as
their own stream.  Weights exceed L2 in every case.  Roofline of an op: the slower of its algorithmic bytes over the copy
bandwidth and its flops over the bf16 GEMM rate.
"""
from __future__ import annotations

import ctypes
import json
import os
from typing import Any, Dict, List

import numpy as np

from . import _lib
from . import compute_graph as cg
from .decoder import DecoderConfig, Q8Decoder
from .hybrid import HybridConfig, HybridDecoder

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
NAMES = {getattr(cg, n): n[3:].lower() for n in dir(cg) if n.startswith("OP_") and isinstance(getattr(cg, n), int)}


def peaks() -> Dict[str, Any]:
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            r = json.load(f)
        return {"hbm_gbs": float(r["hbm_gbs"]), "bf16_tflops": float(r["bf16_tflops"]), "kind": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "kind": "fallback"}


def _stack(width, delta_heads, dim, heads, mla_dim, rot, vdim, q_rank, kv_rank, ff, depth, every, moe=None):
    """`every`-th layer attends, the others are recurrent; `moe` = (experts, top, ff) makes every second feed-forward routed."""
    layers = []
    for i in range(depth):
        if (i + 1) % every == 0:
            L = {"type": "latent_attention", "mixer": {
                "heads": heads, "dim": mla_dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": (mla_dim + rot) ** -0.5,
                "rot": {"base": 10000.0, "dims": rot, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
        else:
            L = {"type": "general_delta", "mixer": {"heads": delta_heads, "dim": dim}}
        if moe and i % 2 == 1:
            L["mlp"] = {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2], "limit": 7.0}}
        else:
            L["mlp"] = {"kind": "dense", "ff": ff, "limit": 7.0}
        layers.append(L)
    return {"architecture": "Punilix", "vocab": 32000, "width": width, "norm": {"groups": 4, "eps": 1e-5}, "logit_softcap": 30.0, "layers": layers}


def _somipel(width, heads, kv_heads, dim, lstm_heads, lstm_dim, lstm_vdim, ff, depth, attention_only=False):
    """Layers in fours: gated attention, the same reading its keys and values, attention whose values are its keys, recurrence."""
    layers = []
    for i in range(depth):
        kind = i % 4
        attn = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5}
        if kind == 3 and not attention_only:
            L = {"type": "mlstm", "mixer": {"heads": lstm_heads, "dim": lstm_dim, "vdim": lstm_vdim, "gate_cap": 15.0}}
        elif kind == 2:
            L = {"type": "attention_2", "mixer": dict(attn, q_temp={"coef": 0.1, "every": 1024})}
        else:
            L = {"type": "attention", "mixer": dict(attn, bias_max=128, **({"kv_from": i - 1} if kind == 1 else {}))}
        layers.append(dict(L, mlp={"kind": "dense", "ff": ff}))
    return {"architecture": "Somipel", "vocab": 32000, "width": width, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "layers": layers}


# name → (layer-list stacks, closest Q8 model, prompt)
_W4096, _W2048 = _stack(4096, 32, 128, 32, 128, 64, 128, 1536, 512, 11008, 8, 4), _stack(2048, 16, 128, 16, 128, 64, 128, 1024, 512, 5632, 16, 2)
_LLAMA_4096 = DecoderConfig("llama", 32000, 2176, 4096, 32, 8, 11008)
CASES = {
    "w4096": ({"punilix": _W4096}, _LLAMA_4096, 2048),
    "w2048": ({"punilix": _W2048}, DecoderConfig("deepseek", 32000, 1280, 2048, 16, 16, 5632, 1024, 512), 1024),
    "w2048_experts": ({"punilix": _stack(2048, 32, 64, 16, 128, 64, 128, 1024, 512, 5632, 16, 4, moe=(64, 4, 1408))},
                      DecoderConfig("llama", 32000, 1280, 2048, 16, 16, 5632), 1024),
    "somipel_w4096": ({"somipel": _somipel(4096, 32, 8, 128, 16, 128, 256, 11008, 8), "punilix": _W4096}, _LLAMA_4096, 2048),
    "somipel_w2048": ({"somipel": _somipel(2048, 32, 32, 64, 8, 128, 256, 5632, 16), "punilix": _W2048},
                      DecoderConfig("llama", 32000, 1280, 2048, 32, 16, 5632), 1024),
}
# decode attention where the cache is long enough to be streamed: the context is taken as given (its rows are zeros)
LONG_CASES = {
    "context32k": ({"punilix": _stack(2048, 16, 128, 16, 128, 64, 128, 1024, 512, 5632, 4, 1)}, DecoderConfig("deepseek", 32000, 32832, 2048, 16, 4, 5632, 1024, 512), 32768),
    "somipel_context32k": ({"somipel": _somipel(2048, 16, 4, 128, 8, 128, 256, 5632, 3, attention_only=True)},
                           DecoderConfig("llama", 32000, 32832, 2048, 16, 3, 5632), 32768),
}
DTYPES = {"punilix": "bf16 weights and latent cache, fp32 rows", "somipel": "bf16 weights and cache, fp32 rows and state"}


def layer_list(rec, max_seq: int) -> HybridDecoder:
    dec = HybridDecoder(HybridConfig.parse(rec, max_seq, lambda n: 32 if n.endswith(".rel") else 64), dtype="bf16")
    dec.load_synthetic(5, 0.02)
    return dec


def split_ops(stream: np.ndarray) -> List[np.ndarray]:
    out, at = [], 0
    while at < stream.size:
        n = cg.OP_METADATA[int(stream[at])][0]
        out.append(stream[at:at + n])
        at += n
    return out


def weight_dims(dec) -> Dict[int, tuple]:
    """Buffer id → (K, N) of every weight object."""
    if isinstance(dec, HybridDecoder):
        return dict(dec.weight_dims)
    plan = {o: (k, sum(p[3] for p in parts)) for o, k, parts in dec._shard_plan()}
    plan["Wlm"] = (dec.cfg.d_model, dec.v_local)
    return {i: plan[name.split(".")[0]] for name, i in dec.ids.items() if name.split(".")[0] in plan}


def op_cost(op: np.ndarray, dims: Dict[int, tuple], q8: bool, context: int, kv_bytes: int, tok: np.ndarray, tables: Dict[int, np.ndarray]):
    """(algorithmic bytes, flops) of one op, or None for bookkeeping ops."""
    c = [int(v) for v in op]
    code = c[0]

    def w_bytes(k, n):
        return k * n + (k + 31) // 32 * n * 4 if q8 else 2 * k * n
    if code in (cg.OP_Q8_LINEAR, cg.OP_Q8_LINEAR_LN, cg.OP_Q8_SWIGLU, cg.OP_BF16_LINEAR, cg.OP_BF16_LINEAR_SUM):
        at_w, at_m = {cg.OP_Q8_LINEAR: (6, 14), cg.OP_Q8_LINEAR_LN: (7, 15), cg.OP_Q8_SWIGLU: (6, 13), cg.OP_BF16_LINEAR: (14, 21),
                      cg.OP_BF16_LINEAR_SUM: (14, 21)}[code]
        w, m = c[at_w], c[at_m]
        k, n = dims[w]
        n2 = 2 * n if code == cg.OP_Q8_SWIGLU else n
        sums = 8 * m * k if code == cg.OP_BF16_LINEAR_SUM and c[31] >= 0 else 0          # the residual row read, the sum written
        return w_bytes(k, n2) + 4 * m * (k + n) + sums, 2 * m * k * n2
    if code == cg.OP_BF16_BLOCK_LINEAR:
        k, n = dims[c[5]]
        return 2 * k * n + 4 * c[11] * (c[6] * k + n), 2 * c[11] * k * n
    if code in (cg.OP_ATTN_DECODE, cg.OP_ATTN_PREFILL):
        B, H, hd = c[14], c[15], c[16]
        T = c[17] if code == cg.OP_ATTN_PREFILL else 1
        pairs = B * H * (T * (context - T) + T * (T + 1) // 2)
        return 2 * B * H * hd * kv_bytes * context, 4 * hd * pairs
    if code == cg.OP_ATTN_LATENT:
        B, T, H, dim, rot, R = c[19:25]
        pairs = B * H * (T * (context - T) + T * (T + 1) // 2)
        return B * (R + rot) * kv_bytes * context + 4 * B * T * H * (2 * R + rot), 2 * pairs * (2 * R + rot)
    if code == cg.OP_ATTN_LATENT_CHUNK:
        B, T, H, dim, rot, R, vdim = c[18:25]
        pairs = B * H * (T * (context - T) + T * (T + 1) // 2)
        return B * (R + rot) * kv_bytes * context + 4 * B * T * H * (dim + rot + vdim), 2 * pairs * (dim + rot + vdim) + 2 * B * context * R * H * (dim + vdim)
    if code == cg.OP_ATTN_GROUPED:
        B, T, H, G, dim, vdim = c[19:25]
        pairs = B * H * (T * (context - T) + T * (T + 1) // 2)
        row = dim * kv_bytes + 4 if c[13] < 0 else (dim + vdim) * kv_bytes
        return B * G * row * context + 4 * B * T * H * (dim + vdim), 2 * pairs * (dim + vdim)
    if code == cg.OP_MLSTM:
        B, T, H, dim, vdim = c[16:21]
        return B * (2 * 4 * H * dim * vdim + 4 * T * H * 2 * (dim + vdim)), B * T * H * 5 * dim * vdim
    if code == cg.OP_DELTA_RULE:
        B, T, H, dim = c[16:20]
        return B * (2 * 4 * H * dim * dim + 4 * T * H * dim * 6), B * T * H * (7 * dim * dim + 2 * dim * dims[c[9]][0])
    if code == cg.OP_TABLE_EXPERTS:
        top, ff, d, m = c[10], c[14], c[22], c[23]
        used = len(np.unique(tables[c[8]][tok[:m]]))
        return used * 2 * 3 * ff * d + 4 * m * (2 * d), 6 * m * top * ff * d
    return None


def time_stream(lib, stream: np.ndarray, iters: int, warmup: int = 3) -> float:
    stream = np.ascontiguousarray(stream)
    for _ in range(max(3, warmup)):
        _lib.check(lib.deepj_cuda_flush_ops(stream.ctypes.data, stream.size))
    _lib.check(lib.deepj_cuda_timer_begin())
    for _ in range(iters):
        _lib.check(lib.deepj_cuda_flush_ops_async(stream.ctypes.data, stream.size))
    ms = ctypes.c_float(0)
    _lib.check(lib.deepj_cuda_timer_end(ctypes.byref(ms)))
    return ms.value / iters


def by_op(dec, stream: np.ndarray, context: int, tok: np.ndarray, pk, iters: int) -> Dict[str, Any]:
    q8 = not isinstance(dec, HybridDecoder)
    dims = weight_dims(dec)
    kv_bytes = (4 if dec.kv_dtype == "f32" else 2) if q8 else (2 if dec.dtype == "bf16" else 4)
    tables = {} if q8 else {dec.ids[n]: t for n, t in dec.tables.items()}
    groups: Dict[str, Dict[str, Any]] = {}
    for op in split_ops(stream):
        cost = op_cost(op, dims, q8, context, kv_bytes, tok, tables)
        if cost is None:
            continue
        g = groups.setdefault(NAMES[int(op[0])], {"ops": [], "us_roof": 0.0})
        g["ops"].append(op)
        g["us_roof"] += 1e6 * max(cost[0] / (pk["hbm_gbs"] * 1e9), cost[1] / (pk["bf16_tflops"] * 1e12))
    out = {}
    for name, g in groups.items():
        us = 1e3 * time_stream(dec.lib, np.concatenate(g["ops"]), iters)
        out[name] = {"launch_groups": len(g["ops"]), "us": round(us, 1), "us_roofline": round(g["us_roof"], 1), "of_roofline": round(g["us_roof"] / us, 3)}
    return out


def measure(dec, prompt: int, steps: int, warmup: int, seed: int, pk) -> Dict[str, Any]:
    tok = np.random.default_rng(seed).integers(0, dec.cfg.vocab_size, size=prompt)
    lib = dec.lib
    best = None
    for _ in range(4):                     # the first builds the buffers, the second captures the graph
        dec.reset()
        _lib.check(lib.deepj_cuda_synchronize())
        _lib.check(lib.deepj_cuda_timer_begin())
        nxt = dec.prefill(tok.reshape(1, -1))
        ms = ctypes.c_float(0)
        _lib.check(lib.deepj_cuda_timer_end(ctypes.byref(ms)))
        best = ms.value if best is None else min(best, ms.value)
    dec.set_tokens(nxt)
    dec.step_device(max(3, warmup))
    _lib.check(lib.deepj_cuda_timer_begin())
    dec.step_device(steps, sync=False)
    ms = ctypes.c_float(0)
    _lib.check(lib.deepj_cuda_timer_end(ctypes.byref(ms)))
    step_ms = ms.value / steps
    ctx = dec.position
    decode = by_op(dec, dec._build(feed_back=False), ctx, tok, pk, 20)
    T = min(prompt, dec._chunk_tokens())
    dec.reset()
    dec.prefill(tok.reshape(1, -1))
    dec.reset()
    chunk = by_op(dec, dec._prefill_streams[T], T, tok, pk, 5)
    return {"prefill": {"tokens": prompt, "ms": round(best, 3), "tokens_per_s": round(prompt / best * 1e3), "ops": chunk},
            "decode": {"context": ctx, "ms_per_step": round(step_ms, 4), "tokens_per_s": round(1e3 / step_ms, 1), "ops": decode},
            "device_error": dec.stats()["device_error"]}


def measure_long(dec, context: int, steps: int, pk) -> Dict[str, Any]:
    dec.reset()
    dec.set_position(context)
    dec.set_tokens([1])
    dec.step_device(3)
    step_ms = time_stream(dec.lib, dec._build(feed_back=False), max(4, min(steps, 40)))
    dec.set_position(context)
    return {"decode": {"context": context, "ms_per_step": round(step_ms, 4), "tokens_per_s": round(1e3 / step_ms, 1),
                       "ops": by_op(dec, dec._build(feed_back=False), context, np.zeros(1, dtype=np.int64), pk, 20)},
            "device_error": dec.stats()["device_error"]}


def main(case: str = "", steps: int = 64, warmup: int = 8, clocks=None) -> None:
    pk = peaks()
    line: Dict[str, Any] = {"metric": "layers_prefill_and_decode", "peaks": pk, "data": "synthetic", "steps": steps, "warmup": max(3, warmup), "cases": {}}
    for name, (stacks, near, prompt) in CASES.items():
        if case and name != case:
            continue
        sampler = clocks() if clocks else None
        if sampler:
            sampler.start()
            sampler.wait_ready()
        res = {}
        for label, rec in stacks.items():
            dec = layer_list(rec, near.max_seq_len)
            res[label] = dict(measure(dec, prompt, steps, warmup, 1, pk), dtype=DTYPES[label])
            dec.close()
        q = Q8Decoder(near, id_base=2 << 24)
        q.load_synthetic(5, 0.02)
        res[f"{near.kind}_q8"] = dict(measure(q, prompt, steps, warmup, 1, pk), dtype="q8 weights, fp32 rows and cache")
        q.close()
        if sampler:
            res["clocks"] = sampler.stop()
        line["cases"][name] = res
    for name, (stacks, near, context) in LONG_CASES.items():
        if case and name != case:
            continue
        res = {}
        for label, rec in stacks.items():
            dec = layer_list(rec, near.max_seq_len)
            res[label] = measure_long(dec, context, steps, pk)
            dec.close()
        q = Q8Decoder(near, id_base=2 << 24)
        q.load_synthetic(5, 0.02)
        res[f"{near.kind}_q8"] = measure_long(q, context, steps, pk)
        q.close()
        line["cases"][name] = res
    print(json.dumps(line), flush=True)
