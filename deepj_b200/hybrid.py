"""Decoders whose configuration lists their layers one by one: every layer names its mixer and its feed-forward.

`DESIGNS` says, per architecture, what the layer types mean, how a feed-forward's (gate, up) pairs are joined and how a
layer is put together:

  parallel (Punilix)    with h = norm(x), x ← x + mixer(h) + feed_forward(h).  All projections that read h are one bf16
                        weight and one launch (op 77: the norm is staged with the row, the gated feed-forward's pairs are
                        finished in the epilogue), and so are the two that write the residual: [W_o ‖ W_down] over [mixed
                        heads, gated values].
  post_norm (Somipel)   x ← x + c·norm1(mixer(x)), then x ← x + c·norm2(feed_forward(x)).  A sublayer's output is normed
                        and added where the next sublayer's projection stages its row (op 83), which also leaves the new
                        residual row for the one after it; only the last sum of a pass is a launch of its own (op 84).

Between its projections a mixer runs its own ops; head norms and output gates are part of the output projection's staging:

  GeneralDelta       op 79 (the recurrence)
  LatentAttention    W_uq on the normed query latent, the queries taken into the latent space (op 78), op 80, values (op 78)
  GroupedAttention   op 85: norms, cache append and attention over grouped heads
  MatrixLstm         op 86 (the recurrence)

A feed-forward is dense or table-routed experts (op 81), or absent.  A token step and a prompt chunk record the same
sequence of ops with different row counts.  Another mechanism is another class with the same methods.

dtype "bf16": bf16 weights and latent cache; rows are fp32 between ops, the many-row kernels round their operand to bf16.
dtype "f32": the same weights, every product in fp32, fp32 cache.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Mapping, NamedTuple, Optional, Tuple

import numpy as np

from . import _lib
from .compute_graph import (OP_ADD_SCALAR_INPLACE, OP_ARGMAX_ROWS, OP_ATTN_GROUPED, OP_ATTN_LATENT, OP_ATTN_LATENT_CHUNK, OP_BF16_BLOCK_LINEAR, OP_BF16_LINEAR,
                            OP_BF16_LINEAR_SUM, OP_COPY, OP_DELTA_RULE, OP_EMBED_GATHER, OP_MLSTM, OP_NORM_ADD, OP_SAMPLE_TOPK, OP_TABLE_EXPERTS, float_bits)
from .decoder import scaled_rope_tables
from .runner import StreamDecoder


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _positive(rec: Mapping[str, Any], *names: str) -> List[int]:
    out = []
    for n in names:
        v = rec[n]
        if not isinstance(v, int) or v <= 0:
            raise ValueError(f"{n} must be a positive integer, got {v!r}")
        out.append(v)
    return out


# ───────────── configuration ─────────────

@dataclass(frozen=True)
class GeneralDelta:
    """Generalized delta rule with per-channel decay and removal."""
    heads: int
    dim: int
    rank: int            # of the decay's low-rank projection

    @classmethod
    def parse(cls, rec: Mapping[str, Any], rows_of: Callable[[str], Optional[int]]) -> "GeneralDelta":
        heads, dim = _positive(rec, "heads", "dim")
        rank = rows_of("mix.w1")
        if rank is None:
            raise ValueError("the decay rank of a general_delta layer comes from its weights")
        return cls(heads, dim, rank)

    @property
    def out_width(self) -> int:
        return self.heads * self.dim

    def tensors(self, d: int) -> Dict[str, Tuple[int, ...]]:
        n = self.out_width
        t: Dict[str, Tuple[int, ...]] = {f"mix.{k}": (n, d) for k in "rkvga"}
        t.update({"mix.a.b": (n,), "mix.w1": (self.rank, d), "mix.w2": (n, self.rank), "mix.w0": (n,), "mix.norm": (n,), "mix.o": (d, n)})
        return t

    def fields(self) -> List[Tuple[str, int]]:
        """What the input projection produces per token: (tensor, rows)."""
        return [(f"mix.{k}", self.out_width) for k in "rkvga"] + [("mix.w1", self.rank)]

    def buffers(self, M: int) -> Dict[str, int]:
        return {"mix": M * self.out_width}

    def alloc(self, dec: "HybridDecoder", l: int) -> None:
        dec._f32(f"state.{l}", dec.B * self.out_width * self.dim)

    def load(self, dec: "HybridDecoder", l: int, get) -> None:
        dec._f32(f"abias.{l}", self.out_width, get("mix.a.b"))
        dec._f32(f"w0.{l}", self.out_width, get("mix.w0"))
        dec._f32(f"onorm.{l}", self.out_width, get("mix.norm"))
        dec._weight(f"w2.{l}", self.rank, self.out_width, [("mix.w2", 0, 1, 0)], get)

    def emit(self, op, dec: "HybridDecoder", l: int, buf: Dict[str, int], B: int, T: int) -> None:
        I, at, ld = dec.ids, dec._offsets[l], dec._in_rows[l]
        op("delta", OP_DELTA_RULE, buf["proj"], at["mix.r"], at["mix.k"], at["mix.v"], at["mix.a"], at["mix.w1"], ld, I[f"abias.{l}"], I[f"w2.{l}"],
           I[f"w0.{l}"], I[f"state.{l}"], I["pos"], buf["mix"], 0, self.out_width, B, T, self.heads, self.dim)

    def out_operand(self, dec: "HybridDecoder", l: int, buf: Dict[str, int]) -> List[int]:
        """x … ldgate of the output projection (op 77): each head over its root mean square, a gain, the gate."""
        n = self.out_width
        return [buf["mix"], 0, n, dec.ids[f"onorm.{l}"], self.heads, float_bits(dec.cfg.eps), buf["proj"], dec._offsets[l]["mix.g"], dec._in_rows[l]]


@dataclass(frozen=True)
class LatentAttention:
    """Causal attention over one cached latent row per position."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    base: float
    scaling: Optional[Tuple[Tuple[str, float], ...]]

    @classmethod
    def parse(cls, rec: Mapping[str, Any], rows_of: Callable[[str], Optional[int]]) -> "LatentAttention":
        heads, dim, rot_dim, vdim, q_rank, kv_rank = _positive(rec, "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")
        rot = rec["rot"]
        if rot["dims"] != rot_dim or rot_dim % 2 != 0:
            raise ValueError("rot.dims must equal rot_dim and be even")
        sc = rot.get("scaling")
        scaling = None if sc is None else tuple((k, float(sc[k])) for k in ("factor", "original", "fast", "slow"))
        return cls(heads, dim, rot_dim, vdim, q_rank, kv_rank, float(rec["scale"]), float(rot["base"]), scaling)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def tensors(self, d: int) -> Dict[str, Tuple[int, ...]]:
        H, R = self.heads, self.kv_rank
        return {"mix.dq": (self.q_rank, d), "mix.dq.norm": (self.q_rank,), "mix.uq": (H * (self.dim + self.rot_dim), self.q_rank),
                "mix.dkv": (R + self.rot_dim, d), "mix.dkv.norm": (R,), "mix.uk": (H * self.dim, R), "mix.uv": (H * self.vdim, R),
                "mix.g": (self.out_width, d), "mix.o": (d, self.out_width)}

    def fields(self) -> List[Tuple[str, int]]:
        return [("mix.dq", self.q_rank), ("mix.dkv", self.kv_rank + self.rot_dim), ("mix.g", self.out_width)]

    def buffers(self, M: int) -> Dict[str, int]:
        H = self.heads
        return {"mix": M * self.out_width, "q": M * H * (self.dim + self.rot_dim), "qc": M * H * self.kv_rank, "ctx": M * H * self.kv_rank}

    def alloc(self, dec: "HybridDecoder", l: int) -> None:
        i = dec._new_id()
        _lib.check(dec.lib.deepj_cuda_latent_alloc(i, dec.B, dec.cfg.max_seq_len, self.kv_rank + self.rot_dim, int(dec.dtype == "bf16")))
        dec.ids[f"cache.{l}"] = i
        key = f"rot {self.rot_dim} {self.base} {self.scaling}"
        if key + " cos" not in dec.ids:
            cos, sin = scaled_rope_tables(self.rot_dim, dec.cfg.max_seq_len, self.base, dict(self.scaling) if self.scaling else None)
            dec._f32(key + " cos", cos.size, cos)
            dec._f32(key + " sin", sin.size, sin)

    def load(self, dec: "HybridDecoder", l: int, get) -> None:
        H, R = self.heads, self.kv_rank
        dec._f32(f"dqnorm.{l}", self.q_rank, get("mix.dq.norm"))
        dec._f32(f"dkvnorm.{l}", R, get("mix.dkv.norm"))
        dec._weight(f"uq.{l}", self.q_rank, H * (self.dim + self.rot_dim), [("mix.uq", 0, 1, 0)], get)

        def transposed(name):            # queries enter the latent space: W_uk of every head transposed, [heads · kv_rank][dim]
            a = get(name)
            if isinstance(a, tuple):     # generated on the device: any order will do
                return H * R, self.dim, a[2]
            return np.ascontiguousarray(a.reshape(H, self.dim, R).transpose(0, 2, 1)).reshape(H * R, self.dim)

        dec._weight(f"ukT.{l}", self.dim, H * R, [("mix.uk", 0, 1, 0)], transposed)
        if self.expands(dec):
            dec._weight(f"uk.{l}", R, H * self.dim, [("mix.uk", 0, 1, 0)], get)
        dec._weight(f"uv.{l}", R, H * self.vdim, [("mix.uv", 0, 1, 0)], get)

    def expands(self, dec: "HybridDecoder") -> bool:
        """Whether prompt chunks run over expanded keys and values (op 82)."""
        return (dec.dtype == "bf16" and all(n % 8 == 0 for n in (self.dim, self.rot_dim, self.vdim, self.kv_rank)) and self.dim + self.rot_dim <= 256 and
                self.vdim <= 128)

    def emit(self, op, dec: "HybridDecoder", l: int, buf: Dict[str, int], B: int, T: int) -> None:
        I, at, ld, M = dec.ids, dec._offsets[l], dec._in_rows[l], B * T
        H, R, qw = self.heads, self.kv_rank, self.heads * (self.dim + self.rot_dim)
        eps = float_bits(dec.cfg.eps)
        key = f"rot {self.rot_dim} {self.base} {self.scaling}"
        dec._linear(op, "q_up", [buf["proj"], at["mix.dq"], ld, I[f"dqnorm.{l}"], 1, eps, -1, 0, 0], self.q_rank, None, I[f"uq.{l}"],
                    None, (buf["q"], qw), M, qw)
        if self.expands(dec) and T >= EXPAND_MIN_TOKENS:
            op("attn", OP_ATTN_LATENT_CHUNK, buf["q"], 0, qw, buf["proj"], at["mix.dkv"], ld, I[f"dkvnorm.{l}"], eps, I[f"cache.{l}"], I["pos"],
               I[key + " cos"], I[key + " sin"], I[f"uk.{l}"], I[f"uv.{l}"], buf["mix"], 0, self.out_width, B, T, H, self.dim, self.rot_dim, R, self.vdim,
               float_bits(self.scale))
            return
        op("q_latent", OP_BF16_BLOCK_LINEAR, buf["q"], 0, qw, self.dim + self.rot_dim, I[f"ukT.{l}"], H, buf["qc"], 0, H * R, R, M)
        op("attn", OP_ATTN_LATENT, buf["q"], 0, qw, buf["qc"], 0, H * R, buf["proj"], at["mix.dkv"], ld, I[f"dkvnorm.{l}"], eps, I[f"cache.{l}"],
           I["pos"], I[key + " cos"], I[key + " sin"], buf["ctx"], 0, H * R, B, T, H, self.dim, self.rot_dim, R, float_bits(self.scale))
        op("values", OP_BF16_BLOCK_LINEAR, buf["ctx"], 0, H * R, R, I[f"uv.{l}"], H, buf["mix"], 0, self.out_width, self.vdim, M)

    def out_operand(self, dec: "HybridDecoder", l: int, buf: Dict[str, int]) -> List[int]:
        return [buf["mix"], 0, self.out_width, -1, 0, 0, buf["proj"], dec._offsets[l]["mix.g"], dec._in_rows[l]]


EXPAND_MIN_TOKENS = 48      # chunks from here on expand the context's keys and values; shorter ones attend in the latent space


def distance_buckets(rows: int, far: float, limit: int) -> np.ndarray:
    """Table row for distances 0, 1, … up to the first that has the last row, or `limit` of them: one row per distance in
    the first half, logarithmic up to `far` in the second."""
    half = rows // 2
    if rows < 2 or far <= half:
        raise ValueError("the distance table needs two rows and a largest distance beyond its first half")
    out: List[int] = []
    while len(out) < limit and (not out or out[-1] < rows - 1):
        n = len(out)
        # the quotient of logarithms can come out just below a whole number it equals
        out.append(n if n < half else min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9)))
    return np.asarray(out, dtype=np.int64)


@dataclass(frozen=True)
class GroupedAttention:
    """Causal attention of grouped query heads, queries and keys RMS-normed per head.  Options: projection biases, a sigmoid
    output gate, a learned bias by distance, a query factor by position, a sink in the softmax's denominator, values that are
    the keys as projected, another layer's keys and values."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    biases: bool = False
    gated: bool = False
    keys_are_values: bool = False
    sink: bool = False
    rel_rows: int = 0                                   # rows of the distance bias table, 0 = none
    rel_far: float = 0.0
    q_temp: Optional[Tuple[float, float]] = None        # (coefficient, positions per step of the logarithm's argument)
    kv_from: Optional[int] = None

    @classmethod
    def parse(cls, rec: Mapping[str, Any], rows_of: Callable[[str], Optional[int]], distance_bias: bool = False, **options: bool) -> "GroupedAttention":
        heads, kv_heads, dim = _positive(rec, "heads", "kv_heads", "dim")
        vdim = dim if options.get("keys_are_values") and "vdim" not in rec else _positive(rec, "vdim")[0]
        if heads % kv_heads:
            raise ValueError("kv_heads must divide heads")
        if options.get("keys_are_values") and vdim != dim:
            raise ValueError("values that are the keys have the keys' size")
        rel_rows, far = 0, 0.0
        if distance_bias:
            rel_rows, far = rows_of("mix.rel") or 0, float(rec["bias_max"])
            distance_buckets(rel_rows, far, 1)
        temp = rec.get("q_temp")
        if temp is not None:
            temp = (float(temp["coef"]), float(temp["every"]))
            if not temp[1] > 0:
                raise ValueError("q_temp.every must be positive")
        return cls(heads, kv_heads, dim, vdim, float(rec["scale"]), rel_rows=rel_rows, rel_far=far, q_temp=temp, kv_from=rec.get("kv_from"), **options)

    def check_source(self, l: int, layers) -> None:
        """The layer whose keys and values this one reads comes earlier, has its own, and the same shapes."""
        if self.kv_from is None:
            return
        src = layers[self.kv_from][0] if isinstance(self.kv_from, int) and 0 <= self.kv_from < l else None
        same = ("kv_heads", "dim", "vdim", "keys_are_values")
        if not isinstance(src, GroupedAttention) or src.kv_from is not None or any(getattr(src, k) != getattr(self, k) for k in same):
            raise ValueError(f"layer {l}: kv_from must name an earlier layer with keys and values of its own and the same head sizes")

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def tensors(self, d: int) -> Dict[str, Tuple[int, ...]]:
        own = {"q": self.heads * self.dim}
        t: Dict[str, Tuple[int, ...]] = {"mix.q.norm": (self.dim,), "mix.o": (d, self.out_width)}
        if self.kv_from is None:
            t["mix.k.norm"] = (self.dim,)
            own["k"] = self.kv_heads * self.dim
            if not self.keys_are_values:
                own["v"] = self.kv_heads * self.vdim
        for name, n in own.items():
            t[f"mix.{name}"] = (n, d)
            if self.biases:
                t[f"mix.{name}.b"] = (n,)
        if self.rel_rows:
            t["mix.rel"] = (self.rel_rows, self.heads)
        if self.gated:
            t["mix.g"] = (self.out_width, d)
        return t

    def fields(self) -> List[Tuple[str, int]]:
        t = self.tensors(1)
        return [(n, t[n][0]) for n in ("mix.q", "mix.k", "mix.v", "mix.g") if n in t]

    def field_biases(self) -> List[str]:
        return [n for n in ("mix.q", "mix.k", "mix.v") if n + ".b" in self.tensors(1)]

    def buffers(self, M: int) -> Dict[str, int]:
        return {"mix": M * self.out_width}

    def alloc(self, dec: "HybridDecoder", l: int) -> None:
        if self.kv_from is None:
            half, n, S = int(dec.dtype == "bf16"), dec.B * self.kv_heads, dec.cfg.max_seq_len
            for name, width in (("keys", self.dim),) + (() if self.keys_are_values else (("values", self.vdim),)):
                i = dec._new_id()
                _lib.check(dec.lib.deepj_cuda_latent_alloc(i, n, S, (width + 15) // 16 * 16, half))
                dec.ids[f"{name}.{l}"] = i
            if self.keys_are_values:
                dec._f32(f"kscale.{l}", n * ((S + 63) // 64 * 64))
        if self.q_temp and f"temp {self.q_temp}" not in dec.ids:
            coef, every = self.q_temp
            steps = np.floor((np.arange(dec.cfg.max_seq_len, dtype=np.float64) + 1.0) / every)
            dec._f32(f"temp {self.q_temp}", steps.size, 1.0 + coef * np.log(steps + 1.0))

    def load(self, dec: "HybridDecoder", l: int, get) -> None:
        dec._f32(f"qnorm.{l}", self.dim, get("mix.q.norm"))
        if self.kv_from is None:
            dec._f32(f"knorm.{l}", self.dim, get("mix.k.norm"))
        if self.rel_rows:
            rows = distance_buckets(self.rel_rows, self.rel_far, dec.cfg.max_seq_len)
            table = get("mix.rel")
            by_distance = np.zeros((rows.size, self.heads)) if isinstance(table, tuple) else np.asarray(table)[rows]
            dec._f32(f"rel.{l}", by_distance.size, np.ascontiguousarray(by_distance.T))

    def emit(self, op, dec: "HybridDecoder", l: int, buf: Dict[str, int], B: int, T: int) -> None:
        I, at, own = dec.ids, dec._offsets[l], self.kv_from is None
        src = l if own else self.kv_from
        rel_len = distance_buckets(self.rel_rows, self.rel_far, dec.cfg.max_seq_len).size if self.rel_rows else 0
        op("attn", OP_ATTN_GROUPED, buf["proj"], at["mix.q"], at["mix.k"] if own else -1, at.get("mix.v", -1), dec._in_rows[l], I[f"qnorm.{l}"],
           I[f"knorm.{src}"] if own or self.keys_are_values else -1, float_bits(dec.cfg.eps), I[f"temp {self.q_temp}"] if self.q_temp else -1,
           I[f"rel.{l}"] if self.rel_rows else -1, rel_len, I[f"keys.{src}"], -1 if self.keys_are_values else I[f"values.{src}"],
           I[f"kscale.{src}"] if self.keys_are_values else -1, I["pos"], buf["mix"], 0, self.out_width, B, T, self.heads, self.kv_heads, self.dim, self.vdim,
           float_bits(self.scale), int(self.sink))

    def out_operand(self, dec: "HybridDecoder", l: int, buf: Dict[str, int]) -> List[int]:
        gate = [buf["proj"], dec._offsets[l]["mix.g"], dec._in_rows[l]] if self.gated else [-1, 0, 0]
        return [buf["mix"], 0, self.out_width, -1, 0, 0] + gate


@dataclass(frozen=True)
class MatrixLstm:
    """Matrix memory per head with exponential input and forget gates and a running maximum."""
    heads: int
    dim: int
    vdim: int
    cap: float

    @classmethod
    def parse(cls, rec: Mapping[str, Any], rows_of: Callable[[str], Optional[int]]) -> "MatrixLstm":
        cap = float(rec["gate_cap"])
        if not cap > 0:
            raise ValueError("gate_cap must be positive")
        return cls(*_positive(rec, "heads", "dim", "vdim"), cap)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def tensors(self, d: int) -> Dict[str, Tuple[int, ...]]:
        H, n = self.heads, self.out_width
        return {"mix.q": (H * self.dim, d), "mix.k": (H * self.dim, d), "mix.v": (n, d), "mix.g": (n, d), "mix.i": (H, d), "mix.f": (H, d),
                "mix.i.b": (H,), "mix.f.b": (H,), "mix.norm": (n,), "mix.o": (d, n)}

    def fields(self) -> List[Tuple[str, int]]:
        t = self.tensors(1)
        return [(f"mix.{n}", t[f"mix.{n}"][0]) for n in "qkvgif"]

    def field_biases(self) -> List[str]:
        return ["mix.i", "mix.f"]

    def buffers(self, M: int) -> Dict[str, int]:
        return {"mix": M * self.out_width}

    def alloc(self, dec: "HybridDecoder", l: int) -> None:
        dec._f32(f"state.{l}", dec.B * self.out_width * self.dim)
        dec._f32(f"normaliser.{l}", 2 * dec.B * self.heads * (self.dim + 1))

    def load(self, dec: "HybridDecoder", l: int, get) -> None:
        dec._f32(f"onorm.{l}", self.out_width, get("mix.norm"))

    def emit(self, op, dec: "HybridDecoder", l: int, buf: Dict[str, int], B: int, T: int) -> None:
        I, at = dec.ids, dec._offsets[l]
        op("mlstm", OP_MLSTM, buf["proj"], *(at[f"mix.{n}"] for n in "qkvif"), dec._in_rows[l], float_bits(self.cap), float_bits(self.dim ** -0.5),
           I[f"state.{l}"], I[f"normaliser.{l}"], I["pos"], buf["mix"], 0, self.out_width, B, T, self.heads, self.dim, self.vdim, int(dec.dtype == "f32"))

    def out_operand(self, dec: "HybridDecoder", l: int, buf: Dict[str, int]) -> List[int]:
        return [buf["mix"], 0, self.out_width, dec.ids[f"onorm.{l}"], self.heads, float_bits(dec.cfg.eps), buf["proj"], dec._offsets[l]["mix.g"], dec._in_rows[l]]


RECURRENT = (GeneralDelta, MatrixLstm)
PAIR_CLAMP, PAIR_SILU = 0, 1            # how a feed-forward joins its (gate, up) pairs (op 83)


class Design(NamedTuple):
    """What an architecture's configuration means."""
    block: str                          # "parallel" | "post_norm"
    pair: int
    mixers: Mapping[str, Callable[[Mapping[str, Any], Callable[[str], Optional[int]]], Any]]      # layer type → parser


DESIGNS = {
    "Punilix": Design("parallel", PAIR_CLAMP, {"general_delta": GeneralDelta.parse, "latent_attention": LatentAttention.parse}),
    "Somipel": Design("post_norm", PAIR_SILU, {
        "attention": lambda rec, rows_of: GroupedAttention.parse(rec, rows_of, distance_bias=True, biases=True, gated=True),
        "attention_2": lambda rec, rows_of: GroupedAttention.parse(rec, rows_of, keys_are_values=True, sink=True),
        "mlstm": MatrixLstm.parse}),
}


@dataclass(frozen=True)
class DenseFF:
    ff: int
    limit: float             # of the clamped pair

    def tensors(self, d: int) -> Dict[str, Tuple[int, ...]]:
        return {"mlp.gate": (self.ff, d), "mlp.up": (self.ff, d), "mlp.down": (d, self.ff)}


@dataclass(frozen=True)
class TableExperts:
    ff: int
    limit: float
    experts: int
    top: int
    vocab: int

    def tensors(self, d: int) -> Dict[str, Tuple[int, ...]]:
        t: Dict[str, Tuple[int, ...]] = {"mlp.table": (self.vocab, self.top)}
        for e in range(self.experts):
            t.update({f"mlp.e{e}.gate": (self.ff, d), f"mlp.e{e}.up": (self.ff, d), f"mlp.e{e}.down": (d, self.ff)})
        return t


def parse_ff(rec: Optional[Mapping[str, Any]], vocab: int, pair: int = PAIR_CLAMP):
    if rec is None:
        return None
    if rec["kind"] == "dense":
        return DenseFF(*_positive(rec, "ff"), limit=float(rec["limit"]) if pair == PAIR_CLAMP else 0.0)
    if rec["kind"] == "moe" and pair == PAIR_CLAMP:
        experts, top = _positive(rec["router"], "experts", "top")
        if top > experts:
            raise ValueError("a token cannot use more experts than there are")
        return TableExperts(*_positive(rec["expert"], "ff"), limit=float(rec["expert"]["limit"]), experts=experts, top=top, vocab=vocab)
    raise ValueError(f"unknown feed-forward kind {rec['kind']!r}")


@dataclass(frozen=True)
class HybridConfig:
    vocab_size: int
    d_model: int
    norm_groups: int
    eps: float
    logit_softcap: float                 # 0 = none
    max_seq_len: int
    layers: Tuple[Tuple[Any, Any], ...] = field(default=())      # (mixer, feed-forward or None)
    block: str = "parallel"
    pair: int = PAIR_CLAMP
    residual_mult: float = 1.0           # of a sublayer's output, post_norm blocks

    @classmethod
    def parse(cls, rec: Mapping[str, Any], max_seq_len: int, rank_of: Callable[[str], Optional[int]]) -> "HybridConfig":
        """From a config.json record; `rank_of(tensor)` gives the first dimension of a weight that only its shape tells."""
        design = DESIGNS[rec["architecture"]]
        vocab, width = _positive(rec, "vocab", "width")
        groups, = _positive(dict(rec["norm"], groups=rec["norm"].get("groups", 1)), "groups")
        if width % groups:
            raise ValueError("norm.groups must divide width")
        if max_seq_len <= 0:
            raise ValueError("maxSeqLen must be > 0")
        layers = []
        for i, L in enumerate(rec["layers"]):
            if L["type"] not in design.mixers:
                raise ValueError(f"unknown layer type {L['type']!r}")
            mixer = design.mixers[L["type"]](L["mixer"], lambda name, i=i: rank_of(f"l{i}.{name}"))
            if isinstance(mixer, GroupedAttention):
                mixer.check_source(i, layers)
            layers.append((mixer, parse_ff(L["mlp"], vocab, design.pair)))
        return cls(vocab, width, groups, float(rec["norm"]["eps"]), float(rec.get("logit_softcap") or 0.0), int(max_seq_len), tuple(layers),
                   design.block, design.pair, float(rec["residual_mult"]) if design.block == "post_norm" else 1.0)

    def tensors(self) -> Dict[str, Tuple[int, ...]]:
        """Every tensor of a checkpoint and its shape."""
        d = self.d_model
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        for i, (mixer, ff) in enumerate(self.layers):
            out[f"l{i}.norm1"] = (d,)
            if self.block == "post_norm" and ff is not None:
                out[f"l{i}.norm2"] = (d,)
            for part in (mixer, ff):
                if part is not None:
                    out.update({f"l{i}.{n}": s for n, s in part.tensors(d).items()})
        out.update({"final.norm": (d,), "head": (self.vocab_size, d)})
        return out


# ───────────── the decoder ─────────────

class HybridDecoder(StreamDecoder):
    CHUNK_MIN = 2

    def __init__(self, cfg: HybridConfig, batch: int = 1, device: int = 0, id_base: int = 1 << 24, dtype: str = "bf16"):
        if dtype not in ("bf16", "f32"):
            raise ValueError("dtype must be 'bf16' or 'f32'")
        super().__init__(cfg, batch, device, id_base)
        self.dtype = dtype
        self.weight_dims: Dict[int, Tuple[int, int]] = {}         # bf16 object → (K, N)
        self.tables: Dict[str, np.ndarray] = {}
        self.REWINDS = not any(isinstance(m, RECURRENT) for m, _ in cfg.layers)
        # the input projection's rows per layer: every field starts at a multiple of eight, the gated pairs come last
        self._offsets: List[Dict[str, int]] = []
        self._in_rows: List[int] = []
        for mixer, _ in cfg.layers:
            at, n = {}, 0
            for name, rows in mixer.fields():
                at[name] = n
                n += pad8(rows)
            self._offsets.append(at)
            self._in_rows.append(n)
        for name, n in (("tok", self.B), ("pos", self.B), ("logits", self.B * cfg.vocab_size), ("next", self.B), ("r", self.B)):
            self._f32(name, n)
        self._step_buf = {name: self._f32("", n) for name, n in self._row_buffers(self.B).items()}
        self.ids["x"] = self._step_buf["x"]
        for l, (mixer, _) in enumerate(cfg.layers):
            mixer.alloc(self, l)

    def _row_buffers(self, M: int) -> Dict[str, int]:
        sizes = {"x": M * self.cfg.d_model}
        for l, (mixer, ff) in enumerate(self.cfg.layers):
            need = dict(mixer.buffers(M), proj=M * self._in_rows[l])
            if self.cfg.block == "post_norm":
                need.update(x2=M * self.cfg.d_model, s=M * self.cfg.d_model)
            if isinstance(ff, DenseFF):
                need["y"] = M * ff.ff
            if isinstance(ff, TableExperts):
                need["x2"] = M * self.cfg.d_model
            for name, n in need.items():
                sizes[name] = max(sizes.get(name, 0), n)
        return sizes

    # ── weights ──
    def _weight(self, name: str, K: int, N: int, parts: List[Tuple[str, int, int, int]], get) -> None:
        """A bf16 weight [N × K] from windows: (tensor, first row, row step, first column)."""
        i = self._new_id()
        _lib.check(self.lib.deepj_cuda_bf16_alloc(i, K, N))
        for tensor, row0, step, col0 in parts:
            a = get(tensor)
            if isinstance(a, tuple):         # (rows, cols, fill): generated on the device
                rows, cols, fill = a
                tmp = self._f32("", rows * cols)
                fill(tmp, rows * cols)
            else:
                rows, cols = a.shape
                tmp = self._f32("", rows * cols, a)
            _lib.check(self.lib.deepj_cuda_bf16_store(i, row0, step, col0, tmp, 0, rows, cols))
            self._release([tmp])
        self.ids[name] = i
        self.weight_dims[i] = (K, N)

    def _load(self, get: Callable[[str], Any], vec: Callable[[str], np.ndarray], table: Callable[[str], np.ndarray]) -> None:
        """`get` yields a matrix (or a recipe for one), `vec` a vector, `table` an integer table."""
        c = self.cfg
        d = c.d_model
        for l, (mixer, ff) in enumerate(c.layers):
            def mine(name, l=l):
                shape = self._shapes[f"l{l}.{name}"]
                return vec(f"l{l}.{name}") if len(shape) == 1 else get(f"l{l}.{name}")
            self._f32(f"norm.{l}", d, mine("norm1"))
            if c.block == "post_norm":
                self._load_post_norm(l, mixer, ff, mine)
                continue
            at, n = self._offsets[l], self._in_rows[l]
            parts = [(name, at[name], 1, 0) for name, _ in mixer.fields()]
            out = [("mix.o", 0, 1, 0)]
            k_out = mixer.out_width
            if isinstance(ff, DenseFF):
                parts += [("mlp.gate", n, 2, 0), ("mlp.up", n + 1, 2, 0)]
                n += 2 * ff.ff
                out.append(("mlp.down", 0, 1, pad8(k_out)))
                k_out = pad8(k_out) + ff.ff
            self._weight(f"in.{l}", d, n, parts, mine)
            self._weight(f"out.{l}", k_out, d, out, mine)
            mixer.load(self, l, mine)
            if isinstance(ff, TableExperts):
                t = np.asarray(table(f"l{l}.mlp.table"))
                if t.min() < 0 or t.max() >= ff.experts:
                    raise ValueError("the expert table names an expert that does not exist")
                self._f32(f"table.{l}", t.size, t.astype(np.float32))
                self.tables[f"table.{l}"] = t
                self._weight(f"up.{l}", d, ff.experts * 2 * ff.ff,
                             [(f"mlp.e{e}.{k}", e * 2 * ff.ff + j, 2, 0) for e in range(ff.experts) for j, k in enumerate(("gate", "up"))], mine)
                self._weight(f"down.{l}", ff.ff, ff.experts * d, [(f"mlp.e{e}.down", e * d, 1, 0) for e in range(ff.experts)], mine)
        self._f32("gF", d, vec("final.norm"))
        self._weight("head", d, c.vocab_size, [("head", 0, 1, 0)], get)
        self.loaded = True

    def _load_post_norm(self, l: int, mixer, ff: Optional[DenseFF], get) -> None:
        d, at, n = self.cfg.d_model, self._offsets[l], self._in_rows[l]
        self._weight(f"in.{l}", d, n, [(name, at[name], 1, 0) for name, _ in mixer.fields()], get)
        if mixer.field_biases():
            bias = np.zeros(n, dtype=np.float32)
            for name in mixer.field_biases():
                b = get(name + ".b")
                bias[at[name]:at[name] + b.size] = b
            self._f32(f"inbias.{l}", n, bias)
        self._weight(f"out.{l}", mixer.out_width, d, [("mix.o", 0, 1, 0)], get)
        mixer.load(self, l, get)
        if ff is not None:
            self._f32(f"norm2.{l}", d, get("norm2"))
            self._weight(f"up.{l}", d, 2 * ff.ff, [("mlp.gate", 0, 2, 0), ("mlp.up", 1, 2, 0)], get)
            self._weight(f"down.{l}", ff.ff, d, [("mlp.down", 0, 1, 0)], get)

    @property
    def _shapes(self) -> Dict[str, Tuple[int, ...]]:
        return self.cfg.tensors()

    def load_weights(self, get: Callable[[str], np.ndarray]) -> None:
        """Upload a checkpoint: `get(tensor)` returns it as numpy ([out × in] matrices), bf16 values widened to fp32."""
        shapes = self._shapes

        def checked(name: str) -> np.ndarray:
            a = np.asarray(get(name))
            if tuple(a.shape) != shapes[name]:
                raise IOError(f"Shape mismatch at parameter {name}: {tuple(a.shape)}, expected {shapes[name]}")
            return a

        self._f32("embed", self.cfg.vocab_size * self.cfg.d_model, checked("embed"))
        self._load(checked, checked, checked)

    def load_synthetic(self, seed: int, std: float) -> None:
        """Random weights of this architecture from the library's counter-based generator, one ordinal per tensor; gains
        are ones, biases zeros, table rows distinct."""
        names = list(self._shapes)
        shapes = self._shapes

        def filler(name):
            ordinal = names.index(name)
            return lambda buf, n: _lib.check(self.lib.deepj_cuda_synth_fill(buf, seed, ordinal, std, 0, n))

        def table(name):
            rng = np.random.default_rng(seed + names.index(name))
            rows, top = shapes[name]
            experts = self.cfg.layers[int(name.split(".")[0][1:])][1].experts
            return np.argsort(rng.random((rows, experts)), axis=1)[:, :top]

        emb = self._f32("embed", self.cfg.vocab_size * self.cfg.d_model)
        filler("embed")(emb, self.cfg.vocab_size * self.cfg.d_model)
        self._load(lambda n: (*shapes[n], filler(n)), lambda n: (np.ones if n.endswith(("norm", "norm1", "norm2")) else np.zeros)(shapes[n], dtype=np.float32), table)

    # ── streams ──
    def _linear(self, op, label, operand: List[int], k1: int, second: Optional[Tuple[int, int]], w: int, residual: Optional[Tuple[int, int]],
                out: Tuple[int, int], M: int, glu_row: int, glu: Optional[Tuple[int, int, float]] = None, softcap: float = 0.0,
                bias: int = -1, pair: int = PAIR_CLAMP, base: Optional[Tuple[int, int, float, int]] = None) -> None:
        """`operand`: x … ldgate of op 77; `second`, `residual`, `out`: (buffer, row stride); `glu` adds the clamp's limit; `base`:
        (residual buffer, row stride, factor, buffer of the sum), the staged row being base + factor · norm(x)."""
        x2, ldx2 = second if second else (-1, 0)
        res, ldr = residual if residual else (-1, 0)
        gb, ldg, limit = glu if glu else (-1, 0, 0.0)
        ints = [*operand, k1, x2, 0, ldx2, w, res, 0, ldr, out[0], 0, out[1], M, glu_row, float_bits(limit), gb, 0, ldg, float_bits(softcap), int(self.dtype == "f32")]
        if bias < 0 and pair == PAIR_CLAMP and base is None:
            op(label, OP_BF16_LINEAR, *ints)
        else:
            tail = [base[0], 0, base[1], float_bits(base[2]), base[3], 0, base[1]] if base else [-1, 0, 0, 0, -1, 0, 0]
            op(label, OP_BF16_LINEAR_SUM, *ints, bias, pair, *tail)

    def _blocks(self, op, buf: Dict[str, int], tok: int, B: int, T: int) -> None:
        """Embedding and every layer for B·T rows (row b·T + t is token pos[b] + t of sequence b)."""
        c, I, M, d = self.cfg, self.ids, B * T, self.cfg.d_model
        eps = float_bits(c.eps)
        op("embed", OP_EMBED_GATHER, I["embed"], tok, buf["x"], M, d, c.vocab_size)
        if c.block == "post_norm":
            self._post_norm_blocks(op, buf, B, T)
            return
        for l, (mixer, ff) in enumerate(c.layers):
            x = [buf["x"], 0, d, I[f"norm.{l}"], c.norm_groups, eps]
            n = self._in_rows[l]
            dense = isinstance(ff, DenseFF)
            self._linear(op, "in", x + [-1, 0, 0], d, None, I[f"in.{l}"], None, (buf["proj"], n), M, n, (buf["y"], ff.ff, ff.limit) if dense else None)
            mixer.emit(op, self, l, buf, B, T)
            if isinstance(ff, TableExperts):
                # the experts read the same residual as the mixer: the output projection writes beside it
                self._linear(op, "out", mixer.out_operand(self, l, buf), mixer.out_width, None, I[f"out.{l}"], (buf["x"], d), (buf["x2"], d), M, d)
                op("experts", OP_TABLE_EXPERTS, *x, tok, I[f"table.{l}"], c.vocab_size, ff.top, ff.experts, I[f"up.{l}"], I[f"down.{l}"], ff.ff,
                   float_bits(ff.limit), buf["x2"], 0, d, buf["x"], 0, d, d, M, int(self.dtype == "f32"))
            else:
                self._linear(op, "out", mixer.out_operand(self, l, buf), mixer.out_width, (buf["y"], ff.ff) if dense else None, I[f"out.{l}"],
                             (buf["x"], d), (buf["x"], d), M, d)

    def _post_norm_blocks(self, op, buf: Dict[str, int], B: int, T: int) -> None:
        """The residual rows alternate between two buffers: a projection reads one, adds the normed sublayer output in "s" that
        is still pending, and leaves the sum in the other."""
        c, I, M, d = self.cfg, self.ids, B * T, self.cfg.d_model
        eps, mult = float_bits(c.eps), c.residual_mult
        x, other = buf["x"], buf["x2"]
        pending: Optional[int] = None            # gain of the norm of what is in "s"

        def read(label, w, out, n, **more):
            nonlocal x, other
            if pending is None:
                operand, base = [x, 0, d, -1, 0, 0, -1, 0, 0], None
            else:
                operand, base = [buf["s"], 0, d, pending, c.norm_groups, eps, -1, 0, 0], (x, d, mult, other)
                x, other = other, x
            self._linear(op, label, operand, d, None, w, None, out, M, n, base=base, **more)

        for l, (mixer, ff) in enumerate(c.layers):
            n = self._in_rows[l]
            read("in", I[f"in.{l}"], (buf["proj"], n), n, bias=I.get(f"inbias.{l}", -1))
            mixer.emit(op, self, l, buf, B, T)
            self._linear(op, "out", mixer.out_operand(self, l, buf), mixer.out_width, None, I[f"out.{l}"], None, (buf["s"], d), M, d)
            pending = I[f"norm.{l}"]
            if ff is not None:
                read("up", I[f"up.{l}"], (-1, 0), 0, glu=(buf["y"], ff.ff, ff.limit), pair=c.pair)
                self._linear(op, "down", [buf["y"], 0, ff.ff, -1, 0, 0, -1, 0, 0], ff.ff, None, I[f"down.{l}"], None, (buf["s"], d), M, d)
                pending = I[f"norm2.{l}"]
        if pending is not None:
            op("sum", OP_NORM_ADD, buf["s"], 0, d, pending, eps, x, 0, d, float_bits(mult), buf["x"], d, M)

    def _head_ops(self, x: int, logits: int, rows: int) -> List[int]:
        s: List[int] = []
        self._head(lambda _label, *ints: s.extend(int(v) for v in ints), x, logits, rows)
        return s

    def _head(self, op, x: int, logits: int, rows: int) -> None:
        c, I = self.cfg, self.ids
        self._linear(op, "lm_head", [x, 0, c.d_model, I["gF"], c.norm_groups, float_bits(c.eps), -1, 0, 0], c.d_model, None, I["head"], None,
                     (logits, c.vocab_size), rows, c.vocab_size, softcap=c.logit_softcap)

    def _build(self, feed_back: bool, sampler: Optional[Tuple[int, float]] = None) -> np.ndarray:
        c, B, I = self.cfg, self.B, self.ids
        s: List[int] = []
        labels: List[str] = []
        bounds: List[Tuple[int, int]] = []

        def op(label, *ints):
            bounds.append((len(s), len(s) + len(ints)))
            s.extend(int(v) for v in ints)
            labels.append(label)

        self._blocks(op, self._step_buf, I["tok"], B, 1)
        self._head(op, I["x"], I["logits"], B)
        if sampler is None:
            op("argmax", OP_ARGMAX_ROWS, I["logits"], I["next"], B, c.vocab_size)
        else:
            op("sample", OP_SAMPLE_TOPK, I["logits"], I["r"], I["next"], B, c.vocab_size, sampler[0], float_bits(sampler[1]))
        op("advance", OP_ADD_SCALAR_INPLACE, I["pos"], float_bits(1.0), B)
        if feed_back:
            op("feed_back", OP_COPY, I["next"], 0, I["tok"], 0, B)
        self._op_labels, self._op_bounds = labels, bounds
        return np.asarray(s, dtype=np.int32)

    def _build_prefill(self, T: int) -> np.ndarray:
        B, I, P, d = self.B, self.ids, self._prefill_ids, self.cfg.d_model
        s: List[int] = []
        self._blocks(lambda _label, *ints: s.extend(int(v) for v in ints), P, P["tok"], B, T)
        for b in range(B):
            s.extend((OP_COPY, P["x"], (b * T + T - 1) * d, I["x"], b * d, d))
        s.extend((OP_ADD_SCALAR_INPLACE, I["pos"], float_bits(float(T)), B))
        return np.asarray(s, dtype=np.int32)

    def _chunk_tokens(self) -> int:
        top = max([ff.top for _, ff in self.cfg.layers if isinstance(ff, TableExperts)] or [1])
        return min(super()._chunk_tokens(), max(1, 65535 // (self.B * top)))

    def _prefill_sizes(self, M: int) -> Dict[str, int]:
        return dict(self._row_buffers(M), tok=M)
