"""Decoders whose configuration lists their layers one by one (Punilix): every layer names its mixer and its feed-forward.

A layer is parallel: with h = norm(x), x ← x + mixer(h) + feed_forward(h).  All projections that read h are one bf16
weight and one launch (op 77: the norm is staged with the row, the gated feed-forward's pairs are finished in the
epilogue), and so are the two that write the residual: [W_o ‖ W_down] over [mixed heads, gated values].  Between them the
mixer runs its own ops:

  general_delta      op 79 (the recurrence); its head norm and output gate are part of the output projection's staging
  latent_attention   W_uq on the normed query latent, the queries taken into the latent space (op 78), op 80, values (op 78)

A feed-forward is dense or table-routed experts (op 81), or absent.  A token step and a prompt chunk record the same
sequence of ops with different row counts.  `MIXERS` maps a configuration's layer type to its class: another mechanism is
another class with the same five methods.

dtype "bf16": bf16 weights and latent cache; rows are fp32 between ops, the many-row kernels round their operand to bf16.
dtype "f32": the same weights, every product in fp32, fp32 cache.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Mapping, Optional, Tuple

import numpy as np

from . import _lib
from .compute_graph import (OP_ADD_SCALAR_INPLACE, OP_ARGMAX_ROWS, OP_ATTN_LATENT, OP_ATTN_LATENT_CHUNK, OP_BF16_BLOCK_LINEAR, OP_BF16_LINEAR, OP_COPY, OP_DELTA_RULE,
                            OP_EMBED_GATHER, OP_SAMPLE_TOPK, OP_TABLE_EXPERTS, float_bits)
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
    def parse(cls, rec: Mapping[str, Any], rank: Optional[int]) -> "GeneralDelta":
        heads, dim = _positive(rec, "heads", "dim")
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
    def parse(cls, rec: Mapping[str, Any], rank: Optional[int]) -> "LatentAttention":
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
MIXERS = {"general_delta": GeneralDelta, "latent_attention": LatentAttention}
RECURRENT = (GeneralDelta,)


@dataclass(frozen=True)
class DenseFF:
    ff: int
    limit: float

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


def parse_ff(rec: Optional[Mapping[str, Any]], vocab: int):
    if rec is None:
        return None
    if rec["kind"] == "dense":
        return DenseFF(*_positive(rec, "ff"), limit=float(rec["limit"]))
    if rec["kind"] == "moe":
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

    @classmethod
    def parse(cls, rec: Mapping[str, Any], max_seq_len: int, rank_of: Callable[[str], Optional[int]]) -> "HybridConfig":
        """From a config.json record; `rank_of(tensor)` gives the first dimension of a weight that only its shape tells."""
        vocab, width = _positive(rec, "vocab", "width")
        groups, = _positive(rec["norm"], "groups")
        if width % groups:
            raise ValueError("norm.groups must divide width")
        if max_seq_len <= 0:
            raise ValueError("maxSeqLen must be > 0")
        layers = []
        for i, L in enumerate(rec["layers"]):
            if L["type"] not in MIXERS:
                raise ValueError(f"unknown layer type {L['type']!r}")
            layers.append((MIXERS[L["type"]].parse(L["mixer"], rank_of(f"l{i}.mix.w1")), parse_ff(L["mlp"], vocab)))
        return cls(vocab, width, groups, float(rec["norm"]["eps"]), float(rec.get("logit_softcap") or 0.0), int(max_seq_len), tuple(layers))

    def tensors(self) -> Dict[str, Tuple[int, ...]]:
        """Every tensor of a checkpoint and its shape."""
        d = self.d_model
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        for i, (mixer, ff) in enumerate(self.layers):
            out[f"l{i}.norm1"] = (d,)
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
        self._load(lambda n: (*shapes[n], filler(n)), lambda n: (np.ones if n.endswith(("norm", "norm1")) else np.zeros)(shapes[n], dtype=np.float32), table)

    # ── streams ──
    def _linear(self, op, label, operand: List[int], k1: int, second: Optional[Tuple[int, int]], w: int, residual: Optional[Tuple[int, int]],
                out: Tuple[int, int], M: int, glu_row: int, glu: Optional[Tuple[int, int, float]] = None, softcap: float = 0.0) -> None:
        x2, ldx2 = second if second else (-1, 0)
        res, ldr = residual if residual else (-1, 0)
        gb, ldg, limit = glu if glu else (-1, 0, 0.0)
        op(label, OP_BF16_LINEAR, *operand, k1, x2, 0, ldx2, w, res, 0, ldr, out[0], 0, out[1], M, glu_row, float_bits(limit), gb, 0, ldg,
           float_bits(softcap), int(self.dtype == "f32"))

    def _blocks(self, op, buf: Dict[str, int], tok: int, B: int, T: int) -> None:
        """Embedding and every layer for B·T rows (row b·T + t is token pos[b] + t of sequence b)."""
        c, I, M, d = self.cfg, self.ids, B * T, self.cfg.d_model
        eps = float_bits(c.eps)
        op("embed", OP_EMBED_GATHER, I["embed"], tok, buf["x"], M, d, c.vocab_size)
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
