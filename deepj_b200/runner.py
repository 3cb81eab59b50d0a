"""The model-independent half of a decoder: device buffers, token steps, prompt chunks, sampling and timing.

A decoder owns its weights, its cache (and recurrent state) and a recorded command stream per shape of work; running
it means flushing those streams through `deepj_cuda_flush_ops` (the library turns a repeated stream into a CUDA
graph).  `StreamDecoder` holds everything that does not depend on the architecture; a subclass records the streams:

  `_build(feed_back, sampler)`   one token of every sequence: embedding … logits, pick, position advance
  `_build_prefill(T)`            a chunk of T tokens of every sequence; leaves the chunk's hidden rows in the "x" chunk
                                 buffer and the last token's in the decode buffer
  `_head_ops(x, logits, rows)`   final norm and LM head on `rows` hidden rows
  `_prefill_sizes(M)`            float buffers a chunk of M rows needs: at least "tok" and "x"
"""
from __future__ import annotations

import ctypes
from typing import Dict, List, Optional, Tuple

import numpy as np

from . import _lib
from .compute_graph import OP_ARGMAX_ROWS, OP_EMBED_GATHER, OP_SAMPLE_TOPK, float_bits


class StreamDecoder:
    """Owns the device-side objects of one model and the streams that run it.

    Buffer ids are taken from `id_base` upwards so they never collide with the ids a
    `ComputeGraph` hands out (those start at 0).
    """

    PREFILL_CHUNK = 2048     # prompt tokens per sequence and pass of the many-row path (enough 128 × 256 tiles for the GEMM to pair them)
    CHUNK_MIN = 32           # prompts shorter than this take one decode step per position
    REWINDS = True           # a position may be set back: everything a step reads of the past sits in a cache indexed by position
    HEAD_ROWS = 64           # hidden rows per pass of the LM head when logits of many positions are wanted

    def __init__(self, cfg, batch: int, device: int, id_base: int):
        self.cfg = cfg
        self.B = int(batch)
        self.lib = _lib.load()
        _lib.check(self.lib.deepj_cuda_init(device))
        self._next_id = id_base
        self._owned: List[int] = []
        self.ids: Dict[str, int] = {}
        self.loaded = False
        self._stream_host: Optional[np.ndarray] = None
        self._stream_dev: Optional[np.ndarray] = None
        self._op_labels: List[str] = []
        self._op_bounds: List[Tuple[int, int]] = []
        self._pin_ptr = None
        self._prefill_ids: Dict[str, int] = {}
        self._prefill_cap = 0
        self._prefill_streams: Dict[int, np.ndarray] = {}
        self.position = 0

    # ── what a subclass records ──
    def _build(self, feed_back: bool, sampler: Optional[Tuple[int, float]] = None) -> np.ndarray:
        raise NotImplementedError

    def _build_prefill(self, T: int) -> np.ndarray:
        raise NotImplementedError

    def _head_ops(self, x: int, logits: int, rows: int) -> List[int]:
        raise NotImplementedError

    def _prefill_sizes(self, M: int) -> Dict[str, int]:
        raise NotImplementedError

    def _chunk_tokens(self) -> int:
        """The most tokens per sequence one chunk may carry."""
        return min(self.PREFILL_CHUNK, max(1, 65535 // self.B))

    def _upload_chunk(self, tokens: np.ndarray) -> None:
        """Token ids [B × T] of the next chunk (row b·T + t)."""
        self._upload(self._prefill_ids["tok"], tokens.astype(np.float32).reshape(-1))

    # ── id / buffer helpers ──
    def _new_id(self) -> int:
        i = self._next_id
        self._next_id += 1
        self._owned.append(i)
        return i

    def _f32(self, name: str, n: int, data: Optional[np.ndarray] = None) -> int:
        i = self._new_id()
        ids = (ctypes.c_int32 * 1)(i)
        sizes = (ctypes.c_int32 * 1)(n)
        _lib.check(self.lib.deepj_cuda_alloc_buffers(ids, sizes, 1))
        if data is not None:
            self._upload(i, data)
        if name:
            self.ids[name] = i
        return i

    def _upload(self, buf_id: int, data: np.ndarray) -> None:
        data = np.ascontiguousarray(data, dtype=np.float32)
        _lib.check(self.lib.deepj_cuda_upload_buffer(buf_id, data.ctypes.data, data.size))

    def _download(self, buf_id: int, n: int) -> np.ndarray:
        out = np.empty(n, dtype=np.float32)
        _lib.check(self.lib.deepj_cuda_download_buffer(buf_id, out.ctypes.data, n))
        return out

    def _release(self, ids: List[int]) -> None:
        arr = (ctypes.c_int32 * len(ids))(*ids)
        _lib.check(self.lib.deepj_cuda_release_buffers(arr, len(ids)))
        for i in ids:
            if i in self._owned:
                self._owned.remove(i)

    # ── streams ──
    def _streams(self):
        if not self.loaded:
            raise RuntimeError("weights are not loaded")
        if self._stream_host is None:
            self._stream_dev = self._build(feed_back=True)
            self._stream_host = self._build(feed_back=False)
        return self._stream_host, self._stream_dev

    # ── stepping ──
    def reset(self) -> None:
        """Start every sequence at position 0 (cache contents are overwritten as it refills)."""
        self._upload(self.ids["pos"], np.zeros(self.B, dtype=np.float32))
        self.position = 0

    def set_position(self, position: int) -> None:
        """Rewind (or advance) every sequence to `position`; cache rows at and beyond it are
        overwritten by the following steps."""
        if position < 0 or position > self.cfg.max_seq_len:
            raise ValueError(f"position {position} outside 0..{self.cfg.max_seq_len}")
        if not self.REWINDS and position not in (0, self.position):
            raise ValueError("a recurrent state cannot be moved to another position: reset() and feed the tokens again")
        self._upload(self.ids["pos"], np.full(self.B, float(position), dtype=np.float32))
        self.position = int(position)

    def _pinned(self) -> Tuple[np.ndarray, np.ndarray]:
        """Page-locked staging for the ids going up and the picks coming down each step ([B] floats each)."""
        if self._pin_ptr is None:
            ptr = ctypes.c_void_p()
            _lib.check(self.lib.deepj_cuda_pinned_alloc(ctypes.byref(ptr), 8 * self.B))
            self._pin_ptr = ptr
            buf = (ctypes.c_float * (2 * self.B)).from_address(ptr.value)
            arr = np.frombuffer(buf, dtype=np.float32)
            self._pin_tok, self._pin_next = arr[:self.B], arr[self.B:]
        return self._pin_tok, self._pin_next

    def set_tokens(self, tokens) -> None:
        t = np.asarray(tokens, dtype=np.int64).reshape(-1)
        if t.size != self.B:
            raise ValueError(f"expected {self.B} token ids, got {t.size}")
        # Embedding.forward range check (transformer/embeddings/Embedding.java:30-32)
        if t.min() < 0 or t.max() >= self.cfg.vocab_size:
            bad = t[(t < 0) | (t >= self.cfg.vocab_size)][0]
            raise ValueError(f"Token id out of range: {int(bad)}")
        tok, _ = self._pinned()
        tok[:] = t
        _lib.check(self.lib.deepj_cuda_upload_buffer(self.ids["tok"], tok.ctypes.data, self.B))

    def step(self, tokens) -> np.ndarray:
        """One token per sequence through host buffers: upload the ids, flush the
        stream (synchronous), download the greedy picks."""
        if self.position >= self.cfg.max_seq_len:
            raise ValueError(f"seqLen {self.position + 1} exceeds maxSeqLen {self.cfg.max_seq_len}")
        host, _ = self._streams()
        self.set_tokens(tokens)
        # enqueue the stream behind the upload and let the download's synchronisation be the only one of the step
        _lib.check(self.lib.deepj_cuda_flush_ops_async(host.ctypes.data, host.size))
        self.position += 1
        _, nxt = self._pinned()
        _lib.check(self.lib.deepj_cuda_download_buffer(self.ids["next"], nxt.ctypes.data, self.B))
        return nxt.astype(np.int64)

    def step_device(self, n_steps: int = 1, sync: bool = True) -> None:
        """n greedy steps with the picked token fed back on the device (no host copies)."""
        if self.position + n_steps > self.cfg.max_seq_len:
            raise ValueError(f"seqLen {self.position + n_steps} exceeds maxSeqLen {self.cfg.max_seq_len}")
        _, dev = self._streams()
        for _ in range(n_steps):
            _lib.check(self.lib.deepj_cuda_flush_ops_async(dev.ctypes.data, dev.size))
        self.position += n_steps
        if sync:
            _lib.check(self.lib.deepj_cuda_synchronize())

    def logits(self) -> np.ndarray:
        """The logits row(s) behind the last pick, [B × vocab]."""
        return self._download(self.ids["logits"], self.B * self.cfg.vocab_size).reshape(self.B, self.cfg.vocab_size)

    def next_tokens(self) -> np.ndarray:
        return self._download(self.ids["next"], self.B).astype(np.int64)

    def _head_stream(self) -> np.ndarray:
        """Final norm + LM head + greedy pick on the hidden state in the decode buffer."""
        I = self.ids
        return np.asarray(self._head_ops(I["x"], I["logits"], self.B) + [OP_ARGMAX_ROWS, I["logits"], I["next"], self.B, self.cfg.vocab_size],
                          dtype=np.int32)

    def _check_tokens(self, p: np.ndarray) -> None:
        if np.any(p < 0) or np.any(p >= self.cfg.vocab_size):
            raise ValueError(f"Token id out of range: {int(p[(p < 0) | (p >= self.cfg.vocab_size)][0])}")
        if self.position + p.shape[1] > self.cfg.max_seq_len:
            raise ValueError(f"seqLen {self.position + p.shape[1]} exceeds maxSeqLen {self.cfg.max_seq_len}")

    def _run_chunk(self, p: np.ndarray) -> None:
        """One chunk [B × T] through the many-row path (buffers of at least T tokens per sequence exist)."""
        T = p.shape[1]
        if T not in self._prefill_streams:
            if len(self._prefill_streams) >= 256:
                self._prefill_streams.clear()
            self._prefill_streams[T] = self._build_prefill(T)
        st = self._prefill_streams[T]
        self._upload_chunk(p)
        _lib.check(self.lib.deepj_cuda_flush_ops(st.ctypes.data, st.size))
        self.position += T

    def prefill(self, prompts, chunked: Optional[bool] = None) -> np.ndarray:
        """Feed the prompt (every sequence the same length) from the current position; returns the greedy pick after its
        last token.  Prompts of CHUNK_MIN tokens or more go through the many-row path in chunks of PREFILL_CHUNK tokens
        per sequence (tensor-core GEMMs, chunk attention); shorter ones one decode step per position."""
        p = np.asarray(prompts, dtype=np.int64).reshape(self.B, -1)
        T_all = p.shape[1]
        if chunked is None:
            chunked = T_all >= self.CHUNK_MIN
        if not chunked or T_all == 0:
            nxt = None
            for t in range(T_all):
                nxt = self.step(p[:, t])
            return nxt
        if not self.loaded:
            raise RuntimeError("weights are not loaded")
        self._check_tokens(p)
        C = min(self._chunk_tokens(), T_all)
        self._ensure_prefill_buffers(C)
        for lo in range(0, T_all, C):
            self._run_chunk(p[:, lo:lo + C])
        hs = self._head_stream()
        _lib.check(self.lib.deepj_cuda_flush_ops(hs.ctypes.data, hs.size))
        return self.next_tokens()

    def feed(self, tokens, want=()) -> np.ndarray:
        """Append `tokens` to the one sequence, from the cache and state that earlier calls left, and return the logits
        behind the places `want` (indices into `tokens`): [len(want) × vocab].  One token is a decode step, more are a
        chunk (or steps, below CHUNK_MIN): the paths `generate` takes."""
        if self.B != 1:
            raise ValueError("feed drives one sequence")
        p = np.asarray(tokens, dtype=np.int64).reshape(1, -1)
        V, T_all = self.cfg.vocab_size, p.shape[1]
        want = [int(i) for i in want]
        if any(i < 0 or i >= T_all for i in want):
            raise ValueError("a wanted place lies outside the tokens")
        rows: Dict[int, np.ndarray] = {}
        if T_all == 0:
            return np.empty((0, V), dtype=np.float32)
        if T_all < max(2, self.CHUNK_MIN):
            for t in range(T_all):
                self.step(p[:, t])
                if t in want:
                    rows[t] = self.logits()[0]
        else:
            self._streams()
            self._check_tokens(p)
            C = min(self._chunk_tokens(), T_all)
            self._ensure_prefill_buffers(C)
            for lo in range(0, T_all, C):
                self._run_chunk(p[:, lo:lo + C])
                here = sorted({i for i in want if lo <= i < lo + C})
                for j in range(0, len(here), self.HEAD_ROWS):
                    part = here[j:j + self.HEAD_ROWS]
                    for i, row in zip(part, self._chunk_logits([i - lo for i in part])):
                        rows[i] = row
        return np.stack([rows[i] for i in want]) if want else np.empty((0, V), dtype=np.float32)

    def _chunk_logits(self, rows: List[int]) -> np.ndarray:
        """Logits of some hidden rows of the chunk that has just run."""
        I, d, V, n = self.ids, self.cfg.d_model, self.cfg.vocab_size, len(rows)
        if "want" not in I:
            self._f32("want", self.HEAD_ROWS)
            self._f32("want_x", self.HEAD_ROWS * d)
            self._f32("want_logits", self.HEAD_ROWS * V)
        self._upload(I["want"], np.asarray(rows, dtype=np.float32))
        s = [OP_EMBED_GATHER, self._prefill_ids["x"], I["want"], I["want_x"], n, d, self._prefill_cap]
        s = np.asarray(s + self._head_ops(I["want_x"], I["want_logits"], n), dtype=np.int32)
        _lib.check(self.lib.deepj_cuda_flush_ops(s.ctypes.data, s.size))
        return self._download(I["want_logits"], n * V).reshape(n, V)

    def _ensure_prefill_buffers(self, C: int) -> None:
        if self._prefill_cap >= C:
            return
        if self._prefill_ids:
            self._release(list(self._prefill_ids.values()))
        self._prefill_ids = {name: self._f32("", n) for name, n in self._prefill_sizes(self.B * C).items()}
        self._prefill_cap = C
        self._prefill_streams = {}

    # ── generation ──
    def generate(self, prompt, max_new_tokens: int, temperature: float = 1.0, top_k: int = 40, seed: int = 0) -> np.ndarray:
        """TextGenerator.generate for batch 1 (models/TextGenerator.java:66-151) with the draw on the device:
        temperature / top-k sampling, one `java.util.Random(seed).nextFloat()` per new token, the logits never
        leave the GPU.  topK = 0 means the whole vocabulary, as in the reference (TextGenerator.java:111-115)."""
        from .jrandom import JavaRandom
        if max_new_tokens < 0:
            raise ValueError("maxNewTokens must be >= 0")
        if not temperature > 0.0:
            raise ValueError("temperature must be > 0")
        if top_k < 0:
            raise ValueError("topK must be >= 0")
        if self.B != 1:
            raise ValueError("generate drives one sequence")
        rnd = JavaRandom(seed)
        c, I = self.cfg, self.ids
        pick = np.asarray([OP_SAMPLE_TOPK, I["logits"], I["r"], I["next"], 1, c.vocab_size, top_k, float_bits(float(temperature))], dtype=np.int32)
        step = self._build(feed_back=False, sampler=(top_k, float(temperature)))
        self.reset()
        self.prefill(np.asarray(prompt).reshape(1, -1))              # leaves the last prompt position's logits on the device
        out = []
        for i in range(max_new_tokens):
            self._upload(I["r"], np.asarray([rnd.next_float()], dtype=np.float32))
            if i == 0:
                _lib.check(self.lib.deepj_cuda_flush_ops(pick.ctypes.data, pick.size))
            else:
                if self.position + 1 > c.max_seq_len:
                    raise ValueError(f"seqLen {self.position + 1} exceeds maxSeqLen {c.max_seq_len}")
                self._upload(I["tok"], np.asarray([out[-1]], dtype=np.float32))
                _lib.check(self.lib.deepj_cuda_flush_ops(step.ctypes.data, step.size))
                self.position += 1
            out.append(int(self.next_tokens()[0]))
        return np.asarray(out, dtype=np.int64)

    def generate_greedy(self, prompt, max_new_tokens: int, keep_logits: bool = False):
        """TextGenerator.generate with topK = 1 (models/TextGenerator.java:66-100)
        for batch 1: returns the new token ids (and the logits row behind each)."""
        if max_new_tokens < 0:
            raise ValueError("maxNewTokens must be >= 0")
        if self.B != 1:
            raise ValueError("generate_greedy drives one sequence")
        self.reset()
        nxt = self.prefill(np.asarray(prompt).reshape(1, -1))
        out, rows = [], []
        for i in range(max_new_tokens):
            if keep_logits:
                rows.append(self.logits()[0].copy())
            tok = int(nxt[0])
            out.append(tok)
            if i + 1 < max_new_tokens:
                nxt = self.step([tok])
        return (np.asarray(out, dtype=np.int64), np.stack(rows) if rows else None) if keep_logits else np.asarray(out, dtype=np.int64)

    # ── measurement ──
    def profile_step(self):
        """Device time of every op of one token step, run op by op as the per-operator stream (also when the
        decoder itself steps with the single-kernel op): [(label, ms)]."""
        if not self.loaded:
            raise RuntimeError("weights are not loaded")
        host = self._build(feed_back=False)
        n = len(self._op_labels) + 1
        ms = np.zeros(n, dtype=np.float32)
        cnt = ctypes.c_int32(0)
        _lib.check(self.lib.deepj_cuda_profile_ops(host.ctypes.data, host.size, ms.ctypes.data, n, ctypes.byref(cnt)))
        self.position += 1
        return list(zip(self._op_labels, ms[: cnt.value].tolist()))

    def time_ops(self, labels, iters: int = 20, warmup: int = 3) -> Tuple[float, int]:
        """Device time of the ops whose label is in `labels`, run back to back as their own stream
        (graph-replayed like the full step, at the current position): (ms per pass, ops per pass)."""
        full = self._build(feed_back=False)
        keep = [full[a:b] for lbl, (a, b) in zip(self._op_labels, self._op_bounds) if lbl in labels]
        if not keep:
            return 0.0, 0
        sub = np.ascontiguousarray(np.concatenate(keep))
        for _ in range(max(warmup, 3)):
            _lib.check(self.lib.deepj_cuda_flush_ops(sub.ctypes.data, sub.size))
        _lib.check(self.lib.deepj_cuda_timer_begin())
        for _ in range(iters):
            _lib.check(self.lib.deepj_cuda_flush_ops_async(sub.ctypes.data, sub.size))
        ms = ctypes.c_float(0)
        _lib.check(self.lib.deepj_cuda_timer_end(ctypes.byref(ms)))
        return ms.value / iters, len(keep)

    def stats(self) -> Dict[str, int]:
        v = (ctypes.c_int64 * 6)()
        _lib.check(self.lib.deepj_cuda_stats(v, 6))
        return {"eager_launches": v[0], "graph_replays": v[1], "graphs_captured": v[2],
                "kernels_per_replay": v[3], "workspace_bytes": v[4], "device_error": v[5]}

    def close(self) -> None:
        if self._pin_ptr is not None:
            self.lib.deepj_cuda_pinned_free(self._pin_ptr)
            self._pin_ptr = None
        if self._owned:
            self._release(list(self._owned))
