"""The ops over bf16 weights (77-82), each mechanism alone, against plain numpy (tests/punilix_ref.py)."""
import numpy as np
import pytest

import punilix_ref as ref
from deepj_b200 import _lib
from deepj_b200.compute_graph import (OP_ATTN_LATENT, OP_ATTN_LATENT_CHUNK, OP_BF16_BLOCK_LINEAR, OP_BF16_LINEAR, OP_DELTA_RULE, OP_TABLE_EXPERTS, float_bits)
from deepj_b200.decoder import scaled_rope_tables
from test_q8_gpu import Dev

pytestmark = pytest.mark.gpu


def bf16(a):
    """Round to bf16, keep fp32 storage."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


class BfDev(Dev):
    def new(self):
        self.next += 1
        self.owned.append(self.next - 1)
        return self.next - 1

    def weight(self, K, N, parts):
        """parts: (matrix, first row, row step, first column)."""
        i = self.new()
        _lib.check(self.lib.deepj_cuda_bf16_alloc(i, K, N))
        for a, row0, step, col0 in parts:
            src = self.buf(a.size, a)
            _lib.check(self.lib.deepj_cuda_bf16_store(i, row0, step, col0, src, 0, a.shape[0], a.shape[1]))
        return i

    def latent(self, B, max_seq, width, half):
        i = self.new()
        _lib.check(self.lib.deepj_cuda_latent_alloc(i, B, max_seq, width, half))
        return i

    def error_word(self):
        import ctypes
        v = (ctypes.c_int64 * 6)()
        _lib.check(self.lib.deepj_cuda_stats(v, 6))
        return v[5]


@pytest.fixture()
def dev():
    d = BfDev(9 << 20)
    yield d
    assert d.error_word() == 0
    d.close()


def pad8(n):
    return (n + 7) // 8 * 8


def near(expected, actual, tol):
    scale = np.abs(expected).max()
    err = np.abs(expected - actual).max()
    assert np.all(np.isfinite(actual)) and err <= tol * scale, (err / scale, tol)


# rows: every GEMV pass size, several passes, the tensor-core form with one and several row tiles; K and N with and without
# whole tiles; 3 norm groups of unequal lane counts
@pytest.mark.parametrize("exact", [1, 0])
@pytest.mark.parametrize("M,k1,k2,N,glu,groups", [
    (1, 320, 0, 96, 96, 2), (1, 4096, 520, 512, 512, 1), (2, 120, 200, 72, 72, 3), (3, 264, 0, 160, 40, 1), (4, 1032, 0, 48, 0, 4), (7, 96, 40, 33, 33, 0),
    (16, 72, 0, 30, 8, 9), (17, 320, 0, 200, 64, 2), (40, 136, 72, 24, 24, 1), (129, 512, 0, 640, 320, 8), (300, 200, 104, 264, 264, 5), (513, 64, 0, 1048, 0, 1)])
def test_linear(dev, exact, M, k1, k2, N, glu, groups):
    rng = np.random.default_rng(M * 7 + k1 + N)
    x, gate = rng.standard_normal((M, k1)) * 2, rng.standard_normal((M, k1))
    x2 = rng.standard_normal((M, k2))
    gamma, eps = 1 + 0.3 * rng.standard_normal(k1), 1e-3
    K = pad8(k1) + k2 if k2 else k1
    W1, W2 = bf16(rng.standard_normal((N, k1)) / np.sqrt(k1)), bf16(rng.standard_normal((N, k2)) / np.sqrt(max(k2, 1)))
    use_gate, cap, limit = groups != 2, (5.0 if glu == N and k2 == 0 else 0.0), 0.75
    res = rng.standard_normal((M, max(glu, 1)))
    use_res = cap == 0.0

    s = ref.rms_norm(x, gamma, eps, groups) if groups else x
    if use_gate:
        s = s * ref.sigmoid(gate)
    rounded = (lambda a: a) if exact or M <= 16 else (lambda a: bf16(a).astype(np.float64))
    y = rounded(s) @ W1.T.astype(np.float64) + (rounded(x2) @ W2.T.astype(np.float64) if k2 else 0)
    plain = y[:, :glu] + (res[:, :glu] if use_res else 0)
    if cap:
        plain = cap * np.tanh(plain / cap)
    gated = ref.gated_clamp(y[:, glu::2], y[:, glu + 1::2], limit)

    ld, ld2, ldg, ldo = k1 + 3, k2 + 5, k1 + 1, glu + 2
    wide = lambda a, ld: np.pad(a, ((0, 0), (0, ld - a.shape[1])), constant_values=7.0)
    xb, gb = dev.buf(M * ld, wide(x, ld)), dev.buf(M * ldg, wide(gate, ldg))
    x2b = dev.buf(M * ld2, wide(x2, ld2)) if k2 else -1
    w = dev.weight(K, N, [(W1, 0, 1, 0)] + ([(W2, 0, 1, pad8(k1))] if k2 else []))
    rb = dev.buf(M * max(glu, 1), res) if use_res and glu else -1
    ob, yb = dev.buf(M * ldo), dev.buf(M * max(N - glu, 2))
    cmd = [OP_BF16_LINEAR, xb, 0, ld, dev.buf(k1, gamma) if groups else -1, groups, float_bits(eps), gb if use_gate else -1, 0, ldg, k1, x2b, 0, ld2, w,
           rb, 0, max(glu, 1), ob if glu else -1, 0, ldo, M, glu, float_bits(limit), yb if glu < N else -1, 0, (N - glu) // 2, float_bits(cap), exact]
    for _ in range(3):          # eager, captured, replayed
        dev.flush(cmd)
    tol = 2e-5 if exact or M <= 16 else 2e-3
    if glu:
        near(plain, dev.get(ob, M * ldo).reshape(M, ldo)[:, :glu], tol)
    if glu < N:
        near(gated, dev.get(yb, M * (N - glu) // 2).reshape(M, -1), tol)


def test_linear_refuses_what_does_not_add_up(dev):
    w = dev.weight(64, 16, [])
    x, o = dev.buf(256), dev.buf(64)
    good = [OP_BF16_LINEAR, x, 0, 64, -1, 0, 0, -1, 0, 0, 64, -1, 0, 0, w, -1, 0, 0, o, 0, 16, 1, 16, 0, -1, 0, 0, 0, 1]
    dev.flush(good)
    for at, value in ((10, 63), (3, 32), (5, 1), (20, 8), (22, 12), (22, 24), (21, 0), (28, 2), (1, 1 << 30), (14, x)):
        bad = list(good)
        bad[at] = value
        with pytest.raises(RuntimeError):
            dev.flush(bad)


@pytest.mark.parametrize("M,H,K,Nb", [(1, 1, 8, 5), (1, 5, 64, 80), (2, 3, 48, 64), (3, 32, 128, 136), (9, 2, 100, 7), (70, 4, 520, 33)])
def test_block_diagonal_linear(dev, M, H, K, Nb):
    rng = np.random.default_rng(H * K + Nb)
    xstr, ostr = K + 3, Nb + 2
    x = rng.standard_normal((M, H, xstr))
    W = bf16(rng.standard_normal((H, Nb, K)))
    want = np.einsum("mhk,hnk->mhn", x[..., :K], W)
    o = dev.buf(M * H * ostr)
    dev.flush([OP_BF16_BLOCK_LINEAR, dev.buf(x.size, x), 0, H * xstr, xstr, dev.weight(K, H * Nb, [(W.reshape(H * Nb, K), 0, 1, 0)]), H, o, 0, H * ostr, ostr, M])
    near(want, dev.get(o, M * H * ostr).reshape(M, H, ostr)[..., :Nb], 1e-5)


# ───────────── generalized delta rule ─────────────

@pytest.mark.parametrize("B,H,dim,rank,portions", [(1, 2, 64, 16, [1] * 9), (1, 1, 16, 3, [5, 2, 1, 7]), (2, 3, 40, 9, [2, 3, 1, 11]), (1, 2, 96, 32, [40, 1, 2]),
                                                   (1, 2, 128, 70, [33, 2, 1, 1, 3, 4, 64]), (1, 1, 200, 8, [3, 1, 12])])
def test_delta_rule(dev, B, H, dim, rank, portions):
    """Portions carry the state; the buffer holds garbage before position 0; one decay per channel runs close to each end
    of its range and one key is zero."""
    rng = np.random.default_rng(dim + rank)
    n, total = H * dim, sum(portions)
    names, at, ld = ["r", "k", "v", "a"], {}, 0
    for f in names:
        at[f] = ld
        ld += n + 5
    at["low"] = ld
    ld += rank + 1
    proj = rng.standard_normal((B, total, ld))
    proj[:, 2 % total, at["k"]:at["k"] + dim] = 0.0
    abias, w0 = rng.standard_normal(n), rng.standard_normal(n)
    w0[0], w0[-1] = 30.0, -30.0
    w2 = bf16(rng.standard_normal((n, rank)))
    field = lambda f, b, t: proj[b, t, at[f]:at[f] + n]
    want = np.zeros((B, total, n))
    for b in range(B):
        S = np.zeros((H, dim, dim))
        for t in range(total):
            decay = np.exp(-np.exp(-0.5) * ref.sigmoid(w2 @ np.tanh(proj[b, t, at["low"]:at["low"] + rank]) + w0))
            removal = ref.sigmoid(field("a", b, t) + abias)
            for h in range(H):
                c = slice(h * dim, (h + 1) * dim)
                S[h], want[b, t, c] = ref.delta_step(S[h], field("r", b, t)[c], field("k", b, t)[c], field("v", b, t)[c], decay[c], removal[c])
    state = dev.buf(B * n * dim, rng.standard_normal(B * n * dim) * 100)
    pb, w2b, ab, w0b, pos, out = (dev.buf(B * total * ld), dev.weight(rank, n, [(w2, 0, 1, 0)]), dev.buf(n, abias), dev.buf(n, w0), dev.buf(B), dev.buf(B * total * n))
    lo = 0
    for T in portions:
        chunk = np.ascontiguousarray(proj[:, lo:lo + T], dtype=np.float32)
        _lib.check(dev.lib.deepj_cuda_upload_buffer(pb, chunk.ctypes.data, chunk.size))
        p = np.full(B, lo, dtype=np.float32)
        _lib.check(dev.lib.deepj_cuda_upload_buffer(pos, p.ctypes.data, B))
        dev.flush([OP_DELTA_RULE, pb, at["r"], at["k"], at["v"], at["a"], at["low"], ld, ab, w2b, w0b, state, pos, out, 0, n, B, T, H, dim])
        near(want[:, lo:lo + T], dev.get(out, B * T * n).reshape(B, T, n), 2e-5)
        lo += T


# ───────────── latent attention ─────────────

def latent_reference(q, qc, kv, gamma, eps, R, rot, base, scaling, scale, rounded):
    """q [T, H, dim + rot], qc [T, H, R], kv [T, R + rot] of one sequence → weighted latents [T, H, R]."""
    T, H = qc.shape[:2]
    c = rounded(ref.rms_norm(kv[:, :R], gamma, eps))
    kr = rounded(ref.rotate_interleaved(kv[:, R:], np.arange(T), rot, base, scaling))
    qr = ref.rotate_interleaved(q[..., -rot:], np.arange(T), rot, base, scaling)
    out = np.zeros((T, H, R))
    for t in range(T):
        s = (qc[t] @ c[:t + 1].T + qr[t] @ kr[:t + 1].T) * scale
        out[t] = ref.softmax_rows(s) @ c[:t + 1]
    return out


@pytest.mark.parametrize("half", [0, 1])
@pytest.mark.parametrize("B,H,dim,rot,R,portions,scaled", [
    (1, 8, 64, 16, 64, [37, 1, 2, 60, 1, 1], True), (1, 3, 24, 8, 48, [1, 5, 2, 30], False), (2, 20, 32, 6, 40, [70, 3, 1], True), (1, 1, 16, 2, 10, [9, 40], False),
    (1, 32, 128, 64, 512, [130, 1, 2], True), (1, 5, 40, 24, 200, [65, 64, 1, 1], True), (1, 64, 16, 32, 128, [200, 1], False)])
def test_latent_attention(dev, half, B, H, dim, rot, R, portions, scaled):
    """Every row of every portion; one key far back and the newest key stand out for some queries, so a key that is missed
    or seen too early shows."""
    rng = np.random.default_rng(H * R + rot + half)
    total, W, qw = sum(portions), R + rot, H * (dim + rot)
    scaling = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0} if scaled else None
    base, scale, eps = 1000.0, 0.7 / np.sqrt(R), 1e-5
    kv = rng.standard_normal((B, total, W))
    q = rng.standard_normal((B, total, H, dim + rot))
    qc = rng.standard_normal((B, total, H, R))
    gamma = 1 + 0.2 * rng.standard_normal(R)
    c = ref.rms_norm(kv[..., :R], gamma, eps)
    for t in range(total):                       # queries that look for their own key, the first key and one in between
        for h, j in ((0, t), (H - 1, 0), (H // 2, t * 2 // 3)):
            if t % 3 == 0:
                qc[:, t, h] = c[:, j] * 12.0 / np.sqrt(R) / scale / np.sqrt(R)
    rounded = (lambda a: bf16(a).astype(np.float64)) if half else (lambda a: a)
    want = np.stack([latent_reference(q[b], qc[b], kv[b], gamma, eps, R, rot, base, scaling, scale, rounded) for b in range(B)])
    max_seq = total + 3
    cos, sin = scaled_rope_tables(rot, max_seq, base, scaling)
    cb, sb, gb, pos = dev.buf(cos.size, cos), dev.buf(sin.size, sin), dev.buf(R, gamma), dev.buf(B)
    cache = dev.latent(B, max_seq, W, half)
    qb, qcb, kvb, out = dev.buf(B * total * qw), dev.buf(B * total * H * R), dev.buf(B * total * (W + 4)), dev.buf(B * total * H * R)
    lo = 0

    def put(i, a):
        a = np.ascontiguousarray(a, dtype=np.float32)
        _lib.check(dev.lib.deepj_cuda_upload_buffer(i, a.ctypes.data, a.size))
    for T in portions:
        put(qb, q[:, lo:lo + T]); put(qcb, qc[:, lo:lo + T]); put(pos, np.full(B, lo))
        put(kvb, np.pad(kv[:, lo:lo + T], ((0, 0), (0, 0), (0, 4))))
        dev.flush([OP_ATTN_LATENT, qb, 0, qw, qcb, 0, H * R, kvb, 0, W + 4, gb, float_bits(eps), cache, pos, cb, sb, out, 0, H * R, B, T, H, dim, rot, R,
                   float_bits(scale)])
        near(want[:, lo:lo + T], dev.get(out, B * T * H * R).reshape(B, T, H, R), 1e-2 if half else 5e-5)
        lo += T


# ───────────── experts ─────────────

@pytest.mark.parametrize("exact", [1, 0])
@pytest.mark.parametrize("M,d,ff,experts,top", [(1, 64, 24, 4, 2), (3, 320, 96, 12, 1), (16, 72, 40, 3, 3), (40, 128, 64, 5, 2), (300, 64, 72, 7, 3), (700, 96, 32, 64, 2)])
def test_table_experts(dev, exact, M, d, ff, experts, top):
    rng = np.random.default_rng(M + d + ff)
    vocab, limit, eps, groups = 50, 0.8, 1e-4, 2
    x, res = rng.standard_normal((M, d)) * 3, rng.standard_normal((M, d))
    gamma = 1 + 0.2 * rng.standard_normal(d)
    table = np.stack([rng.permutation(experts)[:top] for _ in range(vocab)])
    table[7] = np.arange(experts - top, experts)
    tok = rng.integers(0, vocab, size=M)
    w = {"m.table": table}
    for e in range(experts):
        w.update({f"m.e{e}.gate": bf16(rng.standard_normal((ff, d)) / np.sqrt(d)), f"m.e{e}.up": bf16(rng.standard_normal((ff, d)) / np.sqrt(d)),
                  f"m.e{e}.down": bf16(rng.standard_normal((d, ff)) / np.sqrt(ff))})
    want = ref.table_experts(ref.rms_norm(x, gamma, eps, groups), tok, w, "m", limit)
    up = dev.weight(d, experts * 2 * ff, [(w[f"m.e{e}.{k}"], e * 2 * ff + j, 2, 0) for e in range(experts) for j, k in enumerate(("gate", "up"))])
    down = dev.weight(ff, experts * d, [(w[f"m.e{e}.down"], e * d, 1, 0) for e in range(experts)])
    o = dev.buf(M * d)
    cmd = [OP_TABLE_EXPERTS, dev.buf(M * d, x), 0, d, dev.buf(d, gamma), groups, float_bits(eps), dev.buf(M, tok), dev.buf(table.size, table), vocab, top, experts,
           up, down, ff, float_bits(limit), dev.buf(M * d, res), 0, d, o, 0, d, d, M, exact]
    for _ in range(2):
        dev.flush(cmd)
    near(want, dev.get(o, M * d).reshape(M, d) - res, 2e-5 if exact or M <= 16 else 2e-2)


@pytest.mark.parametrize("B,H,dim,rot,R,vdim,portions,scaled", [
    (1, 8, 64, 16, 64, 48, [150, 1, 70], True), (1, 3, 24, 8, 48, 16, [48, 200], False), (2, 5, 40, 24, 200, 72, [65, 64], True),
    (1, 4, 128, 64, 512, 128, [300, 2, 129], True), (1, 2, 192, 64, 128, 104, [130, 1], False)])
def test_latent_attention_of_prompt_chunks(dev, B, H, dim, rot, R, vdim, portions, scaled):
    """Op 82 (expanded keys and values) between portions that op 80 would take: same cache, values against the reference."""
    rng = np.random.default_rng(H * R + rot + vdim)
    total, W, qw = sum(portions), R + rot, H * (dim + rot)
    scaling = {"factor": 8.0, "original": 32, "fast": 16.0, "slow": 2.0} if scaled else None
    base, scale, eps = 5000.0, 1.3 / np.sqrt(dim + rot), 1e-5
    kv, q = rng.standard_normal((B, total, W)), rng.standard_normal((B, total, H, dim + rot))
    gamma = 1 + 0.2 * rng.standard_normal(R)
    uk, uv = bf16(rng.standard_normal((H, dim, R)) / np.sqrt(R)), bf16(rng.standard_normal((H, vdim, R)) / np.sqrt(R))
    c = bf16(ref.rms_norm(kv[..., :R], gamma, eps)).astype(np.float64)
    for t in range(total):                       # some queries look for their own key, the first key, or one in between
        for h, j in ((0, t), (H - 1, 0), (H // 2, t * 2 // 3)):
            if t % 3 == 0:
                for b in range(B):
                    k = uk[h] @ c[b, j]
                    q[b, t, h, :dim] = k * 10.0 / scale / (k @ k)
    want = np.zeros((B, total, H, vdim))
    for b in range(B):
        kr = bf16(ref.rotate_interleaved(kv[b, :, R:], np.arange(total), rot, base, scaling)).astype(np.float64)
        qr = ref.rotate_interleaved(q[b][..., -rot:], np.arange(total), rot, base, scaling)
        k_un, v = np.einsum("hdr,tr->thd", uk, c[b]), np.einsum("hdr,tr->thd", uv, c[b])
        for t in range(total):
            s = (np.einsum("hd,thd->ht", q[b, t, :, :dim], k_un[:t + 1]) + qr[t] @ kr[:t + 1].T) * scale
            want[b, t] = np.einsum("ht,thd->hd", ref.softmax_rows(s), v[:t + 1])
    max_seq = total + 5
    cos, sin = scaled_rope_tables(rot, max_seq, base, scaling)
    cb, sb, gb, pos = dev.buf(cos.size, cos), dev.buf(sin.size, sin), dev.buf(R, gamma), dev.buf(B)
    cache = dev.latent(B, max_seq, W, 1)
    wk, wv = dev.weight(R, H * dim, [(uk.reshape(-1, R), 0, 1, 0)]), dev.weight(R, H * vdim, [(uv.reshape(-1, R), 0, 1, 0)])
    qb, kvb, out = dev.buf(B * total * qw), dev.buf(B * total * W), dev.buf(B * total * H * vdim)
    lo = 0

    def put(i, a):
        a = np.ascontiguousarray(a, dtype=np.float32)
        _lib.check(dev.lib.deepj_cuda_upload_buffer(i, a.ctypes.data, a.size))
    for T in portions:
        put(qb, q[:, lo:lo + T]); put(pos, np.full(B, lo)); put(kvb, kv[:, lo:lo + T])
        dev.flush([OP_ATTN_LATENT_CHUNK, qb, 0, qw, kvb, 0, W, gb, float_bits(eps), cache, pos, cb, sb, wk, wv, out, 0, H * vdim, B, T, H, dim, rot, R, vdim,
                   float_bits(scale)])
        near(want[:, lo:lo + T], dev.get(out, B * T * H * vdim).reshape(B, T, H, vdim), 1.5e-2)
        lo += T
