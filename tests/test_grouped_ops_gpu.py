"""The ops of the post-norm models (83-86), each mechanism alone, against plain numpy (tests/somipel_ref.py)."""
import numpy as np
import pytest

import somipel_ref as ref
from deepj_b200.compute_graph import OP_ATTN_GROUPED, OP_BF16_LINEAR_SUM, OP_MLSTM, OP_NORM_ADD, float_bits
from deepj_b200.hybrid import distance_buckets
from test_bf16_ops_gpu import bf16, dev, near, pad8  # noqa: F401  (dev is a fixture)

pytestmark = pytest.mark.gpu


# every GEMV pass size, several passes, one and several row tiles of the many-row forms; widths that are no multiple of four
@pytest.mark.parametrize("exact", [1, 0])
@pytest.mark.parametrize("M,k,N,glu", [(1, 320, 96, 96), (1, 4096, 512, 0), (2, 122, 72, 72), (3, 264, 160, 40), (4, 90, 48, 0), (7, 96, 33, 33), (16, 72, 30, 8),
                                       (17, 320, 200, 64), (129, 514, 640, 320), (300, 200, 264, 264)])
def test_linear_sum(dev, exact, M, k, N, glu):
    rng = np.random.default_rng(M * 7 + k + N)
    x, base = rng.standard_normal((M, k)) * 3, rng.standard_normal((M, k))
    gamma, eps, mult = 1 + 0.3 * rng.standard_normal(k), 1e-3, 0.35
    W, bias = bf16(rng.standard_normal((N, k)) / np.sqrt(k)), rng.standard_normal(max(glu, 1))
    row = base + mult * ref.rms(x, eps) * gamma
    y = (row if exact or M <= 16 else bf16(row).astype(np.float64)) @ W.T.astype(np.float64)
    plain, gated = y[:, :glu] + bias[:glu], ref.silu(y[:, glu::2]) * y[:, glu + 1::2]
    ld, ldb, ldo, lds = k + 3, k + 2, glu + 2, k + 1
    wide = lambda a, n: np.pad(a, ((0, 0), (0, n - a.shape[1])), constant_values=7.0)
    xb, bb, sb = dev.buf(M * ld, wide(x, ld)), dev.buf(M * ldb, wide(base, ldb)), dev.buf(M * lds)
    w, ob, yb = dev.weight(k, N, [(W, 0, 1, 0)]), dev.buf(M * ldo), dev.buf(M * max(N - glu, 2))
    cmd = [OP_BF16_LINEAR_SUM, xb, 0, ld, dev.buf(k, gamma), 1, float_bits(eps), -1, 0, 0, k, -1, 0, 0, w, -1, 0, 0, ob if glu else -1, 0, ldo, M, glu, 0,
           yb if glu < N else -1, 0, (N - glu) // 2, 0, exact, dev.buf(max(glu, 1), bias) if glu else -1, 1, bb, 0, ldb, float_bits(mult), sb, 0, lds]
    for _ in range(3):          # eager, captured, replayed
        dev.flush(cmd)
    tol = 2e-5 if exact or M <= 16 else 2e-3
    if glu:
        near(plain, dev.get(ob, M * ldo).reshape(M, ldo)[:, :glu], tol)
    if glu < N:
        near(gated, dev.get(yb, M * (N - glu) // 2).reshape(M, -1), tol)
    near(row, dev.get(sb, M * lds).reshape(M, lds)[:, :k], 1e-6)
    assert np.array_equal(dev.get(bb, M * ldb).reshape(M, ldb)[:, :k], base.astype(np.float32))
    out = dev.buf(M * k, base)
    dev.flush([OP_NORM_ADD, xb, 0, ld, cmd[4], float_bits(eps), out, 0, k, float_bits(mult), out, k, M])       # in place
    near(row, dev.get(out, M * k).reshape(M, k), 1e-6)
    for at, value in ((30, 2), (33, k - 1), (35, bb), (31, 1 << 30), (7, xb), (5, 0), (37, k - 1)):
        bad = list(cmd)
        bad[at] = value
        with pytest.raises(RuntimeError):
            dev.flush(bad)


class Attention:
    """One layer's cache and the op on it; rows are [q | k | v] with gaps between the fields."""

    def __init__(self, dev, half, B, H, G, dim, vdim, max_seq, scale, rel=None, far=0, shared=False, sink=False, temp=None, seed=0, eps=1e-4):
        self.__dict__.update(dev=dev, B=B, H=H, G=G, dim=dim, vdim=vdim, scale=scale, rel=rel, far=far, shared=shared, sink=sink, temp=temp, eps=eps)
        rng = np.random.default_rng(seed)
        self.qg, self.kg = 1 + 0.3 * rng.standard_normal(dim), 1 + 0.3 * rng.standard_normal(dim)
        pad16 = lambda n: (n + 15) // 16 * 16
        self.keys = dev.latent(B * G, max_seq, pad16(dim), half)
        self.values = -1 if shared else dev.latent(B * G, max_seq, pad16(vdim), half)
        self.kscale = dev.buf(B * G * ((max_seq + 63) // 64 * 64)) if shared else -1
        self.pos = dev.buf(B)
        self.off_k = H * dim + 3
        self.off_v = self.off_k + G * dim + 1
        self.ld = self.off_v + (0 if shared else G * vdim) + 2
        self.ids = [dev.buf(dim, self.qg), dev.buf(dim, self.kg)]
        self.tab = dev.buf(max_seq, [ref.temperature(p, *temp) for p in range(max_seq)]) if temp else -1
        self.rel_len, self.relb = 0, -1
        if rel is not None:
            rows = distance_buckets(len(rel), far, max_seq)
            self.rel_len, self.relb = rows.size, dev.buf(rows.size * H, rel[rows].T)

    def run(self, start, q, k, v, append=True):
        """q [B, T, H, dim] … at positions start[b] … → [B, T, H, vdim]."""
        d, B, T = self.dev, self.B, q.shape[1]
        rows = np.full((B, T, self.ld), 9.0)
        rows[..., :self.H * self.dim] = q.reshape(B, T, -1)
        rows[..., self.off_k:self.off_k + self.G * self.dim] = k.reshape(B, T, -1)
        if not self.shared:
            rows[..., self.off_v:self.off_v + self.G * self.vdim] = v.reshape(B, T, -1)
        pb, ldo = d.buf(rows.size, rows), self.H * self.vdim + 2
        ob = d.buf(B * T * ldo)
        from deepj_b200 import _lib
        p = np.asarray(start, dtype=np.float32)
        _lib.check(d.lib.deepj_cuda_upload_buffer(self.pos, p.ctypes.data, B))
        cmd = [OP_ATTN_GROUPED, pb, 0, self.off_k if append else -1, -1 if self.shared else self.off_v, self.ld, self.ids[0],
               self.ids[1] if append or self.shared else -1, float_bits(self.eps), self.tab, self.relb, self.rel_len, self.keys, self.values, self.kscale, self.pos, ob, 0, ldo,
               B, T, self.H, self.G, self.dim, self.vdim, float_bits(self.scale), int(self.sink)]
        for _ in range(3):
            d.flush(cmd)
        self.cmd = cmd
        return d.get(ob, B * T * ldo).reshape(B, T, ldo)[..., :-2].reshape(B, T, self.H, self.vdim)

    def reference(self, b, q, k, v, start=0):
        q, k = ref.rms(q[b], self.eps) * self.qg, np.asarray(k[b])
        if self.temp:
            q = q * np.array([ref.temperature(start + t, *self.temp) for t in range(len(q))])[:, None, None]
        bias = None if self.rel is None else (lambda n: self.rel[ref.distance_bucket(n, len(self.rel), self.far)])
        return ref.attend(q, ref.rms(k, self.eps) * self.kg, k if self.shared else v[b], start, self.scale, bias, self.sink)


def data(B, n, H, G, dim, vdim, seed, shared=False):
    rng = np.random.default_rng(seed)
    return rng.standard_normal((B, n, H, dim)), rng.standard_normal((B, n, G, dim)) * 2, rng.standard_normal((B, n, G, dim if shared else vdim))


SHAPES = [  # H, G, dim, vdim, scale: groups of one, of several, of more heads than an operand has rows; sizes off every grid
    (4, 4, 64, 64, 0.4), (6, 2, 48, 80, 0.5), (8, 1, 128, 128, 0.3), (3, 3, 13, 7, 0.9), (20, 1, 40, 24, 0.5), (2, 1, 200, 64, 0.3), (2, 2, 32, 256, 0.5), (34, 2, 16, 16, 0.7),
    (1, 1, 256, 256, 0.25)]


@pytest.mark.parametrize("half", [0, 1])
@pytest.mark.parametrize("H,G,dim,vdim,scale", SHAPES)
@pytest.mark.parametrize("kind", ["bias", "keys", "plain"])
def test_attention(dev, half, H, G, dim, vdim, scale, kind):
    """Whole prompt, portions down to two tokens, single tokens: distance bias, values that are the keys with a sink and a query
    temperature, or neither."""
    shared = kind == "keys"
    vdim = dim if shared else vdim
    n, B = 150, 2
    q, k, v = data(B, n, H, G, dim, vdim, H * 100 + dim, shared)
    rel = np.random.default_rng(dim).standard_normal((10, H)) * 2 if kind == "bias" else None
    a = Attention(dev, half, B, H, G, dim, vdim, 160, scale, rel, 45, shared, shared, (0.7, 11) if shared else None)
    want = np.stack([a.reference(b, q, k, v) for b in range(B)])
    tol = 4e-2 if half else 2e-5
    for cuts in ([n], [65, 1, 2, 17, 1, 1, 33, 30], [2, 3, 1] * 25):
        lo, got = 0, []
        for c in cuts:
            got.append(a.run([lo] * B, q[:, lo:lo + c], k[:, lo:lo + c], v[:, lo:lo + c]))
            lo += c
        near(want[:, :lo], np.concatenate(got, axis=1), tol)


@pytest.mark.parametrize("half", [0, 1])
@pytest.mark.parametrize("kind", ["bias", "keys"])
def test_a_single_key_stands_out(dev, half, kind):
    """A query that matches one far key: first, newest, at the borders of every tile size, just inside and outside of the
    distances where the bias changes; in a prompt and decoded.  The output is that key's value."""
    H, G, dim, vdim, n = 4, 2, 64, 64, 700
    shared = kind == "keys"
    q, k, v = data(1, n, H, G, dim, vdim, 5, shared)
    q *= 0.01
    spots = [0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 255, 511, 512, 640]
    rng = np.random.default_rng(1)
    asks = {}                       # query position → key position
    for j, s in enumerate(spots):
        t = 641 + 4 * j
        asks[t] = s
    for t, s in ((699, 698), (698, 698 - 9), (697, 697 - 10), (696, 696 - 44), (695, 695 - 45), (694, 694)):
        asks[t] = s
    for t, s in asks.items():
        q[0, t] = k[0, s][np.arange(H) // (H // G)]
    rel = rng.standard_normal((10, H)) if kind == "bias" else None
    a = Attention(dev, half, 1, H, G, dim, vdim, 704, 0.45, rel, 45, shared, shared, None, eps=1e-6)
    want = a.reference(0, q, k, v)
    source = k if shared else v
    for t, s in asks.items():       # the reference itself: nearly all weight on that key
        assert np.abs(want[t] - source[0, s][np.arange(H) // (H // G)]).max() < 0.3 * np.abs(source[0, s]).max()
    tol = 2.5e-2 if half else 2e-5
    got = a.run([0], q, k, v)[0]
    near(want, got, tol)
    for t in sorted(asks):          # each decoded: everything before is in the cache
        near(want[t], a.run([t], q[:, t:t + 1], k[:, t:t + 1], v[:, t:t + 1])[0, 0], tol)


@pytest.mark.parametrize("half", [0, 1])
def test_the_sink_takes_weight_and_survives_far_scores(dev, half):
    """Scores far below and far above the sink's zero, in one split and in many."""
    for n in (3, 400):
        q, k, v = data(1, n, 2, 1, 32, 32, n, True)
        a = Attention(dev, half, 1, 2, 1, 32, 32, 512, 1.0, shared=True, sink=True, eps=1e-6)
        k[0, :, 0] = np.abs(k[0, :, 0])
        for sign in (-1.0, 1.0, -0.05):
            q[0, -1, 0], q[0, -1, 1] = sign * np.abs(q[0, -1, 0]), -sign * np.abs(q[0, -1, 0])
            want = a.reference(0, q, k, v)
            got = a.run([0], q, k, v)
            near(want, got[0], 2.5e-2 if half else 2e-5)
            last = a.run([n - 1], q[:, -1:], k[:, -1:], v[:, -1:])[0]
            assert np.abs(last[0] - want[-1]).max() <= (2.5e-2 if half else 2e-5) * np.abs(want).max()


@pytest.mark.parametrize("half", [0, 1])
def test_unequal_positions_used_rows_and_another_layers_cache(dev, half):
    """Sequences of a batch at different positions; a cache that held other keys; a second layer that appends nothing."""
    H, G, dim, vdim, B = 6, 3, 48, 32, 3
    q, k, v = data(B, 300, H, G, dim, vdim, 8)
    rel = np.random.default_rng(3).standard_normal((8, H))
    a = Attention(dev, half, B, H, G, dim, vdim, 320, 0.5, rel, 60)
    a.run([0] * B, *(x[:, ::-1][:, :280] for x in (q, k, v)))           # somebody else's
    start = [130, 17, 257]
    for b in range(B):
        a.run([0] * B, q[:, :start[b]], k[:, :start[b]], v[:, :start[b]])    # the longest comes last for nobody: rows are used again
    a.run([0] * B, q[:, :257], k[:, :257], v[:, :257])
    tol = 2.5e-2 if half else 2e-5
    for T in (1, 2, 20):
        pick = lambda x: np.stack([x[b, start[b]:start[b] + T] for b in range(B)])
        got = a.run(start, pick(q), pick(k), pick(v))
        for b in range(B):
            want = a.reference(b, q[:, :start[b] + T], k[:, :start[b] + T], v[:, :start[b] + T])[start[b]:]
            near(want, got[b], tol)
        # the same keys and values, other queries: what the row holds in the key and value fields is not looked at
        got = a.run(start, pick(q)[:, :, ::-1], np.full_like(pick(k), np.nan), np.full_like(pick(v), np.nan), append=False)
        q2 = q.copy()
        for b in range(B):
            q2[b, start[b]:start[b] + T] = q[b, start[b]:start[b] + T, ::-1]
            want = a.reference(b, q2[:, :start[b] + T], k[:, :start[b] + T], v[:, :start[b] + T])[start[b]:]
            near(want, got[b], tol)


def test_attention_refuses_what_does_not_fit(dev):
    a = Attention(dev, 1, 1, 4, 2, 32, 32, 64, 0.3)
    q, k, v = data(1, 4, 4, 2, 32, 32, 0)
    a.run([0], q, k, v)
    for at, value in ((22, 3), (23, 64), (19, 2), (5, 100), (13, a.pos), (14, a.pos), (7, -1), (11, 1 << 20), (18, 64), (20, 0), (26, 2), (24, 48)):
        bad = list(a.cmd)
        bad[at] = value
        if at == 11:
            bad[10] = a.ids[0]
        with pytest.raises(RuntimeError):
            dev.flush(bad)


class Recurrence:
    def __init__(self, dev, B, H, dim, vdim, cap, exact):
        self.__dict__.update(dev=dev, B=B, H=H, dim=dim, vdim=vdim, cap=cap, exact=exact)
        rng = np.random.default_rng(0)
        self.state = dev.buf(B * H * vdim * dim, rng.standard_normal(B * H * vdim * dim) * 100)          # garbage before position 0
        self.norm = dev.buf(2 * B * H * (dim + 1), rng.standard_normal(2 * B * H * (dim + 1)) * 100)
        self.pos = dev.buf(B)
        self.at = np.cumsum([1, H * dim + 1, H * dim + 2, H * vdim + 1, H + 1, H]).tolist()              # q k v i f, end
        self.ld = self.at[5] + 3

    def run(self, start, q, k, v, i, f):
        d, B, T = self.dev, self.B, q.shape[1]
        rows = np.full((B, T, self.ld), 9.0)
        for at, x in zip(self.at, (q, k, v, i, f)):
            rows[..., at:at + x[0, 0].size] = x.reshape(B, T, -1)
        ldo = self.H * self.vdim + 3
        pb, ob = d.buf(rows.size, rows), d.buf(B * T * ldo)
        from deepj_b200 import _lib
        p = np.full(B, start, dtype=np.float32)
        _lib.check(d.lib.deepj_cuda_upload_buffer(self.pos, p.ctypes.data, B))
        self.cmd = [OP_MLSTM, pb, *self.at[:5], self.ld, float_bits(self.cap), float_bits(self.dim ** -0.5), self.state, self.norm, self.pos, ob, 0, ldo, B, T, self.H,
                    self.dim, self.vdim, self.exact]
        d.flush(self.cmd)
        return d.get(ob, B * T * ldo).reshape(B, T, ldo)[..., :-3].reshape(B, T, self.H, self.vdim)

    def reference(self, b, q, k, v, i, f):
        gate = lambda x: self.cap * np.tanh(x / self.cap)
        state = ref.mlstm_zero({"heads": self.H, "dim": self.dim, "vdim": self.vdim})
        out = np.zeros((q.shape[1], self.H, self.vdim))
        for t in range(q.shape[1]):
            for h in range(self.H):
                state[h], out[t, h] = ref.mlstm_step(state[h], q[b, t, h] * self.dim ** -0.5, k[b, t, h], v[b, t, h], gate(i[b, t, h]), ref.log_sigmoid(gate(f[b, t, h])))
        return out


def recurrence_data(B, T, H, dim, vdim, seed, forget):
    """Keys and queries with a common part, so that the normaliser stays away from zero where single terms cancel."""
    rng = np.random.default_rng(seed)
    common = rng.standard_normal((H, dim)) * 1.5
    q, k = rng.standard_normal((B, T, H, dim)) + common, rng.standard_normal((B, T, H, dim)) + common
    return q, k, rng.standard_normal((B, T, H, vdim)), rng.standard_normal((B, T, H)) * 3, rng.standard_normal((B, T, H)) * 2 + forget


@pytest.mark.parametrize("exact", [1, 0])
@pytest.mark.parametrize("H,dim,vdim,cap", [(2, 48, 64, 10.0), (3, 24, 40, 5.0), (1, 128, 96, 15.0), (2, 21, 10, 3.0), (1, 256, 48, 8.0), (1, 200, 33, 30.0), (1, 300, 16, 10.0)])
def test_recurrence(dev, exact, H, dim, vdim, cap):
    B, T = 2, 150
    tol = 2e-5 if exact else 2e-2
    for forget in (4.0, -6.0, 0.5):           # remembers, forgets at once, between
        x = recurrence_data(B, T, H, dim, vdim, dim + int(forget), forget)
        r = Recurrence(dev, B, H, dim, vdim, cap, exact)
        want = np.stack([r.reference(b, *x) for b in range(B)])
        # a portion's outputs depend on what earlier ones left: token by token, pairs, odd and even portions, the block borders
        for cuts in ([T], [1] * 12, [2] * 10, [63, 1, 2, 17, 1, 64, 2], [32, 33, 31, 5], [16, 15, 65, 1]):
            lo, got = 0, []
            for c in cuts:
                got.append(r.run(lo, *(a[:, lo:lo + c] for a in x)))
                lo += c
            near(want[:, :lo], np.concatenate(got, axis=1), tol)


@pytest.mark.parametrize("exact", [1, 0])
def test_recurrence_extremes(dev, exact):
    """Input gates at both ends of the cap, forget gates that wipe the state in the middle of a block and then keep everything:
    sums of hundreds whose differences matter; a first token that the running maximum's zero outweighs."""
    H, dim, vdim, T = 1, 48, 32, 200
    q, k, v, i, f = recurrence_data(1, T, H, dim, vdim, 3, 0.0)
    i[0, :, 0] = np.where(np.arange(T) % 3 == 0, 40.0, -40.0)
    i[0, :5, 0] = -40.0
    f[0, :, 0] = np.where(np.arange(T) % 50 < 30, -60.0, 60.0)
    r = Recurrence(dev, 1, H, dim, vdim, 14.0, exact)
    want = r.reference(0, q, k, v, i, f)
    for cuts in ([T], [1] * T, [130, 1, 69]):
        lo, got = 0, []
        for c in cuts:
            got.append(r.run(lo, *(a[:, lo:lo + c] for a in (q, k, v, i, f))))
            lo += c
        got = np.concatenate(got, axis=1)[0]
        near(want, got, 5e-5 if exact else 2e-2)
        assert np.abs(got[:5] - want[:5]).max() <= (1e-4 if exact else 3e-2) * max(np.abs(want[:5]).max(), 1e-12)
    for at, value in ((19, 0), (19, 600), (7, 10), (15, 3), (11, r.pos), (21, 2), (8, 0)):
        bad = list(r.cmd)
        bad[at] = value
        with pytest.raises(RuntimeError):
            dev.flush(bad)
