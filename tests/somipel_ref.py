"""Plain, slow numpy restatement of the Somipel decoder, one function per mechanism.

It shares no code with the product package: the tests compare the CUDA path with it.  Everything is float64 unless the
caller asks for another dtype; recurrences loop over tokens, and no function holds state that the caller does not see.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def silu(z):
    return z * sigmoid(z)


def feed_forward(x, w, prefix):
    return (silu(x @ w[prefix + ".gate"].T) * (x @ w[prefix + ".up"].T)) @ w[prefix + ".down"].T


def distance_bucket(n, rows, far):
    """Row of the distance table for a key n tokens back: the first half one row each, the second half logarithmic up to
    `far`, everything beyond in the last."""
    half = rows // 2
    if n < half:
        return n
    # the ratio of two logarithms may come out a hair below a whole number that it equals
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9))


def temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def softmax_with_sink(s):
    """One more score of 0 in the denominator, which carries no value."""
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(-m))


def attend(q, keys, values, start, scale, bias=None, sink=False):
    """q [T, H, dim] at positions start…, keys [n, G, dim], values [n, G, vdim] from position 0; bias(distance) → [H]."""
    T, H, _ = q.shape
    G = keys.shape[1]
    out = np.zeros((T, H, values.shape[2]), dtype=q.dtype)
    table = None if bias is None else np.stack([bias(n) for n in range(start + T)])       # [distance, H]
    for t in range(T):
        n = start + t + 1
        for h in range(H):
            g = h // (H // G)
            s = (keys[:n, g] @ q[t, h]) * scale
            if table is not None:
                s = s + table[n - 1::-1, h] if n > 1 else s + table[:1, h]
            out[t, h] = (softmax_with_sink if sink else softmax)(s) @ values[:n, g]
    return out


def gated_attention(x, w, prefix, m, eps, start, cache):
    """Grouped heads with biased projections, normed queries and keys, a learned bias by distance, a sigmoid output gate.
    `cache` is a list [keys, values] of earlier positions, extended in place, or another layer's that already holds these
    positions (kv_from)."""
    W = lambda n: w[prefix + "." + n]
    H, G, dim, vdim, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], len(x)
    q = rms((x @ W("q").T + W("q.b")).reshape(T, H, dim), eps) * W("q.norm")
    if m.get("kv_from") is None:
        k = rms((x @ W("k").T + W("k.b")).reshape(T, G, dim), eps) * W("k.norm")
        v = (x @ W("v").T + W("v.b")).reshape(T, G, vdim)
        extend(cache, k, v)
    rel = W("rel")
    o = attend(q, cache[0], cache[1], start, m["scale"], lambda n: rel[distance_bucket(n, len(rel), m["bias_max"])])
    return (o.reshape(T, H * vdim) * sigmoid(x @ W("g").T)) @ W("o").T


def extend(cache, k, v):
    if cache:
        cache[0], cache[1] = np.concatenate([cache[0], k]), np.concatenate([cache[1], v])
    else:
        cache.extend([k, v])


def key_value_attention(x, w, prefix, m, eps, start, cache):
    """Grouped heads whose values are the keys as projected; normed queries and keys, a query temperature by position, a
    sink in the denominator."""
    W = lambda n: w[prefix + "." + n]
    H, G, dim, T = m["heads"], m["kv_heads"], m["dim"], len(x)
    q = rms((x @ W("q").T).reshape(T, H, dim), eps) * W("q.norm")
    if m.get("q_temp"):
        q = q * np.array([temperature(start + t, m["q_temp"]["coef"], m["q_temp"]["every"]) for t in range(T)])[:, None, None]
    raw = (x @ W("k").T).reshape(T, G, dim)
    extend(cache, rms(raw, eps) * W("k.norm"), raw)
    o = attend(q, cache[0], cache[1], start, m["scale"], sink=True)
    return o.reshape(T, H * dim) @ W("o").T


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def mlstm_step(state, q, k, v, i, f):
    """One token of one head: state (S [dim, vdim], n [dim], running maximum) → (new state, o [vdim])."""
    S, n, m = state
    new = max(f + m, i)
    keep, add = np.exp(f + m - new), np.exp(i - new)
    S = keep * S + add * np.outer(k, v)
    n = keep * n + add * k
    return (S, n, new), S.T @ q / (max(abs(n @ q), np.exp(-new)) + 1e-6)


def mlstm_zero(m, dtype=np.float64):
    return [(np.zeros((m["dim"], m["vdim"]), dtype=dtype), np.zeros(m["dim"], dtype=dtype), 0.0) for _ in range(m["heads"])]


def mlstm(x, w, prefix, m, eps, state):
    """The whole mixer over x [T, width]; `state` (a list per head) is read and replaced in place."""
    W = lambda n: w[prefix + "." + n]
    H, dim, vdim, cap, T = m["heads"], m["dim"], m["vdim"], m["gate_cap"], len(x)
    q = (x @ W("q").T).reshape(T, H, dim) * dim ** -0.5
    k = (x @ W("k").T).reshape(T, H, dim)
    v = (x @ W("v").T).reshape(T, H, vdim)
    i = cap * np.tanh((x @ W("i").T + W("i.b")) / cap)
    f = log_sigmoid(cap * np.tanh((x @ W("f").T + W("f.b")) / cap))
    o = np.zeros((T, H, vdim), dtype=x.dtype)
    for t in range(T):
        for h in range(H):
            state[h], o[t, h] = mlstm_step(state[h], q[t, h], k[t, h], v[t, h], i[t, h], f[t, h])
    return (rms(o, eps).reshape(T, H * vdim) * W("norm") * sigmoid(x @ W("g").T)) @ W("o").T


class Model:
    """Weights (name → array) and a configuration record; `forward` runs tokens from the state earlier calls left."""

    def __init__(self, config, weights, dtype=np.float64):
        self.c, self.dtype = config, dtype
        self.w = {n: np.asarray(a, dtype=dtype) for n, a in weights.items()}
        self.reset()

    def reset(self):
        self.position = 0
        self.state = [mlstm_zero(L["mixer"], self.dtype) if L["type"] == "mlstm" else [] for L in self.c["layers"]]

    def mixer(self, i, x):
        L, eps = self.c["layers"][i], self.c["norm"]["eps"]
        m, prefix = L["mixer"], f"l{i}.mix"
        if L["type"] == "mlstm":
            return mlstm(x, self.w, prefix, m, eps, self.state[i])
        if L["type"] == "attention_2":
            return key_value_attention(x, self.w, prefix, m, eps, self.position, self.state[i])
        source = i if m.get("kv_from") is None else m["kv_from"]
        return gated_attention(x, self.w, prefix, m, eps, self.position, self.state[source])

    def forward(self, tokens, residuals=None):
        """Logits [T, vocab] of the next tokens; `residuals` (a list) receives the residual stream after every layer."""
        c, w = self.c, self.w
        eps, mult = c["norm"]["eps"], c["residual_mult"]
        x = w["embed"][np.asarray(tokens)].copy()
        for i, L in enumerate(c["layers"]):
            x = x + mult * (rms(self.mixer(i, x), eps) * w[f"l{i}.norm1"])
            if L["mlp"] is not None:
                x = x + mult * (rms(feed_forward(x, w, f"l{i}.mlp"), eps) * w[f"l{i}.norm2"])
            if residuals is not None:
                residuals.append(x.copy())
        self.position += len(tokens)
        return (rms(x, eps) * w["final.norm"]) @ w["head"].T
