"""Plain, slow numpy restatement of the Punilix decoder, one function per mechanism.

It shares no code with the product package: the tests compare the CUDA path with it.  Every function takes and
returns arrays of one dtype (float64 by default, float32 when the caller wants 32-bit rounding), loops over tokens
where the mechanism is sequential, and holds no state that the caller does not see.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms_norm(x, weight, eps, groups=1):
    """x [..., n] cut into `groups` equal consecutive parts, each over its own root mean square; then times weight."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    scale = np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return (parts / scale).reshape(x.shape) * weight


def rotary_frequencies(dims, base, scaling=None):
    """(f_i, factor of cos and sin) for i < dims/2; `scaling` is the YaRN record or None."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if scaling is None:
        return f, 1.0

    def at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(scaling["fast"])), 0)
    hi = min(math.ceil(at(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    factor = scaling["factor"]
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_interleaved(x, positions, dims, base, scaling=None):
    """Rotate the first `dims` entries of x [T, ..., n], pairs (2i, 2i+1), by position · f_i."""
    f, m = rotary_frequencies(dims, base, scaling)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (len(angle),) + (1,) * (x.ndim - 2) + (dims // 2,)
    cos, sin = (np.cos(angle) * m).reshape(shape).astype(x.dtype), (np.sin(angle) * m).reshape(shape).astype(x.dtype)
    out = x.copy()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * cos - b * sin
    out[..., 1:dims:2] = b * cos + a * sin
    return out


def gated_clamp(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, w, prefix, limit):
    return gated_clamp(h @ w[prefix + ".gate"].T, h @ w[prefix + ".up"].T, limit) @ w[prefix + ".down"].T


def table_experts(h, tokens, w, prefix, limit):
    """Each token's experts come from a table row indexed by its id; every one has weight 1 / (row length)."""
    table = w[prefix + ".table"].astype(np.int64)
    out = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[tok]:
            out[t] += feed_forward(h[t:t + 1], w, f"{prefix}.e{e}", limit)[0] / table.shape[1]
    return out


def delta_step(S, r, k, v, decay, removal):
    """One token of the generalized delta rule for one head: S [dk, dv] → (new S, o [dv])."""
    u = k / np.sqrt(np.sum(k * k) + 1e-6)
    S = decay[:, None] * S - (removal * u)[:, None] * (u @ S)[None, :] + np.outer(k, v)
    return S, S.T @ r


def general_delta(h, w, prefix, heads, dim, eps, state=None):
    """The whole mixer over h [T, width]; `state` [heads, dim, dim] is read and updated in place when given."""
    T, W = len(h), lambda name: w[prefix + "." + name]
    r, k, v = (h @ W(n).T for n in "rkv")
    decay = np.exp(-math.exp(-0.5) * sigmoid(np.tanh(h @ W("w1").T) @ W("w2").T + W("w0")))
    removal = sigmoid(h @ W("a").T + W("a.b"))
    S = np.zeros((heads, dim, dim), dtype=h.dtype) if state is None else state
    o = np.zeros((T, heads * dim), dtype=h.dtype)
    for t in range(T):
        for j in range(heads):
            c = slice(j * dim, (j + 1) * dim)
            S[j], o[t, c] = delta_step(S[j], r[t, c], k[t, c], v[t, c], decay[t, c], removal[t, c])
    return (rms_norm(o, W("norm"), eps, groups=heads) * sigmoid(h @ W("g").T)) @ W("o").T


def softmax_rows(s):
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


def latent_attention(h, w, prefix, m, eps, start=0, cache=None):
    """The whole mixer over h [T, width] at positions start…; `cache` is a list of earlier (latent, rotated key) rows
    that is extended in place when given.  `m` is the layer's mixer record."""
    W = lambda name: w[prefix + "." + name]
    H, dim, rd, vd, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T, positions = len(h), np.arange(start, start + len(h))
    rot = m["rot"]
    q = (rms_norm(h @ W("dq").T, W("dq.norm"), eps) @ W("uq").T).reshape(T, H, dim + rd)
    q_rot = rotate_interleaved(q[..., dim:], positions, rot["dims"], rot["base"], rot.get("scaling"))
    kv = h @ W("dkv").T
    c_new = rms_norm(kv[:, :R], W("dkv.norm"), eps)
    k_rot_new = rotate_interleaved(kv[:, R:], positions, rot["dims"], rot["base"], rot.get("scaling"))
    rows = [] if cache is None else cache
    rows.extend(zip(c_new, k_rot_new))
    c, k_rot = np.stack([a for a, _ in rows]), np.stack([b for _, b in rows])
    k_un = (c @ W("uk").T).reshape(-1, H, dim)
    v = (c @ W("uv").T).reshape(-1, H, vd)
    out = np.zeros((T, H, vd), dtype=h.dtype)
    for t in range(T):
        L = start + t + 1
        for j in range(H):
            s = (k_un[:L, j] @ q[t, j, :dim] + k_rot[:L] @ q_rot[t, j]) * m["scale"]
            out[t, j] = softmax_rows(s) @ v[:L, j]
    return (out.reshape(T, H * vd) * sigmoid(h @ W("g").T)) @ W("o").T


class Model:
    """Weights (name → array) and a configuration record; `forward` runs tokens from the state earlier calls left."""

    def __init__(self, config, weights, dtype=np.float64):
        self.c, self.dtype = config, dtype
        self.w = {n: (a if np.issubdtype(np.asarray(a).dtype, np.integer) else np.asarray(a, dtype=dtype)) for n, a in weights.items()}
        self.reset()

    def reset(self):
        self.position = 0
        self.state = [np.zeros((L["mixer"]["heads"], L["mixer"]["dim"], L["mixer"]["dim"]), dtype=self.dtype)
                      if L["type"] == "general_delta" else [] for L in self.c["layers"]]

    def forward(self, tokens, residuals=None):
        """Logits [T, vocab] of the next tokens; `residuals` (a list) receives the residual stream after every layer."""
        c, w = self.c, self.w
        eps, groups = c["norm"]["eps"], c["norm"]["groups"]
        x = w["embed"][np.asarray(tokens)].copy()
        for i, L in enumerate(c["layers"]):
            h = rms_norm(x, w[f"l{i}.norm1"], eps, groups)
            if L["type"] == "general_delta":
                y = general_delta(h, w, f"l{i}.mix", L["mixer"]["heads"], L["mixer"]["dim"], eps, self.state[i])
            else:
                y = latent_attention(h, w, f"l{i}.mix", L["mixer"], eps, self.position, self.state[i])
            f = L["mlp"]
            if f is not None:
                if f["kind"] == "dense":
                    y = y + feed_forward(h, w, f"l{i}.mlp", f["limit"])
                else:
                    y = y + table_experts(h, tokens, w, f"l{i}.mlp", f["expert"]["limit"])
            x = x + y
            if residuals is not None:
                residuals.append(x.copy())
        self.position += len(tokens)
        logits = rms_norm(x, w["final.norm"], eps, groups) @ w["head"].T
        cap = c.get("logit_softcap")
        return cap * np.tanh(logits / cap) if cap else logits
