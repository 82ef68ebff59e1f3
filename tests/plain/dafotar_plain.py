"""Plain, slow implementation of the Dafotar decoder: the oracle of the tests.

It shares no code with ``air_b200``: whole sequences, no cache, no batch, numpy on the CPU, one function per
mechanism.  `dtype` is the precision of the arithmetic (float64 for the oracle, float32 to see what 32-bit rounding
alone does).

The design, in this file's notation.  X is [S, T, E]: S residual streams side by side.

  embedding     X[s] = embed[tokens] for every s.
  sub-layer     u = sum_s r_s X[s];  y = f(ln(u));  X'[t] = sum_s M[s, t] X[s] + o_t y  (all t from the old X): what a
                sub-layer reads, how the streams are mixed behind it and where its output goes are learned numbers.
  norm          ln(x) = (x - mean) / sqrt(var + eps) * w + b, var the mean of the squared deviations.
  input         what a mixer reads: h_t + sum_j w[:, j] h_(t - taps + 1 + j), h = ln(u), zeros ahead of the sequence.
  attention     grouped queries; q and k per head over their root mean square (eps under the root), times a weight;
                the first R numbers of a head of q and k rotated, element i with i + R/2, by position * base^(-2i/R);
                the values of position j rotated over their whole width (m with m + dv/2) by j * base^(-2m/dv) and each
                head's output at position i rotated by -i times the same; score = scale * temp_h * q.k; position i sees
                i - j < window; softmax; Wo.  A layer may take keys and values (normalised and rotated) from an earlier
                layer and brings its own queries.
  mlstm         per head: i = c tanh((Wi h + bi) / c), f = log sigmoid(c tanh((Wf h + bf) / c)), q = Wq h / sqrt(d);
                m' = max(f + m, i);  C' = e^(f + m - m') C + e^(i - m') k v^T;  n' = e^(f + m - m') n + e^(i - m') k;
                o = C'^T q / (max(|n'.q|, e^(-m')) + 1e-6), with C, n and m zero at the start; each head's o over its
                root mean square; all heads times a weight, times sigmoid(Wg h); Wo.
  dense         Wdown(relu(Wgate u) * (Wup u)).
  output        ln(sum_s X[s]), then the token table as the output matrix.
"""
from __future__ import annotations

import numpy as np


# ----------------------------------------------------------------------------- small functions
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w + b


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


# ----------------------------------------------------------------------------- mechanisms
def read_streams(X, r):
    """sum_s r_s X[s]"""
    return np.tensordot(r, X, axes=(0, 0))


def mix_streams(X, M, o, y):
    """X'[t] = sum_s M[s, t] X[s] + o_t y"""
    return np.stack([sum(M[s, t] * X[s] for s in range(len(X))) + o[t] * y for t in range(len(X))])


def input_convolution(h, w):
    """h_t + sum_j w[:, j] h_(t - taps + 1 + j), zeros ahead of the sequence; w [E, taps]."""
    taps = w.shape[1]
    y = h.copy()
    for j in range(taps):
        back = taps - 1 - j
        if back < len(h):
            y[back:] += w[:, j] * h[:len(h) - back]
    return y


def turn(x, positions, dims, base, dtype, sign=1.0):
    """x [T, heads, n]: the first `dims` numbers of every head, element i with i + dims / 2, turned by
    sign * position * base^(-2i/dims)."""
    if dims == 0:
        return x
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)
    angle = sign * np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(angle).astype(dtype)[:, None, :], np.sin(angle).astype(dtype)[:, None, :]
    a, b = x[..., :dims // 2], x[..., dims // 2:dims]
    out = x.copy()
    out[..., :dims // 2] = a * c - b * s
    out[..., dims // 2:dims] = b * c + a * s
    return out


def window_attention(q, k, v, scales, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; scales [H]; position i sees j with 0 <= i - j < window
    (None: all j <= i)."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    hidden = (j > i) | ((i - j >= window) if window else False)
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scales[h]
        s = np.where(hidden, -np.inf, s)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def mixer_attention(w, p, x, m, positions, eps, dtype, shared=None):
    """(output [T, E], (k, v) as a cache holds them).  shared: the (k, v) of an earlier layer."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    R, base = (int(m["rot"]["dims"]), float(m["rot"]["base"])) if m.get("rot") else (0, 1.0)
    wide = dv if m.get("rot") else 0
    q = over_rms((x @ w[p + "q"].T).reshape(T, H, d), eps) * w[p + "q.norm"]
    q = turn(q, positions, R, base, dtype)
    if shared is None:
        k = over_rms((x @ w[p + "k"].T).reshape(T, G, d), eps) * w[p + "k.norm"]
        k = turn(k, positions, R, base, dtype)
        v = turn((x @ w[p + "v"].T).reshape(T, G, dv), positions, wide, base, dtype)
        shared = (k, v)
    k, v = shared
    window = int(m["mask"]["size"]) if m.get("mask") else None
    o = window_attention(q, k, v, dtype(m["scale"]) * w[p + "temp"], window)
    o = turn(o, positions, wide, base, dtype, sign=-1.0)
    return o.reshape(T, H * dv) @ w[p + "o"].T, shared


def mlstm_gates(w, p, x, m):
    """(i, f) [T, H]: the logarithms of the input gate and of the forget gate."""
    c = float(m["gate_cap"])
    i = c * np.tanh((x @ w[p + "i"].T + w[p + "i.b"]) / c)
    f = log_sigmoid(c * np.tanh((x @ w[p + "f"].T + w[p + "f.b"]) / c))
    return i, f


def mlstm_memory(q, k, v, i, f, dtype):
    """q (scaled), k [T, H, d], v [T, H, dv], i, f [T, H] -> o [T, H, dv]."""
    T, H, d = q.shape
    o = np.zeros((T, H, v.shape[2]), dtype=dtype)
    for h in range(H):
        C, n, m = np.zeros((d, v.shape[2]), dtype=dtype), np.zeros(d, dtype=dtype), dtype(0.0)
        for t in range(T):
            new = max(f[t, h] + m, i[t, h])
            keep, take = np.exp(f[t, h] + m - new), np.exp(i[t, h] - new)
            C = keep * C + take * np.outer(k[t, h], v[t, h])
            n = keep * n + take * k[t, h]
            m = new
            o[t, h] = (C.T @ q[t, h]) / (max(abs(n @ q[t, h]), np.exp(-m)) + dtype(1e-6))
    return o


def mixer_mlstm(w, p, x, m, positions, eps, dtype, shared=None):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q = (x @ w[p + "q"].T).reshape(T, H, d) * dtype(d ** -0.5)
    k, v = (x @ w[p + "k"].T).reshape(T, H, d), (x @ w[p + "v"].T).reshape(T, H, dv)
    i, f = mlstm_gates(w, p, x, m)
    o = over_rms(mlstm_memory(q, k, v, i, f, dtype), eps).reshape(T, H * dv)
    return (o * w[p + "norm"] * sigmoid(x @ w[p + "g"].T)) @ w[p + "o"].T, None


MIXERS = {"attention": mixer_attention, "mlstm": mixer_mlstm}


def dense_ff(w, p, u):
    return (np.maximum(u @ w[p + "gate"].T, 0.0) * (u @ w[p + "up"].T)) @ w[p + "down"].T


# ----------------------------------------------------------------------------- the model
def forward(config, weights, tokens, dtype=np.float64, taps=None):
    """Logits [T, vocab] of one sequence.  taps: a list that receives the sum of the streams after every layer."""
    w = {k: (v.astype(dtype) if v.dtype.kind == "f" else v) for k, v in weights.items()}
    eps = dtype(config["norm"]["eps"])
    tokens = np.asarray(tokens)
    positions = np.arange(len(tokens))
    X = np.stack([w["embed"][tokens]] * config["streams"])
    kept = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(read_streams(X, w[p + "hc1.in"]), w[p + "norm1"], w[p + "norm1.b"], eps)
        h = input_convolution(h, w[p + "canon1"])
        y, kept[i] = MIXERS[layer["type"]](w, p + "mix.", h, m, positions, eps, dtype, kept.get(m.get("kv_from")))
        X = mix_streams(X, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        if layer.get("mlp") is not None:
            u = layer_norm(read_streams(X, w[p + "hc2.in"]), w[p + "norm2"], w[p + "norm2.b"], eps)
            X = mix_streams(X, w[p + "hc2.mix"], w[p + "hc2.out"], dense_ff(w, p + "mlp.", u))
        if taps is not None:
            taps.append(X.sum(axis=0))
    return layer_norm(X.sum(axis=0), w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
