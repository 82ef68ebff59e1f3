"""Plain, slow implementation of the Sesulorn decoder: the oracle of the tests.

It shares no code with ``air_b200``: whole sequences, no cache, no batch, numpy on the CPU, one function per
mechanism.  `dtype` is the precision of the arithmetic (float64 for the oracle, float32 to see what 32-bit rounding
alone does).

The design, in this file's notation.  x is the stream [T, E], x0 the embedding's output.

  embedding         x = x0 = embed[tokens].
  order             the layers `start` .. `stop - 1` run `times` times over with the same weights, then the layers behind
                    them follow; ahead of EVERY pass x = Win [x | x0] (loop.in, [E, 2E]).
  layer             n = ln(x);  x += mixer(n) + ff(n);  ln(x) = (x - mean) / sqrt(var + eps) * w + b, var the mean of the
                    squared deviations.
  attention         grouped queries with biases on q, k and v; every head of q and of k over its root mean square, no
                    weight; score = scale q.k + R[bucket(i - j), h], R the layer's table [B, H]; position i sees j <= i;
                    softmax; Wo.  With L = floor(B / 2): bucket(n) = n for n < L, else
                    min(B - 1, L + floor(ln(n / L) / ln(bias_max / L) (B - L))).
  channel_delta     q, k (G x d), v (H x dv): projections, a causal convolution per channel, silu; q and k scaled to unit
                    length per head (x / sqrt(sum x^2 + 1e-6)), q also by d^-1/2; b = sigmoid(Wb n) per head;
                    g = exp(-exp(A_h) softplus(Wa2 (Wa1 n) + dt)) per head AND key channel;
                    S = diag(g) S;  u = b (v - S^T k);  S = S + k u^T;  o = S^T q;
                    o over its root mean square, times w (one vector [dv]), times sigmoid(Wg2 (Wg1 n)); Wo.
  latent_attention  q = Wuq (rms(Wdq n) wq), per head [d plain | r rotated]; (c | kr) = Wdkv n, c = rms(c) wc, kr one
                    rotated key part for all heads; per head k = Wuk c, v = Wuv c;
                    score = scale (q_plain . k + q_rot . kr); position i sees j <= i; softmax; Wo.  Rotation of
                    elements 2m and 2m + 1 by position * base^(-2m/r).
  dense             Wdown(silu(Wgate n) * (Wup n)).
  moe               s = softmax(Wr n); consecutive experts make `count` groups of one size, a group's mark is its largest
                    s, only the `keep` groups with the highest marks take part; of their experts the `top` with the
                    largest s are taken; y = sum_e s_e expert_e(n) + sigmoid(wsg . n) shared(n);
                    expert(u) = Wd (a sigmoid(1.702 a) (b + 1)), a = min(Wg u, limit), b = clamp(Wu u, -limit, limit).
  output            ln(x) with final.norm, then the output matrix.
"""
from __future__ import annotations

import math

import numpy as np


# ----------------------------------------------------------------------------- small functions
def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def softmax_rows(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w + b


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


# ----------------------------------------------------------------------------- attention with a distance bias
def bucket(n, rows, bias_max):
    """The row of the table for a key that stands n positions back."""
    low = rows // 2
    if n < low:
        return n
    return min(rows - 1, low + math.floor(math.log(n / low) / math.log(bias_max / low) * (rows - low)))


def biased_attention(q, k, v, scale, table, bias_max):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; table [B, H]."""
    T, H, _ = q.shape
    G = k.shape[1]
    rows = np.array([bucket(n, len(table), bias_max) for n in range(T)])
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale + table[rows[np.maximum(back, 0)], h]
        out[:, h] = softmax_rows(np.where(back < 0, -np.inf, s)) @ v[:, g]
    return out


def mixer_attention(w, p, x, m, eps, dtype):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q = over_rms((x @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d), eps)
    k = over_rms((x @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d), eps)
    v = (x @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    o = biased_attention(q, k, v, dtype(m["scale"]), w[p + "rel"], m["bias_max"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ----------------------------------------------------------------------------- delta rule with a decay per channel
def short_convolution(x, w):
    """sum_j w[:, j] x_(t - taps + 1 + j), zeros ahead of the sequence; w [channels, taps]."""
    taps = w.shape[1]
    y = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < len(x):
            y[back:] += w[:, j] * x[:len(x) - back]
    return y


def channel_decay(w, p, x, H, d):
    """g [T, H, d]"""
    z = (x @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    return np.exp(-np.exp(w[p + "A_log"])[:, None] * softplus(z).reshape(len(x), H, d))


def delta_memory(q, k, v, g, beta, dtype):
    """q, k [T, G, d], v [T, H, dv], g [T, H, d], beta [T, H] -> o [T, H, dv]"""
    T, H, dv = v.shape
    G, d = k.shape[1:]
    o = np.zeros((T, H, dv), dtype=dtype)
    for h in range(H):
        S, kv = np.zeros((d, dv), dtype=dtype), h // (H // G)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, kv])
            S = S + np.outer(k[t, kv], u)
            o[t, h] = S.T @ q[t, kv]
    return o


def mixer_channel_delta(w, p, x, m, eps, dtype):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q, k, v = (silu(short_convolution(x @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q, k = unit(q.reshape(T, G, d)) * dtype(d ** -0.5), unit(k.reshape(T, G, d))
    o = delta_memory(q, k, v.reshape(T, H, dv), channel_decay(w, p, x, H, d), sigmoid(x @ w[p + "b"].T), dtype)
    gate = sigmoid((x @ w[p + "g1"].T) @ w[p + "g2"].T)
    return ((over_rms(o, eps) * w[p + "norm"]).reshape(T, H * dv) * gate) @ w[p + "o"].T


# ----------------------------------------------------------------------------- latent attention
def turn_neighbours(x, base, dtype):
    """x [T, heads, r]: elements 2m and 2m + 1 of every head turned by position * base^(-2m/r)."""
    r = x.shape[-1]
    f = np.array([float(base) ** (-2.0 * i / r) for i in range(r // 2)], dtype=np.float64)
    angle = np.arange(len(x), dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(angle).astype(dtype)[:, None, :], np.sin(angle).astype(dtype)[:, None, :]
    out = np.empty_like(x)
    a, b = x[..., 0::2], x[..., 1::2]
    out[..., 0::2] = a * c - b * s
    out[..., 1::2] = b * c + a * s
    return out


def causal_softmax(s):
    T = s.shape[0]
    return softmax_rows(np.where(np.arange(T)[None, :] > np.arange(T)[:, None], -np.inf, s))


def mixer_latent(w, p, x, m, eps, dtype):
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = x.shape[0]
    q = ((over_rms(x @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).reshape(T, H, d + r)
    both = x @ w[p + "dkv"].T
    c = over_rms(both[:, :R], eps) * w[p + "dkv.norm"]
    base = m["rot"]["base"] if r else 1.0
    q_rot, k_rot = turn_neighbours(q[..., d:], base, dtype), turn_neighbours(both[:, None, R:], base, dtype)[:, 0]
    k, v = (c @ w[p + "uk"].T).reshape(T, H, d), (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = np.stack([causal_softmax((q[:, h, :d] @ k[:, h].T + q_rot[:, h] @ k_rot.T) * dtype(m["scale"])) @ v[:, h]
                  for h in range(H)], axis=1)
    return o.reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"attention": mixer_attention, "channel_delta": mixer_channel_delta, "latent_attention": mixer_latent}


# ----------------------------------------------------------------------------- feed-forwards
def dense_ff(w, p, u):
    return (silu(u @ w[p + "gate"].T) * (u @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(w, p, u, limit):
    a, b = np.minimum(u @ w[p + "gate"].T, limit), np.clip(u @ w[p + "up"].T, -limit, limit)
    return (a * sigmoid(1.702 * a) * (b + 1.0)) @ w[p + "down"].T


def chosen_experts(s, groups, keep, top):
    """The experts of one token, from its scores s [experts]."""
    size = len(s) // groups
    marks = s.reshape(groups, size).max(axis=1)
    kept = np.argsort(-marks, kind="stable")[:keep]
    open_to = [e for e in range(len(s)) if e // size in kept]
    return sorted(open_to, key=lambda e: (-s[e], e))[:top]


def moe_ff(w, p, u, f, dtype):
    router = f["router"]
    groups = router.get("groups") or dict(count=1, keep=1)
    s = softmax_rows(u @ w[p + "router"].T)
    y = np.zeros((len(u), w[p + "e0.down"].shape[0]), dtype=dtype)
    limit = dtype(f["expert"]["limit"])
    for t in range(len(u)):
        for e in chosen_experts(s[t], groups["count"], groups["keep"], router["top"]):
            y[t] += s[t, e] * clamped_expert(w, f"{p}e{e}.", u[t:t + 1], limit)[0]
    if f.get("shared"):
        y = y + sigmoid(u @ w[p + "shared.sg"].T) * clamped_expert(w, p + "shared.", u, dtype(f["shared"]["limit"]))
    return y


def feed_forward(w, p, u, f, dtype):
    return dense_ff(w, p, u) if f["kind"] == "dense" else moe_ff(w, p, u, f, dtype)


# ----------------------------------------------------------------------------- the model
def layer_order(config):
    """(layer, whether a pass of the repeated stretch begins with it)"""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop or loop["stop"] <= loop["start"]:
        return [(i, False) for i in range(n)]
    passes = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])] * loop["times"]
    return [(i, False) for i in range(loop["start"])] + passes + [(i, False) for i in range(loop["stop"], n)]


def forward(config, weights, tokens, dtype=np.float64, taps=None):
    """Logits [T, vocab] of one sequence.  taps: a list that receives the stream after every layer run."""
    w = {k: (v.astype(dtype) if v.dtype.kind == "f" else v) for k, v in weights.items()}
    eps = dtype(config["norm"]["eps"])
    x = x0 = w["embed"][np.asarray(tokens)]
    for i, begins in layer_order(config):
        if begins:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        layer, p = config["layers"][i], f"l{i}."
        n = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        y = MIXERS[layer["type"]](w, p + "mix.", n, layer["mixer"], eps, dtype)
        if layer.get("mlp") is not None:
            y = y + feed_forward(w, p + "mlp.", n, layer["mlp"], dtype)
        x = x + y
        if taps is not None:
            taps.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
