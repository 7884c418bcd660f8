"""Plain numpy restatement of Gipotar's mechanisms: one function each, whole sequences at once, token by token where a
mechanism is a recurrence; no cache, no chunks, no batching.  Test infrastructure only; shares no code with the library.

Weights come as a dict name -> float array (the tensor names of a model directory), the configuration as the parsed
config.json.  ``dtype`` is the arithmetic type (float64 by default, so that the oracle's own rounding does not matter).
"""
from __future__ import annotations

import numpy as np

from oracle.latent_py import linear, load_dir, rms_norm, rotate_half, sigmoid

UNIT_EPS = 1e-6          # added to the sum of squares of a unit vector


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def norm_about_one(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_norm(x, 1.0 + w, eps)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + UNIT_EPS)


def shift(h):
    """The previous token's row; zeros before the first."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def mix(h, mu):
    return h + (shift(h) - h) * mu


def causal_conv(x, taps):
    """x [n, channels], taps [channels, k]; the last tap belongs to the current token."""
    n, k = len(x), taps.shape[1]
    padded = np.concatenate([np.zeros((k - 1, x.shape[1]), dtype=x.dtype), x])
    return sum(padded[i:i + n] * taps[:, i] for i in range(k))


def causal_softmax(s):
    """s [heads, q, k] with as many queries as keys."""
    n = s.shape[-1]
    s = np.where(np.tril(np.ones((n, n), dtype=bool)), s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def grouped_attention(h, w, p, m, pos):
    """Softmax attention with shared key / value heads; keys and values may differ in length, part of a head is rotated."""
    n, H, G, d, vd = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = linear(h, w[p + ".q"]).reshape(n, H, d), linear(h, w[p + ".k"]).reshape(n, G, d)
    v = linear(h, w[p + ".v"]).reshape(n, G, vd)
    q, k = (rotate_half(t, pos, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    own = np.arange(H) // (H // G)
    a = causal_softmax(np.einsum("qhd,khd->hqk", q, k[:, own]) * m["scale"])
    return linear(np.einsum("hqk,khd->qhd", a, v[:, own]).reshape(n, H * vd), w[p + ".o"])


def decay_of(mix_w, w, p):
    """Per key channel, between 0 and 1: exp(-exp(low-rank function of the token + w0))."""
    return np.exp(-np.exp(linear(np.tanh(linear(mix_w, w[p + ".w1"])), w[p + ".w2"]) + w[p + ".w0"]))


def bonus_recurrence(r, k, v, decay, u):
    """r, k, decay [n, heads, d], v [n, heads, dv], u [heads, d]: the read-out sees the current token through u only."""
    n, H, d = r.shape
    S, out = np.zeros((H, d, v.shape[-1]), dtype=r.dtype), np.empty((n, H, v.shape[-1]), dtype=r.dtype)
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hi,hij->hj", r[t], S + u[:, :, None] * kv)
        S = decay[t][:, :, None] * S + kv
    return out


def time_mixing(h, w, p, m, eps):
    n, H, d = len(h), m["heads"], m["dim"]
    x = {s: mix(h, w[f"{p}.mu.{s}"]) for s in "rkvgw"}
    r, k, v = (linear(x[s], w[f"{p}.{s}"]).reshape(n, H, d) for s in "rkv")
    o = bonus_recurrence(r, k, v, decay_of(x["w"], w, p).reshape(n, H, d), w[p + ".u"])
    o = rms_norm(o, 1.0, eps).reshape(n, H * d) * w[p + ".norm"]
    return linear(o * silu(linear(x["g"], w[p + ".g"])), w[p + ".o"])


def parallel(h, w, p, m, eps, pos):
    return m["left_scale"] * grouped_attention(h, w, p + ".left", m["left"], pos) + m["right_scale"] * time_mixing(h, w, p + ".right", m["right"], eps)


def delta_recurrence(q, k, v, g, beta):
    """q, k [n, heads, d], v [n, heads, dv], g, beta [n, heads]: decay, correct what the state holds for k, read out."""
    n, H, d = q.shape
    S, out = np.zeros((H, d, v.shape[-1]), dtype=q.dtype), np.empty(v.shape, dtype=q.dtype)
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hij,hi->hj", S, q[t])
    return out


def gated_delta(h, w, p, m, eps):
    n, H, G, d, vd = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(linear(h, w[f"{p}.{s}"]), w[f"{p}.{s}.conv"])) for s in "qkv")
    own = np.arange(H) // (H // G)
    q, k = unit(q.reshape(n, G, d))[:, own] * d ** -0.5, unit(k.reshape(n, G, d))[:, own]
    beta = sigmoid(linear(h, w[p + ".b"]))
    g = np.exp(-np.exp(w[p + ".A_log"]) * softplus(linear(h, w[p + ".a"]) + w[p + ".dt_bias"]))
    o = delta_recurrence(q, k, v.reshape(n, H, vd), g, beta)
    o = rms_norm(o, w[p + ".norm"], eps) * silu(linear(h, w[p + ".g"])).reshape(n, H, vd)
    return linear(o.reshape(n, H * vd), w[p + ".o"])


def clamped_glu(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_mlp(h, w, p, limit):
    return linear(clamped_glu(linear(h, w[p + ".gate"]), linear(h, w[p + ".up"]), limit), w[p + ".down"])


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def forward(cfg, w, tokens, dtype=np.float64, layers_out=None):
    """Logits [n, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, dtype=dtype) if v.dtype.kind == "f" else v for k, v in w.items()}
    tokens = np.asarray(tokens)
    pos, eps, rm = np.arange(len(tokens)), cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}"
        h = norm_about_one(x, w[p + ".norm1"], eps)
        x = x + rm * (parallel(h, w, p + ".mix", L["mixer"], eps, pos) if L["type"] == "parallel" else gated_delta(h, w, p + ".mix", L["mixer"], eps))
        if L["mlp"] is not None:
            x = x + rm * dense_mlp(norm_about_one(x, w[p + ".norm2"], eps), w, p + ".mlp", L["mlp"]["limit"])
        if layers_out is not None:
            layers_out.append(x.copy())
    return softcap(linear(norm_about_one(x, w["final.norm"], eps), w["head"]), cfg["logit_softcap"])


__all__ = ["forward", "load_dir"]
