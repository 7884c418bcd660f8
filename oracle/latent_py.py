"""Plain numpy restatement of the layer-list designs (Falivik): one function per mechanism, whole sequences at once, no
cache, no batching tricks.  Test infrastructure only; shares no code with the library.

Weights come as a dict name -> float array (the tensor names of a model directory), the configuration as the parsed
config.json.  ``dtype`` is the arithmetic type (float64 by default, so that the oracle's own rounding does not matter).
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np


def rms_norm(x, weight, eps):
    """x over sqrt(mean x^2 + eps), scaled element by element."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def linear(x, w):
    """Rows of x through a weight stored [out, in]."""
    return x @ w.T


def relu_squared(z):
    return np.square(np.maximum(z, 0.0))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def rotate_half(x, pos, base, dims):
    """Rotate the first ``dims`` entries of the last axis; entry i pairs with entry i + dims / 2.
    x: [n, ..., d], pos: [n] absolute positions."""
    half = dims // 2
    freq = np.power(float(base), -2.0 * np.arange(half) / dims)
    ang = pos.astype(np.float64)[:, None] * freq[None, :]
    ang = ang.reshape((len(pos),) + (1,) * (x.ndim - 2) + (half,))
    c, s = np.cos(ang).astype(x.dtype), np.sin(ang).astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def window_mask(n_q, n_k, size, pos0=0):
    """True where query pos0 + i may see key j: the last `size` positions up to its own."""
    d = (pos0 + np.arange(n_q))[:, None] - np.arange(n_k)[None, :]
    return (d >= 0) & (d < size)


def sink_softmax(scores, mask, sink):
    """scores [H, q, k]; the denominator has one more term exp(sink[h]) that carries no value."""
    s = np.where(mask[None], scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - top))


def latent_kv(h, w, p, mix, eps, pos):
    """What a layer with its own latent projection caches: the normed latent and the shared rotated key part."""
    kv = linear(h, w[p + ".dkv"])
    r = mix["kv_rank"]
    c = rms_norm(kv[:, :r], w[p + ".dkv.norm"], eps)
    kr = rotate_half(kv[:, r:], pos, mix["rot"]["base"], mix["rot"]["dims"])
    return c, kr


def latent_attention(h, w, p, mix, eps, pos, c, kr):
    """h [n, width] is the mixer's input, (c, kr) the latents it attends to (its own or another layer's)."""
    n, H, d, rd, vd = len(h), mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    q = linear(rms_norm(linear(h, w[p + ".dq"]), w[p + ".dq.norm"], eps), w[p + ".uq"]).reshape(n, H, d + rd)
    qn, qr = q[..., :d], rotate_half(q[..., d:], pos, mix["rot"]["base"], mix["rot"]["dims"])
    k = linear(c, w[p + ".uk"]).reshape(n, H, d)
    v = linear(c, w[p + ".uv"]).reshape(n, H, vd)
    s = (np.einsum("qhd,khd->hqk", qn, k) + np.einsum("qhd,kd->hqk", qr, kr)) * mix["scale"]
    a = sink_softmax(s, window_mask(n, n, mix["mask"]["size"]), w[p + ".sink"])
    o = np.einsum("hqk,khd->qhd", a, v).reshape(n, H * vd)
    return linear(o * sigmoid(linear(h, w[p + ".g"])), w[p + ".o"])


def dense_mlp(h, w, p):
    return linear(relu_squared(linear(h, w[p + ".up"])), w[p + ".down"])


def side_input(x, e, w, p, eps):
    """The per-layer token input: what is added to the residual stream x for the layer's table rows e."""
    y = linear(gelu_tanh(linear(x, w[p + ".gate"])) * e, w[p + ".proj"])
    return rms_norm(y, w[p + ".norm"], eps)


def forward(cfg, w, tokens, dtype=np.float64, layers_out=None):
    """Logits [n, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, dtype=dtype) if v.dtype.kind == "f" else v for k, v in w.items()}
    tokens = np.asarray(tokens)
    pos = np.arange(len(tokens))
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens]
    latents = {}
    for i, L in enumerate(cfg["layers"]):
        p, mix = f"l{i}", L["mixer"]
        h1 = rms_norm(x, w[p + ".norm1"], eps)
        src = mix.get("kv_from")
        if src is None:
            latents[i] = latent_kv(h1, w, p + ".mix", mix, eps, pos)
            src = i
        add = latent_attention(h1, w, p + ".mix", mix, eps, pos, *latents[src])
        if L["mlp"] is not None:
            add = add + dense_mlp(rms_norm(x, w[p + ".norm2"], eps), w, p + ".mlp")
        x = x + add
        sd = cfg["token_side"]["dim"]
        x = x + side_input(x, w["side.embed"][tokens][:, i * sd:(i + 1) * sd], w, p + ".side", eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return linear(rms_norm(x, w["final.norm"], eps), w["head"])


def load_dir(path):
    """(config, tensors as float32) of a model directory."""
    path = Path(path)
    cfg = json.loads((path / "config.json").read_text())
    raw = (path / "model.safetensors").read_bytes()
    n = int.from_bytes(raw[:8], "little")
    head, body, w = json.loads(raw[8:8 + n]), memoryview(raw)[8 + n:], {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        if t["dtype"] == "BF16":
            v = (np.frombuffer(body[a:b], dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        else:
            v = np.frombuffer(body[a:b], dtype={"F32": "<f4", "F16": "<f2", "I32": "<i4"}[t["dtype"]])
        w[name] = v.reshape(t["shape"])
    return cfg, w
