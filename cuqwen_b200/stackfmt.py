"""Model directories of the layer-list designs: configuration builder, random weights, safetensors writer (numpy only)."""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np


def to_bf16(a) -> np.ndarray:
    """Round float32 to bfloat16 (nearest, ties to even); the bits as uint16."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(b) -> np.ndarray:
    return (np.asarray(b).astype(np.uint32) << 16).view(np.float32)


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, ff, scale=None, base=10000.0, kv_from=None) -> dict:
    """One entry of a Falivik configuration's layer list; ff None: no feed-forward."""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "scale": float((dim + rot_dim) ** -0.5 if scale is None else scale), "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def falivik_config(vocab, width, side_dim, layers, eps=1e-6) -> dict:
    return {"architecture": "Falivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side_dim}, "layers": layers}


def falivik_shapes(cfg) -> dict:
    """Tensor names and shapes that a configuration asks for."""
    W, sd, V, n = cfg["width"], cfg["token_side"]["dim"], cfg["vocab"], len(cfg["layers"])
    out = {"embed": (V, W), "side.embed": (V, n * sd)}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        H, d, r, v, q, k = (m[x] for x in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
        out.update({p + "norm1": (W,), p + "mix.dq": (q, W), p + "mix.dq.norm": (q,), p + "mix.uq": (H * (d + r), q)})
        if m.get("kv_from") is None:
            out.update({p + "mix.dkv": (k + r, W), p + "mix.dkv.norm": (k,)})
        out.update({p + "mix.uk": (H * d, k), p + "mix.uv": (H * v, k), p + "mix.sink": (H,), p + "mix.g": (H * v, W), p + "mix.o": (W, H * v)})
        if L["mlp"] is not None:
            out.update({p + "norm2": (W,), p + "mlp.up": (L["mlp"]["ff"], W), p + "mlp.down": (W, L["mlp"]["ff"])})
        out.update({p + "side.gate": (sd, W), p + "side.proj": (W, sd), p + "side.norm": (W,)})
    out.update({"final.norm": (W,), "head": (V, W)})
    return out


def parallel_layer(heads, kv_heads, dim, vdim, rot_dims, right_heads, right_dim, ff, scale=None, base=10000.0, left_scale=1.0, right_scale=1.0, limit=7.0) -> dict:
    """Entry of a Gipotar configuration's layer list: softmax attention beside time mixing; ff None: no feed-forward."""
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit},
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(dim ** -0.5 if scale is None else scale), "rot": {"base": base, "dims": rot_dims}},
                      "right": {"heads": right_heads, "dim": right_dim}, "left_scale": left_scale, "right_scale": right_scale}}


def delta_layer(heads, kv_heads, dim, vdim, conv, ff, limit=7.0) -> dict:
    """Entry of a Gipotar configuration's layer list: gated delta rule; ff None: no feed-forward."""
    return {"type": "delta", "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def gipotar_config(vocab, width, layers, eps=1e-6, residual_mult=1.0, embed_scale=1.0, softcap=30.0) -> dict:
    return {"architecture": "Gipotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "residual_mult": residual_mult, "logit_softcap": softcap, "layers": layers}


def gipotar_shapes(cfg, rank=16) -> dict:
    """Tensor names and shapes that a configuration asks for; rank: length of the decay's thin matrices (one for all layers, or one a layer)."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W)}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        out[p + "norm1"] = (W,)
        if L["type"] == "parallel":
            a, t, n = m["left"], m["right"], rank if isinstance(rank, int) else rank[i]
            l, r, R = p + "mix.left.", p + "mix.right.", t["heads"] * t["dim"]
            out.update({l + "q": (a["heads"] * a["dim"], W), l + "k": (a["kv_heads"] * a["dim"], W), l + "v": (a["kv_heads"] * a["vdim"], W), l + "o": (W, a["heads"] * a["vdim"])})
            out.update({r + "mu." + s: (W,) for s in "rkvgw"} | {r + s: (R, W) for s in "rkvg"})
            out.update({r + "w1": (n, W), r + "w2": (R, n), r + "w0": (R,), r + "u": (t["heads"], t["dim"]), r + "norm": (R,), r + "o": (W, R)})
        else:
            H, G, d, v, c, q = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], p + "mix."
            out.update({q + "q": (G * d, W), q + "q.conv": (G * d, c), q + "k": (G * d, W), q + "k.conv": (G * d, c), q + "v": (H * v, W), q + "v.conv": (H * v, c), q + "b": (H, W), q + "a": (H, W),
                        q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (v,), q + "g": (H * v, W), q + "o": (W, H * v)})
        if L["mlp"] is not None:
            f = L["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
    out.update({"final.norm": (W,), "head": (V, W)})
    return out


def vector_law(cfg, name):
    """(mean, deviation) of a vector or of a small table of random weights; None for a matrix (N(0, 1 / columns))."""
    last = name.split(".")[-1]
    if cfg["architecture"] == "Falivik":
        return (1.0, 0.1) if "norm" in last else (0.0, 1.0) if last in ("sink", "embed") else None
    if "norm" in last:                                     # the layers' norms are stored about zero, a mixer's own about one
        return (1.0, 0.1) if ".mix." in name else (0.0, 0.1)
    return {"embed": (0.0, 1.0), "w0": (-3.0, 1.0), "u": (0.5, 0.3), "A_log": (-1.0, 0.7), "dt_bias": (-1.0, 0.7), "conv": (0.0, 0.5)}.get(last, (0.5, 0.25) if ".mu." in name else None)


def random_weights(cfg, seed: int, block: int | None = None, rank=16) -> dict:
    """bfloat16 weights (uint16 bits) of a configuration, by vector_law.
    block: draw that many values once and repeat them (large models, where drawing every value would take minutes)."""
    rng = np.random.default_rng(seed)
    pool = to_bf16(rng.standard_normal(block, dtype=np.float32)) if block else None
    w = {}
    for name, shape in (falivik_shapes(cfg) if cfg["architecture"] == "Falivik" else gipotar_shapes(cfg, rank)).items():
        n, law = int(np.prod(shape)), vector_law(cfg, name)
        mean, s = law or (0.0, shape[1] ** -0.5)
        if mean:
            w[name] = to_bf16(mean + s * rng.standard_normal(shape))
        elif pool is not None and n > block:
            w[name] = np.resize(np.roll(to_bf16(s * from_bf16(pool)), int(rng.integers(block))), n).reshape(shape)
        else:
            w[name] = to_bf16(s * rng.standard_normal(shape, dtype=np.float32))
    return w


def write_model_dir(path, cfg, weights) -> Path:
    """config.json and model.safetensors (weights: name -> uint16 bfloat16 bits)."""
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg, indent=1))
    head, off = {}, 0
    for name, a in weights.items():
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + a.nbytes]}
        off += a.nbytes
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path / "model.safetensors", "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h)
        for a in weights.values():
            f.write(np.ascontiguousarray(a).tobytes())
    return path
