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


def random_weights(cfg, seed: int, block: int | None = None) -> dict:
    """bfloat16 weights (uint16 bits): matrices N(0, 1 / columns), embeddings and sinks N(0, 1), norms 1 + N(0, 0.1).
    block: draw that many values once and repeat them (large models, where drawing every value would take minutes)."""
    rng = np.random.default_rng(seed)
    pool = to_bf16(rng.standard_normal(block, dtype=np.float32)) if block else None
    w = {}
    for name, shape in falivik_shapes(cfg).items():
        n = int(np.prod(shape))
        if name.endswith("norm") or name.endswith("norm1") or name.endswith("norm2"):
            w[name] = to_bf16(1.0 + 0.1 * rng.standard_normal(shape))
            continue
        s = 1.0 if len(shape) == 1 or name.endswith("embed") else shape[1] ** -0.5
        if pool is not None and n > block:
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
