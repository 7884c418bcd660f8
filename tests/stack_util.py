"""Small configurations, weights and comparisons for the tests of the layer-list designs."""
from __future__ import annotations

import numpy as np

from cuqwen_b200 import stackfmt as F
from oracle import latent_py as L

# Largest error of a position and mean error, both as root mean square over the vocabulary of the difference of the
# mean-free logits, relative to the standard deviation of all logits.
LIMIT = {"float32": (2e-5, 5e-6), "bfloat16": (4e-2, 8e-3)}


def small(vocab=97, width=104, side=12, window=9, layers=2):
    """Heads, ranks and lengths that are no multiple of a tile; the second layer attends to the first one's latents."""
    return F.falivik_config(vocab, width, side, [F.latent_layer(3, 24, 8, 16, 40, 48, window, 72, kv_from=0 if i == 1 else None) for i in range(layers)])


def odd():
    """Lengths that are no multiple of eight, layers that differ in everything, no feed-forward in one, latents shared."""
    ll = F.latent_layer
    return F.falivik_config(101, 100, 10, [ll(3, 20, 12, 28, 36, 44, 7, 72), ll(2, 13, 12, 19, 27, 44, 30, None, kv_from=0), ll(1, 9, 2, 5, 11, 13, 64, 33, base=500.0)], eps=1e-5)


def tiles():
    """Several 64-column blocks per head part, more heads than one tile of the decode attention, wide layers."""
    ll = F.latent_layer
    return F.falivik_config(300, 512, 64, [ll(5, 64, 32, 128, 192, 256, 100, 1024), ll(18, 136, 72, 200, 320, 520, 200, 640)])


def weights(cfg, seed, sharp=1.0):
    """bfloat16 bits and their float32 values; sharp scales the query projections, so that a few keys carry the attention."""
    w = F.random_weights(cfg, seed)
    if sharp != 1.0:
        for k in w:
            if k.endswith("mix.uq"):
                w[k] = F.to_bf16(F.from_bf16(w[k]) * sharp)
    return w, {k: F.from_bf16(v) for k, v in w.items()}


def errors(got, want):
    """Error of every position, see LIMIT."""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()


def check(got, want, act, factor=1.0):
    e = errors(got, want)
    top, mean = LIMIT[act]
    assert np.isfinite(e).all() and e.max() <= top * factor and e.mean() <= mean * factor, f"{act}: max {e.max():.2e} at {int(e.argmax())}, mean {e.mean():.2e}"
    return e


def run_portions(eng, toks, sizes, pos0=0):
    """All logits of a sequence fed in portions of the given sizes (the last one repeats)."""
    out, i, k = [], 0, 0
    while i < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - i)
        out.append(eng.extend(toks[i:i + n], pos0 + i, range(n)))
        i += n
        k += 1
    return np.concatenate(out)


__all__ = ["F", "L", "LIMIT", "small", "odd", "tiles", "weights", "errors", "check", "run_portions"]
