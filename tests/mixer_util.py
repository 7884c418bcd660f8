"""Small Gipotar configurations, weights and comparisons."""
from __future__ import annotations

import numpy as np

from cuqwen_b200 import stackfmt as F
from oracle import mixers_py as M
from stack_util import check, errors, run_portions

P, D = F.parallel_layer, F.delta_layer


def small():
    """One layer of each kind, grouped heads in both, sizes that are no multiple of a tile."""
    return F.gipotar_config(99, 104, [P(6, 2, 24, 40, 16, 3, 24, 88, base=5000.0, left_scale=0.7, right_scale=1.3, limit=1.5), D(4, 2, 24, 16, 4, 72, limit=0.9)], eps=1e-5, residual_mult=0.6,
                            embed_scale=3.0, softcap=9.0)


def odd():
    """Lengths that are no multiple of eight, layers that differ in everything, one tap and many, no feed-forward in some, rotation of a
    part (also of two entries), of all and of none."""
    ls = [D(3, 1, 13, 21, 1, None), P(4, 4, 22, 9, 6, 2, 11, 37, base=300.0, left_scale=1.4, right_scale=0.5, limit=0.8), D(6, 3, 5, 30, 7, 50, limit=2.5), P(6, 3, 10, 17, 10, 5, 7, None, left_scale=0.9, right_scale=-1.1),
          P(2, 1, 7, 12, 0, 1, 30, 11, limit=5.0), D(2, 2, 40, 3, 2, 19)]
    return F.gipotar_config(101, 100, ls, eps=3e-5, residual_mult=0.45, embed_scale=2.5, softcap=20.0)


def ones():
    """Everything that can be 1 is."""
    return F.gipotar_config(50, 40, [P(1, 1, 8, 1, 2, 1, 1, 1), D(1, 1, 1, 1, 1, 1), P(1, 1, 1, 8, 0, 1, 8, 24), D(1, 1, 8, 8, 2, None)], softcap=50.0)


def wide():
    """Long heads, many of them, several blocks in every dimension."""
    return F.gipotar_config(300, 512, [D(6, 2, 128, 96, 4, 640), P(20, 1, 96, 160, 64, 5, 64, 704), D(2, 1, 200, 256, 3, None), P(4, 2, 160, 256, 160, 2, 136, 320)], residual_mult=0.5, embed_scale=4.0, softcap=15.0)


RANKS = {"small": 12, "odd": [0, 5, 0, 19, 1, 0], "ones": [1, 0, 3, 0], "wide": 40}
MAKERS = {"small": small, "odd": odd, "ones": ones, "wide": wide}


def weights(name, seed, sharp=1.0):
    """Configuration, bfloat16 bits and their float32 values.  sharp scales the attention's queries, so that a few keys carry it."""
    cfg = MAKERS[name]()
    w = F.random_weights(cfg, seed, rank=RANKS[name])
    for k in w:
        if k.endswith("left.q") and sharp != 1.0:
            w[k] = F.to_bf16(F.from_bf16(w[k]) * sharp)
    return cfg, w, {k: F.from_bf16(v) for k, v in w.items()}


def causal_window(n):
    return np.tril(np.ones((n, n), dtype=bool))


__all__ = ["F", "M", "P", "D", "RANKS", "MAKERS", "small", "odd", "ones", "wide", "weights", "check", "errors", "run_portions"]
