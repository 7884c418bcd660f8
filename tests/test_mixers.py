"""Gipotar without a GPU: what the library reads from config.json and refuses, the oracle's mechanisms against a second statement of
the same thing."""
from __future__ import annotations

import copy
import json

import numpy as np
import pytest

from cuqwen_b200 import CuQwenError
from cuqwen_b200 import engine as E
from mixer_util import F, M, MAKERS, odd, small, weights
from oracle import latent_py


def describe(tmp_path, cfg) -> list:
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return E.describe(tmp_path).splitlines()


def test_every_size_and_constant_is_read_from_the_configuration(built, tmp_path):
    cfg = odd()
    text = describe(tmp_path, cfg)
    assert text[0] == "design Gipotar" and f"vocab {cfg['vocab']}" in text and f"width {cfg['width']}" in text
    top = dict(t.split() for t in text[:9])
    assert float(top["norm_eps"]) == cfg["norm"]["eps"] and float(top["residual_mult"]) == cfg["residual_mult"] and float(top["embed_scale"]) == cfg["embedding"]["scale"]
    assert float(top["logit_softcap"]) == cfg["logit_softcap"]
    for i, L in enumerate(cfg["layers"]):
        f = text[9 + i].split()
        got, m = {k: float(v) for k, v in zip(f[3::2], f[4::2])}, L["mixer"]
        assert f[:3] == ["layer", str(i), L["type"]]
        if L["type"] == "parallel":
            a, t = m["left"], m["right"]
            want = {"left_heads": a["heads"], "left_kv_heads": a["kv_heads"], "left_dim": a["dim"], "left_vdim": a["vdim"], "score_scale": a["scale"], "rot_dims": a["rot"]["dims"], "rot_base": a["rot"]["base"],
                    "right_heads": t["heads"], "right_dim": t["dim"], "left_scale": m["left_scale"], "right_scale": m["right_scale"]}
        else:
            want = dict(m)
        want["ff"] = L["mlp"]["ff"] if L["mlp"] else 0
        if L["mlp"]:
            want["limit"] = L["mlp"]["limit"]
        for k, v in want.items():
            assert got[k] == pytest.approx(v, rel=1e-7), (i, k)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="latent_attention"), lambda c: c["layers"][0].pop("type"), lambda c: c["layers"][0]["mixer"].pop("left"), lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=5), lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26),
    lambda c: c["layers"][0]["mixer"].pop("right_scale"), lambda c: c["layers"][0]["mixer"]["right"].update(heads=0), lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][1]["mixer"].update(conv=0), lambda c: c["layers"][1]["mlp"].update(kind="sparse"), lambda c: c["layers"][1]["mlp"].pop("limit"), lambda c: c["layers"][1]["mlp"].update(limit=-1.0),
    lambda c: c.update(layers=[]), lambda c: c.pop("norm"), lambda c: c.update(logit_softcap=-2.0), lambda c: c["embedding"].update(scale="big")])
def test_configurations_that_are_refused(built, tmp_path, change):
    cfg = copy.deepcopy(small())
    change(cfg)
    with pytest.raises(CuQwenError) as e:
        describe(tmp_path, cfg)
    assert e.value.code == 4


@pytest.mark.parametrize("name", sorted(MAKERS))
def test_model_directory_round_trip(tmp_path, name):
    cfg, w, wf = weights(name, 3)
    F.write_model_dir(tmp_path, cfg, w)
    cfg2, w2 = latent_py.load_dir(tmp_path)
    assert cfg2 == cfg and set(w2) == set(w) and all(np.array_equal(w2[k], wf[k]) for k in w)


# ---- the oracle's mechanisms ------------------------------------------------------------------------------------------------
rng = np.random.default_rng(0)


def test_norm_is_stored_about_zero():
    x, w = rng.standard_normal((3, 8)), rng.standard_normal(8)
    assert np.allclose(M.norm_about_one(x, w, 0.1), x * (1 + w) / np.sqrt((x * x).sum(-1, keepdims=True) / 8 + 0.1))


def test_mixes_start_from_zeros():
    h, mu = rng.standard_normal((4, 5)), rng.random(5)
    y = M.mix(h, mu)
    assert np.allclose(y[0], h[0] * (1 - mu)) and np.allclose(y[2], h[2] * (1 - mu) + h[1] * mu)


def test_convolution_is_numpys():
    x, taps = rng.standard_normal((9, 3)), rng.standard_normal((3, 4))
    assert np.allclose(M.causal_conv(x, taps), np.stack([np.convolve(x[:, c], taps[c][::-1])[:9] for c in range(3)], axis=1))


def test_bonus_recurrence_is_a_weighted_sum_over_the_past():
    n, H, d = 7, 2, 3
    r, k, v, w, u = *rng.standard_normal((3, n, H, d)), rng.random((n, H, d)), rng.standard_normal((H, d))
    got = M.bonus_recurrence(r, k, v, w, u)
    for t in range(n):
        want = np.einsum("hi,hi->h", r[t] * u, k[t])[:, None] * v[t]
        for s in range(t):
            want = want + np.einsum("hi,hi->h", r[t] * np.prod(w[s + 1:t], axis=0), k[s])[:, None] * v[s]
        assert np.allclose(got[t], want)


def test_delta_recurrence_stores_and_corrects():
    n, H, d, dv = 5, 1, 4, 3
    k = np.zeros((n, H, d))
    for t, i in enumerate([0, 1, 0, 2, 1]):
        k[t, 0, i] = 1.0
    v, one, q = rng.standard_normal((n, H, dv)), np.ones((n, H)), k.copy()
    o = M.delta_recurrence(q, k, v, one, one)                          # full steps, no decay: what is asked for is what was just stored
    assert np.allclose(o, v)
    q[4, 0] = k[2, 0]                                                   # an older key is still there ...
    assert np.allclose(M.delta_recurrence(q, k, v, one, one)[4], v[2])
    assert np.allclose(M.delta_recurrence(q, k, v, one * 0.5, one)[4], v[2] * 0.25)      # ... unless it has decayed
    S = np.zeros((d, dv))                                               # against the matrix form of the transition
    g, b, k, q = rng.random((n, 1)), rng.random((n, 1)), M.unit(rng.standard_normal((n, H, d))), rng.standard_normal((n, H, d))
    got = M.delta_recurrence(q, k, v, g, b)
    for t in range(n):
        kk = k[t, 0]
        S = g[t] * (np.eye(d) - b[t] * np.outer(kk, kk)) @ S + b[t] * np.outer(kk, v[t, 0])
        assert np.allclose(got[t, 0], S.T @ q[t, 0])


def test_grouped_heads_share_keys():
    cfg, _, w = weights("small", 1)
    m, h = cfg["layers"][0]["mixer"]["left"], rng.standard_normal((6, cfg["width"]))
    full = dict(m, kv_heads=m["heads"])
    rep = m["heads"] // m["kv_heads"]
    ww = {k: v.astype(np.float64) for k, v in w.items()}
    for s, n in (("k", m["dim"]), ("v", m["vdim"])):
        a = w[f"l0.mix.left.{s}"].astype(np.float64).reshape(m["kv_heads"], n, -1)
        ww[f"l0.mix.left.{s}"] = np.repeat(a, rep, axis=0).reshape(m["heads"] * n, -1)
    pos = np.arange(6)
    assert np.allclose(M.grouped_attention(h, w, "l0.mix.left", m, pos), M.grouped_attention(h, ww, "l0.mix.left", full, pos))


def test_gated_unit_and_cap():
    g, u = np.array([-3.0, 0.5, 9.0]), np.array([-9.0, 0.5, 9.0])
    s = lambda z: 1 / (1 + np.exp(-z))
    assert np.allclose(M.clamped_glu(g, u, 2.0), [-3 * s(-5.106) * -1, 0.5 * s(0.851) * 1.5, 2 * s(3.404) * 3])
    assert np.allclose(M.softcap(np.array([0.0, 1.0, 1e6]), 4.0), [0, 4 * np.tanh(0.25), 4])
    assert np.allclose(M.softplus(np.array([-50.0, 0.0, 800.0])), [0, np.log(2), 800.0], atol=1e-12) and np.allclose(np.linalg.norm(M.unit(rng.standard_normal((4, 6))), axis=-1), 1)


def test_layers_without_feed_forward_have_no_second_norm():
    names = F.gipotar_shapes(odd(), [0, 5, 0, 19, 1, 0])
    assert "l0.norm2" not in names and "l3.mlp.up" not in names and "l1.norm2" in names and names["l3.mix.right.w1"] == (19, 100)
