"""Model directories without a GPU: what the library reads from config.json, what it refuses, the oracle's mechanisms, the
command lines."""
from __future__ import annotations

import copy
import importlib.machinery
import importlib.util
import json
from pathlib import Path

import numpy as np
import pytest

from cuqwen_b200 import CuQwenError
from cuqwen_b200 import engine as E
from cuqwen_b200 import generate
from stack_util import F, L, odd, small, weights

ROOT = Path(__file__).resolve().parent.parent


def describe(tmp_path, cfg) -> str:
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return E.describe(tmp_path)


def test_every_size_is_read_from_the_configuration(built, tmp_path):
    cfg = odd()
    text = describe(tmp_path, cfg).splitlines()
    assert text[:6] == ["design Falivik", f"vocab {cfg['vocab']}", f"width {cfg['width']}", "layers 3", "norm_eps 1e-05", "side_dim 10"]
    for i, L_ in enumerate(cfg["layers"]):
        f = text[6 + i].split()
        got = dict(zip(f[3::2], f[4::2]))
        m = L_["mixer"]
        assert f[:3] == ["layer", str(i), "latent_attention"]
        for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"):
            assert got[k] == str(m[k])
        assert got["window"] == str(m["mask"]["size"]) and got["kv_from"] == str(m.get("kv_from", -1)) and got["ff"] == str(L_["mlp"]["ff"] if L_["mlp"] else 0)
        assert float(got["scale"]) == pytest.approx(m["scale"], rel=1e-7) and float(got["rot_base"]) == m["rot"]["base"]


@pytest.mark.parametrize("change,code", [
    (lambda c: c.update(architecture="Nonesuch"), 4), (lambda c: c.pop("architecture"), 4), (lambda c: c.update(width=0), 4), (lambda c: c.update(vocab=1.5), 4),
    (lambda c: c.update(layers=[]), 4), (lambda c: c["layers"][0].update(type="other"), 4), (lambda c: c["layers"][0]["mixer"].pop("heads"), 4),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=7), 4), (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4), 4),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), 4), (lambda c: c["layers"][1]["mixer"].update(kv_rank=40), 4),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=123.0), 4), (lambda c: c["layers"][0]["mlp"].update(kind="other"), 4),
    (lambda c: c["layers"][0]["mixer"].update(kv_from=0), 4)])
def test_configurations_that_are_refused(built, tmp_path, change, code):
    cfg = copy.deepcopy(small())
    change(cfg)
    with pytest.raises(CuQwenError) as e:
        describe(tmp_path, cfg)
    assert e.value.code == code


def test_a_latent_may_not_come_from_a_layer_that_borrows_one(built, tmp_path):
    cfg = small(layers=3)
    cfg["layers"][2]["mixer"]["kv_from"] = 1
    with pytest.raises(CuQwenError):
        describe(tmp_path, cfg)


def test_broken_files_are_io_errors(built, tmp_path):
    with pytest.raises(CuQwenError) as e:
        E.describe(tmp_path / "nowhere")
    assert e.value.code == 2
    for text in ("", "{", "[1, 2", '{"a": tru}', '{"architecture": "Falivik"} x'):
        (tmp_path / "config.json").write_text(text)
        with pytest.raises(CuQwenError) as e:
            E.describe(tmp_path)
        assert e.value.code == 2


def test_json_forms(built, tmp_path):
    cfg = small()
    text = json.dumps(cfg).replace('"Falivik"', '"\\u0046alivik"')          # escapes, unknown keys, nested lists, white space
    (tmp_path / "config.json").write_text(' \n{"x": [1, [2.5e-3, {"y": null}], "\\"\\\\", true], ' + text[1:].replace(",", " ,\t") + "\n")
    assert "design Falivik" in E.describe(tmp_path)


def test_model_directory_round_trip(tmp_path):
    cfg = odd()
    w, wf = weights(cfg, 5)
    F.write_model_dir(tmp_path, cfg, w)
    cfg2, w2 = L.load_dir(tmp_path)
    assert cfg2 == cfg and set(w2) == set(w) == set(F.falivik_shapes(cfg))
    for k in w:
        assert np.array_equal(w2[k], wf[k])


# ---- the oracle's mechanisms, each against a second statement of the same thing -----------------------------------------
def test_rotation_keeps_inner_products_relative():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 1, 12))
    for d in (0, 1, 5):
        s = [float(np.sum(L.rotate_half(q, np.array([p + d]), 100.0, 12) * L.rotate_half(k, np.array([p]), 100.0, 12))) for p in (0, 3, 77)]
        assert np.allclose(s, s[0])
    x = rng.standard_normal((1, 12))
    y = L.rotate_half(x, np.array([2]), 100.0, 8)
    assert np.array_equal(y[:, 8:], x[:, 8:])
    z = (x[0, 1] + 1j * x[0, 5]) * np.exp(2j * 100.0 ** (-2 / 8))             # pair (1, 1 + dims / 2)
    assert np.allclose([y[0, 1], y[0, 5]], [z.real, z.imag])


def test_window_sees_itself_and_size_minus_one_before():
    m = L.window_mask(6, 6, 3)
    assert [list(np.flatnonzero(r)) for r in m] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4], [3, 4, 5]]
    assert np.array_equal(L.window_mask(2, 6, 3, pos0=4), m[4:])


def test_sink_is_a_key_without_value():
    rng = np.random.default_rng(1)
    s, sink = rng.standard_normal((2, 1, 4)), np.array([0.3, -0.7])
    p = L.sink_softmax(s, np.ones((1, 4), bool), sink)
    full = np.concatenate([s, np.broadcast_to(sink[:, None, None], (2, 1, 1))], axis=-1)
    full = np.exp(full) / np.exp(full).sum(axis=-1, keepdims=True)
    assert np.allclose(p, full[..., :-1]) and (p.sum(axis=-1) < 1).all()


def test_latents_carry_the_keys_and_values():
    """Scores and outputs through W_uk / W_uv equal those against the latents themselves (what decoding relies on)."""
    rng = np.random.default_rng(2)
    c, wk, wv, q, p = rng.standard_normal((7, 10)), rng.standard_normal((6, 10)), rng.standard_normal((5, 10)), rng.standard_normal(6), rng.random(7)
    assert np.allclose(L.linear(c, wk) @ q, c @ (wk.T @ q)) and np.allclose(p @ L.linear(c, wv), L.linear(p @ c, wv))


def test_norm_relu_gelu_sigmoid_values():
    x = np.array([[3.0, -4.0]])
    assert np.allclose(L.rms_norm(x, np.array([2.0, 1.0]), 0.0), [[6 / np.sqrt(12.5), -4 / np.sqrt(12.5)]])
    assert np.allclose(L.rms_norm(np.zeros((1, 2)), np.ones(2), 1e-6), 0)
    assert np.allclose(L.relu_squared(np.array([-2.0, 3.0])), [0, 9])
    assert np.allclose(L.gelu_tanh(np.array([0.0, 1.0])), [0, 0.841192], atol=1e-6) and np.allclose(L.sigmoid(np.array([0.0, 2.0])), [0.5, 1 / (1 + np.exp(-2))])


def test_layers_without_feed_forward_have_no_second_norm():
    names = F.falivik_shapes(odd())
    assert "l1.norm2" not in names and "l1.mlp.up" not in names and "l1.mix.dkv" not in names and "l0.mix.dkv" in names


# ---- command lines -------------------------------------------------------------------------------------------------------
def load_script(name):
    loader = importlib.machinery.SourceFileLoader(name, str(ROOT / "bin" / name))
    mod = importlib.util.module_from_spec(importlib.util.spec_from_loader(name, loader))
    loader.exec_module(mod)
    return mod


def test_trace_run_keeps_one_sequence():
    r = load_script("trace_run").Requests()
    assert r.begin("a", 3) == 0 and r.begin("a", 2) == 3
    with pytest.raises(ValueError):
        r.begin("b", 1)
    r.end("other")
    r.end("a")
    assert r.begin("b", 4) == 0 and r.begin("b", 1) == 4


def test_generate_command_line(tmp_path):
    a = generate.parser().parse_args(["--model", "m", "--tokens", "1,2 3", "-n", "4"])
    assert a.dtype == "bfloat16" and a.n == 4
    with pytest.raises(SystemExit):
        generate.main(["--model", str(tmp_path)])
    with pytest.raises(SystemExit):
        generate.main(["--model", str(tmp_path / "file.bin"), "--tokens", "1"])
