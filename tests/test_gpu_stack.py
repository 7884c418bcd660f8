"""The layer-list designs on the GPU against the plain numpy oracle: each kernel alone, then whole models - prompts, decoding,
portions, sequences one after another, window and tile borders, generation."""
from __future__ import annotations

import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from cuqwen_b200 import CuQwenError
from cuqwen_b200 import engine as E
from cuqwen_b200 import kernels as K
from gpu_util import Pool, dev
from stack_util import F, L, check, errors, odd, run_portions, small, tiles, weights

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
ACTS = ["float32", "bfloat16"]
PORTIONS = [2, 3, 17, 1, 1, 40, 2, 64, 1, 33]


def act_array(a, act):
    """Activations as the kernels take them, and the values they then hold."""
    if act == "float32":
        return np.ascontiguousarray(a, dtype=np.float32), np.asarray(a, dtype=np.float32).astype(np.float64)
    b = F.to_bf16(a)
    return b, F.from_bf16(b).astype(np.float64)


def read_act(buf, act, shape):
    if act == "float32":
        return buf.numpy(np.float32).reshape(shape).astype(np.float64)
    return F.from_bf16(buf.numpy(np.uint16)).reshape(shape).astype(np.float64)


def near(got, want, act, scale=1.0):
    tol = (2e-5 if act == "float32" else 1e-2) * scale
    lim = tol * (np.abs(want) + np.sqrt(np.mean(want * want)))
    bad = np.abs(got - want) > lim
    assert np.isfinite(got).all() and not bad.any(), f"{int(bad.sum())} of {bad.size}, max {np.abs(got - want).max():.3e}"


# ---- kernels alone ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("n,rows,cols,cols2", [(1, 72, 104, 0), (1, 1000, 256, 72), (1, 2600, 640, 1024), (2, 72, 104, 40), (5, 24, 8, 0), (130, 264, 192, 72), (300, 1096, 520, 0), (257, 64, 1000, 264)])
def test_linear(built, act, n, rows, cols, cols2):
    rng = np.random.default_rng(n + rows)
    pool = Pool()
    ai = E.ACT_ID[act]
    es = 4 if act == "float32" else 2

    def mat(c):
        w = F.to_bf16(rng.standard_normal((rows, c)) * c ** -0.5)
        pad = np.zeros((rows, -(-c // 128) * 128), np.uint16)
        pad[:, :c] = w
        return pool.p(pad), pad.shape[1], F.from_bf16(w).astype(np.float64)

    x, xv = act_array(rng.standard_normal((n, cols)), act)
    w, pitch, wv = mat(cols)
    acc = xv @ wv.T
    second = None
    if cols2:
        x2, x2v = act_array(rng.standard_normal((n, cols2)), act)
        w2, p2, w2v = mat(cols2)
        second = (pool.p(x2), cols2, w2, p2, cols2)
        acc = acc + x2v @ w2v.T
    sd, vocab = rows - 3, 11
    side = F.to_bf16(rng.standard_normal((vocab, sd + 5)))
    tok = rng.integers(0, vocab, n).astype(np.int32)
    e = np.zeros((n, rows))
    e[:, :sd] = F.from_bf16(side)[tok][:, :sd]
    base = rng.standard_normal((n, rows)).astype(np.float32)
    px, ps, pt = pool.p(x), pool.p(side), pool.p(tok)
    for epi, want in ((K.LIN_F32, acc), (K.LIN_ACT, acc), (K.LIN_RELU2, L.relu_squared(acc)), (K.LIN_ADD, base + acc), (K.LIN_GELU_SIDE, L.gelu_tanh(acc) * e)):
        f32 = epi in (K.LIN_F32, K.LIN_ADD)
        out = dev(base) if epi == K.LIN_ADD else E.DevBuf(n * rows * (4 if f32 else es))
        K.linear(ai, epi, px, cols, w, pitch, cols, n, rows, out, rows, second=second, side=(ps, sd + 5, sd, pt) if epi == K.LIN_GELU_SIDE else None)
        E.sync()
        near(read_act(out, "float32" if f32 else act, (n, rows)), want, "float32" if f32 else act)


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("width", [8, 100, 1536, 3000, 9000])
def test_norm_rows_and_the_added_token_input(built, act, width):
    rng = np.random.default_rng(width)
    n, ld, eps = 3, -(-width // 8) * 8, 1e-3
    x, y, w0, w1, wy = (np.zeros((r, ld), np.float32) for r in (n, n, 1, 1, 1))
    for a in (x, y, w0, w1, wy):
        a[:, :width] = rng.standard_normal((len(a), width))
    bx, pool = dev(x), Pool()
    outs = [E.DevBuf(n * ld * (4 if act == "float32" else 2)) for _ in range(2)]
    K.norm_rows(E.ACT_ID[act], bx, ld, width, eps, n, y=pool.p(y), y_w=pool.p(wy), outs=[(pool.p(w0), outs[0]), (pool.p(w1), outs[1])], ldo=ld)
    E.sync()
    want = x[:, :width].astype(np.float64) + L.rms_norm(y[:, :width].astype(np.float64), wy[0, :width], eps)
    near(bx.numpy(np.float32).reshape(n, ld)[:, :width].astype(np.float64), want, "float32")
    for o, w in zip(outs, (w0, w1)):
        got = read_act(o, act, (n, ld))
        near(got[:, :width], L.rms_norm(want, w[0, :width], eps), act)
        assert not got[:, width:].any()


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("qr,kr,rd", [(40, 24, 6), (2500, 600, 64)])
def test_latent_rows_and_rotation_far_out(built, act, qr, kr, rd):
    rng = np.random.default_rng(qr)
    n, eps, base, pos0 = 4, 1e-6, 10000.0, 30000
    krp, rp, qp = (-(-v // 8) * 8 for v in (kr, rd, qr))
    raw = np.zeros((n, qp + krp + rp), np.float32)
    raw[:, :qr], raw[:, qp:qp + kr], raw[:, qp + krp:qp + krp + rd] = rng.standard_normal((n, qr)), rng.standard_normal((n, kr)), rng.standard_normal((n, rd))
    wq, wk = rng.standard_normal(qp).astype(np.float32), rng.standard_normal(krp).astype(np.float32)
    es, pool = 4 if act == "float32" else 2, Pool()
    rows = pos0 + n
    rot = E.DevBuf(rows * rd * 4)
    K.rot_table(rot, rows, rd, base)
    cq, cache, src = E.DevBuf(n * qp * es), E.DevBuf(rows * (krp + rp) * es), dev(raw)
    K.latent_rows(E.ACT_ID[act], src, raw.shape[1], pool.p(wq), cq, qp, qr, src.ptr + qp * 4, pool.p(wk), cache, krp + rp, kr, krp, rd, rot, eps, pos0, n)
    E.sync()
    near(read_act(cq, act, (n, qp))[:, :qr], L.rms_norm(raw[:, :qr].astype(np.float64), wq[:qr], eps), act)
    got = read_act(cache, act, (rows, krp + rp))
    near(got[pos0:, :kr], L.rms_norm(raw[:, qp:qp + kr].astype(np.float64), wk[:kr], eps), act)
    near(got[pos0:, krp:krp + rd], L.rotate_half(raw[:, qp + krp:qp + krp + rd].astype(np.float64), np.arange(pos0, rows), base, rd), act)
    assert not got[:pos0].any()


def attention_case(seed, n, nk, heads, d, rd, vd, window, spike):
    """Random queries and keys; with a spike the query at position p and the key p - spike agree, so that one score stands out."""
    rng = np.random.default_rng(seed)
    pos0 = nk - n
    q, kn, kr, v = rng.standard_normal((n, heads, d + rd)), rng.standard_normal((nk, heads, d)), rng.standard_normal((nk, rd)), rng.standard_normal((nk, heads, vd))
    if spike is not None:
        for i in range(0, n, 2):
            if pos0 + i - spike >= 0:
                q[i, :, :d] = 3.0 * kn[pos0 + i - spike]
    return q, kn, kr, v, rng.standard_normal(heads) * 2, rng.standard_normal((n, heads, vd)), pos0


def attention_oracle(q, kn, kr, v, sink, gate, pos0, window, scale, d):
    s = (np.einsum("qhd,khd->hqk", q[..., :d], kn) + np.einsum("qhd,kd->hqk", q[..., d:], kr)) * scale
    m = L.window_mask(len(q), len(kn), window if window else 1 << 30, pos0)
    if sink is None:
        sink = np.full(q.shape[1], -np.inf)
    o = np.einsum("hqk,khd->qhd", L.sink_softmax(s, m, sink), v)
    return o if gate is None else o * L.sigmoid(gate)


@pytest.mark.parametrize("act,impl", [("float32", 1), ("bfloat16", 1), ("bfloat16", 0)])
@pytest.mark.parametrize("n,nk,heads,d,rd,vd,window,sinks,gated", [
    (1, 1, 2, 24, 8, 16, 0, True, True), (2, 130, 3, 64, 16, 32, 65, True, True), (200, 200, 2, 24, 8, 16, 64, True, True), (131, 400, 2, 128, 64, 128, 129, True, False),
    (70, 333, 1, 136, 72, 200, 100, False, True), (140, 300, 2, 40, 32, 48, 0, True, True), (65, 65, 1, 8, 8, 8, 1, True, True), (130, 260, 2, 64, 64, 256, 256, False, False)])
def test_attention_windows_sink_and_gate(built, act, impl, n, nk, heads, d, rd, vd, window, sinks, gated):
    w = window or nk
    for spike in (None, w - 1, w):                       # the score that stands out: nowhere, the last key inside, the first key outside the window
        q, kn, kr, v, sink, gate, pos0 = attention_case(n + nk, n, nk, heads, d, rd, vd, window, spike)
        arr = [act_array(a, act) for a in (q, kn, kr, v)]
        pool = Pool()
        out = E.DevBuf(n * heads * vd * (4 if act == "float32" else 2))
        sk, gt = sink.astype(np.float32) if sinks else None, gate.astype(np.float32) if gated else None
        scale = (d + rd) ** -0.5
        K.latent_attention(E.ACT_ID[act], impl, *[pool.p(a[0]) for a in arr], pool.p(sk), pool.p(gt), out, n, pos0, nk, heads, d, rd, vd, window, scale)
        E.sync()
        args = (*[a[1] for a in arr], None if sk is None else sk.astype(np.float64), None if gt is None else gt.astype(np.float64), pos0)
        want = attention_oracle(*args, window, scale, d)
        got = read_act(out, act, want.shape)
        near(got, want, act, 2.0)
        if spike is not None and window > 1 and nk > window + 1:                # a window that is one token off would show
            for wrong in (window - 1, window + 1):
                off = attention_oracle(*args, wrong, scale, d)
                if np.abs(off - want).max() > 0.2:
                    break
            else:
                raise AssertionError("the case cannot tell a window that is one token off")


def test_bad_arguments_are_refused(built):
    b = E.DevBuf(1 << 16)
    for call in (lambda: K.linear(0, 0, b, 100, b, 128, 100, 1, 8, b, 8), lambda: K.linear(2, 0, b, 8, b, 128, 8, 1, 8, b, 8), lambda: K.linear(0, 4, b, 8, b, 128, 8, 1, 8, b, 8),
                 lambda: K.norm_rows(0, b, 12, 10, 1e-6, 1), lambda: K.latent_attention(1, 0, b, b, b, b, None, None, b, 1, 0, 1, 1, 8, 8, 8, 0, 1.0),
                 lambda: K.latent_attention(0, 0, b, b, b, b, None, None, b, 2, 0, 1, 1, 8, 8, 8, 0, 1.0), lambda: K.rot_table(b, 4, 3, 10.0)):
        with pytest.raises(CuQwenError) as e:
            call()
        assert e.value.code == 1


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory, built):
    """name -> (directory, config, float weights, tokens, oracle logits), made on first use."""
    made = {}
    makers = {"small": (small, 1.0, 150), "odd": (odd, 1.0, 150), "tiles": (tiles, 1.0, 330), "sharp": (lambda: small(window=64), 3.0, 260), "one": (lambda: small(layers=1, window=33), 3.0, 140)}

    def get(name):
        if name not in made:
            mk, sharp, n = makers[name]
            cfg = mk()
            w, wf = weights(cfg, 11, sharp)
            d = F.write_model_dir(tmp_path_factory.mktemp(name), cfg, w)
            toks = np.random.default_rng(3).integers(0, cfg["vocab"], n)
            made[name] = (d, cfg, wf, toks, L.forward(cfg, wf, toks))
        return made[name]
    return get


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("name", ["small", "odd", "tiles", "sharp"])
def test_prompt_decoding_and_portions_agree_with_the_oracle(models, act, name):
    d, cfg, _, toks, want = models(name)
    eng = E.Engine.open(d, act=act, max_seq_len=len(toks))
    f = 2.0 if name == "sharp" else 1.0
    whole = eng.extend(toks, 0, range(len(toks)))
    check(whole, want, act, f)
    check(run_portions(eng, toks, [1]), want, act, f)                      # token by token from the first one
    for sizes in (PORTIONS, [2], [65, 2, 1, 64]):
        check(run_portions(eng, toks, sizes), want, act, f)
    # only some places asked for, none in most portions
    n = len(toks) - 3
    eng.extend(toks[:50], 0)
    eng.prefill(toks[50:n], 50)
    check(eng.extend(toks[n:], n, [0, 2]), want[[n, n + 2]], act, f)
    eng.close()


@pytest.mark.parametrize("act", ACTS)
def test_first_tokens(models, act):
    d, _, _, toks, want = models("small")
    for n in (1, 2, 3):
        eng = E.Engine.open(d, act=act, max_seq_len=16)
        check(eng.extend(toks[:n], 0, range(n)), want[:n], act)
        eng.close()


@pytest.mark.parametrize("act", ACTS)
def test_what_is_cached_does_not_outlive_its_sequence(models, act):
    """A long sequence, then shorter ones in the same rows; every answer equals that of a fresh engine."""
    d, cfg, wf, toks, want = models("small")
    eng = E.Engine.open(d, act=act, max_seq_len=len(toks))
    run_portions(eng, toks, PORTIONS)
    for seed, n in ((1, 40), (2, 7), (3, 90)):
        t = np.random.default_rng(seed).integers(0, cfg["vocab"], n)
        got = run_portions(eng, t, [n // 2, 1])
        fresh = E.Engine.open(d, act=act, max_seq_len=len(toks))
        assert np.array_equal(got, run_portions(fresh, t, [n // 2, 1]))
        fresh.close()
        check(got, L.forward(cfg, wf, t), act)
    eng.close()


def planted(cfg, change):
    c = copy.deepcopy(cfg)
    for layer in c["layers"]:
        change(layer["mixer"])
    return c


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("name", ["sharp", "one"])
def test_mistakes_planted_in_the_oracle_show(models, act, name):
    """The engine sides with the right oracle where a wrong window, sink, rotation, gate or latent would move the logits: both
    for prompts and for decoded tokens."""
    d, cfg, wf, toks, want = models(name)
    eng = E.Engine.open(d, act=act, max_seq_len=len(toks))
    got = {"prompt": eng.extend(toks, 0, range(len(toks))), "decoded": run_portions(eng, toks, [1])}
    eng.close()
    wrong = {"window + 1": (planted(cfg, lambda m: m["mask"].update(size=m["mask"]["size"] + 1)), wf), "window - 1": (planted(cfg, lambda m: m["mask"].update(size=m["mask"]["size"] - 1)), wf),
             "rotation base": (planted(cfg, lambda m: m["rot"].update(base=m["rot"]["base"] * 1.3)), wf), "scale": (planted(cfg, lambda m: m.update(scale=m["scale"] * 1.1)), wf),
             "no sink": (cfg, {k: v - 30 if k.endswith("sink") else v for k, v in wf.items()}), "no gate": (cfg, {k: v * 0 if k.endswith("mix.g") else v for k, v in wf.items()}),
             "side input": (cfg, {k: v * 0.9 if k.endswith("side.norm") else v for k, v in wf.items()}), "dq norm": (cfg, {k: v * 0 + 1 if k.endswith("dq.norm") else v for k, v in wf.items()}),
             "dkv norm": (cfg, {k: v * 0 + 1 if k.endswith("dkv.norm") else v for k, v in wf.items()}), "norm2": (cfg, {k: v * 0 + 1 if k.endswith("norm2") else v for k, v in wf.items()})}
    if name == "sharp":
        c = copy.deepcopy(cfg)
        c["layers"][1]["mixer"]["kv_from"] = None
        own = {k.replace("l0.", "l1."): v for k, v in wf.items() if "l0.mix.dkv" in k}
        wrong["latents of its own"] = (c, {**wf, **own})
    for what, (c, w) in wrong.items():
        bad = L.forward(c, w, toks)
        at = int(errors(bad, want).argmax())
        for how, g in got.items():
            e_right, e_wrong = errors(g, want)[at], errors(g, bad)[at]
            assert e_wrong > 4 * e_right, f"{what}, {how}: {e_right:.2e} from the right oracle, {e_wrong:.2e} from the wrong one"


@pytest.mark.parametrize("act", ACTS)
def test_long_decoding_and_keys_that_left_every_window(models, act):
    """400 tokens decoded one by one past windows of 9: what lies before the last window no longer matters."""
    d, cfg, wf, _, _ = models("small")
    rng = np.random.default_rng(9)
    a, b = rng.integers(0, cfg["vocab"], (2, 420))
    b[200:] = a[200:]
    eng = E.Engine.open(d, act=act, max_seq_len=420)
    out = []
    for t in (a, b):
        eng.prefill(t[:20], 0)
        out.append(np.concatenate([eng.extend(t[i:i + 1], i, [0]) for i in range(20, 420)]))
    eng.close()
    check(out[0], L.forward(cfg, wf, a)[20:], act)
    assert np.array_equal(out[0][200:], out[1][200:])                     # 2 layers x 8 tokens back: position 216 on sees equal tokens only
    assert not np.array_equal(out[0][180:196], out[1][180:196])


def test_portions_longer_than_a_chunk(models):
    """More tokens than go through the layers together, wanted places on both sides of the border; bfloat16."""
    d, cfg, wf, _, _ = models("small")
    n = 2100
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], n)
    eng = E.Engine.open(d, max_seq_len=n)
    places = [0, 1, 63, 64, 127, 128, 1000, 2040, 2046, 2047, 2048, 2049, 2055, 2056, 2099]
    got = eng.extend(toks, 0, places)
    ref = np.concatenate([L.forward(cfg, wf, toks[max(0, p - 40):p + 1])[-1:] for p in places if p >= 100])     # positions enter relatively; 40 tokens reach past both windows
    check(got[[i for i, p in enumerate(places) if p >= 100]], ref, "bfloat16", 1.5)
    assert errors(got[:4], L.forward(cfg, wf, toks[:65])[places[:4]]).max() < 0.05
    again = eng.extend(toks[:129], 0, places[:6])
    assert errors(again, got[:6].astype(np.float64)).max() < 0.03
    eng.close()


@pytest.mark.parametrize("act", ACTS)
def test_generation_through_step_decode_and_command_line(models, act):
    d, cfg, wf, _, _ = models("small")
    prompt, n = [5, 17, 3, 88, 41, 2, 60], 24
    eng = E.Engine.open(d, act=act, max_seq_len=64)
    gen = eng.generate(prompt, n)
    seq = prompt + [int(t) for t in gen]
    lg = L.forward(cfg, wf, seq)
    tie = 1e-4 if act == "float32" else 0.1
    for i, t in enumerate(gen):                                            # every token is the oracle's best, or within rounding of it
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= tie * lg.std()
    eng.prefill(prompt[:-1], 0)
    assert np.array_equal(eng.step_loop(prompt[-1], len(prompt) - 1, n), gen)
    # the repetition penalty over what has been seen, on float32 logits
    pen = eng.generate(prompt, 8, penalise=True)
    seen = list(prompt)
    for t in pen:
        row = L.forward(cfg, wf, seen)[-1]
        ids = sorted(set(seen))
        row[ids] = np.where(row[ids] < 0, row[ids] * 1.1, row[ids] / 1.1)
        assert row.max() - row[t] <= tie * lg.std()
        seen.append(int(t))
    eng.close()
    r = subprocess.run([sys.executable, "-m", "cuqwen_b200.generate", "--model", str(d), "--dtype", act, "--tokens", ",".join(map(str, prompt)), "-n", str(n)], cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == [int(t) for t in gen]


def test_graph_pdl_and_plain_launches_agree(models):
    d, _, _, toks, _ = models("small")
    out = []
    for flags in (0, E.FLAG_NO_PDL, E.FLAG_NO_GRAPH, E.FLAG_NO_PDL | E.FLAG_NO_GRAPH):
        eng = E.Engine.open(d, max_seq_len=64, flags=flags)
        eng.prefill(toks[:30], 0)
        out.append(eng.decode_n(int(toks[30]), 30, 12))
        us = eng.profile_step(1, 42)
        assert len(us) == eng.step_launches and (us > 0).all()
        eng.close()
    assert all(np.array_equal(o, out[0]) for o in out)


def test_calls_that_are_refused(models, tmp_path):
    d, cfg, wf, toks, _ = models("small")
    eng = E.Engine.open(d, max_seq_len=32)
    for call in (lambda: eng.extend([cfg["vocab"]], 0, [0]), lambda: eng.extend(toks[:33], 0), lambda: eng.extend(toks[:4], 30), lambda: eng.extend(toks[:4], 0, [2, 1]), lambda: eng.extend(toks[:4], 0, [4]),
                 lambda: eng.step(0, 32), lambda: eng.kv_fill_normal(4, 1), lambda: eng.ptr("WQ")):
        with pytest.raises(CuQwenError) as e:
            call()
        assert e.value.code == 1
    with pytest.raises(CuQwenError):
        eng.load("x.bin")
    eng.close()
    w, _ = weights(cfg, 1)
    for change, code in ((lambda w: w.pop("l0.mix.uk"), 4), (lambda w: w.update({"head": w["head"][:-1]}), 4)):
        bad = dict(w)
        change(bad)
        F.write_model_dir(tmp_path, cfg, bad)
        with pytest.raises(CuQwenError) as e:
            E.Engine.open(tmp_path)
        assert e.value.code == code
    F.write_model_dir(tmp_path, cfg, w)
    raw = (tmp_path / "model.safetensors").read_bytes()
    (tmp_path / "model.safetensors").write_bytes(raw[:-10])
    with pytest.raises(CuQwenError) as e:
        E.Engine.open(tmp_path)
    assert e.value.code == 2


@pytest.mark.parametrize("act", ACTS)
def test_trace_run_replays_a_trace(models, tmp_path, act):
    d, cfg, _, toks, want = models("odd")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:30].tolist(), "want": [29, 3]}], "end": []}, {"step": 1, "entries": [{"id": "a", "tokens": toks[30:31].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[:2].tolist(), "want": []}], "end": []}, {"step": 3, "entries": [{"id": "b", "tokens": toks[2:9].tolist(), "want": [6]}], "end": ["b"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(d), "--dtype", act, "--out", str(tmp_path), "--max-tokens", "40"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    V = cfg["vocab"]
    for step, rows in ((0, [29, 3]), (1, [30]), (3, [8])):
        check(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(-1, V), want[rows], act, 2.0)
    assert not (tmp_path / "2.f32").exists()


def test_extend_on_a_weight_file_of_the_table(built, tmp_path):
    """The same call on a model of the table: prefill between the wanted places, a step at each."""
    from cuqwen_b200 import binfmt
    cfg = dict(vocab=512, dim=256, inter=512, layers=2, heads=4, kv=2, hd=64, tied=False)
    binfmt.write_model(tmp_path / "m.bin", cfg, binfmt.INT8, binfmt.random_tensors(cfg, seed=3))
    out = []
    for whole in (True, False):
        eng = E.Engine(E.custom_params(cfg["vocab"], cfg["dim"], cfg["inter"], cfg["layers"], cfg["heads"], cfg["kv"], cfg["hd"], "int8", max_seq_len=64))
        eng.load(str(tmp_path / "m.bin"))
        toks = np.random.default_rng(1).integers(0, 512, 20)
        if whole:
            out.append(eng.extend(toks, 0, [4, 5, 19]))
        else:
            rows = []
            for i, t in enumerate(toks):
                eng.step(int(t), i)
                rows.append(eng.read("LOGITS").astype(np.float32))
            out.append(np.stack(rows)[[4, 5, 19]])
        eng.close()
    assert errors(out[0], out[1].astype(np.float64)).max() < 5e-3
