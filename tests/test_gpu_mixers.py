"""Gipotar on the GPU against the plain numpy oracle: each kernel alone, then whole models - prompts, decoding, portions, sequences one
after another, far keys, long decoding, generation."""
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
from gpu_util import Pool, dev, dint
from mixer_util import F, M, check, errors, run_portions, weights
from test_gpu_stack import act_array, near, read_act

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
ACTS = ["float32", "bfloat16"]
PORTIONS = [2, 3, 17, 1, 1, 40, 2, 64, 1, 33]
f32 = lambda a: np.ascontiguousarray(a, dtype=np.float32)


def f32_pair(rng, *shape, scale=1.0):
    a = f32(scale * rng.standard_normal(shape))
    return a, a.astype(np.float64)


def pieces(n, sizes):
    out, i = [], 0
    while i < n:
        m = min(sizes[min(len(out), len(sizes) - 1)], n - i)
        out.append((i, m))
        i += m
    return out


# ---- kernels alone ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("act,epi", [("float32", "add"), ("bfloat16", "add"), ("float32", "cap"), ("bfloat16", "cap"), ("bfloat16", "glu"), ("float32", "decay"), ("bfloat16", "decay")])
@pytest.mark.parametrize("n,rows,cols", [(1, 48, 104), (1, 1008, 256), (1, 2608, 640), (2, 48, 104), (130, 272, 192), (300, 1104, 520), (257, 64, 1000)])
def test_epilogues_with_constants(built, act, epi, n, rows, cols):
    if (act, epi, n) == ("bfloat16", "decay", 1):
        pytest.skip("one token's decays are time_mix_step's")
    rng = np.random.default_rng(rows + n)
    pitch, ldx = -(-cols // 128) * 128, cols
    x, xv = act_array(rng.standard_normal((n, cols)), act)
    w = np.zeros((rows, pitch), np.uint16)
    w[:, :cols] = F.to_bf16(rng.standard_normal((rows, cols)) * cols ** -0.5 * 3)
    acc = xv @ F.from_bf16(w[:, :cols]).astype(np.float64).T
    pool = Pool()
    code = {"add": K.LIN_ADD, "cap": K.LIN_CAP, "glu": K.LIN_GLU, "decay": K.LIN_DECAY}[epi]
    c0, c1 = {"add": (0.37, 0), "cap": (2.5, 0), "glu": (1.2, 1.3), "decay": (0, 0)}[epi]
    bias = f32(rng.standard_normal(rows) - 1)
    if epi == "glu":
        out = E.DevBuf(n * rows)
        t = acc.reshape(n, rows // 16, 2, 8)
        g, u = np.minimum(t[:, :, 0], c0), np.clip(t[:, :, 1], -c0, c0)
        want = (g * M.sigmoid(c1 * g) * (u + 1)).reshape(n, rows // 2)
        ldo = rows // 2
    else:
        y = f32(rng.standard_normal((n, rows)))
        out, ldo = dev(y), rows
        want = y + c0 * acc if epi == "add" else np.exp(-np.exp(acc + bias)) if epi == "decay" else c0 * np.tanh(acc / c0)
    K.linear_epi(E.ACT_ID[act], code, pool.p(x), ldx, pool.p(w), pitch, cols, n, rows, out, ldo, c0, c1, pool.p(bias))
    E.sync()
    if epi == "glu":
        near(read_act(out, act, want.shape), want, act)
    else:
        near(out.numpy(np.float32).reshape(n, rows).astype(np.float64), want, "float32", 4.0)


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("width,n_mix", [(100, 5), (1024, 1), (3333, 3), (8, 0)])
def test_mixes_with_the_previous_token(built, act, width, n_mix):
    rng = np.random.default_rng(width)
    n, ld, eps = 11, -(-width // 8) * 8, 1e-5
    x, w, mu = np.zeros((n, ld), np.float32), np.zeros(ld, np.float32), np.zeros((max(n_mix, 1), ld), np.float32)
    x[:, :width], w[:width], mu[:, :width] = rng.standard_normal((n, width)), 1 + rng.standard_normal(width), rng.random((max(n_mix, 1), width))
    h = M.rms_norm(x[:, :width].astype(np.float64), w[:width].astype(np.float64), eps)
    ring, tail, es, pool = dev(np.full((2, ld), 7.0, np.float32)), E.DevBuf(ld * 4), 4 if act == "float32" else 2, Pool()
    for i, m in pieces(n, [3, 1, 1, 2, 9]):
        out = E.DevBuf((n_mix + 1) * m * ld * es)
        K.shift_mix(E.ACT_ID[act], pool.p(x[i:i + m].copy()), ld, pool.p(w), width, eps, pool.p(mu), n_mix, ring, tail, out, i, m)
        E.sync()
        got = read_act(out, act, (n_mix + 1, m, ld))
        near(got[0][:, :width], h[i:i + m], act)
        for j in range(n_mix):
            near(got[j + 1][:, :width], M.mix(h, mu[j, :width].astype(np.float64))[i:i + m], act)
        assert not got[:, :, width:].any()
    near(ring.numpy(np.float32).reshape(2, ld)[(n - 1) & 1, :width].astype(np.float64), h[-1], "float32")


def attention_oracle(raw, heads, kv, dim, vd, rot, base, scale, wrong=None):
    """wrong: 'first' hides the first key from every later query, 'own' the query's own."""
    n, a, b = len(raw), heads * dim, (heads + kv) * dim
    pos, own = np.arange(n), np.arange(heads) // (heads // kv)
    q, k, v = raw[:, :a].reshape(n, heads, dim), raw[:, a:b].reshape(n, kv, dim), raw[:, b:].reshape(n, kv, vd)
    if rot:
        q, k = M.rotate_half(q, pos, base, rot), M.rotate_half(k, pos, base, rot)
    s = np.einsum("qhd,khd->hqk", q, k[:, own]) * scale
    if wrong == "first":
        s[:, 1:, 0] = -1e30
    elif wrong == "own":
        s[:, np.arange(1, n), np.arange(1, n)] = -1e30
    return np.einsum("hqk,khd->qhd", M.causal_softmax(s), v[:, own])


@pytest.mark.parametrize("act,impl", [("float32", 1), ("bfloat16", 1), ("bfloat16", 0), ("bfloat16", 2)])
@pytest.mark.parametrize("n,heads,kv,dim,vd,rot", [(3, 1, 1, 8, 8, 0), (70, 6, 2, 24, 40, 16), (150, 4, 4, 96, 160, 50), (200, 34, 2, 64, 32, 64), (131, 2, 1, 136, 256, 6), (330, 20, 1, 128, 128, 128)])
@pytest.mark.parametrize("stands_out", [None, "first", "own"])
def test_grouped_attention(built, act, impl, n, heads, kv, dim, vd, rot, stands_out):
    """stands_out: every second query agrees with the very first key, or with its own."""
    rng = np.random.default_rng(n)
    a, b = heads * dim, (heads + kv) * dim
    raw = f32(rng.standard_normal((n, b + kv * vd)))
    if stands_out == "first":                                              # along entries that hardly rotate or do not
        raw[:, a:b].reshape(n, kv, dim)[0, :, rot - 1 if rot else 0] = 9.0
        raw[::2, :a].reshape(-1, heads, dim)[:, :, rot - 1 if rot else 0] = 9.0
    elif stands_out == "own":
        raw[::2, :a] = 2.0 * np.repeat(raw[::2, a:b].reshape(-1, kv, dim), heads // kv, axis=1).reshape(-1, a)
    base, scale, oscale = 1e7, dim ** -0.5, 0.75
    want = oscale * attention_oracle(raw.astype(np.float64), heads, kv, dim, vd, rot, base, scale)
    es, max_seq, pool = 4 if act == "float32" else 2, n + 5, Pool()
    rotb = E.DevBuf(max(max_seq * rot * 4, 16))
    if rot:
        K.rot_table(rotb, max_seq, rot, base)
    q, cache, out, scratch = E.DevBuf(n * a * es), E.DevBuf(kv * max_seq * (dim + vd) * es), E.DevBuf(n * heads * vd * es), E.DevBuf(148 * heads * (vd + 4) * 4)
    got = []
    for i, m in pieces(n, [2, n // 3 or 1, n // 2] if impl != 2 else [1]):
        K.grouped_attention(E.ACT_ID[act], impl, pool.p(raw[i:i + m]), q, cache, max_seq, rotb if rot else None, rot, out, scratch, m, i, pool.p(dint(i)), heads, kv, dim, vd, scale, oscale)
        E.sync()
        got.append(read_act(out, act, (n, heads, vd))[:m])
    got = np.concatenate(got)
    near(got, want, act, 3.0)
    if stands_out:
        bad = oscale * attention_oracle(raw.astype(np.float64), heads, kv, dim, vd, rot, base, scale, stands_out)
        assert np.abs(bad - want)[2::2].max() > 0.2 and np.abs(got - bad).max() > 0.1


@pytest.mark.parametrize("heads,dim,n", [(1, 8, 5), (3, 24, 70), (2, 40, 40), (5, 64, 150), (2, 96, 33), (3, 128, 64), (1, 192, 20), (2, 256, 50), (1, 504, 35)])
def test_time_mixing(built, heads, dim, n):
    rng = np.random.default_rng(dim)
    W = heads * dim
    (r, r64), (k, k64), (v, v64), (z, z64) = (f32_pair(rng, n, W) for _ in range(4))
    u, u64 = f32_pair(rng, W)
    z = f32(np.exp(-np.exp(z64 - 3)))
    hd = lambda a: a.reshape(-1, heads, dim)
    seg_state, seg_decay = E.DevBuf(16 * W * dim * 4), E.DevBuf(16 * W * 4)
    want = M.bonus_recurrence(hd(r64), hd(k64), hd(v64), hd(z.astype(np.float64)), u64.reshape(heads, dim)).reshape(n, W)
    for sizes, seg in (([n], 0), ([1], 0), ([2, 15, 16, 17, 1, 33], 0), ([n], -(-n // 9)), ([3, n], -(-n // 2)), ([n], 16 if n > 16 else n - 1)):
        pool, state, got = Pool(), dev(np.full(W * dim, 3.0, np.float32)), []          # what an earlier sequence left does not matter
        for i, m in pieces(n, sizes):
            o = E.DevBuf(m * W * 4)
            K.time_mix(*[pool.p(a[i:i + m]) for a in (r, k, v, z)], pool.p(u), state, o, heads, dim, m, i, seg, seg_state, seg_decay)
            E.sync()
            got.append(o.numpy(np.float32).reshape(m, W))
        near(np.concatenate(got).astype(np.float64), want, "float32", 3.0)


@pytest.mark.parametrize("heads,dim,rank,n", [(1, 8, 1, 5), (3, 24, 12, 30), (5, 64, 64, 20), (2, 128, 33, 12), (2, 200, 100, 9), (1, 504, 7, 6)])
def test_time_mixing_of_single_tokens(built, heads, dim, rank, n):
    rng = np.random.default_rng(dim + 1)
    W, pitch = heads * dim, -(-rank // 128) * 128
    raw, raw64 = f32_pair(rng, n, 4 * W + rank)
    w2 = np.zeros((W, pitch), np.uint16)
    w2[:, :rank] = F.to_bf16(rng.standard_normal((W, rank)) * rank ** -0.5)
    (w0, w064), (u, u64), (norm, norm64) = f32_pair(rng, W), f32_pair(rng, W), f32_pair(rng, W)
    w0, w064 = w0 - 2, w064 - 2
    r, k, v, g = (raw64[:, i * W:(i + 1) * W].reshape(n, heads, dim) for i in range(4))
    decay = np.exp(-np.exp(np.tanh(raw64[:, 4 * W:]) @ F.from_bf16(w2[:, :rank]).astype(np.float64).T + w064)).reshape(n, heads, dim)
    o = M.rms_norm(M.bonus_recurrence(r, k, v, decay, u64.reshape(heads, dim)), 1.0, 1e-5).reshape(n, W) * norm64 * M.silu(g.reshape(n, W)) * 0.6
    pool, state, out, got = Pool(), dev(np.full(W * dim, 3.0, np.float32)), E.DevBuf(W * 2), []
    for t in range(n):
        K.time_mix_step(pool.p(raw[t].copy()), pool.p(w2), pitch, rank, pool.p(w0), pool.p(u), pool.p(norm), state, out, heads, dim, 1e-5, 0.6, pool.p(dint(t)))
        E.sync()
        got.append(read_act(out, "bfloat16", (W,)))
    near(np.stack(got), o, "bfloat16")


def delta_case(heads, kv, dim, vd, taps, n):
    rng = np.random.default_rng(dim + vd)
    kc, vc, hp = kv * dim, heads * vd, -(-heads // 8) * 8
    raw, raw64 = f32_pair(rng, n, 2 * kc + 2 * vc + 2 * hp)
    conv, conv64 = f32_pair(rng, 2 * kc + vc, taps, scale=0.6)
    al, dt, norm = rng.standard_normal(heads) * 0.7 - 1, rng.standard_normal(heads) * 0.7 - 1, f32(rng.standard_normal(vd))
    al, dt = f32(al), f32(dt)
    x = M.silu(M.causal_conv(raw64[:, :2 * kc + vc], conv64))
    own = np.arange(heads) // (heads // kv)
    q, k = M.unit(x[:, :kc].reshape(n, kv, dim))[:, own] * dim ** -0.5, M.unit(x[:, kc:2 * kc].reshape(n, kv, dim))[:, own]
    a0 = 2 * kc + 2 * vc
    g = np.exp(-np.exp(al.astype(np.float64)) * M.softplus(raw64[:, a0:a0 + heads] + dt.astype(np.float64)))
    o = M.delta_recurrence(q, k, x[:, 2 * kc:].reshape(n, heads, vd), g, M.sigmoid(raw64[:, a0 + hp:a0 + hp + heads]))
    gated = M.rms_norm(o, norm.astype(np.float64), 1e-5) * M.silu(raw64[:, 2 * kc + vc:a0].reshape(n, heads, vd))
    return raw, f32(conv.T.copy()), f32(np.exp(al)), dt, norm, o, gated, 2 * kc + vc


DELTA = [(1, 1, 8, 8, 1, 6), (4, 2, 24, 16, 4, 70), (2, 2, 64, 64, 4, 100), (6, 3, 40, 96, 3, 50), (3, 1, 128, 128, 4, 64), (2, 1, 200, 256, 9, 40), (1, 1, 504, 24, 2, 35), (9, 3, 32, 200, 4, 20)]


@pytest.mark.parametrize("heads,kv,dim,vd,taps,n", DELTA)
def test_gated_delta_rule(built, heads, kv, dim, vd, taps, n):
    raw, conv, a_exp, dt, norm, want, _, ch = delta_case(heads, kv, dim, vd, taps, n)
    for sizes in ([n], [1], [2, 15, 16, 17, 1, 3]):
        pool, state, ring, got = Pool(), dev(np.full(heads * vd * dim, 3.0, np.float32)), dev(np.full((taps, ch), 5.0, np.float32)), []
        for i, m in pieces(n, sizes):
            o = E.DevBuf(m * heads * vd * 4)
            K.delta(pool.p(raw[i:i + m].copy()), pool.p(conv), taps, ring, pool.p(a_exp), pool.p(dt), E.DevBuf(m * kv * 2 * dim * 4), E.DevBuf(m * heads * vd * 4), E.DevBuf((m + 3) // 4 * heads * 128), state, o, heads, kv, dim, vd, m, i)
            E.sync()
            got.append(o.numpy(np.float32).reshape(m, heads, vd))
        near(np.concatenate(got).astype(np.float64), want, "float32", 4.0)


@pytest.mark.parametrize("heads,kv,dim,vd,taps,n", DELTA)
def test_gated_delta_rule_of_single_tokens(built, heads, kv, dim, vd, taps, n):
    raw, conv, a_exp, dt, norm, _, want, ch = delta_case(heads, kv, dim, vd, taps, n)
    pool, state, ring, out, got = Pool(), dev(np.full(heads * vd * dim, 3.0, np.float32)), dev(np.full((taps, ch), 5.0, np.float32)), E.DevBuf(heads * vd * 2), []
    for t in range(n):
        K.delta_step(pool.p(raw[t].copy()), pool.p(conv), taps, ring, pool.p(a_exp), pool.p(dt), pool.p(norm), state, out, heads, kv, dim, vd, 1e-5, pool.p(dint(t)))
        E.sync()
        got.append(read_act(out, "bfloat16", (heads, vd)))
    near(np.stack(got), want, "bfloat16", 1.5)


def test_bad_arguments_are_refused(built):
    b = E.DevBuf(1 << 16)
    for call in (lambda: K.linear_epi(0, K.LIN_F32, b, 8, b, 128, 8, 1, 16, b, 16, 1, 0, None), lambda: K.linear_epi(1, K.LIN_GLU, b, 8, b, 128, 8, 1, 16, b, 8, 1, 0, None), lambda: K.linear_epi(0, K.LIN_GLU, b, 8, b, 128, 8, 1, 24, b, 16, 1, 0, None),
                 lambda: K.linear_epi(0, K.LIN_CAP, b, 8, b, 128, 8, 1, 16, b, 16, 0, 0, None), lambda: K.shift_mix(0, b, 12, b, 10, 1e-6, b, 1, b, b, b, 0, 1),
                 lambda: K.grouped_attention(1, 0, b, b, b, 8, None, 0, b, None, 1, 0, None, 2, 1, 8, 8, 1.0, 1.0), lambda: K.grouped_attention(0, 2, b, b, b, 8, None, 0, b, b, 2, 0, b, 2, 1, 8, 8, 1.0, 1.0),
                 lambda: K.grouped_attention(0, 0, b, b, b, 8, None, 0, b, None, 1, 0, None, 3, 2, 8, 8, 1.0, 1.0), lambda: K.grouped_attention(0, 0, b, b, b, 8, None, 0, b, None, 4, 5, None, 2, 1, 8, 8, 1.0, 1.0),
                 lambda: K.time_mix(b, b, b, b, b, b, b, 1, 520, 1, 0, 0, None, None), lambda: K.time_mix(b, b, b, b, b, b, b, 1, 8, 4, 0, 2, None, None), lambda: K.time_mix_step(b, b, 128, 1, b, b, b, b, b, 1, 12, 1e-6, 1.0, b),
                 lambda: K.delta(b, b, 0, b, b, b, b, b, b, b, b, 2, 1, 8, 8, 1, 0), lambda: K.delta_step(b, b, 4, b, b, b, b, b, b, 3, 2, 8, 8, 1e-6, b)):
        with pytest.raises(CuQwenError) as e:
            call()
        assert e.value.code == 1


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory, built):
    """name -> (directory, config, float weights, tokens, oracle logits), made on first use."""
    made = {}
    lengths = {"small": 150, "odd": 150, "ones": 60, "wide": 300, "sharp": 260}

    def get(name):
        if name not in made:
            cfg, w, wf = weights("small" if name == "sharp" else name, 11, 4.0 if name == "sharp" else 1.0)
            d = F.write_model_dir(tmp_path_factory.mktemp(name), cfg, w)
            toks = np.random.default_rng(3).integers(0, cfg["vocab"], lengths[name])
            made[name] = (d, cfg, wf, toks, M.forward(cfg, wf, toks))
        return made[name]
    return get


FACTOR = {"small": 1.0, "odd": 2.0, "ones": 4.0, "wide": 1.5, "sharp": 2.0}      # ones: a head of one value has nothing but its sign left after its norm


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("name", ["small", "odd", "ones", "wide", "sharp"])
def test_prompt_decoding_and_portions_agree_with_the_oracle(models, act, name):
    d, cfg, _, toks, want = models(name)
    eng = E.Engine.open(d, act=act, max_seq_len=len(toks))
    f = FACTOR[name]
    check(eng.extend(toks, 0, range(len(toks))), want, act, f)
    check(run_portions(eng, toks, [1]), want, act, f)                      # token by token from the first one
    for sizes in (PORTIONS, [2], [65, 2, 1, 64]):
        check(run_portions(eng, toks, sizes), want, act, f)
    # only some places asked for, none in most portions
    n = len(toks) - 3
    eng.extend(toks[:30], 0)
    eng.prefill(toks[30:n], 30)
    check(eng.extend(toks[n:], n, [0, 2]), want[[n, n + 2]], act, f)
    eng.close()


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("name", ["small", "odd"])
def test_first_tokens(models, act, name):
    d, _, _, toks, want = models(name)
    eng = E.Engine.open(d, act=act, max_seq_len=16)
    for n in (1, 2, 3, 5):
        check(eng.extend(toks[:n], 0, range(n)), want[:n], act, 2 * FACTOR[name])
    eng.close()


@pytest.mark.parametrize("act", ACTS)
def test_states_and_rows_do_not_outlive_their_sequence(models, act):
    """A long sequence, then shorter ones in the same rows and states; every answer equals that of a fresh engine."""
    d, cfg, wf, toks, want = models("odd")
    eng = E.Engine.open(d, act=act, max_seq_len=len(toks))
    run_portions(eng, toks, PORTIONS)
    for seed, n in ((1, 40), (2, 7), (3, 90), (4, 1)):
        t = np.random.default_rng(seed).integers(0, cfg["vocab"], n)
        sizes = [max(n // 2, 1), 1]
        got = run_portions(eng, t, sizes)
        fresh = E.Engine.open(d, act=act, max_seq_len=len(toks))
        assert np.array_equal(got, run_portions(fresh, t, sizes))
        fresh.close()
        check(got, M.forward(cfg, wf, t), act, 2 * FACTOR["odd"])
    eng.close()


@pytest.mark.parametrize("act", ACTS)
def test_mistakes_planted_in_the_oracle_show(models, act):
    """The engine sides with the right oracle where a constant, a weight or a state that is left out would move the logits: in prompts,
    in decoded tokens and in portions."""
    d, cfg, wf, toks, want = models("sharp")
    eng = E.Engine.open(d, act=act, max_seq_len=len(toks))
    got = {"prompt": eng.extend(toks, 0, range(len(toks))), "decoded": run_portions(eng, toks, [1]), "portions": run_portions(eng, toks, PORTIONS)}
    eng.close()

    def cfg_with(change):
        c = copy.deepcopy(cfg)
        change(c, c["layers"][0]["mixer"], c["layers"][1])
        return c, wf

    def w_with(change):
        return cfg, {k: change(k, v) for k, v in wf.items()}
    wrong = {
        "rotation base": cfg_with(lambda c, m, l: m["left"]["rot"].update(base=6500.0)), "rotated dims": cfg_with(lambda c, m, l: m["left"]["rot"].update(dims=24)),
        "score scale": cfg_with(lambda c, m, l: m["left"].update(scale=m["left"]["scale"] * 1.1)), "left scale": cfg_with(lambda c, m, l: m.update(left_scale=0.8)),
        "right scale": cfg_with(lambda c, m, l: m.update(right_scale=1.1)), "limit": cfg_with(lambda c, m, l: l["mlp"].update(limit=1.1)), "eps": cfg_with(lambda c, m, l: c["norm"].update(eps=0.05)),
        "residual": cfg_with(lambda c, m, l: c.update(residual_mult=0.63)), "embedding": cfg_with(lambda c, m, l: c["embedding"].update(scale=2.7)), "cap": cfg_with(lambda c, m, l: c.update(logit_softcap=11.0)),
        "no bonus": w_with(lambda k, v: v * 0 if k.endswith(".u") else v), "decay": w_with(lambda k, v: v + 0.3 if k.endswith(".w0") else v), "no low-rank decay": w_with(lambda k, v: v * 0 if k.endswith(".w2") else v),
        "no mix": w_with(lambda k, v: v * 0 if ".mu." in k else v), "delta decay": w_with(lambda k, v: v + 0.4 if k.endswith("A_log") else v), "time step": w_with(lambda k, v: v + 0.4 if k.endswith("dt_bias") else v),
        "one tap less": w_with(lambda k, v: np.concatenate([v[:, :1] * 0, v[:, 1:]], axis=1) if k.endswith(".conv") else v), "delta norm": w_with(lambda k, v: v * 0 + 1 if k == "l1.mix.norm" else v),
        "step size": w_with(lambda k, v: v * 0 if k.endswith("mix.b") else v), "norms about one": w_with(lambda k, v: v * 0 if k.endswith("norm1") else v)}
    for what, (c, w) in wrong.items():
        bad = M.forward(c, w, toks)
        at = int(errors(bad, want).argmax())
        for how, g in got.items():
            e_right, e_wrong = errors(g, want)[at], errors(g, bad)[at]
            assert e_wrong > 3 * e_right, f"{what}, {how}: {e_right:.2e} from the right oracle, {e_wrong:.2e} from the wrong one"


def far_model(tmp_path_factory):
    """One parallel layer whose attention looks for a token's own kind: a key of the same token id stands out however far back it is."""
    cfg = F.gipotar_config(64, 64, [F.parallel_layer(2, 1, 64, 48, 0, 1, 8, None, scale=1.0)], embed_scale=1.0, softcap=50.0)
    w = F.random_weights(cfg, 8, rank=3)
    eye = np.eye(64, dtype=np.float32)
    w["embed"], w["l0.mix.left.k"], w["l0.mix.left.q"], w["l0.norm1"] = F.to_bf16(8 * eye), F.to_bf16(eye), F.to_bf16(0.25 * np.concatenate([eye, eye])), F.to_bf16(np.zeros(64))
    return F.write_model_dir(tmp_path_factory.mktemp("far"), cfg, w), cfg, {k: F.from_bf16(v) for k, v in w.items()}


@pytest.mark.parametrize("act", ACTS)
def test_keys_far_away_and_at_tile_borders(tmp_path_factory, built, act):
    d, cfg, wf = far_model(tmp_path_factory)
    n = 700
    eng = E.Engine.open(d, act=act, max_seq_len=n)
    for place in (0, 1, 63, 64, 127, 128, 255, 256, 511, 600):
        toks = np.random.default_rng(place).integers(1, 64, n)
        toks[place] = 0
        asked = [p for p in (place + 1, place + 2, 640, 650, n - 1) if p > place]
        toks[asked] = 0                                                    # the same id again: attends to `place` and to itself
        want, without = M.forward(cfg, wf, toks)[asked], toks.copy()
        without[place] = 5
        bad = M.forward(cfg, wf, without)[asked]
        assert errors(bad, want)[0] > 0.15
        whole = eng.extend(toks, 0, asked)
        check(whole, want, act, 1.5)
        eng.prefill(toks[:asked[-2]], 0)                                   # the last two decoded
        for p in range(asked[-2], n):
            lg = eng.extend(toks[p:p + 1], p, [0])
            if p in asked:
                check(lg, want[asked.index(p)][None], act, 1.5)
    eng.close()


@pytest.mark.parametrize("act", ACTS)
def test_long_decoding(models, act):
    d, cfg, wf, _, _ = models("small")
    toks = np.random.default_rng(9).integers(0, cfg["vocab"], 620)
    eng = E.Engine.open(d, act=act, max_seq_len=620)
    eng.prefill(toks[:20], 0)
    got = np.concatenate([eng.extend(toks[i:i + 1], i, [0]) for i in range(20, 620)])
    eng.close()
    want = M.forward(cfg, wf, toks)[20:]
    e = check(got, want, act)
    assert e[-100:].mean() < 3 * e[:100].mean() + 1e-6                     # rounding does not pile up in the states


@pytest.mark.parametrize("act", ACTS)
def test_portions_longer_than_a_chunk(models, act):
    """More tokens than go through the layers together; the first tokens after the border are one and several."""
    d, cfg, wf, _, _ = models("small")
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], 2100)
    want = M.forward(cfg, wf, toks)
    eng = E.Engine.open(d, act=act, max_seq_len=2100)
    for n in (2100, 2049):
        places = [p for p in (0, 1, 63, 64, 1000, 2046, 2047, 2048, 2049, 2055, 2099) if p < n]
        check(eng.extend(toks[:n], 0, places), want[places], act, 1.5)
        if n < 2100:
            check(eng.extend(toks[n:n + 1], n, [0]), want[n][None], act, 1.5)
        eng.prefill(toks[:2049], 0)
        check(eng.extend(toks[2049:2052], 2049, [0, 1, 2]), want[2049:2052], act, 1.5)
    eng.close()


def test_a_recurrence_goes_on_where_it_stands_or_starts_over(models):
    d, _, _, toks, want = models("small")
    eng = E.Engine.open(d, max_seq_len=64)
    eng.prefill(toks[:10], 0)
    for call in (lambda: eng.extend(toks[:2], 9, [0]), lambda: eng.extend(toks[:1], 11, [0]), lambda: eng.step(1, 4), lambda: eng.decode_n(1, 11, 2), lambda: eng.prefill(toks[:3], 5), lambda: eng.profile_step(1, 2)):
        with pytest.raises(CuQwenError) as e:
            call()
        assert e.value.code == 8 and "10" in str(e.value)
    check(eng.extend(toks[10:12], 10, [0, 1]), want[10:12], "bfloat16", 2.0)           # a refused call has changed nothing
    check(eng.extend(toks[:1], 0, [0]), want[:1], "bfloat16", 2.0)
    check(eng.extend(toks[1:2], 1, [0]), want[1:2], "bfloat16", 2.0)
    eng.close()


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("name", ["small", "odd"])
def test_generation_through_step_decode_and_command_line(models, act, name):
    d, cfg, wf, _, _ = models(name)
    prompt, n = [5, 17, 3, 88, 41, 2, 60], 24
    eng = E.Engine.open(d, act=act, max_seq_len=64)
    gen = eng.generate(prompt, n)
    seq = prompt + [int(t) for t in gen]
    lg = M.forward(cfg, wf, seq)
    tie = 1e-4 if act == "float32" else 0.1
    for i, t in enumerate(gen):                                            # every token is the oracle's best, or within rounding of it
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= tie * lg.std()
    eng.prefill(prompt[:-1], 0)
    assert np.array_equal(eng.step_loop(prompt[-1], len(prompt) - 1, n), gen)
    assert np.array_equal(eng.generate(prompt[:1], 5)[:1], eng.generate(prompt[:1], 1))
    pen = eng.generate(prompt, 8, penalise=True)
    seen = list(prompt)
    for t in pen:
        row = M.forward(cfg, wf, seen)[-1]
        ids = sorted(set(seen))
        row[ids] = np.where(row[ids] < 0, row[ids] * 1.1, row[ids] / 1.1)
        assert row.max() - row[t] <= tie * lg.std()
        seen.append(int(t))
    eng.close()
    r = subprocess.run([sys.executable, "-m", "cuqwen_b200.generate", "--model", str(d), "--dtype", act, "--tokens", ",".join(map(str, prompt)), "-n", str(n)], cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == [int(t) for t in gen]


def test_graph_pdl_and_plain_launches_agree(models):
    d, _, _, toks, _ = models("odd")
    out = []
    for flags in (0, E.FLAG_NO_PDL, E.FLAG_NO_GRAPH, E.FLAG_NO_PDL | E.FLAG_NO_GRAPH):
        eng = E.Engine.open(d, max_seq_len=64, flags=flags)
        eng.prefill(toks[:30], 0)
        out.append(eng.decode_n(int(toks[30]), 30, 12))
        us = eng.profile_step(1, 42)
        assert len(us) == eng.step_launches and (us > 0).all()
        eng.close()
    assert all(np.array_equal(o, out[0]) for o in out)


def test_weights_that_do_not_fit_are_refused(models, tmp_path):
    _, cfg, _, _, _ = models("small")
    _, w, _ = weights("small", 1)
    for change in (lambda w: w.pop("l0.mix.right.w1"), lambda w: w.pop("l1.mix.A_log"), lambda w: w.update({"l0.mix.right.w2": w["l0.mix.right.w2"][:, :-1]}), lambda w: w.update({"l1.mix.k.conv": w["l1.mix.k.conv"][:, :-1]}),
                   lambda w: w.update({"l0.mix.right.u": w["l0.mix.right.u"].reshape(-1)}), lambda w: w.update({"l0.mlp.gate": w["l0.mlp.gate"][:-1]})):
        bad = dict(w)
        change(bad)
        F.write_model_dir(tmp_path, cfg, bad)
        with pytest.raises(CuQwenError) as e:
            E.Engine.open(tmp_path)
        assert e.value.code == 4


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
        check(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(-1, V), want[rows], act, 2 * FACTOR["odd"])
