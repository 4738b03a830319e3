"""Gobesun on the GPU against the plain implementation: every operator alone, whole prompts, portions, decoding
through cache and state, slots, greedy generation through the loop and the command line."""
import json
import os
import subprocess

import numpy as np
import pytest

from litnicelm_b200 import formats
from litnicelm_b200.plugin import (ModelSession, NativeError, bf16_product_host, delta_host, grouped_attention_host,
                                   residual_norm_host)
from oracle import gobesun as og
from oracle import mitilix as om
import gobesun_util as gu

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DRIVER = os.path.join(ROOT, "litnicelm_b200", "litnice_b200_run")
DTYPES = ["float32", "bfloat16"]


def rounded(a):
    return formats.from_bf16_bits(formats.to_bf16_bits(np.asarray(a, np.float32)))


def rms_rel(got, want):
    return float(np.sqrt(((got - want) ** 2).mean() / (want ** 2).mean()))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, folder, tokens, plain logits of every position, errors allowed per position)"""
    base = tmp_path_factory.mktemp("gobesun")
    made = {}

    def get(name):
        if name not in made:
            cfg, w, folder = gu.build(name, base)
            t = gu.tokens(cfg, 330, 11)
            want = og.forward(cfg, w, t)
            made[name] = (cfg, w, folder, t, want, gu.allowed(cfg, w, t, want))
        return made[name]

    return get


# ---- operators ----

@pytest.mark.parametrize("engine,m", [(0, 1), (0, 7), (0, 12), (0, 64), (1, 3), (1, 300)])
@pytest.mark.parametrize("n,k", [(16, 64), (70, 40), (272, 1100), (6, 7)])
def test_gated_product(engine, m, n, k):
    rng = np.random.default_rng(m * 1000 + n + k)
    a, w = rounded(rng.standard_normal((m, k))), rounded(2.0 * rng.standard_normal((n, k)) * k ** -0.5)
    c = a.astype(np.float64) @ w.T.astype(np.float64)
    want = og.gelu_tanh(c[:, 0::2]) * c[:, 1::2]
    got = bf16_product_host(a, w, engine, n_half=n, act="gelu_tanh", gated=True)
    assert np.abs(got - want).max() < 2 ** -7 * np.abs(want).max()
    half = n // 4 * 2                     # pairs in front, floats behind them
    got = bf16_product_host(a, w, engine, n_half=half, act="gelu_tanh", gated=True)
    assert np.abs(got[:, :half // 2] - want[:, :half // 2]).max() < 2 ** -7 * np.abs(want).max()
    assert np.abs(got[:, half // 2:] - c[:, half:]).max() < 2e-5 * max(1.0, k ** 0.5)


@pytest.mark.parametrize("d", [24, 33, 100, 1024, 1028, 2048, 4096, 8192, 9000])
def test_residual_norm(d):
    rng = np.random.default_rng(d)
    x, y = (3.0 * rng.standard_normal((2, 5, d))).astype(np.float32)
    after, before = (0.3 * rng.standard_normal((2, d))).astype(np.float32)
    for base in (1.0, 0.0):
        wx = x + om.rms_normalise(y.astype(np.float64), 1e-2) * (base + after)
        wh = om.rms_normalise(wx, 1e-2) * (base + before)
        gx, gh = residual_norm_host(x, y, after, before, base, 1e-2)
        assert np.abs(gx - wx).max() < 1e-5 * np.abs(wx).max() and np.abs(gh - wh).max() < 1e-5 * np.abs(wh).max()
        gx, gh = residual_norm_host(x, y, after, before, base, 1e-2, dtype="bfloat16")
        assert np.abs(gx - wx).max() < 1e-5 * np.abs(wx).max() and np.abs(gh - wh).max() < 2 ** -8 * np.abs(wh).max()
    gx, gh = residual_norm_host(x, None, None, before, 1.0, 1e-6)
    assert np.array_equal(gx, x)
    assert np.abs(gh - og.centred_rms_norm(x.astype(np.float64), before, 1e-6)).max() < 1e-5 * np.abs(gh).max()
    gx, gh = residual_norm_host(x, y, after, None, 1.0, 1e-6)
    assert gh is None and not np.array_equal(gx, x)


def delta_case(seed, streams, n, heads, groups, dim, vdim, taps):
    rng = np.random.default_rng(seed)
    c = 2 * groups * dim + heads * vdim
    return {"rows": rounded(rng.standard_normal((streams, n, c + heads * vdim))),
            "ba": rng.standard_normal((streams, n, 2 * heads)).astype(np.float32),
            "conv": rounded(rng.standard_normal((c, taps)) * taps ** -0.5),
            "a_log": rng.uniform(-5.0, 1.0, heads).astype(np.float32),
            "dt_bias": (0.5 * rng.standard_normal(heads)).astype(np.float32),
            "norm": (1.0 + 0.2 * rng.standard_normal(vdim)).astype(np.float32)}


def plain_delta(x, eps, heads, groups, dim, vdim, round_conv=False):
    """(outputs, states) of the plain rule on projected rows; round_conv: convolved vectors rounded to bfloat16."""
    x = {k: v.astype(np.float64) for k, v in x.items()}
    outs, states = [], []
    c = 2 * groups * dim + heads * vdim
    for rows, ba in zip(x["rows"], x["ba"]):
        n = len(rows)
        y = og.silu(og.causal_channel_conv(rows[:, :c], x["conv"]))
        if round_conv:
            y = rounded(y).astype(np.float64)
        q = og.unit_vector(y[:, :groups * dim].reshape(n, groups, dim)) * dim ** -0.5
        k = og.unit_vector(y[:, groups * dim:2 * groups * dim].reshape(n, groups, dim))
        v = y[:, 2 * groups * dim:].reshape(n, heads, vdim)
        beta, log_g = og.sigmoid(ba[:, :heads]), og.log_decay(ba[:, heads:], x["a_log"], x["dt_bias"])
        s = np.zeros((heads, dim, vdim))
        o = np.stack([og.delta_rule(q[:, h * groups // heads], k[:, h * groups // heads], v[:, h], beta[:, h], log_g[:, h],
                                    s[h]) for h in range(heads)], axis=1)
        outs.append(og.gated_head_norm(o, rows[:, c:].reshape(n, heads, vdim), x["norm"], eps).reshape(n, -1))
        states.append(s)
    return np.stack(outs), np.stack(states)


DELTA_SHAPES = [  # streams, n, heads, groups, dim, vdim, taps
    (1, 1, 1, 1, 16, 16, 1),
    (2, 9, 6, 3, 48, 80, 3),
    (1, 70, 3, 1, 20, 28, 2),
    (3, 64, 2, 2, 48, 16, 3),
    (1, 200, 2, 1, 64, 128, 4),
    (2, 130, 4, 4, 128, 128, 5),
    (1, 140, 2, 1, 128, 64, 22),
    (1, 90, 1, 1, 160, 144, 4),
    (1, 150, 2, 1, 256, 48, 4),
    (1, 33, 2, 2, 272, 80, 2),
    (8, 70, 12, 6, 32, 256, 3),
    (2, 150, 3, 3, 80, 100, 3),
    (1, 700, 2, 1, 128, 128, 4),
]


@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_rule_in_32_bit(shape):
    streams, n, heads, groups, dim, vdim, taps = shape
    x = delta_case(sum(shape), *shape)
    want, state = plain_delta(x, 1e-4, heads, groups, dim, vdim)
    for portions in ([n], [1] * min(n, 9) + ([n - 9] if n > 9 else []), [2] * (n // 2) + [1] * (n % 2)):
        got, s = delta_host(**x, eps=1e-4, heads=heads, groups=groups, dim=dim, vdim=vdim, portions=portions)
        assert np.abs(got - want).max() < 1e-4 * np.abs(want).max()
        assert np.abs(s - state).max() < 1e-5 * np.abs(state).max()


@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_rule_in_chunks_equals_token_by_token(shape):
    """bfloat16: the chunked form leaves the state of the plain rule on the same convolved vectors, in 32-bit; so do
    single tokens, short portions, and any mixture."""
    streams, n, heads, groups, dim, vdim, taps = shape
    x = delta_case(sum(shape) + 1, *shape)
    want, state = plain_delta(x, 1e-4, heads, groups, dim, vdim, round_conv=True)
    cuts = [[n], [1] * n if n < 80 else [n - 40] + [1] * 40, [5] * (n // 5) + [1] * (n % 5)]
    if n > 60:
        cuts += [[20, 1, 17, n - 38], [2, 50, 3, n - 55], [n - 19, 19]]
    for portions in cuts:
        got, s = delta_host(**x, eps=1e-4, heads=heads, groups=groups, dim=dim, vdim=vdim, portions=portions, dtype="bfloat16")
        assert rms_rel(s, state) < 2e-3, portions      # a convolved value may round the other way here and there
        assert rms_rel(got, want) < 6e-3, portions
    a, s1 = delta_host(**x, eps=1e-4, heads=heads, groups=groups, dim=dim, vdim=vdim, portions=[n], dtype="bfloat16")
    b, s2 = delta_host(**x, eps=1e-4, heads=heads, groups=groups, dim=dim, vdim=vdim, dtype="bfloat16",
                       portions=[16] * (n // 16) + ([n % 16] if n % 16 else []))
    assert np.abs(s1 - s2).max() < 3e-5 * np.abs(s2).max()
    assert np.abs(a - b).max() < 2 ** -6 * np.abs(b).max() and rms_rel(a, b) < 3e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [40, 64, 65, 129, 300])
def test_a_far_write_is_read_back(dtype, n):
    """Slow decay and small steps except at one early token: a query with its key, far behind it, finds its value."""
    heads = groups = 1
    dim, vdim = 32, 48
    x = delta_case(n, 1, n, heads, groups, dim, vdim, 1)
    x["conv"] = np.ones_like(x["conv"])
    x["a_log"][:] = -12.0
    x["ba"][:, :, 0] = -9.0
    at = 7
    x["ba"][0, at, 0] = 9.0
    x["rows"][0, -1, :dim] = x["rows"][0, at, dim:2 * dim]
    want, state = plain_delta(x, 1e-6, heads, groups, dim, vdim)
    got, s = delta_host(**x, eps=1e-6, heads=heads, groups=groups, dim=dim, vdim=vdim, dtype=dtype)
    assert rms_rel(got[0, -1], want[0, -1]) < (1e-4 if dtype == "float32" else 2e-2)
    v = og.silu(x["rows"][0, at, 2 * dim:2 * dim + vdim].astype(np.float64))
    found = want[0, -1] / og.silu(x["rows"][0, -1, 2 * dim + vdim:].astype(np.float64)) / x["norm"]
    assert np.corrcoef(found, v)[0, 1] > 0.99      # the value does stand out
    x["rows"][0, at, 2 * dim:2 * dim + vdim] *= -1.0
    other = delta_host(**x, eps=1e-6, heads=heads, groups=groups, dim=dim, vdim=vdim, dtype=dtype)[0]
    assert rms_rel(other[0, -1], want[0, -1]) > 0.5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decays_from_none_to_total(dtype):
    """Some tokens wipe the state (factors that underflow), others keep all of it; repeated keys."""
    heads, groups, dim, vdim, n = 2, 1, 64, 32, 190
    x = delta_case(5, 1, n, heads, groups, dim, vdim, 2)
    x["a_log"][:] = [3.0, -3.0]
    x["ba"][0, :, heads] = -30.0
    x["ba"][0, [20, 64, 127, 128, 150], heads] = 60.0
    x["ba"][0, 100:120, heads] = -2.0
    x["rows"][0, 70:110, dim:2 * dim] = x["rows"][0, 70, dim:2 * dim]
    want, state = plain_delta(x, 1e-5, heads, groups, dim, vdim, round_conv=dtype == "bfloat16")
    got, s = delta_host(**x, eps=1e-5, heads=heads, groups=groups, dim=dim, vdim=vdim, dtype=dtype)
    assert np.isfinite(got).all()
    assert rms_rel(s, state) < (1e-5 if dtype == "float32" else 2e-3)
    assert rms_rel(got, want) < (1e-4 if dtype == "float32" else 8e-3)


def attention_case(seed, streams, t, heads, groups, dim, vdim, rot):
    rng = np.random.default_rng(seed)
    rows = rounded(rng.standard_normal((streams, t, (heads + groups) * dim + groups * vdim)))
    qw, kw = (rounded(1.0 + 0.3 * rng.standard_normal(n * dim)) for n in (heads, groups))
    turns = og.yarn_frequencies(rot) / np.pi if rot else np.empty(0)
    return rows, qw, kw, turns, og.yarn_amplitude(rot) if rot else 1.0


def plain_attention(rows, n, qw, kw, eps, rot, heads, groups, dim, vdim, scale, size):
    qs, ks, outs = [], [], []
    for x in rows.astype(np.float64):
        t = len(x)
        q = og.plain_rms_norm(x[:, :heads * dim], qw, eps).reshape(t, heads, dim)
        k = og.plain_rms_norm(x[:, heads * dim:(heads + groups) * dim], kw, eps).reshape(t, groups, dim)
        at = np.arange(t, dtype=np.float64)
        if rot:
            q, k = og.rotate(q, at, rot), og.rotate(k, at, rot)
        v = x[:, (heads + groups) * dim:].reshape(t, groups, vdim)
        qs.append(q[t - n:].reshape(n, -1))
        ks.append(k.reshape(t, -1))
        outs.append(og.grouped_attention(q, k, v, scale, size)[t - n:].reshape(n, -1))
    return np.stack(qs), np.stack(ks), np.stack(outs)


ROT = {"dims": 16, "base": 700.0, "scaling": {"factor": 3.0, "original": 128, "fast": 20.0, "slow": 1.0}}
ATT_TOL = {0: 3e-6, 1: 1e-2, 2: 1.2e-2}


@pytest.mark.parametrize("engine", [0, 1, 2])
@pytest.mark.parametrize("streams,t,n,heads,groups,dim,vdim,size,rot", [
    (1, 1, 1, 3, 3, 16, 32, 9, ROT),
    (2, 70, 3, 6, 2, 32, 16, 64, dict(ROT, dims=32)),
    (1, 200, 5, 4, 1, 48, 80, 65, ROT),
    (1, 150, 150, 2, 2, 64, 32, 44, ROT),
    (3, 137, 137, 1, 1, 16, 16, 1000, {"dims": 16, "base": 100.0}),
    (2, 300, 129, 4, 2, 128, 128, 100, ROT),
    (1, 260, 20, 2, 1, 80, 144, 128, ROT),
    (1, 400, 131, 2, 1, 256, 256, 7, ROT),
    (1, 40, 40, 2, 2, 32, 32, 1, None),
    (1, 1300, 3, 3, 1, 32, 48, 1250, ROT),
    (1, 700, 300, 9, 1, 20, 12, 256, dict(ROT, dims=6)),
    (2, 90, 40, 24, 2, 16, 208, 33, ROT),
])
def test_grouped_attention(engine, streams, t, n, heads, groups, dim, vdim, size, rot):
    rows, qw, kw, turns, amp = attention_case(t + n + dim, streams, t, heads, groups, dim, vdim, rot)
    scale = 1.7 * dim ** -0.5
    wq, wk, want = plain_attention(rows, n, qw, kw, 1e-3, rot, heads, groups, dim, vdim, scale, size)
    q, k, got = grouped_attention_host(engine, rows, n, qw, kw, 1e-3, turns, amp, heads, groups, dim, vdim, scale, "chunk", size)
    tol = 5e-6 if engine == 0 else 2 ** -8
    assert np.abs(q - wq).max() < tol * np.abs(wq).max() and np.abs(k - wk).max() < tol * np.abs(wk).max()
    assert rms_rel(got, want) < ATT_TOL[engine]
    assert np.abs(got - want).max() < 10 * ATT_TOL[engine] * np.abs(want).max()


@pytest.mark.parametrize("engine", [0, 1, 2])
@pytest.mark.parametrize("size", [1, 2, 16, 63, 64, 65, 100, 128, 129])
@pytest.mark.parametrize("place", ["own", "chunk's first", "before the chunk", "chunk's first, seen by its last"])
def test_one_key_that_stands_out_at_the_chunk_edge(engine, size, place):
    """One query is a large multiple of one key: its own, the first of its chunk, or the last before the chunk (which
    must then change nothing)."""
    heads, groups, dim, vdim, t = 2, 1, 32, 48, 300
    n = 150 if engine == 2 else 140
    rows, qw, kw, turns, amp = attention_case(size, 1, t, heads, groups, dim, vdim, None)
    first = (t - 20) // size * size                # a chunk that starts inside the rows looked at
    i = first + size - 1 if place.endswith("last") and first + size <= t else max(first, min(t - 20, first + size - 1))
    j = {"own": i, "before the chunk": first - 1}.get(place, first)
    k = og.plain_rms_norm(rows[0, :, heads * dim:(heads + groups) * dim].astype(np.float64), kw, 1e-3)
    rows[0, i, :heads * dim] = rounded(np.tile(k[j], heads) / qw)
    wq, wk, want = plain_attention(rows, n, qw, kw, 1e-3, None, heads, groups, dim, vdim, 0.9, size)
    q, kk, got = grouped_attention_host(engine, rows, n, qw, kw, 1e-3, turns, amp, heads, groups, dim, vdim, 0.9, "chunk", size)
    r = i - (t - n)
    value = np.tile(rows[0, j, (heads + groups) * dim:], heads)
    assert rms_rel(got[0, r], want[0, r]) < 4 * ATT_TOL[engine]
    if place == "before the chunk":
        assert rms_rel(want[0, r], value) > 0.5
    else:
        assert rms_rel(want[0, r], value) < 0.2    # the key does stand out
    assert rms_rel(got, want) < 2 * ATT_TOL[engine]


@pytest.mark.parametrize("engine", [0, 1, 2])
@pytest.mark.parametrize("size", [1, 7, 64, 100])
def test_the_same_kernels_with_a_sliding_window(engine, size):
    heads, groups, dim, vdim, t, n = 4, 2, 32, 32, 260, 90
    rows, qw, kw, turns, amp = attention_case(size, 2, t, heads, groups, dim, vdim, ROT)
    q, k, got = grouped_attention_host(engine, rows, n, qw, kw, 1e-5, turns, amp, heads, groups, dim, vdim, 0.4, "window", size)
    for s in range(2):
        v = rows[s, :, (heads + groups) * dim:].reshape(t, groups, vdim).astype(np.float64)
        for h in (0, 3):
            kh, vh = k[s].reshape(t, groups, dim)[:, h // 2].astype(np.float64), v[:, h // 2]
            for r in (0, 41, n - 1):
                i = t - n + r
                w = om.window_softmax(0.4 * kh[:i + 1] @ q[s, r, h * dim:(h + 1) * dim], i, size)
                assert rms_rel(got[s, r, h * vdim:(h + 1) * vdim], w @ vh[:i + 1]) < 2 * ATT_TOL[engine]


def test_angles_far_into_a_sequence():
    """Angles of many turns (as at positions in the millions) keep their digits."""
    heads, groups, dim, vdim, t = 1, 1, 16, 16, 50
    rows, qw, kw, _, _ = attention_case(1, 1, t, heads, groups, dim, vdim, None)
    turns = np.array([40000.123456789, 3333.7, 0.25, 1e-6])
    q, k, _ = grouped_attention_host(0, rows, t, qw, kw, 1e-6, turns, 1.25, heads, groups, dim, vdim, 0.25, "chunk", 10)
    x = og.plain_rms_norm(rows[0, :, :dim].astype(np.float64), qw, 1e-6)
    a = np.pi * np.fmod(np.arange(t)[:, None] * turns[None, :], 2.0)
    want = x.copy()
    want[:, :4] = 1.25 * (x[:, :4] * np.cos(a) - x[:, 4:8] * np.sin(a))
    want[:, 4:8] = 1.25 * (x[:, 4:8] * np.cos(a) + x[:, :4] * np.sin(a))
    assert np.abs(q[0] - want).max() < 3e-6 * np.abs(want).max()


# ---- whole model ----

@pytest.mark.parametrize("name", list(gu.CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt(models, name, dtype):
    cfg, w, folder, t, want, tol = models(name)
    with ModelSession(folder, dtype, 3) as s:
        got = s.forward(t, all_rows=True)[0]
        assert (gu.logit_error(got, want) < tol[dtype]).all()
        last = s.forward(np.stack([t[:90], t[5:95], t[100:190]]))
        for row, a in zip(last, (0, 5, 100)):
            ref = og.forward(cfg, w, t[a:a + 90])
            assert gu.logit_error(row[None], ref[-1:]) < gu.allowed(cfg, w, t[a:a + 90], ref)[dtype][-1]
        probs = s.inspect(t[:50])
        p = np.exp(want[49] - want[49].max())
        assert np.abs(probs[0] - p / p.sum()).max() < 2 * tol[dtype][49]


@pytest.mark.parametrize("name", list(gu.CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[2], [3, 2, 37, 16], [1], [100, 1, 9, 66], [150, 1, 1, 1, 1, 70], [64], [17, 63]])
def test_portions(models, name, dtype, sizes):
    cfg, w, folder, t, want, tol = models(name)
    t = t[:130] if sizes in ([1], [2]) else t[:240]
    with ModelSession(folder, dtype, 2) as s:
        at, i = 0, 0
        while at < len(t):
            n = min(sizes[i % len(sizes)], len(t) - at)
            got = s.extend(1, t[at:at + n], range(n))
            err = gu.logit_error(got, want[at:at + n])
            assert (err < tol[dtype][at:at + n]).all(), (at, int((err / tol[dtype][at:at + n]).argmax()))
            at += n
            i += 1


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_interleaved_released_and_used_again(models, dtype):
    cfg, w, folder, t, want, tol = models("mixed")
    other = gu.tokens(cfg, 150, 99)
    with ModelSession(folder, dtype, 3) as s:
        alone = [s.extend(0, t[a:a + 30], [29]) for a in range(0, 150, 30)]
        s.release(0)
        s.extend(2, other[:140], [])
        for k, a in enumerate(range(0, 150, 30)):   # the same cuts between steps of other sequences
            s.extend(1, other[a:a + 30], [])
            got = s.extend(0, t[a:a + 30], [29])
            assert np.array_equal(got, alone[k])
            s.extend(2, other[k:k + 1], [])
        s.release(2)                                # a slot that held a longer sequence
        for k, a in enumerate(range(0, 150, 30)):
            assert np.array_equal(s.extend(2, t[a:a + 30], [29]), alone[k])
        s.release(2)                                # and one that starts with a single token
        one = s.extend(2, t[:1], [0])
        assert gu.logit_error(one, want[:1]) < tol[dtype][0]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_matches_the_whole_pass(models, dtype):
    """Token by token past every chunk's edge, the caches growing on the way."""
    for name in ("mixed", "edge"):
        cfg, w, folder, t, want, tol = models(name)
        with ModelSession(folder, dtype) as s:
            s.extend(0, t[:3], [])
            for p in range(3, 330):
                err = gu.logit_error(s.extend(0, t[p:p + 1], [0]), want[p:p + 1])
                assert err < tol[dtype][p], p


def test_prompt_in_more_than_one_portion_of_the_scheduler(models):
    """A prompt longer than the rows of one step."""
    cfg, w, folder, t, want, tol = models("odd")
    long = np.concatenate([gu.tokens(cfg, 40000, 3)])
    with ModelSession(folder, "bfloat16") as s:
        a = s.forward(long)[0]
        s.extend(0, long[:39000], [])
        b = s.extend(0, long[39000:], [999])[0]
        assert gu.logit_error(a[None], b[None]) < 0.05


def follow(cfg, w, prompt, toks):
    """The generated tokens are the plain implementation's first maxima, near ties apart."""
    lg = og.forward(cfg, w, list(prompt) + [int(v) for v in toks[:-1]])[len(prompt) - 1:]
    for i, tok in enumerate(toks):
        assert lg[i].max() - lg[i][tok] < 1e-3, i


@pytest.mark.parametrize("name", ["mixed", "odd", "edge"])
def test_greedy_generation_through_the_loop(models, name):
    cfg, w, folder, t, want, tol = models(name)
    prompts = np.stack([t[:21], t[40:61], t[90:111]])
    with ModelSession(folder, "float32", 3) as s:
        toks = s.generate(prompts, 110)
        assert toks.shape == (3, 110)
        for p, g in zip(prompts, toks):
            follow(cfg, w, p, g)
        assert toks[0][:8].tolist() == og.greedy(cfg, w, prompts[0], 8)
        s.upload_prompts(prompts)                     # the same in two runs
        assert s.run(40) == 40 and s.run(70) == 110
        assert np.array_equal(s.download_tokens(110), toks)
    for p, g in zip(prompts, toks):                   # every stream alone
        with ModelSession(folder, "float32", 1) as s:
            alone = s.generate(p, 110)[0]
            follow(cfg, w, p, alone)
            assert np.array_equal(alone[:20], g[:20])


def test_bfloat16_generation_is_the_forward_pass_of_its_own_tokens(models):
    """Each greedy token is the maximum of the whole-pass logits of what precedes it (near ties apart), the same with
    and without graphs."""
    cfg, w, folder, t, want, tol = models("mixed")
    p = t[:77]
    outs = []
    for graphs in ("1", "0"):
        os.environ["LITNICE_B200_GRAPHS"] = graphs
        try:
            with ModelSession(folder, "bfloat16", 2) as s:
                outs.append(s.generate(np.stack([p, t[100:177]]), 150))
                seq = np.concatenate([p, outs[-1][0]])
                lg = s.forward(seq, all_rows=True)[0][len(p) - 1:-1]
        finally:
            del os.environ["LITNICE_B200_GRAPHS"]
        picked = lg[np.arange(150), outs[-1][0]]
        assert (lg.max(-1) - picked).max() < 0.3
    assert np.array_equal(outs[0], outs[1])


def test_many_streams_and_sampling(models):
    """More streams than the few-row products take, and sampled ones: each equals its own run with the same seed."""
    cfg, w, folder, t, want, tol = models("mixed")
    prompts = np.stack([gu.tokens(cfg, 12, 500 + i) for i in range(70)])
    seeds = np.arange(70, dtype=np.uint32) + 5
    with ModelSession(folder, "float32", 70) as s:
        toks = s.generate(prompts, 9, temp=0.9, top_k=20, top_p=0.95, seeds=seeds)
    with ModelSession(folder, "float32", 1) as s:
        same = sum(np.array_equal(s.generate(prompts[i], 9, temp=0.9, top_k=20, top_p=0.95, seeds=seeds[i:i + 1])[0],
                                  toks[i]) for i in range(0, 70, 7))
    assert same >= 9
    with ModelSession(folder, "bfloat16", 70) as s:
        s.keep_step_logits(True)
        toks = s.generate(prompts, 5)
        lg = s.read_step_logits(5, 70)
    for i in (0, 33, 69):
        ref = og.forward(cfg, w, list(prompts[i]) + list(toks[i][:4]))[11:]
        seq = list(prompts[i]) + list(toks[i][:4])
        assert (gu.logit_error(lg[:, i], ref) < gu.allowed(cfg, w, np.array(seq), og.forward(cfg, w, seq))["bfloat16"][11:]).all()


def test_bad_calls_are_errors(models, tmp_path):
    cfg, w, folder, t, want, tol = models("odd")
    with ModelSession(folder, "bfloat16") as s:
        with pytest.raises(NativeError, match="out of range"):
            s.extend(0, [3, cfg["vocab"]], [])
        assert (gu.logit_error(s.extend(0, t[:9], range(9)), want[:9]) < tol["bfloat16"][:9]).all()
    for name in ("l1.mix.q.norm", "l2.mix.v.conv", "l0.norm1b"):
        broken = dict(w)
        del broken[name]
        formats.write_model_folder(str(tmp_path / "a"), cfg, broken)
        with pytest.raises(NativeError, match=name):
            ModelSession(str(tmp_path / "a"))
    broken = dict(w)
    broken["l0.mix.g"] = w["l0.mix.g"][:-1]
    formats.write_model_folder(str(tmp_path / "b"), cfg, broken)
    with pytest.raises(NativeError, match="l0.mix.g has shape"):
        ModelSession(str(tmp_path / "b"))
    broken = dict(w)
    broken["l0.mix.A_log"] = np.array(w["l0.mix.A_log"])
    broken["l0.mix.A_log"][1] = np.inf
    formats.write_model_folder(str(tmp_path / "c"), cfg, broken)
    with pytest.raises(NativeError, match="not finite"):
        ModelSession(str(tmp_path / "c"))


def test_command_line_generates_and_replays(models, tmp_path):
    cfg, w, folder, t, want, tol = models("mixed")
    ids = ",".join(str(int(v)) for v in t[:30])
    out = str(tmp_path / "out.i32")
    p = subprocess.run([DRIVER, "infer", "--model", folder, "--dtype", "float32", "--ids", ids, "--max_new", "40",
                        "--out-ids-file", out], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    toks = np.fromfile(out, np.int32)
    assert len(toks) == 40
    follow(cfg, w, t[:30], toks)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:31].tolist(), "want": [0, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[31:33].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[33:34].tolist(), "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": t[:100].tolist(), "want": [99, 7]}], "end": ["y"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "100"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "1.f32").exists()
    for step, places in ((0, [0, 30]), (2, [33]), (3, [99, 7])):
        got = np.fromfile(str(tmp_path / f"{step}.f32"), "<f4").reshape(len(places), -1)
        assert gu.logit_error(got, want[places]).max() < tol["float32"][0]
