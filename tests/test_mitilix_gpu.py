"""Mitilix on the GPU against the plain implementation: every operator alone, whole prompts, portions, decoding
through the cache, slots, greedy generation through the loop and the command line."""
import json
import os
import subprocess

import numpy as np
import pytest

from litnicelm_b200 import formats
from litnicelm_b200.plugin import (ModelSession, NativeError, bf16_product_host, latent_attention_host, rms_canon_host)
from oracle import mitilix as om
import mitilix_util as mu

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DRIVER = os.path.join(ROOT, "litnicelm_b200", "litnice_b200_run")


def rounded(a):
    return formats.from_bf16_bits(formats.to_bf16_bits(np.asarray(a, np.float32)))


def rms_rel(got, want):
    return float(np.sqrt(((got - want) ** 2).mean() / (want ** 2).mean()))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, folder, tokens, plain logits of every position, greedy memo)"""
    base = tmp_path_factory.mktemp("mitilix")
    made = {}

    def get(name):
        if name not in made:
            cfg, w, folder = mu.build(name, base)
            t = mu.tokens(cfg, min(cfg["max_positions"] - 20, 330), 11)
            made[name] = (cfg, w, folder, t, om.forward(cfg, w, t))
        return made[name]

    return get


# ---- operators ----

@pytest.mark.parametrize("engine,m", [(0, 1), (0, 5), (0, 8), (0, 9), (0, 17), (0, 64), (1, 1), (1, 130), (1, 300)])
@pytest.mark.parametrize("n,k", [(16, 64), (70, 40), (200, 333), (272, 1000), (13, 7)])
def test_product(engine, m, n, k):
    rng = np.random.default_rng(m * 1000 + n + k)
    a, w = rounded(rng.standard_normal((m, k))), rounded(rng.standard_normal((n, k)) * k ** -0.5)
    want = a.astype(np.float64) @ w.T.astype(np.float64)
    got = bf16_product_host(a, w, engine)
    assert np.abs(got - want).max() < 2e-5 * max(1.0, k ** 0.5)
    c = rng.standard_normal((m, n)).astype(np.float32)
    assert np.abs(bf16_product_host(a, w, engine, c=c) - (want + c)).max() < 2e-5 * max(1.0, k ** 0.5)
    got = bf16_product_host(a, w, engine, n_half=n, act="gelu")
    assert np.abs(got - om.gelu_exact(want)).max() < 2 ** -8 * np.abs(want).max()
    half = n // 2 & ~7
    got = bf16_product_host(a, w, engine, n_half=half, c=c)
    if half:
        assert np.abs(got[:, :half] - want[:, :half]).max() < 2 ** -8 * np.abs(want).max()
    assert np.abs(got[:, half:] - (want + c)[:, half:]).max() < 2e-5 * max(1.0, k ** 0.5)


def test_product_over_many_tiles_and_a_long_k():
    rng = np.random.default_rng(5)
    for m, n, k in ((900, 4100, 192), (2300, 2056, 72), (200, 130, 5000)):
        a, w = rounded(rng.standard_normal((m, k))), rounded(rng.standard_normal((n, k)) * k ** -0.5)
        assert rms_rel(bf16_product_host(a, w, 1), a.astype(np.float64) @ w.T.astype(np.float64)) < 1e-4


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9, 13])
@pytest.mark.parametrize("n,d,portions", [(1, 24, None), (37, 100, None), (37, 100, [1, 2, 3, 2, 11, 8, 9, 1]),
                                          (40, 260, [2] * 20), (40, 33, [16, 24])])
def test_norm_and_input_convolution(taps, n, d, portions):
    rng = np.random.default_rng(taps * 100 + n + d)
    x = (3.0 * rng.standard_normal((n, d))).astype(np.float32)
    w1, w2 = (rng.standard_normal((d, taps)).astype(np.float32) for _ in range(2))
    h = om.scalar_rms_norm(x.astype(np.float64), 0.7, 1e-2)
    want = [om.with_input_conv(h, w.astype(np.float64)) for w in (w1, w2)]
    got = rms_canon_host(x, 0.7, 1e-2, w1, w2, portions)
    for g, t in zip(got, want):
        assert np.abs(g - t).max() < 1e-5 * np.abs(t).max()
    half = rms_canon_host(x, 0.7, 1e-2, w1, None, portions, dtype="bfloat16")[0]
    assert np.abs(half - want[0]).max() < 2 ** -8 * np.abs(want[0]).max()


def attention_case(seed, streams, t, n, heads, dim, vdim, rank):
    rng = np.random.default_rng(seed)
    dkv = rounded(rng.standard_normal((streams, t, rank)) * 2.0)
    gain = rounded(1.0 + 0.2 * rng.standard_normal(rank))
    uk = rounded(rng.standard_normal((heads * dim, rank)) * rank ** -0.5)
    uv = rounded(rng.standard_normal((heads * vdim, rank)) * rank ** -0.5)
    q = rounded(rng.standard_normal((streams, n, heads * dim)))
    return dkv, gain, uk, uv, q


def plain_attention(q, dkv, gain, eps, uk, uv, heads, dim, vdim, scale, window):
    """The last n positions, through the plain implementation with identity W_q and W_o."""
    out = []
    t, n = dkv.shape[1], q.shape[1]
    for s in range(q.shape[0]):
        c = om.vector_rms_norm(dkv[s].astype(np.float64), gain.astype(np.float64), eps)
        a = np.zeros((t, heads * dim))
        a[t - n:] = q[s]
        out.append(om.latent_attention(a, c, np.eye(heads * dim), uk.astype(np.float64), uv.astype(np.float64),
                                       np.eye(heads * vdim), heads, dim, vdim, scale, window)[t - n:])
    return np.stack(out)


ATT_TOL = {0: 3e-6, 1: 8e-3, 2: 8e-3, 3: 1.2e-2}


@pytest.mark.parametrize("engine", [0, 1, 2, 3])
@pytest.mark.parametrize("streams,t,n,heads,dim,vdim,rank,window", [
    (1, 1, 1, 3, 16, 32, 24, 9),
    (2, 70, 3, 17, 32, 16, 40, 64),       # the window is one chunk of keys
    (1, 200, 5, 2, 48, 80, 64, 65),       # one key more than a chunk
    (1, 150, 150, 2, 64, 32, 56, 44),
    (3, 137, 137, 1, 16, 16, 16, 1000),   # window beyond the context
    (2, 300, 129, 2, 128, 128, 136, 100), # a portion in the middle, ragged tiles
    (1, 260, 20, 1, 80, 144, 32, 128),    # two slabs of the head, wide values
    (1, 400, 131, 1, 256, 256, 64, 7),
    (1, 40, 40, 2, 32, 32, 512, 1),       # sees itself only
    (1, 2300, 3, 3, 32, 48, 72, 2200),    # more splits of the window than a cluster has CTAs
    (2, 700, 30, 18, 16, 16, 264, 650),   # several tiles per split, two groups of heads
])
def test_latent_attention(engine, streams, t, n, heads, dim, vdim, rank, window):
    if engine == 2 and streams * n > 64:
        n = 64 // streams
    dkv, gain, uk, uv, q = attention_case(t + n + dim, streams, t, n, heads, dim, vdim, rank)
    scale = 1.7 * dim ** -0.5
    want = plain_attention(q, dkv, gain, 1e-3, uk, uv, heads, dim, vdim, scale, window)
    got = latent_attention_host(engine, q, dkv, gain, 1e-3, uk, uv, heads, dim, vdim, scale, window)
    assert rms_rel(got, want) < ATT_TOL[engine]
    assert np.abs(got - want).max() < 10 * ATT_TOL[engine] * np.abs(want).max()


@pytest.mark.parametrize("engine", [0, 1, 2, 3])
@pytest.mark.parametrize("window", [1, 2, 7, 63, 64, 65, 127, 128, 129, 200])
@pytest.mark.parametrize("back", ["newest", "inside", "outside"])
def test_one_key_that_stands_out_at_the_window_edge(engine, window, back):
    """The query of the last position is a large multiple of one key: of its own position, of the oldest position
    the window shows, or of the first one it hides (which must then change nothing)."""
    heads, dim, vdim, rank, t = 2, 32, 48, 40, 230
    n = 40 if engine == 3 else 2
    dkv, gain, uk, uv, q = attention_case(window, 1, t, n, heads, dim, vdim, rank)
    i = t - 1
    j = {"newest": i, "inside": i - window + 1, "outside": i - window}[back]
    dkv[0, :, 0] *= 0.05                # one latent coordinate that only this position uses
    dkv[0, j] = 0.0
    dkv[0, j, 0] = 2.0
    c = om.vector_rms_norm(dkv[0].astype(np.float64), gain.astype(np.float64), 1e-3)
    keys = c @ uk.T.astype(np.float64)
    q[0, -1] = rounded(3.0 * keys[j])
    want = plain_attention(q, dkv, gain, 1e-3, uk, uv, heads, dim, vdim, 0.5, window)
    got = latent_attention_host(engine, q, dkv, gain, 1e-3, uk, uv, heads, dim, vdim, 0.5, window)
    value = (c @ uv.T.astype(np.float64))[j]
    assert rms_rel(got[0, -1], want[0, -1]) < 4 * ATT_TOL[engine]
    if back != "outside":
        assert rms_rel(want[0, -1], value) < 0.2      # the key does stand out
    else:
        assert rms_rel(want[0, -1], value) > 0.5


def test_tensor_core_attention_with_growing_and_shrinking_scores():
    """Row maxima that keep rising (accumulators rescaled) and that fall (nothing to do) over many key tiles."""
    heads, dim, vdim, rank, t = 1, 64, 64, 64, 1100
    dkv, gain, uk, uv, q = attention_case(3, 1, t, t, heads, dim, vdim, rank)
    c = om.vector_rms_norm(dkv[0].astype(np.float64), gain.astype(np.float64), 1e-3)
    keys = c @ uk.T.astype(np.float64)
    for spikes in (range(60, 1100, 130), range(1000, 0, -130)):
        for g, j in enumerate(spikes):
            q[0, :, :] += rounded(0.12 * (g + 1) * keys[j])
    q = rounded(q)
    want = plain_attention(q, dkv, gain, 1e-3, uk, uv, heads, dim, vdim, 0.5, 900)
    got = latent_attention_host(3, q, dkv, gain, 1e-3, uk, uv, heads, dim, vdim, 0.5, 900)
    assert rms_rel(got, want) < 2e-2


# ---- whole model ----

@pytest.mark.parametrize("name", list(mu.CONFIGS))
@pytest.mark.parametrize("dtype,tol", [("float32", mu.F32_TOL), ("bfloat16", mu.BF16_TOL)])
def test_whole_prompt(models, name, dtype, tol):
    cfg, w, folder, t, want = models(name)
    with ModelSession(folder, dtype, 3) as s:
        got = s.forward(t, all_rows=True)[0]
        assert mu.logit_error(got, want).max() < tol
        last = s.forward(np.stack([t[:90], t[5:95], t[100:190]]))
        assert np.abs(last[0] - got[89]).max() < 30 * tol * np.abs(got).max() / 3
        probs = s.inspect(t[:50])
        p = np.exp(want[49] - want[49].max())
        assert np.abs(probs[0] - p / p.sum()).max() < 2 * tol


@pytest.mark.parametrize("name", list(mu.CONFIGS))
@pytest.mark.parametrize("dtype,tol", [("float32", mu.F32_TOL), ("bfloat16", mu.BF16_TOL)])
@pytest.mark.parametrize("sizes", [[2], [3, 2, 37, 16], [1], [100, 1, 9, 66], [150, 1, 1, 1, 1, 70]])
def test_portions(models, name, dtype, tol, sizes):
    cfg, w, folder, t, want = models(name)
    t = t[:120] if sizes in ([1], [2]) else t[:240]
    with ModelSession(folder, dtype, 2) as s:
        at, i = 0, 0
        while at < len(t):
            n = min(sizes[i % len(sizes)], len(t) - at)
            got = s.extend(1, t[at:at + n], range(n))
            err = mu.logit_error(got, want[at:at + n])
            assert err.max() < tol, (at, int(err.argmax()))
            at += n
            i += 1


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_interleaved_released_and_used_again(models, dtype):
    cfg, w, folder, t, want = models("mixed")
    other = mu.tokens(cfg, 150, 99)
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
        assert s.extend(1, other[:2], [1, 0]).shape == (2, cfg["vocab"])


def test_wanted_places_come_in_the_asked_order(models):
    cfg, w, folder, t, want = models("odd")
    with ModelSession(folder, "float32") as s:
        got = s.extend(0, t[:40], [30, 2, 39])
        assert mu.logit_error(got, want[[30, 2, 39]]).max() < mu.F32_TOL


@pytest.mark.parametrize("dtype,tol", [("float32", mu.F32_TOL), ("bfloat16", mu.BF16_TOL)])
def test_long_decoding_matches_the_whole_pass(models, dtype, tol):
    """Token by token far past every window, the caches growing on the way."""
    cfg, w, folder, t, want = models("mixed")
    with ModelSession(folder, dtype) as s:
        s.extend(0, t[:3], [])
        for p in range(3, 330 if dtype == "bfloat16" else 290):
            err = mu.logit_error(s.extend(0, t[p:p + 1], [0]), want[p:p + 1])
            assert err.max() < tol, p


def follow(cfg, w, prompt, toks):
    """The generated tokens are the plain implementation's first maxima, near ties apart."""
    lg = om.forward(cfg, w, list(prompt) + [int(v) for v in toks[:-1]])[len(prompt) - 1:]
    for i, tok in enumerate(toks):
        assert lg[i].max() - lg[i][tok] < 1e-3, i


@pytest.mark.parametrize("name", ["mixed", "odd", "heads"])
def test_greedy_generation_through_the_loop(models, name):
    cfg, w, folder, t, want = models(name)
    prompts = np.stack([t[:21], t[40:61], t[90:111]])
    with ModelSession(folder, "float32", 3) as s:
        toks = s.generate(prompts, 110)
        assert toks.shape == (3, 110)
        for p, g in zip(prompts, toks):
            follow(cfg, w, p, g)
        assert toks[0][:12].tolist() == om.greedy(cfg, w, prompts[0], 12)
        s.upload_prompts(prompts)                     # the same in two runs
        assert s.run(40) == 40 and s.run(70) == 110
        assert np.array_equal(s.download_tokens(110), toks)
    for p, g in zip(prompts, toks):                   # every stream alone
        with ModelSession(folder, "float32", 1) as s:
            assert np.array_equal(s.generate(p, 110)[0], g)


def test_bfloat16_generation_is_the_forward_pass_of_its_own_tokens(models):
    """Each greedy token is the maximum of the whole-pass logits of what precedes it (near ties apart), with and
    without graphs, and the step's logits are those of the whole pass."""
    cfg, w, folder, t, want = models("mixed")
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
    """More streams than the few-row products take, sampled: each equals its own run with the same seed."""
    cfg, w, folder, t, want = models("heads")
    prompts = np.stack([mu.tokens(cfg, 12, 500 + i) for i in range(70)])
    seeds = np.arange(70, dtype=np.uint32) + 5
    with ModelSession(folder, "float32", 70) as s:
        toks = s.generate(prompts, 9, temp=0.9, top_k=20, top_p=0.95, seeds=seeds)
        again = s.generate(prompts, 9, temp=0.9, top_k=20, top_p=0.95, seeds=seeds)
        assert np.array_equal(toks, again)
    with ModelSession(folder, "float32", 1) as s:
        same = sum(np.array_equal(s.generate(prompts[i], 9, temp=0.9, top_k=20, top_p=0.95, seeds=seeds[i:i + 1])[0],
                                  toks[i]) for i in range(0, 70, 7))
    assert same >= 9
    with ModelSession(folder, "bfloat16", 70) as s:
        s.keep_step_logits(True)
        toks = s.generate(prompts, 5)
        lg = s.read_step_logits(5, 70)
    for i in (0, 33, 69):
        ref = om.forward(cfg, w, list(prompts[i]) + list(toks[i][:4]))[11:]
        assert mu.logit_error(lg[:, i], ref).max() < mu.BF16_TOL


def test_positions_end_where_the_table_ends(models):
    cfg, w, folder, t, want = models("plain")
    with ModelSession(folder, "float32") as s:
        toks = s.generate(t[:200], 500)[0]
        assert len(toks) == cfg["max_positions"] - 200
        follow(cfg, w, t[:200], toks)
        s.extend(0, t[:200], [])
        with pytest.raises(NativeError, match="exceed 260 positions"):
            s.extend(0, t[:61], [])


def test_bad_calls_are_errors(models, tmp_path):
    cfg, w, folder, t, want = models("odd")
    with ModelSession(folder, "bfloat16") as s:
        with pytest.raises(NativeError, match="out of range"):
            s.extend(0, [3, cfg["vocab"]], [])
        with pytest.raises(NativeError):
            s.extend(1, [3], [])
        with pytest.raises(NativeError, match="wanted"):
            s.extend(0, [3], [1])
        with pytest.raises(NativeError, match="model folder"):
            s.load_params(np.zeros(16, np.uint8))
        assert mu.logit_error(s.extend(0, t[:9], range(9)), want[:9]).max() < mu.BF16_TOL
    broken = dict(w)
    del broken["l1.mix.uk"]
    formats.write_model_folder(str(tmp_path / "a"), cfg, broken)
    with pytest.raises(NativeError, match="l1.mix.uk"):
        ModelSession(str(tmp_path / "a"))
    broken = dict(w)
    broken["l0.mlp.up"] = w["l0.mlp.up"][:, :-1]
    formats.write_model_folder(str(tmp_path / "b"), cfg, broken)
    with pytest.raises(NativeError, match="l0.mlp.up has shape"):
        ModelSession(str(tmp_path / "b"))
    broken = dict(w)
    broken["head"] = np.array(w["head"])
    broken["head"][3, 4] = np.inf
    formats.write_model_folder(str(tmp_path / "c"), cfg, broken)
    with pytest.raises(NativeError, match="not finite"):
        ModelSession(str(tmp_path / "c"))


def test_command_line_generates_and_replays(models, tmp_path):
    cfg, w, folder, t, want = models("mixed")
    ids = ",".join(str(int(v)) for v in t[:30])
    out = str(tmp_path / "out.i32")
    p = subprocess.run([DRIVER, "infer", "--model", folder, "--dtype", "float32", "--ids", ids, "--max_new", "40",
                        "--out-ids-file", out], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    toks = np.fromfile(out, np.int32)
    assert len(toks) == 40
    follow(cfg, w, t[:30], toks)
    p = subprocess.run([DRIVER, "inspect", "--model", folder, "--ids", ids], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0 and "Argmax" in p.stdout, p.stderr
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
        assert mu.logit_error(got, want[places]).max() < mu.F32_TOL
