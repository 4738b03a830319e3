"""Gobesun without a GPU: the plain implementation's own properties, the model-folder formats, and what the
library refuses before it touches a device."""
import copy
import json
import math
import os

import numpy as np
import pytest

from litnicelm_b200 import formats, plugin
from oracle import gobesun as og
import gobesun_util as gu
from test_mitilix_cpu import create, lib  # noqa: F401


# ---- the plain implementation ----

def test_delta_rule_on_orthonormal_keys_is_a_lookup():
    k = np.eye(4)[[0, 1, 2, 3, 1]]
    v = np.arange(10.0).reshape(5, 2) + 1.0
    beta = np.array([1.0, 1.0, 0.5, 1.0, 1.0])
    o = og.delta_rule(k, k, v, beta, np.zeros(5))
    assert np.allclose(o[:2], v[:2])            # the read sees the token's own write
    assert np.allclose(o[2], 0.5 * v[2])
    assert np.allclose(o[4], v[4])              # a key written again: its old value is taken out first
    s = np.zeros((4, 2))
    og.delta_rule(k[:3], k[:3], v[:3], beta[:3], np.zeros(3), s)
    assert np.allclose(og.delta_rule(k[3:], k[3:], v[3:], beta[3:], np.zeros(2), s), o[3:])


def test_decay_comes_before_the_write():
    k = np.array([[1.0, 0.0], [1.0, 0.0]])
    o = og.delta_rule(k, k, np.array([[2.0], [0.0]]), np.array([1.0, 0.25]), np.log([0.5, 0.5]))
    assert np.allclose(o[:, 0], [2.0, 1.0 - 0.25 * 1.0])


def test_chunk_sees_its_own_positions_only():
    p = og.chunk_softmax(np.zeros(10), 7, 3)
    assert np.allclose(p, [0, 0, 0, 0, 0, 0, 0.5, 0.5, 0, 0])
    assert np.allclose(og.chunk_softmax(np.zeros(10), 6, 3), np.eye(10)[6])
    assert np.allclose(og.chunk_softmax(np.zeros(3), 2, 100), [1 / 3] * 3)


def test_rotation_keeps_relative_positions_and_scales_by_the_amplitude():
    rot = {"dims": 6, "base": 40.0, "scaling": {"factor": 4.0, "original": 60, "fast": 3.0, "slow": 0.5}}
    rng = np.random.default_rng(1)
    x, y = rng.standard_normal((2, 1, 1, 8))
    dots = [float((og.rotate(x, np.array([a]), rot)[..., :6] * og.rotate(y, np.array([a - 5.0]), rot)[..., :6]).sum())
            for a in (5.0, 700.0)]
    assert abs(dots[0] - dots[1]) < 1e-9
    r = og.rotate(x, np.array([3.0]), rot)
    assert np.array_equal(r[..., 6:], x[..., 6:])
    amp = 0.1 * math.log(4.0) + 1.0
    assert np.isclose(np.linalg.norm(r[..., :6]), amp * np.linalg.norm(x[..., :6]))


def test_slow_pairs_are_divided_and_fast_ones_kept():
    rot = {"dims": 64, "base": 10000.0}
    plain = og.yarn_frequencies(rot)
    turns = 1000 * plain / (2 * math.pi)
    f = og.yarn_frequencies(dict(rot, scaling={"factor": 4.0, "original": 1000, "fast": 30.0, "slow": 2.0}))
    assert np.allclose(f[turns > 40], plain[turns > 40])
    assert np.allclose(f[turns < 1.2], plain[turns < 1.2] / 4.0)
    mid = (turns < 20) & (turns > 4)
    assert (f[mid] < plain[mid]).all() and (f[mid] > plain[mid] / 4.0).all()


def test_layers_of_the_loop_run_in_a_row():
    assert og.layer_order(gu.CONFIGS["mixed"]) == [0, 1, 2, 1, 2, 3]
    assert og.layer_order(gu.CONFIGS["odd"]) == [0, 0, 0, 1, 2]
    assert og.layer_order(gu.CONFIGS["wide"]) == [0, 1, 2]


def test_activations():
    z = np.array([-3.0, 0.0, 0.7, 4.0])
    assert np.allclose(og.silu(z), z / (1 + np.exp(-z)))
    assert np.allclose(og.softplus(z), np.log(1 + np.exp(z)))
    assert np.allclose(og.gelu_tanh(np.array([1.0, -1.0])), [0.8411919906082768, -0.15880800939172324])
    assert og.softplus(np.array([800.0]))[0] == 800.0


def test_prefix_of_a_sequence_does_not_see_what_follows():
    cfg = gu.CONFIGS["mixed"]
    w = formats.gobesun_random_weights(cfg, 3)
    t = gu.tokens(cfg, 60, 1)
    assert np.allclose(og.forward(cfg, w, t)[:45], og.forward(cfg, w, t[:45]), atol=1e-11)


# ---- formats ----

def test_safetensors_round_trip(tmp_path):
    cfg, w, folder = gu.build("odd", tmp_path)
    raw = open(os.path.join(folder, "model.safetensors"), "rb").read()
    n = int.from_bytes(raw[:8], "little")
    header = json.loads(raw[8:8 + n])
    assert set(header) == set(formats.gobesun_shapes(cfg)) == set(w)
    for name, e in header.items():
        assert tuple(e["shape"]) == formats.gobesun_shapes(cfg)[name]


# ---- the library's checks on a folder (before a device is needed) ----

def test_registry_names_the_design(lib):  # noqa: F811
    assert "Gobesun" in plugin.architectures()


@pytest.mark.parametrize("change,words", [
    (lambda c: c["layers"][0].update(type="ring"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=50), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"].update(dim=600), "size"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c.pop("embedding"), "embedding"),
    (lambda c: c.update(width=1.5), "integer"),
    (lambda c: c.update(layers=[]), "no layers"),
])
def test_bad_configurations_are_refused(lib, tmp_path, change, words):  # noqa: F811
    cfg = copy.deepcopy(gu.CONFIGS["mixed"])
    change(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    rc, msg = create(lib, tmp_path)
    assert rc == -4 and words in msg
