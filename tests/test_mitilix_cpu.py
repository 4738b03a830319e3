"""Mitilix without a GPU: the plain implementation's own properties, the model-folder formats, and what the
library refuses before it touches a device."""
import copy
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

from litnicelm_b200 import formats, plugin
from oracle import mitilix as om
import mitilix_util as mu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DRIVER = os.path.join(ROOT, "litnicelm_b200", "litnice_b200_run")


@pytest.fixture(scope="module")
def lib():
    if not os.path.exists(plugin.LIB_PATH) or not os.path.exists(DRIVER):
        import __graft_entry__
        __graft_entry__.build()
    return plugin.load_library()


# ---- the plain implementation ----

def test_convolution_reads_zeros_before_the_sequence():
    h = np.arange(1.0, 6.0)[:, None] * np.array([[1.0, 10.0]])
    w = np.array([[0.5, 2.0, 1.0], [0.0, 0.0, 3.0]])
    y = om.causal_channel_conv(h, w)
    assert y[0].tolist() == [1.0, 30.0]
    assert y[1].tolist() == [2.0 * 1 + 2.0, 60.0]
    assert y[4].tolist() == [0.5 * 3 + 2.0 * 4 + 5.0, 150.0]


def test_window_keeps_the_last_size_tokens():
    s = np.zeros(10)
    p = om.window_softmax(s, 7, 3)
    assert np.allclose(p, [0, 0, 0, 0, 0, 1 / 3, 1 / 3, 1 / 3, 0, 0])
    assert np.allclose(om.window_softmax(s[:2], 1, 3), [0.5, 0.5])
    assert np.allclose(om.window_softmax(s, 4, 1), np.eye(10)[4])


def test_norms_put_eps_inside_the_root():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(om.scalar_rms_norm(x, 2.0, 3.5), x * 2.0 / 4.0)
    assert np.allclose(om.vector_rms_norm(x, np.array([1.0, 5.0]), 3.5), [[0.75, 5.0]])


def test_gelu_is_the_error_function_form():
    assert np.allclose(om.gelu_exact(np.array([0.0, 1.0, -1.0, 3.0])), [0.0, 0.8413447460685429, -0.15865525393145707,
                                                                         2.9959503061044])


def test_prefix_of_a_sequence_does_not_see_what_follows():
    cfg = mu.CONFIGS["mixed"]
    w = formats.mitilix_random_weights(cfg, 3)
    t = mu.tokens(cfg, 40, 1)
    whole = om.forward(cfg, w, t)
    assert np.allclose(whole[:25], om.forward(cfg, w, t[:25]), atol=1e-12)


# ---- formats ----

def test_safetensors_round_trip(tmp_path):
    cfg, w, folder = mu.build("odd", tmp_path)
    raw = open(os.path.join(folder, "model.safetensors"), "rb").read()
    n = int.from_bytes(raw[:8], "little")
    header = json.loads(raw[8:8 + n])
    assert set(header) == set(formats.mitilix_shapes(cfg))
    for name, e in header.items():
        a, b = e["data_offsets"]
        got = formats.from_bf16_bits(np.frombuffer(raw[8 + n + a:8 + n + b], np.uint16)).reshape(e["shape"])
        assert e["shape"] == list(w[name].shape) and np.array_equal(got, w[name])


# ---- the library's checks on a folder (before a device is needed) ----

def create(lib, folder, dtype=0):
    h = C.c_void_p()
    lib.litnice_b200_session_create_model.argtypes = [C.c_char_p, C.c_int32, C.c_int32, C.c_int32, C.POINTER(C.c_void_p)]
    rc = lib.litnice_b200_session_create_model(str(folder).encode(), dtype, 1, -1, C.byref(h))
    lib.litnice_b200_last_error.restype = C.c_char_p
    lib.litnice_b200_last_error.argtypes = [C.c_void_p]
    msg = lib.litnice_b200_last_error(h).decode()
    if h:
        lib.litnice_b200_session_destroy.argtypes = [C.c_void_p]
        lib.litnice_b200_session_destroy(h)
    return rc, msg


def test_registry_names_the_design(lib):
    assert "Mitilix" in plugin.architectures()
    p = subprocess.run([DRIVER, "designs"], capture_output=True, text=True, timeout=60)
    assert p.returncode == 0 and "Mitilix" in p.stdout.strip().split(",")


@pytest.mark.parametrize("change,words", [
    (lambda c: c.update(architecture="Nothing"), "unknown architecture"),
    (lambda c: c["layers"][0].update(type="ring"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),      # layer 2 has no latents of its own
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "kv_from"),      # another rank
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["canon"].update(taps=0), "taps"),
    (lambda c: c.update(width=1.5), "integer"),
    (lambda c: c.update(layers=[]), "no layers"),
])
def test_bad_configurations_are_refused(lib, tmp_path, change, words):
    cfg = copy.deepcopy(mu.CONFIGS["mixed"])
    change(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    rc, msg = create(lib, tmp_path)
    assert rc == -4 and words in msg


def test_broken_files_are_refused(lib, tmp_path):
    rc, msg = create(lib, tmp_path / "absent")
    assert rc == -4 and "cannot open" in msg
    (tmp_path / "config.json").write_text('{"architecture": "Mitilix", ')
    assert create(lib, tmp_path)[0] == -4
    (tmp_path / "config.json").write_text(json.dumps(mu.CONFIGS["odd"]))
    (tmp_path / "model.safetensors").write_bytes(b"\x10\x00\x00\x00\x00\x00\x00\x00{}")
    rc, msg = create(lib, tmp_path)
    assert rc == -4 and "longer than the file" in msg
    assert create(lib, tmp_path, dtype=7)[0] == -1


def test_trace_command_rejects_bad_usage(lib, tmp_path):
    run = os.path.join(ROOT, "bin", "trace_run")
    assert os.access(run, os.X_OK)
    p = subprocess.run([run, "--model", str(tmp_path / "absent"), "--dtype", "bfloat16", "--out", str(tmp_path),
                        "--max-tokens", "8"], capture_output=True, text=True, stdin=subprocess.DEVNULL, timeout=600)
    assert p.returncode == 1 and "cannot open" in p.stderr
    p = subprocess.run([run, "--model", str(tmp_path), "--dtype", "int4", "--out", str(tmp_path)], capture_output=True,
                       text=True, stdin=subprocess.DEVNULL, timeout=600)
    assert p.returncode == 1 and "--dtype" in p.stderr
