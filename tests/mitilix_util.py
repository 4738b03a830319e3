"""Small Mitilix models for the tests: configurations, weights, error measures."""
import numpy as np

from litnicelm_b200 import formats


def layer(heads, dim, vdim, kv_rank, window, ff=None, kv_from=None, scale=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "window": window, "ff": ff,
            "kv_from": kv_from, "scale": dim ** -0.5 if scale is None else scale}


CONFIGS = {
    # unequal layers: windows of several lengths, a shared cache read through a longer window than the one of
    # the layer that fills it, layers without feed-forward, sizes the tensor-core attention takes
    "mixed": formats.mitilix_config(96, 200, 700, [
        layer(3, 32, 16, 40, 24, ff=160),
        layer(2, 48, 64, 24, 130),
        layer(5, 16, 32, 40, 70, ff=72, kv_from=0, scale=0.3),
        layer(1, 64, 48, 24, 5, ff=104, kv_from=1),
    ], taps=4, eps=1e-5),
    # nothing a multiple of 8: the sizes only the any-size attention takes; a window of one token
    "odd": formats.mitilix_config(100, 131, 300, [
        layer(3, 20, 12, 22, 17, ff=90),
        layer(2, 9, 7, 13, 1),
        layer(4, 10, 30, 22, 60, ff=50, kv_from=0, scale=0.5),
    ], taps=6, eps=1e-3),
    # no convolution memory (one tap), one head, equal value and key sizes, a window beyond every context
    "plain": formats.mitilix_config(64, 72, 260, [
        layer(1, 32, 32, 32, 100000, ff=64),
        layer(1, 32, 32, 16, 2, ff=64, scale=1.0),
    ], taps=1, eps=1e-6),
    # many heads over one latent: two groups of 16 heads in the few-row kernels
    "heads": formats.mitilix_config(128, 96, 400, [
        layer(20, 16, 16, 72, 90, ff=256),
        layer(20, 16, 16, 72, 33, ff=128, kv_from=0),
    ], taps=2, eps=1e-6),
}


def build(name, tmp_path, seed=7):
    """(config, weights, folder) of one of the models above, the folder written."""
    cfg = CONFIGS[name]
    w = formats.mitilix_random_weights(cfg, seed)
    folder = str(tmp_path / name)
    formats.write_model_folder(folder, cfg, w)
    return cfg, w, folder


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


def logit_error(got, want):
    """Root mean square over the vocabulary of the mean-free difference, per position, over the logits' own."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


F32_TOL = 2e-5
BF16_TOL = 4e-2
