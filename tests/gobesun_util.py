"""Small Gobesun models for the tests: configurations, weights, error measures."""
import numpy as np

from litnicelm_b200 import formats
from litnicelm_b200.formats import chunk_attention_layer as attention, delta_layer as delta
from oracle import gobesun as og
from mitilix_util import logit_error, tokens  # noqa: F401

YARN = {"factor": 8.0, "original": 96, "fast": 12.0, "slow": 1.5}

CONFIGS = {
    # unequal layers of both kinds, shared key heads, chunks of several lengths, a loop in the middle
    "mixed": formats.gobesun_config(96, 200, [
        delta(6, 3, 32, 48, 3, ff=120),
        attention(4, 2, 48, 32, 40, {"dims": 24, "base": 5000.0, "scaling": YARN}),
        delta(4, 4, 16, 64, 4),
        attention(6, 1, 32, 32, 100, {"dims": 32, "base": 100.0}, scale=0.3, ff=88),
    ], loop=(1, 3, 2), embed_scale=3.5, eps=1e-5),
    # nothing a multiple of 8; taps 1 and 2; a first layer that runs three times
    "odd": formats.gobesun_config(100, 131, [
        delta(3, 1, 20, 28, 2),
        attention(3, 3, 18, 22, 17, {"dims": 10, "base": 300.0, "scaling": dict(YARN, factor=2.5)}, ff=50),
        delta(2, 2, 9, 7, 1, ff=30),
    ], loop=(0, 1, 3), embed_scale=1.0, eps=1e-3),
    # heads beyond 128 elements, many taps, a chunk beyond every context, one head for all, no layer repeated
    "wide": formats.gobesun_config(72, 90, [
        delta(2, 1, 128, 128, 4, ff=64),
        attention(2, 1, 160, 144, 100000, {"dims": 160, "base": 10000.0}),
        delta(2, 2, 144, 160, 6),
    ], loop=(1, 1, 5), embed_scale=8.0, eps=1e-6),
    # a chunk of one position (every query sees itself only), twelve query heads on one key head, the last layers looped
    "edge": formats.gobesun_config(64, 72, [
        attention(12, 1, 16, 16, 64, {"dims": 8, "base": 50.0, "scaling": dict(YARN, factor=1.0)}, ff=48),
        attention(2, 2, 32, 32, 1, {"dims": 2, "base": 10.0}, scale=1.0),
        delta(1, 1, 64, 32, 4, ff=96),
    ], loop=(1, 3, 2), embed_scale=2.0, eps=1e-6),
}


def build(name, tmp_path, seed=7):
    """(config, weights, folder) of one of the models above, the folder written."""
    cfg = CONFIGS[name]
    w = formats.gobesun_random_weights(cfg, seed)
    folder = str(tmp_path / name)
    formats.write_model_folder(folder, cfg, w)
    return cfg, w, folder


def nearest(a):
    return formats.from_bf16_bits(formats.to_bf16_bits(np.asarray(a, np.float32))).astype(np.float64)


def toward_zero(a):
    return (np.ascontiguousarray(a, np.float32).view(np.uint32) & 0xFFFF0000).view(np.float32).astype(np.float64)


def allowed(cfg, w, t, want):
    """dtype -> largest logit_error of every position. Heads' outputs are divided by their own size, so where one happens
    to be small, rounding moves the position more: bfloat16 is allowed a few times what rounding alone does there."""
    moved = np.maximum(logit_error(og.forward(cfg, w, t, cast=nearest), want),
                       0.7 * logit_error(og.forward(cfg, w, t, cast=toward_zero), want))
    return {"float32": np.full(len(t), 3e-5), "bfloat16": 0.025 + 3.0 * moved}
