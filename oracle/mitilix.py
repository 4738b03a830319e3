"""Plain, slow implementation of the Mitilix decoder in numpy, for the tests of the CUDA path.

One function per mechanism, written from the equations in double precision; nothing here is
shared with the product path. Weights are a dict name -> array (linear weights [out, in]).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np

_erf = np.vectorize(math.erf, otypes=[np.float64])


def rms_normalise(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def scalar_rms_norm(x: np.ndarray, gain: float, eps: float) -> np.ndarray:
    """RMS norm whose gain is one number for all coordinates."""
    return rms_normalise(x, eps) * gain


def vector_rms_norm(x: np.ndarray, gain: np.ndarray, eps: float) -> np.ndarray:
    """RMS norm with a gain per coordinate."""
    return rms_normalise(x, eps) * gain


def causal_channel_conv(h: np.ndarray, w: np.ndarray) -> np.ndarray:
    """y[t, c] = sum_j w[c, j] h[t - (taps - 1) + j, c], zeros before the first row."""
    taps = w.shape[1]
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(taps):
            u = t - (taps - 1) + j
            if u >= 0:
                y[t] += w[:, j] * h[u]
    return y


def with_input_conv(h: np.ndarray, w: np.ndarray) -> np.ndarray:
    return h + causal_channel_conv(h, w)


def gelu_exact(z: np.ndarray) -> np.ndarray:
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def dense_feed_forward(a: np.ndarray, up: np.ndarray, down: np.ndarray) -> np.ndarray:
    return gelu_exact(a @ up.T) @ down.T


def latent(a: np.ndarray, w_dkv: np.ndarray, gain: np.ndarray, eps: float) -> np.ndarray:
    """The compressed row per position: what a cache has to keep."""
    return vector_rms_norm(a @ w_dkv.T, gain, eps)


def window_softmax(scores: np.ndarray, i: int, size: int) -> np.ndarray:
    """Weights of query i over keys 0..len-1: softmax over 0 <= i - j < size, zero elsewhere."""
    j = np.arange(scores.shape[-1])
    seen = (i - j >= 0) & (i - j < size)
    w = np.zeros_like(scores)
    s = scores[..., seen]
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    w[..., seen] = e / e.sum(axis=-1, keepdims=True)
    return w


def latent_attention(a: np.ndarray, c: np.ndarray, w_q: np.ndarray, w_uk: np.ndarray, w_uv: np.ndarray,
                     w_o: np.ndarray, heads: int, dim: int, vdim: int, scale: float, size: int) -> np.ndarray:
    """a [T, width] queries' input, c [T, kv_rank] latents of the same positions."""
    n = a.shape[0]
    q = (a @ w_q.T).reshape(n, heads, dim)
    k = (c @ w_uk.T).reshape(n, heads, dim)
    v = (c @ w_uv.T).reshape(n, heads, vdim)
    out = np.zeros((n, heads, vdim))
    for i in range(n):
        scores = np.einsum("hd,jhd->hj", q[i], k[:i + 1]) * scale
        p = window_softmax(scores, i, size)
        out[i] = np.einsum("hj,jhe->he", p, v[:i + 1])
    return out.reshape(n, heads * vdim) @ w_o.T


def embed(tokens: np.ndarray, table: np.ndarray, pos: np.ndarray) -> np.ndarray:
    return table[tokens] + pos[:len(tokens)]


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, layers_out: Optional[List[np.ndarray]] = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence; layers_out receives the residual stream after every layer."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(np.asarray(tokens), w["embed"], w["pos"])
    latents: Dict[int, np.ndarray] = {}
    for i, entry in enumerate(cfg["layers"]):
        m, p = entry["mixer"], f"l{i}."
        h = scalar_rms_norm(x, float(w[p + "norm1"]), eps)
        a = with_input_conv(h, w[p + "canon1"])
        if m.get("kv_from") is None:
            latents[i] = latent(a, w[p + "mix.dkv"], w[p + "mix.dkv.norm"], eps)
            c = latents[i]
        else:
            c = latents[m["kv_from"]]
        y = latent_attention(a, c, w[p + "mix.q"], w[p + "mix.uk"], w[p + "mix.uv"], w[p + "mix.o"], m["heads"],
                             m["dim"], m["vdim"], m["scale"], m["mask"]["size"])
        if entry.get("mlp") is not None:
            y = y + dense_feed_forward(with_input_conv(h, w[p + "canon2"]), w[p + "mlp.up"], w[p + "mlp.down"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return scalar_rms_norm(x, float(w["final.norm"]), eps) @ w["head"].T


def greedy(cfg: dict, w: Dict[str, np.ndarray], prompt, steps: int) -> List[int]:
    """First-maximum greedy continuation, the whole sequence recomputed for every token."""
    seq = [int(t) for t in prompt]
    for _ in range(steps):
        seq.append(int(np.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]
