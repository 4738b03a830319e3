"""Plain, slow implementation of the Gobesun decoder in numpy, for the tests of the CUDA path.

One function per mechanism, written from the equations in double precision; nothing here is
shared with the product path. Weights are a dict name -> array (linear weights [out, in]).

``cast`` (the identity unless given) is applied to what a served model may hold in 16 bits: inputs and
results of the matrix products, convolved vectors, rotated queries and keys. With a rounding function it
shows how far rounding alone moves each position.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np


def exact(x: np.ndarray) -> np.ndarray:
    return x


def rms_normalise(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def centred_rms_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    """RMS norm whose stored weight is the gain minus one."""
    return rms_normalise(x, eps) * (1.0 + w)


def plain_rms_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    return rms_normalise(x, eps) * w


def sigmoid(z: np.ndarray) -> np.ndarray:
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


def softplus(z: np.ndarray) -> np.ndarray:
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z: np.ndarray) -> np.ndarray:
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


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


def unit_vector(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def log_decay(a: np.ndarray, a_log: np.ndarray, dt_bias: np.ndarray) -> np.ndarray:
    """Logarithm of the factor that shrinks a head's state at a token."""
    return -np.exp(a_log) * softplus(a + dt_bias)


def delta_rule(q: np.ndarray, k: np.ndarray, v: np.ndarray, beta: np.ndarray, log_g: np.ndarray,
               state: Optional[np.ndarray] = None) -> np.ndarray:
    """One head, token by token: q, k [T, dim], v [T, vdim], beta, log_g [T]; state [dim, vdim] is updated in place."""
    s = np.zeros((k.shape[1], v.shape[1])) if state is None else state
    out = np.zeros_like(v)
    for t in range(v.shape[0]):
        s *= math.exp(log_g[t])
        u = beta[t] * (v[t] - k[t] @ s)
        s += np.outer(k[t], u)
        out[t] = q[t] @ s
    return out


def gated_head_norm(o: np.ndarray, gate: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    """o, gate [T, heads, vdim]."""
    return rms_normalise(o, eps) * w * silu(gate)


def delta_mixer(h: np.ndarray, w: Dict[str, np.ndarray], p: str, m: dict, eps: float, cast=exact) -> np.ndarray:
    n, heads, kv, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (cast(silu(causal_channel_conv(cast(h @ w[p + t].T), w[p + t + ".conv"]))) for t in "qkv")
    q = unit_vector(q.reshape(n, kv, dim)) * dim ** -0.5
    k = unit_vector(k.reshape(n, kv, dim))
    v = v.reshape(n, heads, vdim)
    beta = sigmoid(h @ w[p + "b"].T)
    log_g = log_decay(h @ w[p + "a"].T, w[p + "A_log"], w[p + "dt_bias"])
    o = np.stack([delta_rule(q[:, i * kv // heads], k[:, i * kv // heads], v[:, i], beta[:, i], log_g[:, i])
                  for i in range(heads)], axis=1)
    o = gated_head_norm(o, cast(h @ w[p + "g"].T).reshape(n, heads, vdim), w[p + "norm"], eps)
    return cast(o.reshape(n, heads * vdim)) @ w[p + "o"].T


def yarn_frequencies(rot: dict) -> np.ndarray:
    """Angle per position of every pair, the slow ones divided by the factor."""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if sc is None:
        return f

    def place(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp)


def yarn_amplitude(rot: dict) -> float:
    sc = rot.get("scaling")
    return 1.0 if sc is None else 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x: np.ndarray, positions: np.ndarray, rot: dict) -> np.ndarray:
    """x [T, heads, dim]: the first rot dims of each head, dimension i turned together with i + dims / 2."""
    half = rot["dims"] // 2
    angle = positions[:, None] * yarn_frequencies(rot)[None, :]
    c, s = (f(angle)[:, None, :] * yarn_amplitude(rot) for f in (np.cos, np.sin))
    y = x.copy()
    u, v = x[..., :half], x[..., half:2 * half]
    y[..., :half] = u * c - v * s
    y[..., half:2 * half] = v * c + u * s
    return y


def chunk_softmax(scores: np.ndarray, i: int, size: int) -> np.ndarray:
    """Weights of query i over keys 0..len-1: softmax over the keys j <= i of its own chunk, zero elsewhere."""
    j = np.arange(scores.shape[-1])
    seen = (j <= i) & (j // size == i // size)
    w = np.zeros_like(scores)
    s = scores[..., seen]
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    w[..., seen] = e / e.sum(axis=-1, keepdims=True)
    return w


def grouped_attention(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float, size: int) -> np.ndarray:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]; query head h reads key head h // (H / G)."""
    n, heads = q.shape[:2]
    per = heads // k.shape[1]
    out = np.zeros((n, heads, v.shape[2]))
    for h in range(heads):
        kh, vh = k[:, h // per], v[:, h // per]
        for i in range(n):
            out[i, h] = chunk_softmax((kh[:i + 1] @ q[i, h]) * scale, i, size) @ vh[:i + 1]
    return out


def attention_mixer(h: np.ndarray, w: Dict[str, np.ndarray], p: str, m: dict, eps: float, cast=exact) -> np.ndarray:
    n, heads, kv, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = plain_rms_norm(cast(h @ w[p + "q"].T), w[p + "q.norm"], eps).reshape(n, heads, dim)
    k = plain_rms_norm(cast(h @ w[p + "k"].T), w[p + "k.norm"], eps).reshape(n, kv, dim)
    v = cast(h @ w[p + "v"].T).reshape(n, kv, vdim)
    at = np.arange(n, dtype=np.float64)
    o = grouped_attention(cast(rotate(q, at, m["rot"])), cast(rotate(k, at, m["rot"])), v, m["scale"], m["mask"]["size"])
    return cast(o.reshape(n, heads * vdim)) @ w[p + "o"].T


def gated_feed_forward(h: np.ndarray, gate: np.ndarray, up: np.ndarray, down: np.ndarray, cast=exact) -> np.ndarray:
    return cast(gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def layer_order(cfg: dict) -> List[int]:
    """Indices of the layers in the order they run."""
    lp = cfg["loop"]
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, len(cfg["layers"])))


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, layers_out: Optional[List[np.ndarray]] = None,
            cast=exact) -> np.ndarray:
    """Logits [T, vocab] of one sequence; layers_out receives the residual stream after every layer run."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i in layer_order(cfg):
        e, p = cfg["layers"][i], f"l{i}."
        mixer = {"delta": delta_mixer, "attention": attention_mixer}[e["type"]]
        h = cast(centred_rms_norm(x, w[p + "norm1"], eps))
        x = x + centred_rms_norm(mixer(h, w, p + "mix.", e["mixer"], eps, cast), w[p + "norm1b"], eps)
        if e.get("mlp") is not None:
            h = cast(centred_rms_norm(x, w[p + "norm2"], eps))
            f = gated_feed_forward(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"], cast)
            x = x + centred_rms_norm(f, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return cast(centred_rms_norm(x, w["final.norm"], eps)) @ w["head"].T


def greedy(cfg: dict, w: Dict[str, np.ndarray], prompt, steps: int) -> List[int]:
    """First-maximum greedy continuation, the whole sequence recomputed for every token."""
    seq = [int(t) for t in prompt]
    for _ in range(steps):
        seq.append(int(np.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]
