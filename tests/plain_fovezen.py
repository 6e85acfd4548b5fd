"""A plain, slow Fovezen model: whole sequences, no cache, float64, one function a mechanism.

Fovezen is a decoder-only model that carries several residual streams instead of one. All of them start as the token's
embedding row; a sublayer reads a weighted sum of the streams, normed by an RMS norm whose stored weight w stands for the
scale 1 + w, and afterwards every stream becomes a mixture of the old streams plus its own share of the sublayer's output
(hyper-connections with stored weights). The last norm reads the sum of the streams. Three kinds of mixers: ``mamba2`` (a
matrix state per head with one data-dependent decay a token and head, behind a short causal convolution), ``attention``
(grouped-query softmax attention, queries and keys normed over their whole projections, rotated halves with frequencies
stretched by wavelength) and ``parallel`` (softmax attention over a sliding window with short convolutions, a norm a head
and softly capped scores, beside a gated linear attention with a decay a key channel; half the sum of their normed
outputs). Feed-forward: a gated unit with clamped gate and up values. A run of layers may repeat with the same weights.
This file shares no code with the ``celeg_b200`` package: it takes the configuration as the dict that config.json holds
and the weights as a dict of arrays.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence

import numpy as np


def as_float64(tensors) -> Dict[str, np.ndarray]:
    """{name: torch tensor} -> {name: float64 array}."""
    import torch
    return {name: value.to(torch.float64).numpy() for name, value in tensors.items()}


# ------------------------------------------------------------------------- small functions
def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def rms_scaled(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x: np.ndarray, stored: np.ndarray, eps: float) -> np.ndarray:
    """The blocks' norm: the stored weight lies around zero and stands for 1 + itself."""
    return rms_scaled(x, eps) * (1.0 + stored)


def causal_convolution(u: np.ndarray, taps: np.ndarray, bias: Optional[np.ndarray] = None) -> np.ndarray:
    """u [tokens, channels], taps [channels, n]: the last tap meets the token itself, zeros before the start."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, u.shape[1])), u], axis=0)
    out = np.zeros_like(u)
    for j in range(n):
        out += padded[j:j + u.shape[0]] * taps[:, j]
    return out if bias is None else out + bias


# -------------------------------------------------------------------------------- mamba2
def decayed_states(keys, values, decays, queries) -> np.ndarray:
    """One head's read-outs [tokens, vdim]: S <- diag(decay) S + key value^T from S = 0, then S^T query. ``decays`` has one
    number a token, or one a token and key channel."""
    state = np.zeros((keys.shape[1], values.shape[1]), dtype=np.float64)
    out = np.zeros((keys.shape[0], values.shape[1]), dtype=np.float64)
    for t in range(keys.shape[0]):
        state = np.reshape(decays[t], (-1, 1)) * state + np.outer(keys[t], values[t])
        out[t] = state.T @ queries[t]
    return out


def mamba2(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> np.ndarray:
    heads, vdim, states, groups = (int(mixer[name]) for name in ("heads", "vdim", "state", "groups"))
    inner, tokens = heads * vdim, h.shape[0]
    rows = h @ tensors[base + "in"].T
    z = rows[:, :inner]
    convolved = silu(causal_convolution(rows[:, inner:2 * inner + 2 * groups * states], tensors[base + "conv"],
                                        tensors[base + "conv.b"]))
    x = convolved[:, :inner].reshape(tokens, heads, vdim)
    b = convolved[:, inner:inner + groups * states].reshape(tokens, groups, states)
    c = convolved[:, inner + groups * states:].reshape(tokens, groups, states)
    step = softplus(rows[:, 2 * inner + 2 * groups * states:] + tensors[base + "dt_bias"])
    decay = np.exp(-np.exp(tensors[base + "A_log"]) * step)
    y = np.zeros((tokens, heads, vdim), dtype=np.float64)
    for head in range(heads):
        group = head // (heads // groups)
        y[:, head] = decayed_states(step[:, head, None] * b[:, group], x[:, head], decay[:, head], c[:, group])
        y[:, head] += tensors[base + "D"][head] * x[:, head]
    gated = y.reshape(tokens, inner) * silu(z)
    parts = int(mixer["norm_groups"])
    normed = rms_scaled(gated.reshape(tokens, parts, inner // parts), eps).reshape(tokens, inner)
    return (normed * tensors[base + "norm"]) @ tensors[base + "o"].T


# -------------------------------------------------------------- gated linear attention
def channel_decays(tensors, base: str, mixer: dict, h: np.ndarray) -> np.ndarray:
    """[tokens, heads * dim]: sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)."""
    z = (h @ tensors[base + "a1"].T) @ tensors[base + "a2"].T + tensors[base + "a2.b"]
    return np.exp(-softplus(-z) / float(mixer["tau"]))


def gated_linear_attention(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> np.ndarray:
    heads, dim, vdim = (int(mixer[name]) for name in ("heads", "dim", "vdim"))
    tokens = h.shape[0]
    q = (h @ tensors[base + "q"].T).reshape(tokens, heads, dim) * dim ** -0.5
    k = (h @ tensors[base + "k"].T).reshape(tokens, heads, dim)
    v = (h @ tensors[base + "v"].T).reshape(tokens, heads, vdim)
    decays = channel_decays(tensors, base, mixer, h).reshape(tokens, heads, dim)
    read = np.stack([decayed_states(k[:, n], v[:, n], decays[:, n], q[:, n]) for n in range(heads)], axis=1)
    normed = (rms_scaled(read, eps) * tensors[base + "norm"]).reshape(tokens, heads * vdim)
    return (normed * silu(h @ tensors[base + "g"].T)) @ tensors[base + "o"].T


# ------------------------------------------------------------------------------ attention
def turn_frequencies(rot: dict) -> np.ndarray:
    """One frequency a pair; with ``scaling`` = {factor, low, high, original} stretched by wavelength."""
    dims = int(rot["dims"])
    plain = float(rot["base"]) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    scaling = rot.get("scaling")
    if not scaling:
        return plain
    factor, low, high, original = (float(scaling[name]) for name in ("factor", "low", "high", "original"))
    out = []
    for f in plain:
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return np.asarray(out, dtype=np.float64)


def rotate(x: np.ndarray, rot: Optional[dict]) -> np.ndarray:
    """x [tokens, heads, dim], token t at position t: pairs (i, i + dims / 2) of the first ``dims`` dimensions turn."""
    if not rot:
        return x
    dims = int(rot["dims"])
    half = dims // 2
    angles = np.arange(x.shape[0], dtype=np.float64)[:, None] * turn_frequencies(rot)[None, :]
    c, s = np.cos(angles)[:, None, :], np.sin(angles)[:, None, :]
    out = x.copy()
    u, v = x[:, :, :half], x[:, :, half:dims]
    out[:, :, :half] = u * c - v * s
    out[:, :, half:dims] = v * c + u * s
    return out


def visible_from(position: int, window: Optional[int]) -> int:
    """The first position that a query at ``position`` sees."""
    return 0 if window is None else max(0, position - window + 1)


def capped(scores: np.ndarray, cap: Optional[float]) -> np.ndarray:
    return scores if cap is None else cap * np.tanh(scores / cap)


def softmax(scores: np.ndarray) -> np.ndarray:
    e = np.exp(scores - scores.max())
    return e / e.sum()


def attend(q, k, v, scale: float, cap: Optional[float] = None, window: Optional[int] = None) -> np.ndarray:
    """q [tokens, heads, dim], k and v [tokens, groups, *]: query head n reads key/value head n // (heads / groups)."""
    tokens, heads = q.shape[:2]
    per = heads // k.shape[1]
    out = np.zeros((tokens, heads, v.shape[2]), dtype=np.float64)
    for head in range(heads):
        group = head // per
        for i in range(tokens):
            first = visible_from(i, window)
            weights = softmax(capped((k[first:i + 1, group] @ q[i, head]) * scale, cap))
            out[i, head] = weights @ v[first:i + 1, group]
    return out.reshape(tokens, -1)


def attention(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> np.ndarray:
    heads, groups, dim, vdim = (int(mixer[name]) for name in ("heads", "kv_heads", "dim", "vdim"))
    tokens = h.shape[0]
    q = rms_scaled(h @ tensors[base + "q"].T, eps) * tensors[base + "q.norm"]
    k = rms_scaled(h @ tensors[base + "k"].T, eps) * tensors[base + "k.norm"]
    v = (h @ tensors[base + "v"].T).reshape(tokens, groups, vdim)
    q = rotate(q.reshape(tokens, heads, dim), mixer.get("rot"))
    k = rotate(k.reshape(tokens, groups, dim), mixer.get("rot"))
    return attend(q, k, v, float(mixer["scale"])) @ tensors[base + "o"].T


def window_attention(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> np.ndarray:
    heads, groups, dim, vdim = (int(mixer[name]) for name in ("heads", "kv_heads", "dim", "vdim"))
    tokens = h.shape[0]
    q, k, v = (causal_convolution(h @ tensors[base + name].T, tensors[base + name + ".conv"]) for name in ("q", "k", "v"))
    q = rms_scaled(q.reshape(tokens, heads, dim), eps) * tensors[base + "q.norm"]
    k = rms_scaled(k.reshape(tokens, groups, dim), eps) * tensors[base + "k.norm"]
    read = attend(q, k, v.reshape(tokens, groups, vdim), float(mixer["scale"]), float(mixer["softcap"]),
                  int(mixer["mask"]["size"]))
    return read @ tensors[base + "o"].T


def side_by_side(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> np.ndarray:
    left = window_attention(tensors, base + "left.", mixer["left"], h, eps)
    right = gated_linear_attention(tensors, base + "right.", mixer["right"], h, eps)
    return 0.5 * (rms_scaled(left, eps) * tensors[base + "left.out"] + rms_scaled(right, eps) * tensors[base + "right.out"])


# ---------------------------------------------------------------------------- feed-forward
def clamped_unit(tensors, base: str, h: np.ndarray, limit: float) -> np.ndarray:
    g = np.minimum(h @ tensors[base + "gate"].T, limit)
    u = np.clip(h @ tensors[base + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ tensors[base + "down"].T


# ----------------------------------------------------------------------- hyper-connections
def gathered(copies: np.ndarray, weights: np.ndarray) -> np.ndarray:
    """copies [streams, tokens, width]: what a sublayer reads, before its norm."""
    return np.tensordot(weights, copies, axes=(0, 0))


def spread(copies: np.ndarray, mix: np.ndarray, out: np.ndarray, y: np.ndarray) -> np.ndarray:
    """New stream t = sum_s mix[s, t] (old stream s) + out[t] y."""
    return np.stack([gathered(copies, mix[:, t]) + out[t] * y for t in range(copies.shape[0])])


# ------------------------------------------------------------------------------- the model
def run_order(config: dict) -> List[int]:
    count = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(count))
    start, stop, times = (int(loop[name]) for name in ("start", "stop", "times"))
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, count))


MIXERS = {"mamba2": mamba2, "attention": attention, "parallel": side_by_side}


def streams(config: dict, tensors: Dict[str, np.ndarray], tokens: Sequence[int]) -> List[np.ndarray]:
    """The sum of the streams after every layer that runs, [tokens, width] each."""
    eps = float(config["norm"]["eps"])
    x = tensors["embed"][np.asarray(tokens)]
    copies = np.stack([x] * int(config["streams"]))
    out = []
    for index in run_order(config):
        base, layer = f"l{index}.", config["layers"][index]
        hc = base + "hc1."
        h = offset_norm(gathered(copies, tensors[hc + "in"]), tensors[base + "norm1"], eps)
        y = MIXERS[layer["type"]](tensors, base + "mix.", layer["mixer"], h, eps)
        copies = spread(copies, tensors[hc + "mix"], tensors[hc + "out"], y)
        if layer.get("mlp") is not None:
            hc = base + "hc2."
            h = offset_norm(gathered(copies, tensors[hc + "in"]), tensors[base + "norm2"], eps)
            y = clamped_unit(tensors, base + "mlp.", h, float(layer["mlp"]["limit"]))
            copies = spread(copies, tensors[hc + "mix"], tensors[hc + "out"], y)
        out.append(copies.sum(axis=0))
    return out


def logits(config: dict, tensors: Dict[str, np.ndarray], tokens: Sequence[int]) -> np.ndarray:
    x = streams(config, tensors, tokens)[-1]
    normed = offset_norm(x, tensors["final.norm"], float(config["norm"]["eps"]))
    return normed @ tensors["head"].T * float(config["logit_scale"])
