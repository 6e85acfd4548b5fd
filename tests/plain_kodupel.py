"""A plain, slow Kodupel model: whole sequences, no cache, float64, one function a mechanism.

Kodupel is a decoder-only model whose blocks norm what a sublayer puts out instead of what it reads:
x <- x + Norm(Mixer(x)), then x <- x + Norm(FeedForward(x)), the norm an RMS norm whose stored weight w stands for the
scale 1 + w. Token rows are the embedding rows times a constant. Two kinds of mixers: ``general_delta`` (a matrix state
per head whose key channels each decay at a rate of their own, from which a share of what lies along the token's unit
key is removed, channel by channel, before the token's own key and value are written) and ``attention`` (grouped-query
softmax attention with biases, a norm per head on queries and keys, a rotation of neighbouring pairs with stretched
frequencies, values of unit root mean square, a one in the softmax's denominator, a sigmoid gate per head; a layer may
read another layer's keys and values). Feed-forward: a mixture of experts with clamped gates, chosen by sigmoid scores
plus a stored correction and weighed by the scores themselves. This file shares no code with the ``celeg_b200`` package:
it takes the configuration as the dict that config.json holds and the weights as a dict of arrays.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np


def as_float64(tensors) -> Dict[str, np.ndarray]:
    """{name: torch tensor} -> {name: float64 array}."""
    import torch
    return {name: value.to(torch.float64).numpy() for name, value in tensors.items()}


# ------------------------------------------------------------------------- small functions
def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def rms_scaled(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x: np.ndarray, stored: np.ndarray, eps: float) -> np.ndarray:
    """The blocks' norm: the stored weight lies around zero and stands for 1 + itself."""
    return rms_scaled(x, eps) * (1.0 + stored)


def embed(config: dict, tensors, tokens: Sequence[int]) -> np.ndarray:
    return tensors["embed"][np.asarray(tokens)] * float(config["embedding"]["scale"])


# -------------------------------------------------------------------------- general delta
def channel_decay(tensors, base: str, h: np.ndarray) -> np.ndarray:
    """[tokens, heads * dim]: exp(-e^(-1/2) sigmoid(W_w2 tanh(W_w1 h) + w0)), between e^(-e^(-1/2)) and 1."""
    z = np.tanh(h @ tensors[base + "w1"].T) @ tensors[base + "w2"].T + tensors[base + "w0"]
    return np.exp(-math.exp(-0.5) * sigmoid(z))


def removal_rate(tensors, base: str, h: np.ndarray) -> np.ndarray:
    return sigmoid(h @ tensors[base + "a"].T + tensors[base + "a.b"])


def delta_states(r, k, v, decay, removal) -> np.ndarray:
    """One head's read-outs [tokens, dim]: S <- diag(w) S - (a u)(u^T S) + k v^T from S = 0, both terms of the old S,
    u = k / sqrt(sum(k^2) + 1e-6); then S^T r."""
    tokens, dim = k.shape
    state = np.zeros((dim, v.shape[1]), dtype=np.float64)
    out = np.zeros((tokens, v.shape[1]), dtype=np.float64)
    for t in range(tokens):
        u = k[t] / math.sqrt(float(k[t] @ k[t]) + 1e-6)
        state = decay[t][:, None] * state - np.outer(removal[t] * u, u @ state) + np.outer(k[t], v[t])
        out[t] = state.T @ r[t]
    return out


def general_delta(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> np.ndarray:
    heads, dim = int(mixer["heads"]), int(mixer["dim"])
    tokens = h.shape[0]
    r, k, v = (h @ tensors[base + name].T for name in ("r", "k", "v"))
    decay, removal = channel_decay(tensors, base, h), removal_rate(tensors, base, h)
    read = np.zeros((tokens, heads * dim), dtype=np.float64)
    for head in range(heads):
        cut = slice(head * dim, (head + 1) * dim)
        read[:, cut] = rms_scaled(delta_states(r[:, cut], k[:, cut], v[:, cut], decay[:, cut], removal[:, cut]), eps)
    return (read * tensors[base + "norm"] * sigmoid(h @ tensors[base + "g"].T)) @ tensors[base + "o"].T


# ------------------------------------------------------------------------------ attention
def turn_frequencies(rot: dict) -> Tuple[np.ndarray, float]:
    """(one frequency a pair, the factor on cosine and sine)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    pairs = np.arange(dims // 2, dtype=np.float64)
    plain = base ** (-2.0 * pairs / dims)
    scaling = rot.get("scaling")
    if not scaling:
        return plain, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
    ramp = np.clip((pairs - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return plain / factor * ramp + plain * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x: np.ndarray, rot: Optional[dict]) -> np.ndarray:
    """x [tokens, heads, dim], token t at position t: pairs (2i, 2i + 1) of the first ``dims`` dimensions turn."""
    if not rot:
        return x
    dims = int(rot["dims"])
    frequencies, magnitude = turn_frequencies(rot)
    out = x.copy()
    for t in range(x.shape[0]):
        c, s = np.cos(t * frequencies) * magnitude, np.sin(t * frequencies) * magnitude
        u, v = x[t, :, 0:dims:2], x[t, :, 1:dims:2]
        out[t, :, 0:dims:2] = u * c - v * s
        out[t, :, 1:dims:2] = v * c + u * s
    return out


def keys_and_values(tensors, base: str, mixer: dict, h: np.ndarray, eps: float) -> Tuple[np.ndarray, np.ndarray]:
    """What the layer's cache holds: keys [tokens, groups, dim] (normed, rotated), values of unit root mean square."""
    groups, dim, vdim = int(mixer["kv_heads"]), int(mixer["dim"]), int(mixer["vdim"])
    k = (h @ tensors[base + "k"].T + tensors[base + "k.b"]).reshape(-1, groups, dim)
    v = (h @ tensors[base + "v"].T + tensors[base + "v.b"]).reshape(-1, groups, vdim)
    return rotate(rms_scaled(k, eps) * tensors[base + "k.norm"], mixer.get("rot")), rms_scaled(v, eps)


def weights_with_one(scores: np.ndarray) -> np.ndarray:
    """exp(s_j) / (1 + sum exp(s_j))."""
    top = max(float(scores.max()), 0.0)
    e = np.exp(scores - top)
    return e / (math.exp(-top) + e.sum())


def attention(tensors, base: str, mixer: dict, h: np.ndarray, k: np.ndarray, v: np.ndarray, eps: float) -> np.ndarray:
    """Query head n reads key/value head n // (heads / kv_heads) of the given keys and values (this layer's or those of
    the layer it shares with)."""
    heads, groups, dim, vdim = (int(mixer[name]) for name in ("heads", "kv_heads", "dim", "vdim"))
    scale, tokens = float(mixer["scale"]), h.shape[0]
    q = (h @ tensors[base + "q"].T + tensors[base + "q.b"]).reshape(tokens, heads, dim)
    q = rotate(rms_scaled(q, eps) * tensors[base + "q.norm"], mixer.get("rot"))
    gate = sigmoid(h @ tensors[base + "g"].T)
    out = np.zeros((tokens, heads, vdim), dtype=np.float64)
    for head in range(heads):
        group = head // (heads // groups)
        for i in range(tokens):
            weights = weights_with_one((k[:i + 1, group] @ q[i, head]) * scale)
            out[i, head] = (weights @ v[:i + 1, group]) * gate[i, head]
    return out.reshape(tokens, heads * vdim) @ tensors[base + "o"].T + tensors[base + "o.b"]


# ---------------------------------------------------------------------------- feed-forward
def clamped_expert(tensors, base: str, h: np.ndarray, limit: float) -> np.ndarray:
    g = np.minimum(h @ tensors[base + "gate"].T, limit)
    u = np.clip(h @ tensors[base + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ tensors[base + "down"].T


def route(tensors, base: str, mlp: dict, h: np.ndarray):
    """(chosen [tokens, top], weights [tokens, top]): sigmoid scores plus the correction choose, the scores weigh."""
    scores = sigmoid(h @ tensors[base + "router"].T)
    chosen = np.argsort(-(scores + tensors[base + "correction"]), axis=-1, kind="stable")[:, :int(mlp["router"]["top"])]
    return chosen, np.take_along_axis(scores, chosen, axis=-1)


def mixture_of_experts(tensors, base: str, mlp: dict, h: np.ndarray) -> np.ndarray:
    chosen, weights = route(tensors, base, mlp, h)
    limit = float(mlp["expert"]["limit"])
    out = np.zeros((h.shape[0], tensors[base + "e0.down"].shape[0]), dtype=np.float64)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weights[t]):
            out[t] += w * clamped_expert(tensors, f"{base}e{int(e)}.", h[t:t + 1], limit)[0]
    return out


# ------------------------------------------------------------------------------- the model
def streams(config: dict, tensors: Dict[str, np.ndarray], tokens: Sequence[int]) -> List[np.ndarray]:
    """The stream after every block, [tokens, width] each."""
    eps = float(config["norm"]["eps"])
    x = embed(config, tensors, tokens)
    out, cached = [], {}
    for index, layer in enumerate(config["layers"]):
        base, mixer = f"l{index}.", layer["mixer"]
        if layer["type"] == "general_delta":
            mixed = general_delta(tensors, base + "mix.", mixer, x, eps)
        elif layer["type"] == "attention":
            source = mixer.get("kv_from")
            if source is None:
                cached[index] = keys_and_values(tensors, base + "mix.", mixer, x, eps)
                source = index
            mixed = attention(tensors, base + "mix.", mixer, x, *cached[source], eps)
        else:
            raise ValueError(layer["type"])
        x = x + offset_norm(mixed, tensors[base + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + offset_norm(mixture_of_experts(tensors, base + "mlp.", layer["mlp"], x), tensors[base + "norm2"], eps)
        out.append(x)
    return out


def logits(config: dict, tensors: Dict[str, np.ndarray], tokens: Sequence[int]) -> np.ndarray:
    x = streams(config, tensors, tokens)[-1]
    return offset_norm(x, tensors["final.norm"], float(config["norm"]["eps"])) @ tensors["head"].T
