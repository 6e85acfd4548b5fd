"""Small Fovezen configurations with weights of the tests' own making, written as model folders.

The sizes differ from one configuration to the next in every respect that the design leaves open (numbers of streams,
widths, head counts, key and value sizes, states, groups, norm groups, taps, ranks of the decay, windows, caps, rotated
dimensions with and without stretched frequencies, which layers repeat, layers without a feed-forward, which mixer comes
first). Weights come from a numpy generator and are rounded to bfloat16, so the float64 plain model and the engine read
the same numbers. They are made so that rounding stays rounding: no norm acts on what nearly vanishes, and the streams do
not cancel in their sum.
"""
from __future__ import annotations

import copy
import json
import math
import os
from typing import Dict, Optional

import numpy as np
import torch


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def rotation(base, dims, factor=None, low=1.0, high=4.0, original=64):
    out = {"base": base, "dims": dims}
    if factor is not None:
        out["scaling"] = {"factor": factor, "low": low, "high": high, "original": original}
    return out


def attention(heads, kv_heads, dim, vdim, rot, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot,
                                           "scale": dim ** -0.5 if scale is None else scale}}


def parallel(left, right):
    """left: (heads, kv_heads, dim, vdim, taps, window, softcap, scale); right: (heads, dim, vdim, tau, rank). The rank is
    the tests' own entry: the reader takes it from the tensors' shapes."""
    heads, kv_heads, dim, vdim, taps, window, softcap, scale = left
    r_heads, r_dim, r_vdim, tau, rank = right
    return {"type": "parallel", "rank": rank, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps, "mask": {"size": window},
                 "softcap": softcap, "scale": scale},
        "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "tau": tau}}}


def with_mlp(layer, ff, limit=1.25):
    layer = copy.deepcopy(layer)
    layer["mlp"] = None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}
    return layer


def config(vocab, width, layers, streams=3, eps=1e-5, logit_scale=1.0, loop=None):
    out = {"architecture": "Fovezen", "vocab": vocab, "width": width, "streams": streams, "logit_scale": logit_scale,
           "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# all three mixers, keys of 16 with values of 24 (stored at one size on the bfloat16 path), a loop over two layers, a
# window shorter than a page, two taps beside four
MIXED = config(160, 64, [
    with_mlp(parallel((4, 2, 16, 24, 4, 11, 5.0, 0.4), (2, 16, 24, 4.0, 12)), 96),
    with_mlp(mamba(4, 16, 24, 2, 2, 2), 80, limit=0.7),
    with_mlp(attention(4, 2, 16, 32, rotation(10000.0, 8, factor=4.0)), None),
    with_mlp(parallel((6, 3, 24, 8, 2, 40, 20.0, 0.3), (3, 24, 8, 1.0, 8)), 64, limit=2.5),
], streams=3, logit_scale=0.7, loop=(1, 3, 2))

# sizes that fit no vector width: a width of 36, seventeen query heads on one key head (more than the split-key kernel
# groups), keys of 12 and values of 7, states of 5 and heads of 7 and 9, five taps, one tap, a rank of 3, five streams
# (more than the product mixes), a window of one, layers that repeat right from the start
ODD = config(50, 36, [
    with_mlp(mamba(3, 7, 5, 1, 5, 3), 20, limit=0.9),
    with_mlp(parallel((17, 1, 12, 7, 3, 1, 2.0, 0.5), (3, 7, 9, 2.0, 3)), None),
    with_mlp(attention(17, 1, 12, 7, rotation(77.0, 6, factor=3.0, low=0.5, high=2.0, original=40), scale=0.5), 12, limit=3.0),
    with_mlp(mamba(2, 9, 6, 2, 1, 1), 28),
], streams=5, eps=1e-6, logit_scale=2.0, loop=(0, 2, 3))

# heads of 64 and of 128 (the tensor-core kernels' sizes), more than one tile of keys and values in the scans, one stream
# only, no loop
WIDE = config(200, 128, [
    with_mlp(mamba(4, 72, 136, 2, 4, 4), 72),
    with_mlp(parallel((8, 1, 64, 64, 4, 96, 30.0, 0.125), (2, 72, 136, 16.0, 40)), 96, limit=1.75),
    with_mlp(attention(3, 3, 128, 64, rotation(20000.0, 64, factor=8.0, original=256)), 64),
    with_mlp(parallel((4, 4, 64, 128, 4, 64, 8.0, 0.3), (1, 130, 20, 8.0, 16)), None),
], streams=1, logit_scale=0.5)

# four streams (the number that steps of few rows mix inside the products), sizes that every fused form takes
EVEN = config(96, 64, [
    with_mlp(mamba(4, 32, 16, 2, 4, 2), 64),
    with_mlp(attention(4, 2, 32, 32, rotation(500.0, 16)), 64, limit=0.5),
    with_mlp(parallel((4, 2, 32, 32, 4, 20, 10.0, 0.3), (2, 32, 32, 16.0, 8)), 64),
    with_mlp(mamba(2, 64, 32, 1, 3, 1), None),
], streams=4, loop=(1, 2, 2))

CONFIGS = {"mixed": (MIXED, 16), "odd": (ODD, 12), "wide": (WIDE, 13), "even": (EVEN, 20)}


def single_layer(layer, ff=None, vocab=96, width=48, streams=2, limit=1.25):
    """A model of one layer, to look at one mechanism alone."""
    return config(vocab, width, [with_mlp(layer, ff, limit)], streams=streams)


def _round(values: np.ndarray) -> torch.Tensor:
    return torch.from_numpy(np.asarray(values, dtype=np.float32)).to(torch.bfloat16)


def make_tensors(raw: dict, seed: int) -> Dict[str, torch.Tensor]:
    rng = np.random.default_rng(seed)
    width, vocab, streams = raw["width"], raw["vocab"], raw["streams"]
    out: Dict[str, torch.Tensor] = {}

    def matrix(name, rows, cols, gain=1.0):
        out[name] = _round(rng.normal(0.0, gain / math.sqrt(cols), size=(rows, cols)))

    def vector(name, size, mean=0.0, std=0.3):
        out[name] = _round(rng.normal(mean, std, size=(size,)))

    def connection(name):
        # every stream keeps most of itself and gets something of every other (more in one direction than back), and all
        # take an output with the same sign: the sum of the streams is no small difference of large numbers
        pull = rng.uniform(-0.1, 0.5, size=(streams, streams)) / max(streams - 1, 1)
        np.fill_diagonal(pull, rng.uniform(0.6, 0.9, size=streams))
        out[name + ".mix"] = _round(pull)
        out[name + ".in"] = _round(rng.uniform(0.2, 1.2, size=(streams,)))
        out[name + ".out"] = _round(rng.uniform(0.2, 0.9, size=(streams,)))

    def softmax(at, m, per_head):
        heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name, rows in (("q", heads * dim), ("k", groups * dim), ("v", groups * vdim)):
            matrix(at + name, rows, width)
            if name != "v":
                vector(at + name + ".norm", dim if per_head else rows, 1.2, 0.3)
            if per_head:
                out[at + name + ".conv"] = _round(rng.normal(0.0, 0.6, size=(rows, m["conv"])))
        matrix(at + "o", width, heads * vdim)

    out["embed"] = _round(rng.normal(0.0, 1.0, size=(vocab, width)))
    for index, layer in enumerate(raw["layers"]):
        base = f"l{index}."
        mix, m = base + "mix.", layer["mixer"]
        vector(base + "norm1", width, 0.0, 0.2)
        connection(base + "hc1")
        if layer["type"] == "mamba2":
            inner, shared = m["heads"] * m["vdim"], m["groups"] * m["state"]
            matrix(mix + "in", 2 * inner + 2 * shared + m["heads"], width)
            out[mix + "conv"] = _round(rng.normal(0.0, 0.6, size=(inner + 2 * shared, m["conv"])))
            vector(mix + "conv.b", inner + 2 * shared)
            # steps and rates so that decays range from almost one to almost nothing
            out[mix + "dt_bias"] = _round(rng.uniform(-4.0, 1.0, size=(m["heads"],)))
            out[mix + "A_log"] = _round(rng.uniform(-2.0, 1.5, size=(m["heads"],)))
            vector(mix + "D", m["heads"], 0.7, 0.4)
            vector(mix + "norm", inner, 1.0, 0.2)
            matrix(mix + "o", width, inner)
        elif layer["type"] == "attention":
            softmax(mix, m, per_head=False)
        else:
            softmax(mix + "left.", m["left"], per_head=True)
            at, r = mix + "right.", m["right"]
            qk, vw = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            for name, rows in (("q", qk), ("k", qk), ("v", vw), ("g", vw)):
                matrix(at + name, rows, width)
            # (a token's key looks like its query: the first tokens' read-outs, which are normed, are not close to nothing)
            out[at + "k"] = _round(0.95 * out[at + "q"].float().numpy() + 0.3 * out[at + "k"].float().numpy())
            matrix(at + "a1", layer["rank"], width)
            matrix(at + "a2", qk, layer["rank"], gain=1.5)
            out[at + "a2.b"] = _round(rng.uniform(-3.0, 5.0, size=(qk,)))
            vector(at + "norm", r["vdim"], 1.0, 0.2)
            matrix(at + "o", width, vw)
            vector(mix + "left.out", width, 1.0, 0.3)
            vector(mix + "right.out", width, 1.0, 0.3)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        vector(base + "norm2", width, 0.0, 0.2)
        connection(base + "hc2")
        name = base + "mlp."
        matrix(name + "gate", mlp["ff"], width, gain=1.5)          # (gates and ups beyond the limit on both sides)
        matrix(name + "up", mlp["ff"], width, gain=1.5)
        matrix(name + "down", width, mlp["ff"])
    vector("final.norm", width, 0.0, 0.2)
    matrix("head", vocab, width)
    return out


def stored(raw: dict) -> dict:
    """The configuration as a folder holds it: without the tests' own entry."""
    out = copy.deepcopy(raw)
    for layer in out["layers"]:
        layer.pop("rank", None)
    return out


def write_model(folder: str, raw: dict, seed: int, tensors: Optional[Dict[str, torch.Tensor]] = None):
    """Writes ``folder`` and returns (config, {name: bfloat16 tensor})."""
    from safetensors.torch import save_file
    tensors = tensors if tensors is not None else make_tensors(raw, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as handle:
        json.dump(stored(raw), handle, indent=1)
    save_file({name: value.contiguous() for name, value in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return raw, tensors
