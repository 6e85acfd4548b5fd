"""Small Kodupel configurations with weights of the tests' own making, written as model folders.

The sizes differ from one configuration to the next in every respect that the design leaves open (widths, head counts,
key and value sizes, ranks of the decay, rotated dimensions with and without stretched frequencies, which layers share
keys and values, numbers of experts and choices, limits, layers without a feed-forward, which mixer comes first). Weights
come from a numpy generator and are rounded to bfloat16, so the float64 plain model and the engine read the same numbers.
A few columns of the embedding hold large signs that sublayers leave alone, and the routers read mostly those: which
experts a token takes hangs on what token it is, and few choices are close calls that bfloat16's rounding could turn.
"""
from __future__ import annotations

import copy
import json
import math
import os
from typing import Dict, Optional

import numpy as np
import torch


def delta(heads, dim, rank):
    """``rank`` is the tests' own entry: the reader takes it from the tensors' shapes."""
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "rank": rank}


def rotation(base, dims, factor=None, original=64, fast=4.0, slow=0.5):
    out = {"base": base, "dims": dims}
    if factor is not None:
        out["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return out


def attention(heads, kv_heads, dim, vdim, rot=None, scale=None, kv_from=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if rot is not None:
        mixer["rot"] = rot
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer}


def moe(experts, top, ff, limit=1.25):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def with_mlp(layer, mlp):
    layer = copy.deepcopy(layer)
    layer["mlp"] = mlp
    return layer


def config(vocab, width, layers, eps=1e-5, scale=None):
    return {"architecture": "Kodupel", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": math.sqrt(width) if scale is None else scale}, "layers": layers}


# both mixers, keys of 16 with values of 32 (stored at one size on the bfloat16 path) and keys of 24 with values of 8, two
# layers that read an earlier layer's keys and values (one right behind it, one behind another layer that owns some)
STRETCHED = rotation(10000.0, 8, factor=4.0)
MIXED = config(160, 64, [
    with_mlp(attention(4, 2, 16, 32, STRETCHED), moe(8, 3, 32)),
    with_mlp(delta(2, 16, 12), moe(6, 1, 40, limit=0.7)),
    with_mlp(attention(4, 2, 16, 32, STRETCHED, scale=0.4, kv_from=0), moe(5, 2, 24, limit=2.5)),
    with_mlp(attention(6, 3, 24, 8, rotation(500.0, 24), scale=0.3), None),
    with_mlp(delta(3, 24, 8), moe(12, 4, 16)),
    with_mlp(attention(6, 3, 24, 8, rotation(500.0, 24), kv_from=3), moe(4, 2, 48)),
    with_mlp(attention(4, 2, 16, 32, STRETCHED, kv_from=0), None),
])

# sizes that fit no vector width: a width of 36, seventeen query heads on one key head (more than the split-key kernel
# groups), keys of 12 and values of 7, three rotated pairs, a rank of 5, head sizes of 20 and 7 in the recurrence, five
# experts all chosen, forty experts (more than a warp), an attention without any rotation
ODD = config(50, 36, [
    with_mlp(delta(3, 7, 5), moe(5, 5, 20, limit=0.9)),
    with_mlp(attention(17, 1, 12, 7, rotation(77.0, 6, factor=3.0, original=40, fast=6.0, slow=1.0)), None),
    with_mlp(delta(1, 20, 1), moe(40, 3, 8)),
    with_mlp(attention(17, 1, 12, 7, rotation(77.0, 6, factor=3.0, original=40, fast=6.0, slow=1.0), scale=0.5, kv_from=1),
             moe(3, 2, 12)),
    with_mlp(attention(2, 2, 10, 10), moe(7, 2, 28, limit=3.0)),
], eps=1e-6, scale=2.0)

# heads of 64 and of 128 (the tensor-core kernels' sizes), 136 in the recurrence (several lanes a column), a grouping of
# eight and of one, all dimensions rotated
WIDE = config(200, 128, [
    with_mlp(attention(8, 1, 64, 128, rotation(1e6, 64, factor=2.0, original=512), scale=0.11), moe(6, 2, 72)),
    with_mlp(delta(2, 136, 40), moe(12, 4, 48)),
    with_mlp(attention(3, 3, 64, 64, rotation(20000.0, 32)), moe(9, 3, 64, limit=1.75)),
    with_mlp(attention(3, 3, 64, 64, rotation(20000.0, 32), scale=0.2, kv_from=2), moe(4, 1, 96)),
    with_mlp(delta(3, 64, 24), None),
    with_mlp(attention(8, 1, 64, 128, rotation(1e6, 64, factor=2.0, original=512), kv_from=0), moe(8, 8, 24)),
])

CONFIGS = {"mixed": (MIXED, 11), "odd": (ODD, 15), "wide": (WIDE, 13)}


TAGS = 8                     # columns of the embedding that the routers read
TAG = 3.0                    # their size in the stream


def single_layer(layer, mlp=None, vocab=96, width=48, scale=None):
    """A model of one layer, to look at one mechanism alone."""
    return config(vocab, width, [with_mlp(layer, mlp)], scale=scale)


def _round(values: np.ndarray) -> torch.Tensor:
    return torch.from_numpy(np.asarray(values, dtype=np.float32)).to(torch.bfloat16)


def make_tensors(raw: dict, seed: int) -> Dict[str, torch.Tensor]:
    rng = np.random.default_rng(seed)
    width, vocab = raw["width"], raw["vocab"]
    out: Dict[str, torch.Tensor] = {}

    def matrix(name, rows, cols, gain=1.0):
        out[name] = _round(rng.normal(0.0, gain / math.sqrt(cols), size=(rows, cols)))

    def vector(name, size, mean=0.0, std=0.3):
        out[name] = _round(rng.normal(mean, std, size=(size,)))

    def block_norm(name):
        values = rng.normal(0.0, 0.2, size=(width,))
        values[:TAGS] = -1.0
        out[name] = _round(values)

    table = rng.normal(0.0, 1.0 / math.sqrt(width), size=(vocab, width))
    table[:, :TAGS] = rng.choice([-1.0, 1.0], size=(vocab, TAGS)) * TAG / raw["embedding"]["scale"]
    out["embed"] = _round(table)
    for index, layer in enumerate(raw["layers"]):
        base = f"l{index}."
        mix, m = base + "mix.", layer["mixer"]
        block_norm(base + "norm1")
        heads, dim = m["heads"], m["dim"]
        if layer["type"] == "general_delta":
            inner, rank = heads * dim, layer["rank"]
            for name in ("r", "k", "v", "g", "a"):
                matrix(mix + name, inner, width)
            vector(mix + "a.b", inner, 0.0, 1.0)
            matrix(mix + "w1", rank, width)
            matrix(mix + "w2", inner, rank, gain=2.0)
            # decays from about 0.6 (a channel that forgets at once) to about 0.999
            out[mix + "w0"] = _round(rng.uniform(-6.0, 2.0, size=(inner,)))
            vector(mix + "norm", inner, 1.0, 0.2)
            matrix(mix + "o", width, inner)
        else:
            groups, vdim = m["kv_heads"], m["vdim"]
            own = m.get("kv_from") is None
            for name, rows in (("q", heads * dim), ("k", groups * dim), ("v", groups * vdim)):
                if name == "q" or own:
                    matrix(mix + name, rows, width)
                    vector(mix + name + ".b", rows)
                    if name != "v":
                        vector(mix + name + ".norm", dim, 1.2, 0.3)
            matrix(mix + "g", heads, width, gain=1.5)
            matrix(mix + "o", width, heads * vdim)
            vector(mix + "o.b", width)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        block_norm(base + "norm2")
        name, experts, ff = base + "mlp.", mlp["router"]["experts"], mlp["expert"]["ff"]
        router = rng.normal(0.0, 0.03 / math.sqrt(width), size=(experts, width))
        router[:, :TAGS] = rng.normal(0.0, 1.5 / (TAG * math.sqrt(TAGS)), size=(experts, TAGS))
        out[name + "router"] = _round(router)
        vector(name + "correction", experts, 0.0, 0.2)
        for e in range(experts):
            matrix(f"{name}e{e}.gate", ff, width, gain=1.5)        # (gates and ups beyond the limit on both sides)
            matrix(f"{name}e{e}.up", ff, width, gain=1.5)
            matrix(f"{name}e{e}.down", width, ff)
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
