"""The Fovezen design as an arrangement of parts.

The model carries several residual streams (``hyper_residual`` blocks): a sublayer reads a weighted sum of them behind an
RMSNorm whose stored weight lies around zero (``rmsnorm`` with ``weight_offset`` 1), and its output enters all of them while
they are mixed (a ``connection`` of kind ``hyper`` a sublayer). Mixers: ``mamba2`` (a matrix state per head with one decay a
token and head), ``prepared_attention`` (norms over the whole q and k projections, rotated halves with frequencies scaled by
wavelength) and ``side_by_side`` of ``prepared_attention`` (short convolutions, norms a head, capped scores, a sliding
window) and ``gated_linear_attention`` (a decay a key channel), half the sum of their normed outputs. Feed-forward:
``swiglu`` with clamped gate and up values. A run of layers may repeat with the same weights: the run order names them
again, with caches of their own each time. Output: the same kind of norm over the sum of the streams, an untied head, a
factor on the logits.

Tensor names: ``embed``, ``final.norm``, ``head``; layer i: ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``l<i>.hc1.*`` and ``l<i>.hc2.*`` (``in``, ``out``, ``mix`` [from, to]); a bias is its matrix's name plus ``.b``.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Mapping

from .errors import ConfigError
from .fovezen import ATTENTION, MAMBA2, PARALLEL, FovezenConfig, FovezenFeedForward, FovezenLayer, SoftmaxConfig
from .registry import Architecture, register_architecture
from .spec import ExecutionEntry, LayerSpec, ModelSpec, PartSpec, TensorRef

GATE_SLOPE = 1.702          # the feed-forward's inner rows: g sigmoid(GATE_SLOPE g) (u + UP_SHIFT)
UP_SHIFT = 1.0
PARALLEL_SCALE = 0.5        # of the sum of a parallel mixer's two normed outputs


def _offset_norm(name: str, width: int, eps: float) -> PartSpec:
    return PartSpec(kind="rmsnorm", params={"width": width, "eps": eps, "weight_offset": 1.0},
                    tensors={"weight": TensorRef(name, (width,))})


def _softmax(attention: SoftmaxConfig, at: str, width: int, eps: float, head_norms: bool) -> PartSpec:
    q_width, k_width = attention.heads * attention.dim, attention.kv_heads * attention.dim
    v_width = attention.kv_heads * attention.vdim
    norm_sizes = (attention.dim, attention.dim) if head_norms else (q_width, k_width)
    tensors = {"q": TensorRef(at + "q", (q_width, width)), "k": TensorRef(at + "k", (k_width, width)),
               "v": TensorRef(at + "v", (v_width, width)), "q_norm": TensorRef(at + "q.norm", (norm_sizes[0],)),
               "k_norm": TensorRef(at + "k.norm", (norm_sizes[1],)),
               "out": TensorRef(at + "o", (width, attention.heads * attention.vdim))}
    if attention.taps is not None:
        for name, rows in (("q", q_width), ("k", k_width), ("v", v_width)):
            tensors[name + "_conv"] = TensorRef(at + name + ".conv", (rows, attention.taps))
    parts = {}
    if attention.rotary is not None:
        scaling = attention.rotary.scaling
        parts["position"] = PartSpec(kind="rope_split_half", params={
            "theta": attention.rotary.base, "rotary_dim": attention.rotary.dims, "head_dim": attention.dim,
            "wavelength_scaling": None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))})
    return PartSpec(kind="prepared_attention", category="mixer",
                    params={"hidden_size": width, "heads": attention.heads, "kv_heads": attention.kv_heads,
                            "dim": attention.dim, "vdim": attention.vdim, "scale": attention.scale, "eps": eps,
                            "head_qk_norm": head_norms, "whole_qk_norm": not head_norms, "window": attention.window,
                            "softcap": attention.softcap, "taps": attention.taps},
                    tensors=tensors, parts=parts)


def _mixer(layer: FovezenLayer, base: str, width: int, eps: float) -> PartSpec:
    mix = base + ".mix."
    if layer.type == MAMBA2:
        m = layer.state_space
        inner, shared = m.heads * m.vdim, m.groups * m.state
        channels = inner + 2 * shared
        return PartSpec(
            kind="mamba2",
            params={"hidden_size": width, "heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups,
                    "taps": m.taps, "norm_groups": m.norm_groups, "eps": eps},
            tensors={"in_proj": TensorRef(mix + "in", (inner + channels + m.heads, width)),
                     "conv": TensorRef(mix + "conv", (channels, m.taps)), "conv_bias": TensorRef(mix + "conv.b", (channels,)),
                     "dt_bias": TensorRef(mix + "dt_bias", (m.heads,)), "a_log": TensorRef(mix + "A_log", (m.heads,)),
                     "direct": TensorRef(mix + "D", (m.heads,)), "norm": TensorRef(mix + "norm", (inner,)),
                     "out": TensorRef(mix + "o", (width, inner))})
    if layer.type == ATTENTION:
        return _softmax(layer.softmax, mix, width, eps, head_norms=False)
    assert layer.type == PARALLEL
    linear, at = layer.linear, mix + "right."
    qk_width, v_width, rank = linear.heads * linear.dim, linear.heads * linear.vdim, linear.decay_rank
    if rank < 1:
        raise ConfigError(f"{base}: the rank of the decay's projection is unknown (the checkpoint gives it as the rows of "
                          f"{at}a1; a configuration without one names it under 'mixer.right.decay_rank')")
    right = PartSpec(
        kind="gated_linear_attention", category="mixer",
        params={"hidden_size": width, "heads": linear.heads, "dim": linear.dim, "vdim": linear.vdim, "tau": linear.tau,
                "eps": eps},
        tensors={"q": TensorRef(at + "q", (qk_width, width)), "k": TensorRef(at + "k", (qk_width, width)),
                 "v": TensorRef(at + "v", (v_width, width)), "gate": TensorRef(at + "g", (v_width, width)),
                 "decay_down": TensorRef(at + "a1", (rank, width)), "decay_up": TensorRef(at + "a2", (qk_width, rank)),
                 "decay_bias": TensorRef(at + "a2.b", (qk_width,)), "norm": TensorRef(at + "norm", (linear.vdim,)),
                 "out": TensorRef(at + "o", (width, v_width))})
    return PartSpec(kind="side_by_side",
                    params={"hidden_size": width, "left_scale": PARALLEL_SCALE, "right_scale": PARALLEL_SCALE, "eps": eps},
                    tensors={"left_norm": TensorRef(mix + "left.out", (width,)), "right_norm": TensorRef(mix + "right.out", (width,))},
                    parts={"left": _softmax(layer.softmax, mix + "left.", width, eps, head_norms=True), "right": right})


def _feed_forward(mlp: FovezenFeedForward, base: str, width: int) -> PartSpec:
    name = base + ".mlp."
    return PartSpec(kind="swiglu", params={"hidden_size": width, "intermediate_size": mlp.ff, "activation": "clamped_silu",
                                           "gate_limit": mlp.limit, "gate_slope": GATE_SLOPE, "up_shift": UP_SHIFT},
                    tensors={"gate": TensorRef(name + "gate", (mlp.ff, width)), "up": TensorRef(name + "up", (mlp.ff, width)),
                             "down": TensorRef(name + "down", (width, mlp.ff))})


def _connection(name: str, streams: int, width: int) -> PartSpec:
    return PartSpec(kind="hyper", category="connection", params={"streams": streams, "width": width},
                    tensors={"take": TensorRef(name + ".in", (streams,)), "give": TensorRef(name + ".out", (streams,)),
                             "mix": TensorRef(name + ".mix", (streams, streams))})


def build_fovezen_spec(config: FovezenConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    layers = []
    for index, layer in enumerate(config.layers):
        base = f"l{index}"
        has_ff = layer.mlp is not None
        connections = {"mixer_connection": _connection(base + ".hc1", config.streams, width)}
        if has_ff:
            connections["feed_forward_connection"] = _connection(base + ".hc2", config.streams, width)
        layers.append(LayerSpec(name=base, arrangement="hyper_residual",
                                mixer_norm=_offset_norm(base + ".norm1", width, eps),
                                mixer=_mixer(layer, base, width, eps),
                                feed_forward_norm=_offset_norm(base + ".norm2", width, eps) if has_ff else None,
                                feed_forward=_feed_forward(layer.mlp, base, width) if has_ff else None,
                                extra_parts=connections))
    spec = ModelSpec(
        architecture=config.model_type, vocab_size=config.vocab, hidden_size=width, max_context=config.max_context,
        embedding=TensorRef("embed", (config.vocab, width)), layers=tuple(layers),
        order=tuple(ExecutionEntry(layer=index) for index in config.run_order()),
        final_norm=_offset_norm("final.norm", width, eps), lm_head=TensorRef("head", (config.vocab, width)),
        eos_token_ids=tuple(config.eos_token_ids), bos_token_id=config.bos_token_id, logits_multiplier=config.logit_scale)
    spec.validate()
    return spec


def fovezen_random_init(config: FovezenConfig, name: str, shape: tuple) -> str:
    """Distribution of a tensor in random-weights mode: matrices N(0, 1/fan-in) (the connections' mixes and weights of what
    a sublayer reads among them), the blocks' stored norm weights and biases small around zero, the mixers' plain norm
    weights and direct shares around 1, taps N(0, 0.5), decay and step parameters N(0, 0.3)."""
    leaf = name.rsplit(".", 1)[-1]
    connection = ".hc1." in name or ".hc2." in name
    if leaf == "conv":
        return "taps"
    if leaf in ("A_log", "dt_bias"):
        return "small"
    if connection:
        return "depth" if leaf == "out" else "fan_in"
    if ".mix." in name and (leaf in ("norm", "D", "out")):
        return "norm"
    return "tiny" if len(shape) == 1 else "fan_in"


def _parse(raw: Mapping[str, Any]) -> FovezenConfig:
    return FovezenConfig.from_dict(raw)


def _resolve(config: FovezenConfig, tensor_shapes: Mapping[str, Any]) -> FovezenConfig:
    """The rank of the decay's projection is the row count of its stored first matrix."""
    layers = []
    for index, layer in enumerate(config.layers):
        name = f"l{index}.mix.right.a1"
        shape = tensor_shapes.get(name)
        if layer.type == PARALLEL and shape is not None:
            if len(shape) != 2:
                raise ConfigError(f"{name} has shape {tuple(shape)}, expected (rank, {config.width})")
            layer = dataclasses.replace(layer, linear=dataclasses.replace(layer.linear, decay_rank=int(shape[0])))
        layers.append(layer)
    return dataclasses.replace(config, layers=tuple(layers))


FOVEZEN = Architecture(name="Fovezen", parse_config=_parse, resolve_config=_resolve,
                       build_spec=build_fovezen_spec, random_init=fovezen_random_init)
register_architecture(FOVEZEN, replace=True)
