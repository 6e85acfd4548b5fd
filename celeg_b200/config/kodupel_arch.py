"""The Kodupel design as an arrangement of parts.

Token rows are embedding rows times a constant. A block norms what its sublayers put out (``output_norm_residual``):
x <- x + Norm(Mixer(x)), x <- x + Norm(FeedForward(x)), the norm an RMSNorm whose stored weight lies around zero
(``rmsnorm`` with ``weight_offset`` 1). Mixers: ``general_delta`` (a matrix state per head, a decay and a removal rate per
key channel) and ``prepared_attention`` (biases on all four projections, an RMS norm per query and key head, rotation of
neighbouring pairs with YaRN frequencies, values of unit root mean square, a one in the softmax's denominator, a sigmoid
gate per head; layers that read another layer's keys and values own no cache: the run order names whose they read).
Feed-forward: ``moe`` with clamped gated experts (``clamped_silu``), sigmoid scores that choose with a stored correction
and weigh without it, not renormalised. Output: the same kind of norm, an untied head.

Tensor names: ``embed``, ``final.norm``, ``head``; layer i: ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
``l<i>.mlp.*``; a bias is its matrix's name plus ``.b``.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Mapping

from .errors import ConfigError
from .kodupel import GENERAL_DELTA, KodupelConfig, KodupelExperts, KodupelLayer
from .registry import Architecture, register_architecture
from .spec import ExecutionEntry, LayerSpec, ModelSpec, PartSpec, TensorRef

GATE_SLOPE = 1.702          # an expert's inner rows: g sigmoid(GATE_SLOPE g) (u + UP_SHIFT)
UP_SHIFT = 1.0


def _offset_norm(name: str, width: int, eps: float) -> PartSpec:
    return PartSpec(kind="rmsnorm", params={"width": width, "eps": eps, "weight_offset": 1.0},
                    tensors={"weight": TensorRef(name, (width,))})


def _mixer(layer: KodupelLayer, base: str, width: int, eps: float) -> PartSpec:
    mix = base + ".mix."
    if layer.type == GENERAL_DELTA:
        inner, rank = layer.heads * layer.dim, layer.decay_rank
        if rank < 1:
            raise ConfigError(f"{base}: the rank of the decay's projection is unknown (the checkpoint gives it as the rows of "
                              f"{mix}w1; a configuration without one names it under 'mixer.decay_rank')")
        tensors = {name: TensorRef(mix + key, (inner, width))
                   for name, key in (("r", "r"), ("k", "k"), ("v", "v"), ("gate", "g"), ("removal", "a"))}
        tensors.update({"removal_bias": TensorRef(mix + "a.b", (inner,)), "decay_down": TensorRef(mix + "w1", (rank, width)),
                        "decay_up": TensorRef(mix + "w2", (inner, rank)), "decay_bias": TensorRef(mix + "w0", (inner,)),
                        "norm": TensorRef(mix + "norm", (inner,)), "out": TensorRef(mix + "o", (width, inner))})
        return PartSpec(kind="general_delta", params={"hidden_size": width, "heads": layer.heads, "dim": layer.dim, "eps": eps},
                        tensors=tensors)
    q_width, k_width, v_width = layer.heads * layer.dim, layer.kv_heads * layer.dim, layer.kv_heads * layer.vdim
    o_width = layer.heads * layer.vdim
    params = {"hidden_size": width, "heads": layer.heads, "kv_heads": layer.kv_heads, "dim": layer.dim, "vdim": layer.vdim,
              "scale": layer.scale, "eps": eps, "head_qk_norm": True, "unit_values": True, "one_in_denominator": True,
              "output_gate": "head", "reads_cache_only": layer.kv_from is not None}
    tensors = {"q": TensorRef(mix + "q", (q_width, width)), "q_bias": TensorRef(mix + "q.b", (q_width,)),
               "q_norm": TensorRef(mix + "q.norm", (layer.dim,)), "gate": TensorRef(mix + "g", (layer.heads, width)),
               "out": TensorRef(mix + "o", (width, o_width)), "out_bias": TensorRef(mix + "o.b", (width,))}
    if layer.kv_from is None:
        tensors.update({"k": TensorRef(mix + "k", (k_width, width)), "k_bias": TensorRef(mix + "k.b", (k_width,)),
                        "k_norm": TensorRef(mix + "k.norm", (layer.dim,)),
                        "v": TensorRef(mix + "v", (v_width, width)), "v_bias": TensorRef(mix + "v.b", (v_width,))})
    parts = {}
    if layer.rotary is not None:
        scaling = layer.rotary.scaling
        parts["position"] = PartSpec(kind="rope_interleaved", params={
            "theta": layer.rotary.base, "rotary_dim": layer.rotary.dims, "head_dim": layer.dim,
            "yarn": None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))})
    return PartSpec(kind="prepared_attention", params=params, tensors=tensors, parts=parts)


def _feed_forward(mlp: KodupelExperts, base: str, width: int) -> PartSpec:
    name = base + ".mlp."
    tensors = {"router": TensorRef(name + "router", (mlp.experts, width)),
               "correction": TensorRef(name + "correction", (mlp.experts,))}
    for expert in range(mlp.experts):
        tensors[f"e{expert}.gate"] = TensorRef(f"{name}e{expert}.gate", (mlp.ff, width))
        tensors[f"e{expert}.up"] = TensorRef(f"{name}e{expert}.up", (mlp.ff, width))
        tensors[f"e{expert}.down"] = TensorRef(f"{name}e{expert}.down", (width, mlp.ff))
    return PartSpec(kind="moe", params={"hidden_size": width, "intermediate_size": mlp.ff, "experts": mlp.experts,
                                        "top": mlp.top, "activation": "clamped_silu", "gated_experts": True,
                                        "gate_limit": mlp.limit, "gate_slope": GATE_SLOPE, "up_shift": UP_SHIFT,
                                        "scores": "sigmoid", "renormalize": False}, tensors=tensors)


def build_kodupel_spec(config: KodupelConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    layers = []
    for index, layer in enumerate(config.layers):
        base = f"l{index}"
        has_ff = layer.mlp is not None
        layers.append(LayerSpec(name=base, arrangement="output_norm_residual",
                                mixer_norm=_offset_norm(base + ".norm1", width, eps),
                                mixer=_mixer(layer, base, width, eps),
                                feed_forward_norm=_offset_norm(base + ".norm2", width, eps) if has_ff else None,
                                feed_forward=_feed_forward(layer.mlp, base, width) if has_ff else None))
    spec = ModelSpec(
        architecture=config.model_type, vocab_size=config.vocab, hidden_size=width, max_context=config.max_context,
        embedding=TensorRef("embed", (config.vocab, width)), layers=tuple(layers),
        order=tuple(ExecutionEntry(layer=index, cache_of=layer.kv_from) for index, layer in enumerate(config.layers)),
        final_norm=_offset_norm("final.norm", width, eps), lm_head=TensorRef("head", (config.vocab, width)),
        eos_token_ids=tuple(config.eos_token_ids), bos_token_id=config.bos_token_id,
        embedding_multiplier=config.embedding_scale)
    spec.validate()
    return spec


def kodupel_random_init(config: KodupelConfig, name: str, shape: tuple) -> str:
    """Distribution of a tensor in random-weights mode: matrices N(0, 1/fan-in), the blocks' stored norm weights, biases
    and corrections small around zero, the mixers' plain norm weights around 1, the decay's bias N(0, 0.3)."""
    leaf = name.rsplit(".", 1)[-1]
    if leaf == "norm" and ".mix." in name:
        return "norm"
    if leaf == "w0":
        return "small"
    return "tiny" if len(shape) == 1 else "fan_in"


def _parse(raw: Mapping[str, Any]) -> KodupelConfig:
    return KodupelConfig.from_dict(raw)


def _resolve(config: KodupelConfig, tensor_shapes: Mapping[str, Any]) -> KodupelConfig:
    """The rank of a general_delta layer's decay projection is the row count of its stored first matrix."""
    layers = []
    for index, layer in enumerate(config.layers):
        shape = tensor_shapes.get(f"l{index}.mix.w1")
        if layer.type == GENERAL_DELTA and shape is not None:
            if len(shape) != 2:
                raise ConfigError(f"l{index}.mix.w1 has shape {tuple(shape)}, expected (rank, {config.width})")
            layer = dataclasses.replace(layer, decay_rank=int(shape[0]))
        layers.append(layer)
    return dataclasses.replace(config, layers=tuple(layers))


KODUPEL = Architecture(name="Kodupel", parse_config=_parse, resolve_config=_resolve,
                       build_spec=build_kodupel_spec, random_init=kodupel_random_init)
register_architecture(KODUPEL, replace=True)
