"""Typed configuration of the Kodupel design, read from config.json (``"architecture": "Kodupel"``).

Keys: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``layers`` (a list; each entry has ``type`` =
general_delta | attention, the mixer's sizes and constants under ``mixer``, and ``mlp`` = {kind: moe, router: {experts,
top}, expert: {ff, limit}} | null). general_delta: ``heads``, ``dim``. attention: ``heads``, ``kv_heads`` (absent: as many
as heads), ``dim``, ``vdim`` (absent: as wide as keys), ``scale`` (absent: 1 / sqrt(dim)), ``rot`` = {base, dims, scaling:
{factor, original, fast, slow} or absent} or absent, ``kv_from`` (absent: the layer projects keys and values of its own;
else the index of an earlier attention layer whose keys and values it reads). Every size and every constant that can
differ between two models of the design comes from here, or from a tensor's shape where config.json is silent (the rank
of the decay's projection; a model yet to be written names it under ``mixer.decay_rank``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .kedesun import YarnRotaryConfig
from .liverax import _positive_int
from .ramosun import DEFAULT_MAX_CONTEXT, _need

GENERAL_DELTA, ATTENTION = "general_delta", "attention"
LAYER_TYPES = (GENERAL_DELTA, ATTENTION)
MOE = "moe"


@dataclass(frozen=True)
class KodupelExperts:
    experts: int
    top: int
    ff: int                                  # an expert's inner size
    limit: float                             # where gate and up are cut off

    @staticmethod
    def from_dict(raw: Mapping[str, Any], where: str) -> "KodupelExperts":
        kind = _need(raw, "kind", where)
        if kind != MOE:
            raise ConfigError(f"{where}: unknown kind {kind!r}; known: {MOE}")
        router, expert = _need(raw, "router", where), _need(raw, "expert", where)
        experts, top = _positive_int(router, "experts", where + ".router"), _positive_int(router, "top", where + ".router")
        if top > experts:
            raise ConfigError(f"{where}.router: top {top} exceeds the {experts} experts")
        limit = float(_need(expert, "limit", where + ".expert"))
        if limit <= 0:
            raise ConfigError(f"{where}.expert: a limit of {limit}")
        return KodupelExperts(experts=experts, top=top, ff=_positive_int(expert, "ff", where + ".expert"), limit=limit)

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": MOE, "router": {"experts": self.experts, "top": self.top},
                "expert": {"ff": self.ff, "limit": self.limit}}


@dataclass(frozen=True)
class KodupelLayer:
    type: str
    heads: int
    dim: int
    mlp: Optional[KodupelExperts] = None
    decay_rank: int = 0                            # general_delta; 0: not known yet
    kv_heads: int = 0                              # attention
    vdim: int = 0
    scale: float = 1.0
    rotary: Optional[YarnRotaryConfig] = None
    kv_from: Optional[int] = None

    @staticmethod
    def from_dict(raw: Mapping[str, Any], index: int) -> "KodupelLayer":
        where = f"layers[{index}]"
        kind = _need(raw, "type", where)
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}: unknown layer type {kind!r}; known: {', '.join(LAYER_TYPES)}")
        mixer, at = _need(raw, "mixer", where), where + ".mixer"
        mlp = raw.get("mlp")
        heads, dim = _positive_int(mixer, "heads", at), _positive_int(mixer, "dim", at)
        common = dict(type=kind, heads=heads, dim=dim,
                      mlp=None if mlp is None else KodupelExperts.from_dict(mlp, where + ".mlp"))
        if kind == GENERAL_DELTA:
            rank = _positive_int(mixer, "decay_rank", at) if mixer.get("decay_rank") is not None else 0
            return KodupelLayer(**common, decay_rank=rank)
        kv_heads = _positive_int(mixer, "kv_heads", at) if mixer.get("kv_heads") is not None else heads
        if heads % kv_heads:
            raise ConfigError(f"{at}: {heads} heads are not a multiple of {kv_heads} kv_heads")
        rot, kv_from = mixer.get("rot"), mixer.get("kv_from")
        if kv_from is not None:
            if isinstance(kv_from, bool) or int(kv_from) != kv_from or not 0 <= kv_from < index:
                raise ConfigError(f"{at}: 'kv_from' must name an earlier layer, got {kv_from!r}")
            kv_from = int(kv_from)
        return KodupelLayer(
            **common, kv_heads=kv_heads, vdim=_positive_int(mixer, "vdim", at) if mixer.get("vdim") is not None else dim,
            scale=float(mixer["scale"]) if mixer.get("scale") is not None else dim ** -0.5,
            rotary=None if rot is None else YarnRotaryConfig.from_dict(rot, dim, at + ".rot"), kv_from=kv_from)

    def to_dict(self) -> Dict[str, Any]:
        mixer: Dict[str, Any] = {"heads": self.heads, "dim": self.dim}
        if self.type == GENERAL_DELTA:
            if self.decay_rank:
                mixer["decay_rank"] = self.decay_rank
        else:
            mixer.update(kv_heads=self.kv_heads, vdim=self.vdim, scale=self.scale)
            if self.rotary is not None:
                mixer["rot"] = self.rotary.to_dict()
            if self.kv_from is not None:
                mixer["kv_from"] = self.kv_from
        return {"type": self.type, "mixer": mixer, "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class KodupelConfig:
    vocab: int
    width: int
    layers: Tuple[KodupelLayer, ...]
    norm_eps: float
    embedding_scale: float
    max_context: int = DEFAULT_MAX_CONTEXT
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    model_type: str = "Kodupel"

    @staticmethod
    def from_dict(raw: Mapping[str, Any]) -> "KodupelConfig":
        layers_raw = _need(raw, "layers", "config.json")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        eos = raw.get("eos_token_id")
        eos_ids = tuple(int(e) for e in eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
        context = raw.get("max_context")
        eps = float(_need(_need(raw, "norm", "config.json"), "eps", "norm"))
        if eps <= 0:
            raise ConfigError("norm.eps must be positive")
        layers = tuple(KodupelLayer.from_dict(layer, index) for index, layer in enumerate(layers_raw))
        for index, layer in enumerate(layers):
            if layer.kv_from is None:
                continue
            source = layers[layer.kv_from]
            if source.type != ATTENTION or source.kv_from is not None:
                raise ConfigError(f"layers[{index}].mixer: 'kv_from' {layer.kv_from} is no attention layer with keys and "
                                  f"values of its own")
            if (source.kv_heads, source.dim, source.vdim) != (layer.kv_heads, layer.dim, layer.vdim):
                raise ConfigError(f"layers[{index}].mixer: reads keys and values of {source.kv_heads} x {source.dim} / "
                                  f"{source.vdim}, its own sizes are {layer.kv_heads} x {layer.dim} / {layer.vdim}")
        return KodupelConfig(
            vocab=_positive_int(raw, "vocab", "config.json"), width=_positive_int(raw, "width", "config.json"),
            layers=layers, norm_eps=eps, embedding_scale=float(_need(_need(raw, "embedding", "config.json"), "scale", "embedding")),
            max_context=DEFAULT_MAX_CONTEXT if context is None else int(context), eos_token_ids=eos_ids,
            bos_token_id=None if raw.get("bos_token_id") is None else int(raw["bos_token_id"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.model_type, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": [layer.to_dict() for layer in self.layers],
                "max_context": self.max_context}


__all__ = ["ATTENTION", "GENERAL_DELTA", "MOE", "KodupelExperts", "KodupelLayer", "KodupelConfig"]
