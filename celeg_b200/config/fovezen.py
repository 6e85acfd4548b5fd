"""Typed configuration of the Fovezen design, read from config.json (``"architecture": "Fovezen"``).

Keys: ``vocab``, ``width``, ``norm.eps``, ``streams`` (how many residual streams; absent: one, with connections of its own
all the same), ``logit_scale`` (absent: 1), ``layers`` (a list; each entry has ``type`` = mamba2 | attention | parallel, the
mixer's sizes and constants under ``mixer``, and ``mlp`` = {kind: dense, ff, limit} | null), ``loop`` = {start, stop, times}
(absent: every layer runs once). mamba2: ``heads``, ``vdim``, ``state``, ``groups``, ``conv``, ``norm_groups``. attention:
``heads``, ``kv_heads`` (absent: as many as heads), ``dim``, ``vdim`` (absent: as wide as keys), ``scale`` (absent: 1 /
sqrt(dim)), ``rot`` = {base, dims, scaling: {factor, low, high, original} or absent} or absent. parallel: ``left`` = an
attention's keys without ``rot``, and ``conv``, ``softcap``, ``mask.size`` (absent: none of it), ``right`` = {heads, dim,
vdim, tau}. Every size and every constant that can differ between two models of the design comes from here, or from a
tensor's shape where config.json is silent (the rank of the decay's projection in ``right``; a model yet to be written
names it under ``right.decay_rank``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .liverax import _positive_int
from .ramosun import DEFAULT_MAX_CONTEXT, RotaryConfig, _need

MAMBA2, ATTENTION, PARALLEL = "mamba2", "attention", "parallel"
LAYER_TYPES = (MAMBA2, ATTENTION, PARALLEL)
MAX_TAPS, MAX_STREAMS = 16, 16


def _positive(mapping: Mapping[str, Any], key: str, where: str) -> float:
    value = float(_need(mapping, key, where))
    if not value > 0:
        raise ConfigError(f"{where}: '{key}' must be positive, got {value!r}")
    return value


def _taps(mapping: Mapping[str, Any], where: str) -> int:
    taps = _positive_int(mapping, "conv", where)
    if taps > MAX_TAPS:
        raise ConfigError(f"{where}: {taps} taps exceed {MAX_TAPS}")
    return taps


@dataclass(frozen=True)
class FovezenFeedForward:
    ff: int
    limit: float                             # where gate and up are cut off

    @staticmethod
    def from_dict(raw: Mapping[str, Any], where: str) -> "FovezenFeedForward":
        kind = _need(raw, "kind", where)
        if kind != "dense":
            raise ConfigError(f"{where}: unknown kind {kind!r}; known: dense")
        return FovezenFeedForward(ff=_positive_int(raw, "ff", where), limit=_positive(raw, "limit", where))

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    @staticmethod
    def from_dict(raw: Mapping[str, Any], where: str) -> "StateSpaceConfig":
        heads, vdim = _positive_int(raw, "heads", where), _positive_int(raw, "vdim", where)
        groups = _positive_int(raw, "groups", where) if raw.get("groups") is not None else 1
        if heads % groups:
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {groups} groups")
        norm_groups = _positive_int(raw, "norm_groups", where) if raw.get("norm_groups") is not None else 1
        if (heads * vdim) % norm_groups:
            raise ConfigError(f"{where}: {heads * vdim} channels are not a multiple of {norm_groups} norm_groups")
        return StateSpaceConfig(heads=heads, vdim=vdim, state=_positive_int(raw, "state", where), groups=groups,
                                taps=_taps(raw, where), norm_groups=norm_groups)

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.taps,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class SoftmaxConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[RotaryConfig] = None
    taps: Optional[int] = None               # None: no short convolutions
    softcap: Optional[float] = None
    window: Optional[int] = None             # None: every earlier position is visible

    @staticmethod
    def from_dict(raw: Mapping[str, Any], where: str, side: bool) -> "SoftmaxConfig":
        """``side``: the left half of a parallel mixer (convolutions, capped scores, a window, no rotation)."""
        heads, dim = _positive_int(raw, "heads", where), _positive_int(raw, "dim", where)
        kv_heads = _positive_int(raw, "kv_heads", where) if raw.get("kv_heads") is not None else heads
        if heads % kv_heads:
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
        vdim = _positive_int(raw, "vdim", where) if raw.get("vdim") is not None else dim
        scale = float(raw["scale"]) if raw.get("scale") is not None else dim ** -0.5
        fields: Dict[str, Any] = {}
        if side:
            fields["taps"] = _taps(raw, where) if raw.get("conv") is not None else None
            fields["softcap"] = _positive(raw, "softcap", where) if raw.get("softcap") is not None else None
            mask = raw.get("mask")
            fields["window"] = None if mask is None else _positive_int(mask, "size", where + ".mask")
        elif raw.get("rot") is not None:
            fields["rotary"] = RotaryConfig.from_dict(raw["rot"], dim, where + ".rot")
        return SoftmaxConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, **fields)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale}
        if self.rotary is not None:
            out["rot"] = self.rotary.to_dict()
        if self.taps is not None:
            out["conv"] = self.taps
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 0                      # 0: not known yet (the checkpoint's tensor gives it)

    @staticmethod
    def from_dict(raw: Mapping[str, Any], where: str) -> "GatedLinearConfig":
        return GatedLinearConfig(
            heads=_positive_int(raw, "heads", where), dim=_positive_int(raw, "dim", where),
            vdim=_positive_int(raw, "vdim", where) if raw.get("vdim") is not None else _positive_int(raw, "dim", where),
            tau=_positive(raw, "tau", where),
            decay_rank=_positive_int(raw, "decay_rank", where) if raw.get("decay_rank") is not None else 0)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}
        if self.decay_rank:
            out["decay_rank"] = self.decay_rank
        return out


@dataclass(frozen=True)
class FovezenLayer:
    type: str
    mlp: Optional[FovezenFeedForward] = None
    state_space: Optional[StateSpaceConfig] = None     # mamba2
    softmax: Optional[SoftmaxConfig] = None            # attention; the left half of parallel
    linear: Optional[GatedLinearConfig] = None         # the right half of parallel

    @staticmethod
    def from_dict(raw: Mapping[str, Any], index: int) -> "FovezenLayer":
        where = f"layers[{index}]"
        kind = _need(raw, "type", where)
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}: unknown layer type {kind!r}; known: {', '.join(LAYER_TYPES)}")
        mixer, at = _need(raw, "mixer", where), where + ".mixer"
        mlp = raw.get("mlp")
        mlp = None if mlp is None else FovezenFeedForward.from_dict(mlp, where + ".mlp")
        if kind == MAMBA2:
            return FovezenLayer(type=kind, mlp=mlp, state_space=StateSpaceConfig.from_dict(mixer, at))
        if kind == ATTENTION:
            return FovezenLayer(type=kind, mlp=mlp, softmax=SoftmaxConfig.from_dict(mixer, at, side=False))
        return FovezenLayer(type=kind, mlp=mlp,
                            softmax=SoftmaxConfig.from_dict(_need(mixer, "left", at), at + ".left", side=True),
                            linear=GatedLinearConfig.from_dict(_need(mixer, "right", at), at + ".right"))

    def to_dict(self) -> Dict[str, Any]:
        if self.type == MAMBA2:
            mixer = self.state_space.to_dict()
        elif self.type == ATTENTION:
            mixer = self.softmax.to_dict()
        else:
            mixer = {"left": self.softmax.to_dict(), "right": self.linear.to_dict()}
        return {"type": self.type, "mixer": mixer, "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class FovezenConfig:
    vocab: int
    width: int
    layers: Tuple[FovezenLayer, ...]
    norm_eps: float
    streams: int = 1
    logit_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None       # start, stop, times
    max_context: int = DEFAULT_MAX_CONTEXT
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    model_type: str = "Fovezen"

    @staticmethod
    def from_dict(raw: Mapping[str, Any]) -> "FovezenConfig":
        layers_raw = _need(raw, "layers", "config.json")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = tuple(FovezenLayer.from_dict(layer, index) for index, layer in enumerate(layers_raw))
        loop = raw.get("loop")
        if loop is not None:
            start, stop, times = (int(_need(loop, key, "loop")) for key in ("start", "stop", "times"))
            if not (0 <= start < stop <= len(layers)) or times < 1:
                raise ConfigError(f"loop: start {start}, stop {stop}, times {times} do not name a run of the "
                                  f"{len(layers)} layers that runs at least once")
            loop = (start, stop, times)
        streams = _positive_int(raw, "streams", "config.json") if raw.get("streams") is not None else 1
        if streams > MAX_STREAMS:
            raise ConfigError(f"config.json: {streams} streams exceed {MAX_STREAMS}")
        eos = raw.get("eos_token_id")
        eos_ids = tuple(int(e) for e in eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
        context = raw.get("max_context")
        return FovezenConfig(
            vocab=_positive_int(raw, "vocab", "config.json"), width=_positive_int(raw, "width", "config.json"), layers=layers,
            norm_eps=_positive(_need(raw, "norm", "config.json"), "eps", "norm"), streams=streams,
            logit_scale=float(raw["logit_scale"]) if raw.get("logit_scale") is not None else 1.0, loop=loop,
            max_context=DEFAULT_MAX_CONTEXT if context is None else int(context), eos_token_ids=eos_ids,
            bos_token_id=None if raw.get("bos_token_id") is None else int(raw["bos_token_id"]))

    def run_order(self) -> Tuple[int, ...]:
        """The layer at every position of the run order."""
        count = len(self.layers)
        if self.loop is None:
            return tuple(range(count))
        start, stop, times = self.loop
        return tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, count))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.model_type, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "streams": self.streams, "logit_scale": self.logit_scale,
                               "layers": [layer.to_dict() for layer in self.layers], "max_context": self.max_context}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out
