"""Typed configuration of the ``Rirulix`` architecture, read from ``config.json``.

``config.json`` names the architecture under ``architecture`` and gives ``width`` (the residual stream), ``vocab``,
``max_positions`` (rows of the learned position table), ``norm`` (``groups``, ``eps``) and ``layers``.  A layer entry gives
``type`` (which mixer: ``attention`` or ``rglru``), ``mixer`` (its sizes and constants) and ``mlp``: null or routed experts
(``{"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}, "shared": {"ff", "limit"}}``; ``shared`` may be
absent).  Layers may differ from one another in every number.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from ..config.reading import ConfigError, require as _require

_NUMBER = (int, float)


def _number(data: Mapping[str, Any], key: str, where: str) -> float:
    value = float(_require(data, key, _NUMBER, where))
    if not math.isfinite(value):
        raise ConfigError(f"{where}.{key} must be finite")
    return value


def _positive_int(data: Mapping[str, Any], key: str, where: str) -> int:
    value = _require(data, key, int, where)
    if value <= 0:
        raise ConfigError(f"{where}: {key} must be positive")
    return value


@dataclass(frozen=True)
class RirulixAttention:
    """Grouped-query attention over a sliding window of ``window`` tokens and the first ``keep_first`` ones, with biases, a
    learned distance bias and, with ``v_mix``, values mixed with the first such layer's."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    keep_first: int
    scale: float
    v_mix: bool

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str) -> "RirulixAttention":
        heads, kv_heads = _positive_int(data, "heads", where), _positive_int(data, "kv_heads", where)
        if heads % kv_heads:
            raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
        mask = _require(data, "mask", dict, where)
        keep_first = 0
        if mask.get("keep_first") is not None:
            keep_first = _require(mask, "keep_first", int, where + ".mask")
            if keep_first < 0:
                raise ConfigError(f"{where}.mask: keep_first must not be negative")
        v_mix = data.get("v_mix", False)
        if v_mix is not None and not isinstance(v_mix, bool):
            raise ConfigError(f"{where}: v_mix must be true or false")
        return cls(heads=heads, kv_heads=kv_heads, dim=_positive_int(data, "dim", where), vdim=_positive_int(data, "vdim", where),
                   window=_positive_int(mask, "size", where + ".mask"), keep_first=keep_first,
                   scale=_number(data, "scale", where), v_mix=bool(v_mix))


@dataclass(frozen=True)
class RirulixRecurrence:
    """A real-gated linear recurrent unit of ``width`` channels in ``blocks`` equal blocks behind a convolution of
    ``taps`` taps."""

    width: int
    blocks: int
    taps: int

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str) -> "RirulixRecurrence":
        width, blocks = _positive_int(data, "width", where), _positive_int(data, "blocks", where)
        if width % blocks:
            raise ConfigError(f"{where}: width must be a multiple of blocks")
        return cls(width, blocks, _positive_int(data, "conv", where))


@dataclass(frozen=True)
class RirulixExperts:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: Optional[int]
    shared_limit: float


RirulixMixer = Union[RirulixAttention, RirulixRecurrence]
_MIXERS = {"attention": RirulixAttention, "rglru": RirulixRecurrence}


def _expert(data: Mapping[str, Any], where: str) -> Tuple[int, float]:
    limit = _number(data, "limit", where)
    if not limit > 0:
        raise ConfigError(f"{where}: limit must be positive")
    return _positive_int(data, "ff", where), limit


def _read_mlp(mlp: Any, where: str) -> Optional[RirulixExperts]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} must be an object or null")
    kind = _require(mlp, "kind", str, where)
    if kind != "moe":
        raise ConfigError(f"{where}: unknown kind '{kind}' (known: moe)")
    router = _require(mlp, "router", dict, where)
    experts, top = _positive_int(router, "experts", where + ".router"), _positive_int(router, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"{where}.router: top must be at most experts")
    ff, limit = _expert(_require(mlp, "expert", dict, where), where + ".expert")
    shared_ff, shared_limit = None, 0.0
    if mlp.get("shared") is not None:
        shared_ff, shared_limit = _expert(_require(mlp, "shared", dict, where), where + ".shared")
    return RirulixExperts(experts, top, ff, limit, shared_ff, shared_limit)


@dataclass(frozen=True)
class RirulixLayer:
    type: str
    mixer: RirulixMixer
    mlp: Optional[RirulixExperts]


@dataclass(frozen=True)
class RirulixConfig:
    width: int
    vocab: int
    max_positions: int
    norm_groups: int
    norm_eps: float
    layers: Tuple[RirulixLayer, ...]

    ARCHITECTURE = "Rirulix"

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "RirulixConfig":
        norm = _require(data, "norm", dict)
        groups = 1 if norm.get("groups") is None else _positive_int(norm, "groups", "norm")
        layers = []
        for index, entry in enumerate(_require(data, "layers", list)):
            where = f"layers[{index}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"{where} must be an object")
            kind = _require(entry, "type", str, where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}: unknown type '{kind}' (known: {sorted(_MIXERS)})")
            mixer = _MIXERS[kind].from_dict(_require(entry, "mixer", dict, where), where + ".mixer")
            layers.append(RirulixLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + ".mlp")))
        cfg = cls(width=_require(data, "width", int), vocab=_require(data, "vocab", int),
                  max_positions=_require(data, "max_positions", int), norm_groups=groups,
                  norm_eps=_number(norm, "eps", "norm"), layers=tuple(layers))
        if cfg.width <= 0 or cfg.vocab <= 0 or cfg.max_positions <= 0 or not cfg.layers:
            raise ConfigError("width, vocab and max_positions must be positive and layers not empty")
        if not cfg.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if cfg.width % cfg.norm_groups:
            raise ConfigError("norm.groups must divide width")
        mixing = {layer.mixer.kv_heads * layer.mixer.vdim for layer in cfg.layers
                  if isinstance(layer.mixer, RirulixAttention) and layer.mixer.v_mix}
        if len(mixing) > 1:
            raise ConfigError(f"layers with v_mix must share one value width (kv_heads * vdim), got {sorted(mixing)}")
        return cfg

    def first_mixing_layer(self) -> Optional[int]:
        """The first layer whose values later layers with ``v_mix`` mix into their own."""
        for index, layer in enumerate(self.layers):
            if isinstance(layer.mixer, RirulixAttention) and layer.mixer.v_mix:
                return index
        return None
