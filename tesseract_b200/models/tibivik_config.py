"""Typed configuration of the ``Tibivik`` architecture, read from ``config.json``.

``config.json`` names the architecture under ``architecture`` and gives ``width`` (of one copy of the residual stream), ``vocab``,
``streams`` (copies of the stream), ``norm.eps``, ``embedding.bigram`` (``buckets``, ``mul_prev``, ``mul_cur``), ``layers`` and, optionally,
``loop`` (``start``, ``stop``, ``times``: layers ``start`` to ``stop - 1`` run ``times`` times in a row).  A layer entry gives ``type`` (which mixer:
``mamba2``, ``parallel`` or ``parallel_2``), ``mixer`` (its sizes and constants) and ``mlp``: null or ``{"kind": "dense", "ff": n}``.  Layers
may differ from one another in every number.
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


def _positive(data: Mapping[str, Any], key: str, where: str) -> float:
    value = _number(data, key, where)
    if not value > 0:
        raise ConfigError(f"{where}.{key} must be positive")
    return value


def _positive_int(data: Mapping[str, Any], key: str, where: str) -> int:
    value = _require(data, key, int, where)
    if value <= 0:
        raise ConfigError(f"{where}: {key} must be positive")
    return value


def _divides(part: int, whole: int, where: str, what: str) -> None:
    if whole % part:
        raise ConfigError(f"{where}: {what}")


@dataclass(frozen=True)
class TibivikRotation:
    dims: int
    base: float

    @classmethod
    def from_dict(cls, data: Optional[Mapping[str, Any]], head_dim: int, where: str) -> Optional["TibivikRotation"]:
        if data is None:
            return None
        dims, base = _require(data, "dims", int, where), _positive(data, "base", where)
        if dims < 0 or dims % 2 or dims > head_dim:
            raise ConfigError(f"{where}: dims must be even and at most the head's {head_dim}")
        return cls(dims, base) if dims else None


@dataclass(frozen=True)
class TibivikAttention:
    """Grouped-query attention: over a sliding window of ``size`` tokens with rotated, normed queries and keys whose projections
    are also the values (``parallel``), or within chunks of ``size`` tokens (``parallel_2``)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    size: int
    scale: float
    rotation: Optional[TibivikRotation]

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str, shares_keys: bool) -> "TibivikAttention":
        heads, kv_heads = _positive_int(data, "heads", where), _positive_int(data, "kv_heads", where)
        _divides(kv_heads, heads, where, "heads must be a multiple of kv_heads")
        dim, vdim = _positive_int(data, "dim", where), _positive_int(data, "vdim", where)
        rotation = None
        if shares_keys:
            if vdim != dim:
                raise ConfigError(f"{where}: values that are keys have the keys' size, got dim {dim} and vdim {vdim}")
            rotation = TibivikRotation.from_dict(data.get("rot"), dim, where + ".rot")
        mask = _require(data, "mask", dict, where)
        return cls(heads, kv_heads, dim, vdim, _positive_int(mask, "size", where + ".mask"), _number(data, "scale", where), rotation)


@dataclass(frozen=True)
class TibivikMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str) -> "TibivikMemory":
        return cls(_positive_int(data, "heads", where), _positive_int(data, "dim", where), _positive_int(data, "vdim", where),
                   _positive(data, "gate_cap", where))


@dataclass(frozen=True)
class TibivikDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str) -> "TibivikDelta":
        heads, kv_heads = _positive_int(data, "heads", where), _positive_int(data, "kv_heads", where)
        _divides(kv_heads, heads, where, "heads must be a multiple of kv_heads")
        return cls(heads, kv_heads, _positive_int(data, "dim", where), _positive_int(data, "vdim", where),
                   _positive_int(data, "conv", where))


@dataclass(frozen=True)
class TibivikStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str) -> "TibivikStateSpace":
        heads, vdim = _positive_int(data, "heads", where), _positive_int(data, "vdim", where)
        groups, norm_groups = _positive_int(data, "groups", where), _positive_int(data, "norm_groups", where)
        _divides(groups, heads, where, "heads must be a multiple of groups")
        _divides(norm_groups, heads * vdim, where, "norm_groups must divide heads * vdim")
        return cls(heads, vdim, _positive_int(data, "state", where), groups, norm_groups, _positive_int(data, "conv", where))


@dataclass(frozen=True)
class TibivikParallel:
    """Two mixers side by side on the same input: attention (left) and a recurrence (right), each result with a weight."""

    left: TibivikAttention
    right: Union[TibivikMemory, TibivikDelta]
    left_scale: float
    right_scale: float


TibivikMixer = Union[TibivikStateSpace, TibivikParallel]


def _read_mixer(kind: str, data: Mapping[str, Any], where: str) -> TibivikMixer:
    if kind == "mamba2":
        return TibivikStateSpace.from_dict(data, where)
    right = {"parallel": TibivikMemory, "parallel_2": TibivikDelta}.get(kind)
    if right is None:
        raise ConfigError(f"{where}: unknown type '{kind}' (known: mamba2, parallel, parallel_2)")
    return TibivikParallel(
        TibivikAttention.from_dict(_require(data, "left", dict, where), where + ".left", shares_keys=kind == "parallel"),
        right.from_dict(_require(data, "right", dict, where), where + ".right"),
        _number(data, "left_scale", where), _number(data, "right_scale", where))


def _read_mlp(mlp: Any, where: str) -> Optional[int]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} must be an object or null")
    kind = _require(mlp, "kind", str, where)
    if kind != "dense":
        raise ConfigError(f"{where}: unknown kind '{kind}' (known: dense)")
    return _positive_int(mlp, "ff", where)


@dataclass(frozen=True)
class TibivikLayer:
    type: str
    mixer: TibivikMixer
    ff: Optional[int]           # the dense feed-forward's size, or None for a layer without one


@dataclass(frozen=True)
class TibivikLoop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class TibivikConfig:
    width: int
    vocab: int
    streams: int
    norm_eps: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: Tuple[TibivikLayer, ...]
    loop: Optional[TibivikLoop]

    ARCHITECTURE = "Tibivik"

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "TibivikConfig":
        layers = []
        for index, entry in enumerate(_require(data, "layers", list)):
            where = f"layers[{index}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"{where} must be an object")
            kind = _require(entry, "type", str, where)
            mixer = _read_mixer(kind, _require(entry, "mixer", dict, where), where + ".mixer")
            layers.append(TibivikLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + ".mlp")))
        if not layers:
            raise ConfigError("layers must not be empty")
        loop = None
        if data.get("loop") is not None:
            raw = _require(data, "loop", dict)
            loop = TibivikLoop(*(_require(raw, key, int, "loop") for key in ("start", "stop", "times")))
            if not (0 <= loop.start <= loop.stop <= len(layers)) or loop.times < 1:
                raise ConfigError("loop: needs 0 <= start <= stop <= number of layers and times >= 1")
        bigram = _require(_require(data, "embedding", dict), "bigram", dict, "embedding")
        where = "embedding.bigram"
        return cls(width=_positive_int(data, "width", "config"), vocab=_positive_int(data, "vocab", "config"),
                   streams=_positive_int(data, "streams", "config"),
                   norm_eps=_positive(_require(data, "norm", dict), "eps", "norm"),
                   buckets=_positive_int(bigram, "buckets", where), mul_prev=_require(bigram, "mul_prev", int, where),
                   mul_cur=_require(bigram, "mul_cur", int, where), layers=tuple(layers), loop=loop)

    def run_order(self) -> Tuple[int, ...]:
        """Layer indices in the order they run."""
        count = len(self.layers)
        if self.loop is None:
            return tuple(range(count))
        looped = tuple(range(self.loop.start, self.loop.stop)) * self.loop.times
        return tuple(range(self.loop.start)) + looped + tuple(range(self.loop.stop, count))
