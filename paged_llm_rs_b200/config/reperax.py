"""Typed configuration of the Reperax decoder.

Its config.json is nested: ``vocab``, ``width``, ``norm.eps``, ``logit_softcap``, ``loop`` (which layers run several times in
a row) and a list ``layers`` whose entries give the mixer's kind (``type``: ``retention`` or ``parallel``), the mixer's sizes
and constants (``mixer``) and the feed-forward (``mlp``: dense, or null).  Every size and every constant that can differ
between two models of the design is read here, but for the inner size of the decay's product in two factors, which only the
tensors tell; nothing about a particular model stands in code.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ConfigError, UnsupportedModelError
from .schema import _take
from .surelorn import _obj, _positive


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    """Grouped-query attention within chunks of the sequence, q and k normed over the whole projection, no rotation."""

    heads: int
    kv_heads: int
    dim: int                   # query / key entries a head
    vdim: int                  # value entries a head
    scale: float               # multiplies q . k
    chunk: int                 # a position sees its own chunk of this many positions only; 0: all before it

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ChunkedAttentionConfig":
        heads, kv = _positive(d, "heads"), _positive(d, "kv_heads")
        if heads % kv:
            raise ConfigError(f"{heads} heads do not group over {kv} kv_heads")
        mask = _obj(d, "mask", optional=True)
        return cls(heads, kv, _positive(d, "dim"), _positive(d, "vdim"), _take(d, "scale", float),
                   _positive(mask, "size") if mask is not None else 0)


@dataclass(frozen=True)
class GatedLinearAttentionConfig:
    """Linear attention with a decay a key entry that depends on the token."""

    heads: int
    dim: int
    vdim: int
    tau: float                 # the decay is sigmoid(z)^(1 / tau)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "GatedLinearAttentionConfig":
        tau = _take(d, "tau", float)
        if not tau > 0:
            raise ConfigError(f"tau must be positive, got {tau}")
        return cls(_positive(d, "heads"), _positive(d, "dim"), _positive(d, "vdim"), tau)


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: ChunkedAttentionConfig
    right: GatedLinearAttentionConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ParallelMixerConfig":
        return cls(ChunkedAttentionConfig.from_dict(_obj(d, "left")), GatedLinearAttentionConfig.from_dict(_obj(d, "right")),
                   _take(d, "left_scale", float), _take(d, "right_scale", float))


@dataclass(frozen=True)
class RetentionConfig:
    """Linear attention with a constant decay a head, q and k rotated in halves."""

    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]   # one a head
    rot_dims: int              # leading entries of each head that are rotated; 0: none
    rot_base: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RetentionConfig":
        heads, dim = _positive(d, "heads"), _positive(d, "dim")
        decay = d.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != heads or \
                not all(isinstance(x, (int, float)) and not isinstance(x, bool) and 0 <= x <= 1 for x in decay):
            raise ConfigError(f"`decay` must list one number from 0 to 1 for each of {heads} heads")
        rot = _obj(d, "rot", optional=True)
        rot_dims, rot_base = (_take(rot, "dims", int), _take(rot, "base", float)) if rot is not None else (0, 10000.0)
        if rot_dims % 2 or not 0 <= rot_dims <= dim:
            raise ConfigError(f"rot.dims {rot_dims} must be even and at most dim {dim}")
        if rot_dims and rot_base <= 0:
            raise ConfigError("rot.base must be positive")
        return cls(heads, dim, _positive(d, "vdim"), tuple(float(x) for x in decay), rot_dims, rot_base)


_MIXERS = {"retention": RetentionConfig, "parallel": ParallelMixerConfig}


@dataclass(frozen=True)
class LoopConfig:
    """Layers start .. stop - 1 run ``times`` times in a row."""

    start: int
    stop: int
    times: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], layers: int) -> "LoopConfig":
        start, stop, times = _take(d, "start", int), _take(d, "stop", int), _positive(d, "times")
        if not 0 <= start < stop <= layers:
            raise ConfigError(f"loop: layers {start} to {stop} are no range of {layers} layers")
        return cls(start, stop, times)


@dataclass(frozen=True)
class ReperaxLayer:
    mixer_kind: str                       # "retention" or "parallel"
    mixer: object
    dense_ff: Optional[int]               # None: the layer has no feed-forward


@dataclass(frozen=True)
class ReperaxConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: Optional[float]
    loop: Optional[LoopConfig]
    layers: Tuple[ReperaxLayer, ...]
    architecture: str = "Reperax"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ReperaxConfig":
        entries = d.get("layers")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("`layers` must list at least one layer")
        layers = []
        for i, e in enumerate(entries):
            if not isinstance(e, Mapping):
                raise ConfigError(f"layers[{i}] must be an object")
            kind = _take(e, "type", str)
            if kind not in _MIXERS:
                raise UnsupportedModelError(f"layers[{i}]: mixer type {kind!r} is not implemented; known: {sorted(_MIXERS)}")
            try:
                mixer = _MIXERS[kind].from_dict(_obj(e, "mixer"))
                mlp = _obj(e, "mlp", optional=True)
                ff = None
                if mlp is not None:
                    mlp_kind = _take(mlp, "kind", str)
                    if mlp_kind != "dense":
                        raise UnsupportedModelError(f"feed-forward kind {mlp_kind!r} is not implemented")
                    ff = _positive(mlp, "ff")
            except ConfigError as err:
                raise ConfigError(f"layers[{i}]: {err}") from None
            layers.append(ReperaxLayer(kind, mixer, ff))
        eps = _take(_obj(d, "norm"), "eps", float)
        if eps <= 0:
            raise ConfigError(f"norm.eps must be positive, got {eps}")
        cap = d.get("logit_softcap")
        if cap is not None:
            cap = _take(d, "logit_softcap", float)
            if not cap > 0:
                raise ConfigError(f"logit_softcap must be positive, got {cap}")
        loop = _obj(d, "loop", optional=True)
        return cls(vocab=_positive(d, "vocab"), width=_positive(d, "width"), norm_eps=eps, logit_softcap=cap,
                   loop=LoopConfig.from_dict(loop, len(layers)) if loop is not None else None, layers=tuple(layers),
                   architecture=_take(d, "architecture", str, "Reperax"))
