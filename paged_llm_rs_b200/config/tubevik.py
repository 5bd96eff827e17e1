"""Typed configuration of the Tubevik decoder.

Its config.json is nested: ``vocab``, ``width``, ``norm.eps``, ``residual_mult``, ``logit_softcap`` and a list ``layers`` whose
entries give the mixer's kind (``type``: ``attention`` or ``parallel``), the mixer's sizes and constants (``mixer``) and the
feed-forward (``mlp``: dense, or null).  Every size and every constant that can differ between two models of the design is read
here, but for the inner sizes of the products in two factors, which only the tensors tell; nothing about a particular model
stands in code.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ConfigError, UnsupportedModelError
from .pamarax import DeltaRuleHalfConfig, _grouped
from .schema import _take
from .surelorn import _obj, _positive


@dataclass(frozen=True)
class YarnConfig:
    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "YarnConfig":
        c = cls(*(_take(d, k, float) for k in ("factor", "original", "fast", "slow")))
        if min(c.factor, c.original, c.fast, c.slow) <= 0:
            raise ConfigError("rot.scaling: factor, original, fast and slow must be positive")
        return c

    def params(self) -> dict:
        return dict(factor=self.factor, original=self.original, fast=self.fast, slow=self.slow)


@dataclass(frozen=True)
class RotationConfig:
    dims: int                  # leading entries of each head that are rotated
    base: float
    scaling: Optional[YarnConfig]

    @classmethod
    def from_dict(cls, d: Optional[Mapping[str, Any]], head: int) -> "RotationConfig":
        if d is None:
            return cls(0, 10000.0, None)
        dims, base = _take(d, "dims", int), _take(d, "base", float)
        if dims % 2 or not 0 <= dims <= head:
            raise ConfigError(f"rot.dims {dims} must be even and at most dim {head}")
        scaling = _obj(d, "scaling", optional=True)
        if dims and (base <= 0 or (scaling is not None and base == 1.0)):
            raise ConfigError("rot.base must be positive, and with rot.scaling not 1")
        return cls(dims, base, YarnConfig.from_dict(scaling) if scaling is not None else None)


def _cap(d: Mapping[str, Any], key: str) -> Optional[float]:
    cap = _take(d, key, float, None)
    if cap is not None and not cap > 0:
        raise ConfigError(f"{key} must be positive, got {cap}")
    return cap


def _mask(d: Mapping[str, Any]) -> int:
    mask = _obj(d, "mask", optional=True)
    return _positive(mask, "size") if mask is not None else 0


@dataclass(frozen=True)
class WindowAttentionConfig:
    """Grouped-query attention inside a sliding window, q and k normed over the whole projection, capped scores, a gate a head."""

    heads: int
    kv_heads: int
    dim: int                   # query / key entries a head
    vdim: int                  # value entries a head
    scale: float               # multiplies q . k
    softcap: Optional[float]   # scores pass cap * tanh(. / cap)
    window: int                # a position sees itself and the window - 1 before it; 0: all before it
    rot: RotationConfig
    kv_from: Optional[int]     # the layer whose keys and values this one attends over (None: its own)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "WindowAttentionConfig":
        heads, kv = _grouped(d)
        dim = _positive(d, "dim")
        return cls(heads, kv, dim, _positive(d, "vdim"), _take(d, "scale", float), _cap(d, "softcap"), _mask(d),
                   RotationConfig.from_dict(_obj(d, "rot", optional=True), dim), _take(d, "kv_from", int, None))


@dataclass(frozen=True)
class ChunkAttentionConfig:
    """Grouped-query attention within chunks of the sequence, q and k normed a head behind their rotation, one more in the
    softmax's denominator."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                 # a position sees its own chunk of this many positions only; 0: all before it
    rot: RotationConfig

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ChunkAttentionConfig":
        heads, kv = _grouped(d)
        dim = _positive(d, "dim")
        return cls(heads, kv, dim, _positive(d, "vdim"), _take(d, "scale", float), _mask(d),
                   RotationConfig.from_dict(_obj(d, "rot", optional=True), dim))


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: ChunkAttentionConfig
    right: DeltaRuleHalfConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ParallelMixerConfig":
        return cls(ChunkAttentionConfig.from_dict(_obj(d, "left")), DeltaRuleHalfConfig.from_dict(_obj(d, "right")),
                   _take(d, "left_scale", float), _take(d, "right_scale", float))


_MIXERS = {"attention": WindowAttentionConfig, "parallel": ParallelMixerConfig}


@dataclass(frozen=True)
class ClampedFeedForwardConfig:
    ff: int
    limit: float               # bounds the gate from above and the up product on both sides

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ClampedFeedForwardConfig":
        kind = _take(d, "kind", str)
        if kind != "dense":
            raise UnsupportedModelError(f"feed-forward kind {kind!r} is not implemented")
        limit = _take(d, "limit", float)
        if not limit > 0:
            raise ConfigError(f"mlp.limit must be positive, got {limit}")
        return cls(_positive(d, "ff"), limit)


@dataclass(frozen=True)
class TubevikLayer:
    mixer_kind: str                       # "attention" or "parallel"
    mixer: object
    mlp: Optional[ClampedFeedForwardConfig]     # None: the layer has no feed-forward


def _check_lender(layers, i: int) -> None:
    """A layer that borrows keys and values: its lender has ones of its own, of the same heads and sizes."""
    m = layers[i].mixer
    if not 0 <= m.kv_from < i or layers[m.kv_from].mixer_kind != "attention":
        raise ConfigError(f"kv_from {m.kv_from} names no earlier attention layer")
    o = layers[m.kv_from].mixer
    if o.kv_from is not None:
        raise ConfigError(f"kv_from {m.kv_from} names a layer that has no keys and values of its own")
    if (o.heads, o.kv_heads, o.dim, o.vdim) != (m.heads, m.kv_heads, m.dim, m.vdim):
        raise ConfigError(f"kv_from {m.kv_from} names a layer of other heads or sizes")


@dataclass(frozen=True)
class TubevikConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: Optional[float]
    layers: Tuple[TubevikLayer, ...]
    architecture: str = "Tubevik"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "TubevikConfig":
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
                mlp = _obj(e, "mlp", optional=True)
                layers.append(TubevikLayer(kind, _MIXERS[kind].from_dict(_obj(e, "mixer")),
                                           ClampedFeedForwardConfig.from_dict(mlp) if mlp is not None else None))
                if kind == "attention" and layers[i].mixer.kv_from is not None:
                    _check_lender(layers, i)
            except ConfigError as err:
                raise ConfigError(f"layers[{i}]: {err}") from None
        eps = _take(_obj(d, "norm"), "eps", float)
        if eps <= 0:
            raise ConfigError(f"norm.eps must be positive, got {eps}")
        return cls(vocab=_positive(d, "vocab"), width=_positive(d, "width"), norm_eps=eps,
                   residual_mult=_take(d, "residual_mult", float, 1.0), logit_softcap=_cap(d, "logit_softcap"), layers=tuple(layers),
                   architecture=_take(d, "architecture", str, "Tubevik"))
