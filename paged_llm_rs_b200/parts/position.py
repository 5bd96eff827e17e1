"""Rotary position encoding (crates/pagedllm/src/model/rope.rs:32-63).

inv_freq[i] = 1 / theta^(2i / rotary_dim); the angle position * inv_freq[i] is
formed in float64 on the host and only float32 cos/sin tables reach the device.
The tables hold each angle once, [max_positions, rotary_dim/2]: dimension i
pairs with i + rotary_dim/2 (rope.rs:96-107), which the kernel that applies
them does.  rotary_dim may be smaller than the head (the rest is not rotated).
"""

from __future__ import annotations

import numpy as np
import torch

from .base import PositionEncoding, register_position_encoding


def rotary_frequencies(dims: int, base: float, scaling=None):
    """(frequencies of the dims / 2 pairs in float64, factor on cos and sin): base^(-2i / dims) and 1, or with ``scaling``
    (factor, original, fast, slow) the YaRN blend of them: a pair that turns more than ``fast`` times within ``original``
    positions keeps its frequency, one that turns fewer than ``slow`` times has it divided by ``factor``, those between go
    linearly from one to the other; cos and sin are then multiplied by 0.1 ln(factor) + 1."""
    i = np.arange(dims // 2, dtype=np.float64)
    f = np.power(np.float64(base), -2.0 * i / dims)
    if scaling is None:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])
    pair = lambda turns: dims * np.log(original / (2.0 * np.pi * float(turns))) / (2.0 * np.log(float(base)))
    lo, hi = max(np.floor(pair(scaling["fast"])), 0.0), min(np.ceil(pair(scaling["slow"])), dims - 1.0)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), float(0.1 * np.log(factor) + 1.0)


class RotaryEncoding(PositionEncoding):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = spec.params
        self.head_dim = int(p["head_dim"])
        self.rotary_dim = int(p.get("rotary_dim", self.head_dim))
        self.theta = float(p["theta"])
        self.max_positions = int(p["max_positions"])
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.cos = self.sin = None

    def _tables(self):
        rt = self.rt
        half = self.rotary_dim // 2
        inv_freq = 1.0 / np.power(np.float64(self.theta), 2.0 * np.arange(half, dtype=np.float64) / self.rotary_dim)
        angle = np.arange(self.max_positions, dtype=np.float64)[:, None] * inv_freq[None, :]
        self.cos = torch.from_numpy(np.cos(angle).astype(np.float32)).to(rt.device)
        self.sin = torch.from_numpy(np.sin(angle).astype(np.float32)).to(rt.device)

    def rotary(self):
        if self.cos is None:
            self._tables()
        return self.cos, self.sin, self.rotary_dim


class NoPositionEncoding(PositionEncoding):
    pass


class SinusoidalEncoding(PositionEncoding):
    """An absolute position vector added to a float32 residual stream right behind the embedding:
    entry 2i is sin(p f_i), entry 2i + 1 is cos(p f_i), f_i = base^(-2i / width).  The frequencies
    are formed in float64 on the host and kept in float32; the angle p f_i is a float32 product
    formed by the kernel, so no table bounds the positions."""

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.width = int(spec.params["width"])
        self.base = float(spec.params.get("base", 10000.0))
        if self.width % 2:
            raise ValueError(f"width {self.width} must be even: a sine pairs with a cosine")
        self.inv_freq = None

    def at_embedding(self, hidden, step):
        if self.inv_freq is None:
            f = np.power(np.float64(self.base), -2.0 * np.arange(self.width // 2, dtype=np.float64) / self.width)
            self.inv_freq = torch.from_numpy(f.astype(np.float32)).to(self.rt.device)
        from ..kernels import ops
        return ops.sinusoid_add(hidden, step.positions, self.inv_freq)


register_position_encoding("rope", RotaryEncoding)
register_position_encoding("none", NoPositionEncoding)
register_position_encoding("sinusoidal", SinusoidalEncoding)
