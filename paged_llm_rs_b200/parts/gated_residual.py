"""Parts that an arrangement of a layer may name beside its mixer, feed-forward and norms.

  residual_gate   a sublayer's result is multiplied, entry by entry, by sigmoid(W h + b), h being the sublayer's normed input;
                  the product with W leaves in the compute dtype, bias, sigmoid and multiplication are float32 in the kernel
                  that adds the result to the stream
  token_shift     a sublayer reads h_t + (h_(t-1) - h_t) * mix instead of h_t; a request's last h is kept in float32 (a
                  ``StateNeed`` slot), zeros before its first token
  pass_vectors    one vector for each pass through layers that run several times
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import Part, StateNeed, register_extra
from .spec import TensorSpec


class ResidualGate(Part):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.hidden, self.width = int(spec.params["hidden_size"]), int(spec.params["width"])
        self.optional = bool(spec.params.get("optional", False))
        self.weight = self.bias = None

    def tensors(self):
        return [TensorSpec(self.prefix, (self.width, self.hidden), optional=self.optional),
                TensorSpec(self._name("b"), (self.width,), "offset", optional=self.optional)]

    def bind(self, tensors):
        self.weight, self.bias = tensors.get(self.prefix), tensors.get(self._name("b"))

    def logits(self, h):
        return ops.linear(h, self.weight, status=self.rt.status)


class TokenShift(Part):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.width = int(spec.params["width"])
        self.mix = None

    def tensors(self):
        return [TensorSpec(self.prefix, (self.width,), "offset")]

    def bind(self, tensors):
        self.mix = tensors[self.prefix]

    def cache_need(self):
        return StateNeed((self.width,), torch.float32)


class PassVectors(Part):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.width, self.times = int(spec.params["width"]), int(spec.params["times"])
        self.table = None

    def tensors(self):
        return [TensorSpec(self.prefix, (self.times, self.width), "offset")]

    def bind(self, tensors):
        self.table = tensors[self.prefix]

    def vector(self, t: int):
        return self.table[t]


register_extra("residual_gate", ResidualGate)
register_extra("token_shift", TokenShift)
register_extra("pass_vectors", PassVectors)
