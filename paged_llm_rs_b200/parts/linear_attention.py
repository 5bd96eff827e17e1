"""Linear attention with decay: recurrent mixers without softmax or denominator whose state is one matrix a head, carried from
token to token in float32 (a ``StateNeed`` slot a request).  With h the mixer's input and S a head's matrix (key entries by
value entries):

    q = W_q h    k = W_k h    v = W_v h                                   (heads x dim, heads x dim, heads x vdim)
    S <- diag(alpha_t) S + k v^T        o = S^T q
    out = W_o (o / rms(o) a head * gain * silu(W_g h))

``retention``: alpha is one constant a head; q and k are rotated on their first ``rot_dims`` entries (entry i with entry
i + rot_dims / 2, by the angle p * rot_base^(-2i / rot_dims)), k then times dim^(-1/2); no gain.

``gated_linear_attention``: alpha is a number a key entry, sigmoid(z)^(1 / tau) with z = W_a2 (W_a1 h) + b; q times dim^(-1/2);
a gain of vdim entries, shared by the heads.  W_a1 h leaves its product in float32 and the second product is formed in
float32 beside the recurrence; how many entries it has only the file knows.

Everything between the stacked input projection and the output projection's input is float32 whatever the compute dtype.  A
step's requests are found through its segment list on the device, so a captured step replays with any requests.
"""

from __future__ import annotations

import numpy as np
import torch

from ..errors import WeightError
from ..kernels import ops
from .base import Mixer, StateNeed, register_mixer
from .spec import TensorSpec

RANDOM_RANK = 16        # the inner size of the decay's product in a model of random weights


class LinearAttention(Mixer):
    """What the two have in common."""

    graph_safe = True

    def __init__(self, spec, rt, position_encodings=None):
        super().__init__(spec, rt)
        p = spec.params
        self.hidden, self.heads, self.dim, self.vdim, self.eps = (int(p["hidden_size"]), int(p["heads"]), int(p["dim"]), int(p["vdim"]),
                                                                  float(p["eps"]))
        self.names = dict(q="q", k="k", v="v", g="g", o="o", norm="norm", a1="a1", a2="a2", a2_b="a2.b")
        self.names.update(p.get("names", {}))
        qk, v = self.heads * self.dim, self.heads * self.vdim
        self.offsets = dict(q_off=0, k_off=qk, v_off=2 * qk, gate_off=2 * qk + v)       # columns of the stacked projection
        self.w_in = self.w_o = None
        # how alpha and the head norm's gain are had, in the kernel's terms
        self.rot, self.inv_freq, self.decay, self.tau, self.gain = 0, None, None, 1.0, None
        self.w_a1 = self.w_a2 = self.a_bias = None
        self.q_scale = self.k_scale = 1.0

    def tensors(self):
        n, W, qk, v = self.names, self.hidden, self.heads * self.dim, self.heads * self.vdim
        return [TensorSpec(self._name(n["q"]), (qk, W)), TensorSpec(self._name(n["k"]), (qk, W)), TensorSpec(self._name(n["v"]), (v, W)),
                TensorSpec(self._name(n["g"]), (v, W)), TensorSpec(self._name(n["o"]), (W, v))]

    def bind(self, tensors):
        t = lambda k: tensors[self._name(self.names[k])]
        self.w_in = torch.cat([t("q"), t("k"), t("v"), t("g")], 0).contiguous()
        self.w_o = t("o")

    def cache_need(self):
        return StateNeed((ops.linear_attention_state_floats(self.heads, self.dim, self.vdim),), torch.float32)

    def forward(self, x, step, cache, writes_cache=True):
        st = self.rt.status
        u = ops.linear(x, self.w_in, status=st)
        a1 = ops.linear(x, self.w_a1, out_dtype=torch.float32, status=st) if self.decay is None else None
        rope = None
        if self.rot and step.max_segment_tokens != 1:       # one table a step for all layers that turn alike
            key = f"rope_table/{self.rot}/{self.rot_base}"
            rope = step.carry.get(key)
            if rope is None:
                rope = step.carry[key] = ops.rope_table(step.positions[:x.shape[0]], self.inv_freq)
        y = torch.empty((x.shape[0], self.heads * self.vdim), dtype=x.dtype, device=x.device)
        ops.linear_attention_mix(u, **self.offsets, q_scale=self.q_scale, k_scale=self.k_scale, rot=self.rot, inv_freq=self.inv_freq,
                                 decay=self.decay, a1=a1, a2=self.w_a2, a_bias=self.a_bias, tau=self.tau, gain=self.gain,
                                 segments=step.segments, max_segment_tokens=step.max_segment_tokens, state=cache, out=y,
                                 heads=self.heads, dim=self.dim, vdim=self.vdim, eps=self.eps, rope=rope)
        out = ops.linear(y, self.w_o, status=st)
        if self.rt.trace is not None:
            for leaf, t in (("in.out", u), ("o.in", y), ("out", out)):
                self.rt.record(self._name(leaf), t)
        return out


class Retention(LinearAttention):
    def __init__(self, spec, rt, position_encodings=None):
        super().__init__(spec, rt, position_encodings)
        p = spec.params
        self.decays = [float(x) for x in p["decay"]]
        self.rot, self.rot_base = int(p.get("rot_dims") or 0), float(p.get("rot_base", 10000.0))
        self.k_scale = self.dim ** -0.5
        if len(self.decays) != self.heads:
            raise ValueError(f"{len(self.decays)} decays for {self.heads} heads")
        if self.rot % 2 or self.rot > self.dim:
            raise ValueError(f"rot_dims {self.rot} must be even and at most dim {self.dim}")

    def bind(self, tensors):
        super().bind(tensors)
        self.decay = torch.tensor(self.decays, dtype=torch.float32, device=self.w_o.device)
        if self.rot:
            f = np.power(np.float64(self.rot_base), -2.0 * np.arange(self.rot // 2, dtype=np.float64) / self.rot)
            self.inv_freq = torch.from_numpy(f.astype(np.float32)).to(self.w_o.device)


class GatedLinearAttention(LinearAttention):
    def __init__(self, spec, rt, position_encodings=None):
        super().__init__(spec, rt, position_encodings)
        self.tau, self.q_scale = float(spec.params["tau"]), self.dim ** -0.5
        if not self.tau > 0:
            raise ValueError("tau must be positive")

    def tensors(self):
        n, W, qk = self.names, self.hidden, self.heads * self.dim
        return super().tensors() + [
            TensorSpec(self._name(n["norm"]), (self.vdim,), "gain"), TensorSpec(self._name(n["a1"]), (None, W), drawn=(RANDOM_RANK, W)),
            TensorSpec(self._name(n["a2"]), (qk, None), drawn=(qk, RANDOM_RANK)), TensorSpec(self._name(n["a2_b"]), (qk,), "offset")]

    def bind(self, tensors):
        super().bind(tensors)
        t = lambda k: tensors[self._name(self.names[k])]
        self.gain, self.w_a1, self.w_a2, self.a_bias = t("norm"), t("a1"), t("a2"), t("a2_b")
        if self.w_a1.shape[0] != self.w_a2.shape[1]:
            raise WeightError(f"{self._name(self.names['a1'])} has {self.w_a1.shape[0]} rows, {self._name(self.names['a2'])} "
                              f"{self.w_a2.shape[1]} columns")


register_mixer("retention", Retention)
register_mixer("gated_linear_attention", GatedLinearAttention)
