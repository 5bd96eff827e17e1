"""Grouped-query attention whose queries and keys are normed before the scores, with the options that designs of this
family combine.

With h the mixer's input, per token at position p and query head a (kv head a // (heads / kv_heads)):

    q = W_q h     k = W_k h     v = W_v h, or (``values_are_keys``) no W_v: v is the raw W_k h;   ``biases``: + b each
    q, k <- norm(q), norm(k)          ``qk_norm``: "head" (each head over its own root mean square, one gain of key_dim
                                      entries shared by the heads), "projection" (all heads of q at once, and all of k,
                                      a gain of the projection's size), "head_after_rotation" (each head, behind the rotation,
                                      no gain) or None
    q <- q * (1 + temp_coef * ln(floor((p + 1) / temp_every) + 1))          (``temp_every`` 0: no such factor)
    q, k <- rot_p(q), rot_p(k)        the first ``rot_dims`` entries of a head, entry i with entry i + rot_dims / 2 (``rot_layout``
                                      "half") or entry 2i with entry 2i + 1 ("pairs"), by the angle p * rot_base^(-2i / rot_dims);
                                      ``rot_scaling``: YaRN's frequencies and factor (parts/position.py); 0: no rotation
    s(p, j) = scale q . k_j           ``softcap``: then cap tanh(s / cap)
    weight(p, j) = exp(s(p, j)) / (sink + sum over seen j' of exp(s(p, j')))
                                      ``sink_one``: sink = 1 = exp(0), as if one more key scored zero and carried nothing; else 0
                                      seen: j <= p; ``window``: and p - j < window; ``chunk``: and j in p's own chunk of that many
                                      positions (0: neither)
    out = W_o ([sum over seen j of weight(p, j) v_j]_a * sigmoid(W_g h)_a)  (``gate`` None: no such factor; ``gate_per`` "entry":
                                      W_g h has an entry for each of the heads' outputs, "head": one a head)

A token's key and value lie side by side in one cache row (``JoinedKVNeed``); the attention itself is the kernel of the
windowed attention with sinks.  A layer may have no keys and values of its own (``keeps`` "nothing"): it attends over an earlier
layer's rows with its own queries and its own window.  A layer whose rows others read further back than itself says so
(``cache_window``: how far back rows are kept; 0: all of them).  Norms, biases, the temperature, angles, scores and weights are
float32 whatever the compute dtype.
"""

from __future__ import annotations

import numpy as np
import torch

from ..errors import KernelError
from ..kernels import ops
from .base import JoinedKVNeed, Mixer, PlanWish, register_mixer, stack_rows
from .position import rotary_frequencies
from .spec import TensorSpec


class NormedQKAttention(Mixer):
    graph_safe = True

    def __init__(self, spec, rt, position_encodings=None):
        super().__init__(spec, rt)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.nh, self.nkv = int(p["num_heads"]), int(p["num_kv_heads"])
        self.dk, self.dv = int(p["key_dim"]), int(p["value_dim"])
        self.scale, self.eps = float(p["scale"]), float(p["eps"])
        self.qk_norm = p.get("qk_norm")
        self.values_are_keys = bool(p.get("values_are_keys", False))
        self.rot, self.rot_base = int(p.get("rot_dims") or 0), float(p.get("rot_base", 10000.0))
        self.rot_layout, self.rot_scaling, self.rot_factor = p.get("rot_layout", "half"), p.get("rot_scaling"), 1.0
        self.temp_coef, self.temp_every = float(p.get("temp_coef") or 0.0), int(p.get("temp_every") or 0)
        self.sink_one = bool(p.get("sink_one", False))
        self.gate = p.get("gate")
        self.gate_per = p.get("gate_per", "entry")
        self.chunk, self.window, self.cap = int(p.get("chunk") or 0), int(p.get("window") or 0), float(p.get("softcap") or 0.0)
        self.cache_window = int(p.get("cache_window", self.window) or 0)
        self.biases, self.keeps = bool(p.get("biases", False)), p.get("keeps", "own")
        if self.rot_layout not in ("half", "pairs"):
            raise ValueError(f"rot_layout {self.rot_layout!r}: 'half' or 'pairs'")
        if self.gate_per not in ("entry", "head") or self.keeps not in ("own", "nothing"):
            raise ValueError(f"gate_per {self.gate_per!r}: 'entry' or 'head'; keeps {self.keeps!r}: 'own' or 'nothing'")
        if self.chunk and (self.window or self.cache_window):
            raise ValueError("a layer sees a window or a chunk, not both")
        if self.cache_window and not 0 < self.window <= self.cache_window:
            raise ValueError(f"rows are kept for {self.cache_window} tokens, but the layer itself sees {self.window or 'all'}")
        if self.qk_norm not in ops.QK_NORMS:
            raise ValueError(f"qk_norm {self.qk_norm!r}: one of {list(ops.QK_NORMS)}")
        if self.gate not in (None,) + tuple(ops.GATE_KINDS):
            raise ValueError(f"gate {self.gate!r}: None or one of {sorted(ops.GATE_KINDS)}")
        if self.nh % self.nkv:
            raise ValueError(f"{self.nh} heads do not group over {self.nkv} kv heads")
        if self.rot % 2 or self.rot > self.dk:
            raise ValueError(f"rot_dims {self.rot} must be even and at most key_dim {self.dk}")
        if self.values_are_keys and self.dv != self.dk:
            raise ValueError(f"the keys are the values, so value_dim {self.dv} must equal key_dim {self.dk}")
        if max(self.dk, self.dv) > 256:
            raise KernelError(f"key_dim {self.dk} / value_dim {self.dv}: the attention kernel takes sizes up to 256")
        self.names = dict(q="q", k="k", v="v", o="o", g="g", q_norm="q.norm", k_norm="k.norm")
        self.names.update(p.get("names", {}))
        for k in ("q", "k", "v"):
            self.names.setdefault(f"{k}_b", self.names[k] + ".b")
        self.w_in = self.w_o = self.q_gain = self.k_gain = self.q_bias = self.k_bias = self.v_bias = self.inv_freq = self.sinks = None
        own = self.keeps == "own"
        self.gates = self.nh * (self.dv if self.gate_per == "entry" else 1) if self.gate else 0
        self.k_off = self.nh * self.dk if own else -1
        self.v_off = self.nh * self.dk + (self.nkv * self.dk if own else 0)
        self.g_off = self.v_off + (0 if self.values_are_keys or not own else self.nkv * self.dv)
        self._need = None

    def _stacked(self):
        keys = [] if self.keeps == "nothing" else ["k"] if self.values_are_keys else ["k", "v"]
        return ["q"] + keys + (["g"] if self.gate else [])

    def _parts_of(self, what):
        """(name, entries) of q, k and v that the layer has."""
        rows = dict(q=self.nh * self.dk, k=self.nkv * self.dk, v=self.nkv * self.dv)
        return [(k, rows[k]) for k in self._stacked() if k in what]

    def tensors(self):
        n, W = self.names, self.hidden
        t = [TensorSpec(self._name(n[k]), (r, W)) for k, r in self._parts_of("qkv") + ([("g", self.gates)] if self.gate else [])]
        t.append(TensorSpec(self._name(n["o"]), (W, self.nh * self.dv)))
        if self.biases:
            t += [TensorSpec(self._name(n[f"{k}_b"]), (r,), "offset") for k, r in self._parts_of("qkv")]
        if self.qk_norm in ("head", "projection"):
            t += [TensorSpec(self._name(n[f"{k}_norm"]), (self.dk if self.qk_norm == "head" else r,), "gain") for k, r in self._parts_of("qk")]
        return t

    def bind(self, tensors):
        n = self.names
        get = lambda k: tensors.get(self._name(n[k]))
        self.w_in = stack_rows([tensors[self._name(n[k])] for k in self._stacked()])
        self.w_o = tensors[self._name(n["o"])]
        if self.biases:
            self.q_bias, self.k_bias, self.v_bias = get("q_b"), get("k_b"), get("v_b")
        if self.qk_norm in ("head", "projection"):
            self.q_gain, self.k_gain = get("q_norm"), get("k_norm")
        if self.rot:
            f, self.rot_factor = rotary_frequencies(self.rot, self.rot_base, self.rot_scaling)
            self.inv_freq = torch.from_numpy(f.astype(np.float32)).to(self.w_o.device)
        if self.sink_one:
            self.sinks = torch.zeros(self.nh, dtype=torch.float32, device=self.w_o.device)      # exp(0) in the denominator

    def cache_need(self):
        if self._need is None:
            self._need = JoinedKVNeed("chunk" if self.chunk else "window" if self.cache_window else "full", self.nkv, self.dk, self.dv,
                                      self.cache_window or None, 0, group_size=self.nh // self.nkv, chunk=self.chunk)
        return self._need

    def plan_wish(self, page_size: int):
        a = (self.nh, self.nkv, self.rt.dtype, self.dk, self.dv)
        return PlanWish(ops.attention_sink_tile_tokens(*a), ops.attention_sink_ctas_per_item(*a), self.nh, self.dv)

    def forward(self, x, step, cache, writes_cache=True):
        kv_pool, gi = cache
        g = step.groups[gi]
        T, st = x.shape[0], self.rt.status
        proj = ops.linear(x, self.w_in, status=st)
        q = torch.empty((T, self.nh * self.dk), dtype=x.dtype, device=x.device)
        ops.normed_qk_kv_write(proj, self.k_off, self.v_off, q, self.q_gain, self.k_gain, self.qk_norm, self.eps, self.temp_coef,
                               self.temp_every, self.inv_freq, self.rot, step.positions, g.slots,
                               kv_pool if writes_cache and self.keeps == "own" else None, self.nh, self.nkv, self.dk, self.dv,
                               self.values_are_keys, st, q_bias=self.q_bias, k_bias=self.k_bias, v_bias=self.v_bias,
                               rot_pairs=self.rot_layout == "pairs", rot_factor=self.rot_factor)
        o = torch.empty((T, self.nh * self.dv), dtype=x.dtype, device=x.device)
        ops.attention_sink(q, kv_pool, g.block_tables, g.plan, o, self.sinks, self.nh, self.nkv, self.dk, self.dv, self.window, 0,
                           self.scale, self.cap, st, chunk=self.chunk)
        if self.gate:
            ops.gate_mul(o, proj[:, self.g_off:self.g_off + self.gates], self.gate, per=self.dv if self.gate_per == "head" else 1)
        out = ops.linear(o, self.w_o, status=st)
        if self.rt.trace is not None:
            for leaf, t in (("q.normed", q), ("o.in", o), ("out", out)):
                self.rt.record(self._name(leaf), t)
        return out


register_mixer("normed_qk_attention", NormedQKAttention)
