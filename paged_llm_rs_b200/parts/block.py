"""The pre-norm residual block: x + mixer(norm(x)), then x + ff(norm(x))
(crates/pagedllm/src/model/mod.rs:117-135).  Each residual add is done by the
norm kernel that follows it: the block hands on the residual stream and the
addition that is still pending."""

from __future__ import annotations

import torch

import torch

from ..kernels import ops
from .base import Block, CompositeNeed, register_block
from .norm import PendingGated


class PreNormResidualBlock(Block):
    def pre_mixer(self, residual, delta):
        return self.norms["mixer"].add_norm(residual, delta)         # residual += delta, in place

    def post_mixer(self, residual, a, step):
        h = self.norms["feed_forward"].add_norm(residual, a)
        out = self.feed_forward.forward(h, step)
        rt = self.mixer.rt
        if rt.trace is not None and self.prefix:
            rt.record(f"{self.prefix}.out", residual + out)          # (otherwise formed by the next norm's kernel)
        return residual, out

    def forward(self, residual, delta, step, cache, writes_cache=True):
        h = self.pre_mixer(residual, delta)
        a = self.mixer.forward(h, step, cache, writes_cache)
        return self.post_mixer(residual, a, step)


class OutputNormResidualBlock(Block):
    """x + norm(mixer(x)), then x + norm(ff(x)): the norm sits on each sublayer's output and the
    sublayers read the stream itself.  The stream is float32 and is added to in place; what is
    handed on beside it is its rounding to the compute dtype (None before the first block, the
    stream itself in a float32 engine), not a pending addition.  A layer may have no feed-forward.
    Its norms are ``StreamRMSNorm``s."""

    def forward(self, stream, rounded, step, cache, writes_cache=True):
        rt = self.mixer.rt
        if rounded is None:
            rounded = stream if rt.dtype == torch.float32 else ops.round_rows(stream, rt.dtype)
        a = self.mixer.forward(rounded, step, cache, writes_cache)
        rounded = self.norms["mixer"].add_into(stream, a)
        if self.feed_forward is not None:
            f = self.feed_forward.forward(rounded, step)
            rounded = self.norms["feed_forward"].add_into(stream, f)
        if rt.trace is not None and self.prefix:
            rt.record(f"{self.prefix}.out", stream)
        return stream, rounded

    def settle(self, stream, rounded):
        return stream, None


class PreNormStreamBlock(Block):
    """x + m mixer(norm(x)), then x + m ff(norm(x)), on a float32 stream: the pre-norm block with its norms
    ``ScaledStreamRMSNorm``s, which add the pending sublayer output (times the model's constant m) into the stream
    and norm the sum into the compute dtype in one kernel.  A layer may have no feed-forward: the mixer's output is
    then what is handed on."""

    def pre_mixer(self, stream, delta):
        return self.norms["mixer"].add_norm(stream, delta)

    def post_mixer(self, stream, a, step):
        out = a
        if self.feed_forward is not None:
            out = self.feed_forward.forward(self.norms["feed_forward"].add_norm(stream, a), step)
        rt = self.mixer.rt
        if rt.trace is not None and self.prefix:
            rt.record(f"{self.prefix}.out", stream + self.norms["mixer"].mult * out.float())
        return stream, out

    def forward(self, stream, delta, step, cache, writes_cache=True):
        h = self.pre_mixer(stream, delta)
        a = self.mixer.forward(h, step, cache, writes_cache)
        return self.post_mixer(stream, a, step)


class SandwichStreamBlock(Block):
    """x + norm_b(mixer(norm_a(x))), then x + norm_d(ff(norm_c(x))), on a float32 stream: every sublayer is normed on the way
    in and on the way out.  Its norms are ``SandwichStreamRMSNorm``s named "mixer", "mixer_out", "feed_forward" and
    "feed_forward_out"; what is handed on beside the stream is the last sublayer's output wrapped by its output norm, so
    that ONE kernel norms it, adds it and norms the sum for the next sublayer.  A feed-forward with a bias on its last
    product leaves that bias to the same kernel.  A layer may have no feed-forward."""

    def pre_mixer(self, stream, pending):
        return self.norms["mixer"].add_norm(stream, pending)

    def post_mixer(self, stream, a, step):
        pending = self.norms["mixer_out"].pending(a)
        if self.feed_forward is not None:
            h = self.norms["feed_forward"].add_norm(stream, pending)
            if hasattr(self.feed_forward, "forward_deferred"):
                f, bias = self.feed_forward.forward_deferred(h, step)
            else:
                f, bias = self.feed_forward.forward(h, step), None
            pending = self.norms["feed_forward_out"].pending(f, bias)
        rt = self.mixer.rt
        if rt.trace is not None and self.prefix:
            x = stream.clone()
            self.norms["mixer_out"].settle(x, pending)
            rt.record(f"{self.prefix}.out", x)
        return stream, pending

    def forward(self, stream, pending, step, cache, writes_cache=True):
        h = self.pre_mixer(stream, pending)
        a = self.mixer.forward(h, step, cache, writes_cache)
        return self.post_mixer(stream, a, step)


class SideBySideGatedStreamBlock(Block):
    """x + g1 * mixer(shift(norm1(x))) + g2 * ff(norm2(x)) on a float32 stream: both sublayers read the same x, each result is
    multiplied by a gate of its normed input (g1 of norm1(x) ahead of the shift, g2 of norm2(x)), and the mixer's input is
    shifted by a token.  Its norms are ``GatedStreamRMSNorm``s named "mixer" and "feed_forward"; its extras "mixer_gate",
    "feed_forward_gate" (``ResidualGate``) and "shift" (``TokenShift``).  A layer may have no feed-forward.  What is handed on
    beside the stream is all that is pending (``PendingGated``): ONE kernel adds it, norms the sum twice and shifts it.  The
    stream that a block is given stays as it is; a run of the layer keeps what its mixer keeps and a row a request."""

    keeps_stream = True

    def __init__(self, mixer, feed_forward, norms, extras=None):
        super().__init__(mixer, feed_forward, norms, extras)
        self.shift, self.gate = self.extras["shift"], self.extras["mixer_gate"]
        self.fed_gate = self.extras["feed_forward_gate"] if feed_forward is not None else None
        self.w_fed = None

    def prepare(self):
        # the feed-forward's first product and its gate's read the same input: one product over both
        if self.feed_forward is not None:
            self.w_fed = torch.cat([self.feed_forward.w_first, self.fed_gate.weight], 0).contiguous()
            n = self.feed_forward.w_first.shape[0]
            self.feed_forward.w_first, self.fed_gate.weight = self.w_fed[:n], self.w_fed[n:]

    def cache_need(self):
        return CompositeNeed((self.mixer.cache_need(), self.shift.cache_need()))

    def owner(self, path):
        return super().owner(path[1:]) if path[:1] == (0,) else self.shift

    def add_ahead(self, stream, pending, embedded, vector):
        pending = pending or PendingGated()
        pending.embedded, pending.vector = embedded, vector
        return stream, pending

    def forward(self, stream, pending, step, cache, writes_cache=True):
        rt, norm1, norm2 = self.mixer.rt, self.norms["mixer"], self.norms["feed_forward"]
        kept, last = cache
        new = lambda: torch.empty(stream.shape, dtype=rt.dtype, device=stream.device)
        h, shifted, h2 = new(), new(), new() if self.feed_forward is not None else None
        x = torch.empty_like(stream) if pending is not None else None
        ops.gated_sum_norm32(stream, norm1.gain, h, norm1.eps, x_out=x, shift=self.shift.mix, shifted=shifted, segments=step.segments,
                             state=last, gain2=norm2.gain if h2 is not None else None, out2=h2,
                             **(pending.arguments() if pending is not None else {}))
        stream = stream if x is None else x
        if hasattr(self.mixer, "forward_terms"):
            terms = self.mixer.forward_terms(shifted, step, kept, writes_cache)
        else:
            terms = [(self.mixer.forward(shifted, step, kept, writes_cache), 1.0)]
        out = PendingGated(terms, (self.gate.logits(h), self.gate.bias))
        if h2 is not None:
            u = ops.linear(h2, self.w_fed, status=rt.status)
            n = self.feed_forward.w_first.shape[0]
            out.fed, out.fed_gate = self.feed_forward.forward_rest(u[:, :n], step), (u[:, n:], self.fed_gate.bias)
        if rt.trace is not None and self.prefix:
            rt.record(f"{self.prefix}.out", norm1.settled(stream, out))
        return stream, out


class SideBySideStreamBlock(Block):
    """x + m (mixer(norm(x)) + ff(norm(x))) on a float32 stream: both sublayers read ONE norm of x.  Its norm is a
    ``TermsStreamNorm`` named "mixer", which holds the model's constant m.  A layer may have no feed-forward.  What is handed on
    beside the stream is what is pending: the mixer's terms (two mixers side by side give one each) and the feed-forward's
    output, with their constants; ONE kernel adds them and norms the sum."""

    def forward(self, stream, pending, step, cache, writes_cache=True):
        rt, norm = self.mixer.rt, self.norms["mixer"]
        h = norm.add_norm(stream, pending)
        if hasattr(self.mixer, "forward_terms"):
            terms = list(self.mixer.forward_terms(h, step, cache, writes_cache))
        else:
            terms = [(self.mixer.forward(h, step, cache, writes_cache), 1.0)]
        if self.feed_forward is not None:
            terms.append((self.feed_forward.forward(h, step), 1.0))
        pending = [(t, norm.mult * c) for t, c in terms]
        if rt.trace is not None and self.prefix:
            rt.record(f"{self.prefix}.out", norm.settled(stream, pending))
        return stream, pending


register_block("side_by_side_gated_stream32", SideBySideGatedStreamBlock)
register_block("side_by_side_stream32", SideBySideStreamBlock)
register_block("prenorm_residual", PreNormResidualBlock)
register_block("prenorm_stream32", PreNormStreamBlock)
register_block("outnorm_residual", OutputNormResidualBlock)
register_block("sandwich_stream32", SandwichStreamBlock)
