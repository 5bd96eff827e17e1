"""The generic decoder: a ModelSpec built from the part registries.

Runs the schedule entry by entry (crates/pagedllm/src/model/mod.rs:315-352 is
the fixed-order original): embedding, each scheduled layer with the cache the
cache manager made for that entry, then the final norm on the wanted rows only
and the head (mod.rs:340-351).
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from . import (attention, block, diff_attention, embedding, feed_forward, gated_residual, latent_attention,  # noqa: F401  (register the parts)
               linear_attention, mamba2, matrix_memory, norm, normed_attention, parallel, position, routed_feed_forward,
               sink_attention)
from .base import (BLOCKS, EMBEDDINGS, EXTRAS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITION_ENCODINGS, Runtime, StepState,
                   make)
from .spec import ModelSpec, TensorSpec


class DecoderModel:
    def __init__(self, spec: ModelSpec, rt: Runtime):
        spec.validate()
        self.spec, self.rt = spec, rt
        self.position_encodings = {name: make(POSITION_ENCODINGS, "position encoding", ps, rt)
                                   for name, ps in spec.position_encodings.items()}
        self.embedding = make(EMBEDDINGS, "embedding", spec.embedding, rt)
        self.blocks = []
        for ls in spec.layers:
            mixer = make(MIXERS, "mixer", ls.mixer, rt, position_encodings=self.position_encodings)
            ff = make(FEED_FORWARDS, "feed-forward", ls.feed_forward, rt) if ls.feed_forward is not None else None
            norms = {k: make(NORMS, "norm", ns, rt) for k, ns in ls.norms.items()}
            if ls.block not in BLOCKS:
                raise KeyError(f"no block arrangement {ls.block!r} is registered; known: {sorted(BLOCKS)}")
            extras = {k: make(EXTRAS, "extra part", es, rt) for k, es in ls.extras.items()}
            self.blocks.append(BLOCKS[ls.block](mixer, ff, norms, **(dict(extras=extras) if extras else {})))
            self.blocks[-1].prefix = ls.prefix
        self.final_norm = make(NORMS, "norm", spec.final_norm, rt)
        self.head = make(HEADS, "head", spec.head, rt)
        self.pass_vectors = make(EXTRAS, "extra part", spec.pass_vectors, rt) if spec.pass_vectors is not None else None
        self.schedule = list(spec.schedule)
        self._runs_twice = len({e.layer for e in self.schedule}) < len(self.schedule)

    def parts(self):
        yield from self.position_encodings.values()
        yield self.embedding
        for b in self.blocks:
            yield b.mixer
            if b.feed_forward is not None:
                yield b.feed_forward
            yield from b.norms.values()
            yield from b.extras.values()
        if self.pass_vectors is not None:
            yield self.pass_vectors
        yield self.final_norm
        yield self.head

    def tensor_specs(self) -> List[TensorSpec]:
        return [t for p in self.parts() for t in p.tensors()]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts():
            p.bind(tensors)
        for b in self.blocks:
            b.prepare()

    def cache_needs(self) -> List[Optional[object]]:
        """Per schedule entry what its block needs of the cache manager; None for
        an entry that reads another entry's cache or needs nothing."""
        return [None if e.reads_cache_of is not None else self.blocks[e.layer].cache_need()
                for e in self.schedule]

    def capturable(self) -> bool:
        """Whether a step of this model can be captured and replayed: every mixer either launches
        fixed kernels only (``graph_safe``) or sits in a block that can be run in halves around it."""
        return all(getattr(b.mixer, "graph_safe", False) or (b.pre_mixer is not None and b.post_mixer is not None)
                   for b in self.blocks)

    def forward(self, step: StepState, caches: List[object], outside=None) -> torch.Tensor:
        """Run the step's tokens; return float32 logits [step.n_wanted, vocab].  ``outside``
        (for a step that is being captured): called as outside(fn, like) for every mixer that is
        not ``graph_safe``; it runs fn() outside the capture, now and at every replay, and returns
        a tensor shaped like ``like`` that holds fn()'s result each time."""
        step.carry = {}
        residual = self.embedding.forward(step.tokens)
        for encoding in self.position_encodings.values():
            residual = encoding.at_embedding(residual, step)
        embedded = None
        if any(e.add_embedding for e in self.schedule):
            embedded = residual if all(b.keeps_stream for b in self.blocks) else residual.clone()
        delta = None
        for i, e in enumerate(self.schedule):
            own = e.reads_cache_of is None
            blk, cache = self.blocks[e.layer], caches[i if own else e.reads_cache_of]
            if e.add_embedding or e.add_pass is not None:
                residual, delta = blk.add_ahead(residual, delta, embedded if e.add_embedding else None,
                                                self.pass_vectors.vector(e.add_pass) if e.add_pass is not None else None)
            if outside is not None and not getattr(blk.mixer, "graph_safe", False):
                h = blk.pre_mixer(residual, delta)
                a = outside(lambda blk=blk, h=h, cache=cache, own=own: blk.mixer.forward(h, step, cache, own), h)
                residual, delta = blk.post_mixer(residual, a, step)
                continue
            residual, delta = blk.forward(residual, delta, step, cache, own)
            if self._runs_twice and self.rt.trace is not None and f"{blk.prefix}.out" in self.rt.trace:
                self.rt.trace[f"run{i}.out"] = self.rt.trace[f"{blk.prefix}.out"]      # (a later run of the layer writes its name again)
        if self.schedule:
            residual, delta = self.blocks[self.schedule[-1].layer].settle(residual, delta)
        if step.n_wanted == 0:
            # A portion in the middle of a prompt runs only to fill the cache (mod.rs:336-346).
            return torch.zeros((0, self.spec.vocab_size), dtype=torch.float32, device=self.rt.device)
        h = self.final_norm.add_norm(residual, delta, rows=step.logit_rows)
        logits = self.head.forward(h)
        self.rt.record("logits", logits)
        return logits


def tensor_specs_of(spec: ModelSpec) -> List[TensorSpec]:
    """The tensors a model of this description reads, without building anything
    on a device (used by the random-weights writer and by weight checks)."""
    return DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32)).tensor_specs()
