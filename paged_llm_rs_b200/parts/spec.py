"""A model as data: which parts each layer is made of and in which order layers run.

An architecture's ``describe(config)`` returns a ``ModelSpec``.  The generic
decoder (``parts/decoder.py``) builds it from the part registries; no part and
no builder code knows which architecture it serves.

The reference assembles one fixed block type in code
(crates/pagedllm/src/model/mod.rs:84-136, 174-257); here the same assembly is a
list, so that a later architecture can give different layers different mixers
and feed-forwards, run a layer twice, or let a layer read another layer's cache.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple


@dataclass(frozen=True)
class TensorSpec:
    """One tensor a part needs from the weight file.

    role decides the dtype it is kept in:
      "matrix"  compute dtype (bfloat16 when serving, float32 on the 32-bit path)
      "gain"    float32 always (norm gains; an exact upcast from bfloat16)
      "matrix32" float32 always (a matrix whose product is formed in float: a router)
      "offset"  float32 always (a vector added to float values: a router's correction)
      "index"   int32 (integer tables)
      "keep"    as stored (a tensor stored in 32-bit stays so)
    A size that only the file knows (the inner size of a product in two factors, say) is None in ``shape``; the part checks
    in ``bind`` that its tensors agree.  ``drawn`` is the whole shape that a random model gets then.
    """

    name: str
    shape: Tuple[Optional[int], ...]
    role: str = "matrix"
    optional: bool = False
    drawn: Optional[Tuple[int, ...]] = None

    def fits(self, shape) -> bool:
        return len(shape) == len(self.shape) and all(a is None or a == b for a, b in zip(self.shape, shape))


@dataclass
class PartSpec:
    """kind picks the class from a registry; params are its sizes and constants;
    prefix is where its tensors live in the weight file."""

    kind: str
    params: Dict[str, Any] = field(default_factory=dict)
    prefix: str = ""


@dataclass
class LayerSpec:
    block: str  # arrangement, e.g. "prenorm_residual"
    mixer: PartSpec
    feed_forward: Optional[PartSpec]  # None: the layer has no feed-forward (for arrangements that allow it)
    norms: Dict[str, PartSpec]  # the norms the arrangement names, e.g. "mixer", "feed_forward"
    prefix: str = ""
    extras: Dict[str, PartSpec] = field(default_factory=dict)  # further parts the arrangement names, e.g. gates on results


@dataclass(frozen=True)
class ScheduleEntry:
    """One run of a layer.  ``layer`` indexes ModelSpec.layers and may appear
    several times in a schedule.  ``reads_cache_of`` names an earlier schedule
    entry whose cache this run attends over instead of writing its own.  Right before it runs, the stream as the embedding
    left it is added to the residual stream (``add_embedding``), and row ``add_pass`` of the model's pass vectors."""

    layer: int
    reads_cache_of: Optional[int] = None
    add_embedding: bool = False
    add_pass: Optional[int] = None


@dataclass
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: List[LayerSpec]
    schedule: List[ScheduleEntry]
    final_norm: PartSpec
    head: PartSpec
    position_encodings: Dict[str, PartSpec] = field(default_factory=dict)
    pass_vectors: Optional[PartSpec] = None     # one vector a pass through layers that run several times

    def validate(self) -> None:
        for i, e in enumerate(self.schedule):
            if not 0 <= e.layer < len(self.layers):
                raise ValueError(f"schedule entry {i} names layer {e.layer}, the model has {len(self.layers)}")
            if e.add_pass is not None and self.pass_vectors is None:
                raise ValueError(f"schedule entry {i} adds a pass vector, the model has none")
            if e.reads_cache_of is not None:
                j = e.reads_cache_of
                if not 0 <= j < i:
                    raise ValueError(f"schedule entry {i} reads the cache of entry {j}, which does not run before it")
                if self.schedule[j].reads_cache_of is not None:
                    raise ValueError(f"schedule entry {i} reads the cache of entry {j}, which owns none")
