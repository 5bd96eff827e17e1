"""Reperax, described as parts.

A decoder whose layers are listed in its configuration and some of which run several times in a row with the same weights
(each run with a cache or state of its own); ahead of each such pass a vector of the pass, and from the second pass on the
embedding's output, is added to the stream.  In a layer (``side_by_side_gated_stream32``) mixer and feed-forward read the same
stream, each through a norm of its own (gains kept as their offset from one), the mixer's input is shifted by a token, and
each result is multiplied by a sigmoid gate of its input before it is added.  The mixers:

  retention   linear attention with a constant decay a head, rotated q and k (``retention``)
  parallel    two mixers on the same input, added with a constant each (``parallel_mixers``): attention within chunks of the
              sequence, q and k normed over the whole projection (``normed_qk_attention``), beside linear attention with a
              decay a key entry (``gated_linear_attention``)

The feed-forward has no gate; its activation is a polynomial of normed powers (``poly_norm_mlp``).  The head is the embedding
table, its logits capped.  Nothing bounds a request's length but float32 positions (exact up to 2^24).

Tensors: ``embed``, ``final.norm``, ``loop.step``, and per layer i ``l<i>.norm1|norm2|shift|rg1|rg1.b|rg2|rg2.b``, ``l<i>.mix.*`` and
``l<i>.mlp.*`` (see the parts for the leaves).
"""

from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.reperax import ReperaxConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 24      # positions enter the rotation as float32


def _attention(W, m, eps):
    return dict(hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
                qk_norm="projection", chunk=m.chunk)


def _linear_attention(W, m, eps):
    return dict(hidden_size=W, heads=m.heads, dim=m.dim, vdim=m.vdim, tau=m.tau, eps=eps)


def _schedule(layers: int, loop):
    """Entries in the order layers run; the first of a pass says what is added ahead of it."""
    if loop is None:
        return [ScheduleEntry(i) for i in range(layers)]
    passes = [ScheduleEntry(i, add_embedding=i == loop.start and t > 0, add_pass=t if i == loop.start else None)
              for t in range(loop.times) for i in range(loop.start, loop.stop)]
    return [ScheduleEntry(i) for i in range(loop.start)] + passes + [ScheduleEntry(i) for i in range(loop.stop, layers)]


def describe_reperax(cfg: ReperaxConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name, **more: PartSpec("rmsnorm_gated_stream32", dict(width=W, eps=eps, one_plus=True, leaf="", **more), name)
    layers = []
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}", L.mixer
        if L.mixer_kind == "retention":
            mixer = PartSpec("retention", dict(hidden_size=W, heads=m.heads, dim=m.dim, vdim=m.vdim, decay=list(m.decay), rot_dims=m.rot_dims,
                                               rot_base=m.rot_base, eps=eps), f"{p}.mix")
        else:
            mixer = PartSpec("parallel_mixers", dict(parts=[
                dict(kind="normed_qk_attention", params=_attention(W, m.left, eps), under="left", scale=m.left_scale),
                dict(kind="gated_linear_attention", params=_linear_attention(W, m.right, eps), under="right", scale=m.right_scale)]), f"{p}.mix")
        # (a layer without feed-forward: a file may hold that sublayer's norm and gate all the same; they are not used)
        unused = dict(optional=True) if L.dense_ff is None else {}
        gate = lambda name, **more: PartSpec("residual_gate", dict(hidden_size=W, width=W, **more), name)
        ff = None
        if L.dense_ff is not None:
            ff = PartSpec("poly_norm_mlp", dict(hidden_size=W, intermediate_size=L.dense_ff, eps=eps), f"{p}.mlp")
        layers.append(LayerSpec(block="side_by_side_gated_stream32", mixer=mixer, feed_forward=ff,
                                norms={"mixer": norm(f"{p}.norm1"), "feed_forward": norm(f"{p}.norm2", **unused)}, prefix=p,
                                extras={"shift": PartSpec("token_shift", dict(width=W), f"{p}.shift"), "mixer_gate": gate(f"{p}.rg1"),
                                        "feed_forward_gate": gate(f"{p}.rg2", **unused)}))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=W,
        vocab_size=cfg.vocab,
        max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab, hidden_size=W, leaf="", stream="float32"), "embed"),
        layers=layers,
        schedule=_schedule(len(layers), cfg.loop),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(vocab_size=cfg.vocab, hidden_size=W, leaf="", softcap=cfg.logit_softcap), "embed"),
        pass_vectors=PartSpec("pass_vectors", dict(width=W, times=cfg.loop.times), "loop.step") if cfg.loop is not None else None,
    )


REPERAX = Architecture(name="Reperax", parse=ReperaxConfig.from_dict, describe=describe_reperax, aliases=("reperax",))
register_architecture(REPERAX)
