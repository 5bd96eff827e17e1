"""Tubevik, described as parts.

A decoder on a float32 stream whose layers are listed in its configuration.  In a layer (``side_by_side_stream32``) mixer and
feed-forward read the same layer norm of the stream and are added to it together, times the model's constant.  The mixers:

  attention   grouped-query attention inside a sliding window (``normed_qk_attention``): biases on q, k and v, q and k normed over
              the whole projection and then rotated in halves with YaRN's frequencies, capped scores, a sigmoid gate a head; a
              layer may attend over an earlier one's keys and values
  parallel    two mixers on the same input, added with a constant each (``parallel_mixers``): attention within chunks of the
              sequence, q and k rotated in pairs and then normed a head, one more in the softmax's denominator
              (``normed_qk_attention``), beside the gated delta rule with a decay a key entry (``channel_gated_delta_rule``)

The feed-forward is gated and clamped.  A layer norm stands behind the embedding and ahead of the head, whose logits are capped.
Nothing bounds a request's length but float32 positions (exact up to 2^24).

Tensors: ``embed``, ``embed.norm``, ``final.norm``, ``head``, and per layer i ``l<i>.norm1``, ``l<i>.mix.*`` and ``l<i>.mlp.*`` (see the
parts for the leaves); a layer norm's bias has its name and ".b".
"""

from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.tubevik import TubevikConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 24      # positions enter the rotation as float32


def _rotation(rot, layout):
    return dict(rot_dims=rot.dims, rot_base=rot.base, rot_layout=layout, rot_scaling=rot.scaling.params() if rot.scaling is not None else None)


def _window_attention(W, m, eps, kept_for):
    return dict(hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
                biases=True, qk_norm="projection", softcap=m.softcap, window=m.window, cache_window=kept_for, gate="sigmoid",
                gate_per="head", keeps="own" if m.kv_from is None else "nothing", **_rotation(m.rot, "half"))


def _chunk_attention(W, m, eps):
    return dict(hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
                qk_norm="head_after_rotation", chunk=m.chunk, sink_one=True, **_rotation(m.rot, "pairs"))


def _delta_rule(W, m, eps):
    return dict(hidden_size=W, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, conv=m.conv, eps=eps)


def _kept_for(layers, i):
    """How many tokens back layer i's keys and values are read, by itself or by a layer that borrows them (0: all)."""
    windows = [L.mixer.window for j, L in enumerate(layers) if L.mixer_kind == "attention" and i in (j, L.mixer.kv_from)]
    return 0 if 0 in windows else max(windows)


def describe_tubevik(cfg: TubevikConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("terms_stream32", dict(width=W, eps=eps, mult=cfg.residual_mult, centered=True, leaf=""), name)
    layers, schedule = [], []
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}", L.mixer
        reads = None
        if L.mixer_kind == "attention":
            reads = m.kv_from
            mixer = PartSpec("normed_qk_attention", _window_attention(W, m, eps, _kept_for(cfg.layers, i) if reads is None else m.window),
                             f"{p}.mix")
        else:
            mixer = PartSpec("parallel_mixers", dict(parts=[
                dict(kind="normed_qk_attention", params=_chunk_attention(W, m.left, eps), under="left", scale=m.left_scale),
                dict(kind="channel_gated_delta_rule", params=_delta_rule(W, m.right, eps), under="right", scale=m.right_scale)]), f"{p}.mix")
        ff = None
        if L.mlp is not None:
            ff = PartSpec("swiglu_mlp", dict(hidden_size=W, intermediate_size=L.mlp.ff, activation="clamped", limit=L.mlp.limit,
                                             names=dict(gate="gate", up="up", down="down")), f"{p}.mlp")
        layers.append(LayerSpec(block="side_by_side_stream32", mixer=mixer, feed_forward=ff, norms={"mixer": norm(f"{p}.norm1")}, prefix=p))
        schedule.append(ScheduleEntry(i, reads_cache_of=reads))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=W,
        vocab_size=cfg.vocab,
        max_positions=MAX_POSITIONS,
        embedding=PartSpec("normed_token_embedding", dict(vocab_size=cfg.vocab, hidden_size=W, eps=eps, leaf="", norm="embed.norm",
                                                          centered=True), "embed"),
        layers=layers,
        schedule=schedule,
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(vocab_size=cfg.vocab, hidden_size=W, leaf="", softcap=cfg.logit_softcap), "head"),
    )


TUBEVIK = Architecture(name="Tubevik", parse=TubevikConfig.from_dict, describe=describe_tubevik, aliases=("tubevik",))
register_architecture(TUBEVIK)
