"""Small Reperax configurations for the tests, and random weights for them.

Sizes differ between the configurations and between the layers of one: heads that share kv heads and heads that do not, key
and value sizes that differ, sizes that are no multiple of a 16-byte vector and sizes the tensor-core attention takes, whole,
partial and no rotation, chunks shorter than a page, chunks that end on a page's border and chunks that no page divides, no
chunks at all, decays of exactly one and of zero beside usual ones, one inner size of the decay's product after another, layers
without a feed-forward, loops over all layers, over some in the middle, over one, run once and three times, and no loop.
Weights are drawn so that scores, decays, gates, the shift and the passes all decide something.
"""

import json
import os

import torch


def retention(heads, dim, vdim, decay=None, rot=None, base=10000.0):
    decay = decay or [1.0 - 2.0 ** -(3 + 2 * i / max(1, heads - 1)) for i in range(heads)]
    m = dict(heads=heads, dim=dim, vdim=vdim, decay=decay)
    if rot:
        m["rot"] = dict(dims=rot, base=base)
    return dict(type="retention", mixer=m)


def left(heads, kv_heads, dim, vdim, chunk=24, scale=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else 1.5 / dim ** 0.5)
    if chunk:
        m["mask"] = dict(size=chunk)
    return m


def right(heads, dim, vdim, tau=8.0):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def parallel(l, r, left_scale=1.0, right_scale=1.0):
    return dict(type="parallel", mixer=dict(left=l, right=r, left_scale=left_scale, right_scale=right_scale))


def dense(ff):
    return dict(kind="dense", ff=ff)


def layer(mix, mlp):
    return dict(mix, mlp=mlp)


def model(vocab, width, layers, eps=1e-6, cap=20.0, loop=None):
    c = dict(architecture="Reperax", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if cap:
        c["logit_softcap"] = cap
    if loop:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


# S: both mixers, a layer with no feed-forward, a loop in the middle, a chunk that no page divides
SMALL = model(200, 64, [
    layer(retention(2, 16, 24, rot=8, base=100.0), dense(96)),
    layer(parallel(left(4, 2, 16, 8, chunk=21), right(3, 8, 16, tau=4.0), 0.7, 1.3), dense(80)),
    layer(retention(3, 8, 8, rot=8, base=50.0), None),
    layer(parallel(left(2, 2, 8, 16, chunk=32), right(2, 16, 8, tau=1.0), 1.1, 0.6), dense(48))], loop=(1, 3, 2))

# O: sizes that are no multiple of eight, chunks shorter than a page, decays of one and zero, one layer run three times, no cap
ODD = model(333, 90, [
    layer(parallel(left(5, 5, 12, 20, chunk=7), right(5, 20, 12, tau=16.0), 1.5, 0.25), None),
    layer(retention(4, 20, 12, decay=[1.0, 0.0, 0.5, 0.97], rot=20, base=1000.0), dense(50)),
    layer(parallel(left(6, 1, 24, 24, chunk=0, scale=0.5), right(1, 12, 36, tau=2.5), 0.3, 2.0), dense(70))], eps=1e-5, cap=None, loop=(1, 2, 3))

# W: sizes the tensor-core attention takes, more query heads than one tile's rows, wide states, all layers looped
WIDE = model(512, 128, [
    layer(parallel(left(20, 1, 32, 64, chunk=48), right(2, 64, 32), 1.0, 1.0), dense(192)),
    layer(retention(2, 64, 128, rot=64), dense(256)),
    layer(parallel(left(8, 2, 64, 32, chunk=100), right(4, 32, 64, tau=16.0), 0.5, 2.0), dense(64))], cap=30.0, loop=(0, 3, 2))

# only recurrent layers and no loop; only side-by-side layers, a loop that runs once
RETENTION_ONLY = model(128, 48, [layer(retention(1, 96, 8, rot=2, base=3.0), dense(64)), layer(retention(6, 8, 24), None)])
PARALLEL_ONLY = model(128, 48, [layer(parallel(left(3, 3, 16, 16, chunk=16), right(1, 16, 16)), dense(64)),
                                layer(parallel(left(8, 2, 8, 8, chunk=40), right(2, 8, 8, tau=3.0), 0.4, 0.9), dense(32))], cap=5.0, loop=(1, 2, 1))

CONFIGS = dict(small=SMALL, odd=ODD, wide=WIDE, retention_only=RETENTION_ONLY, parallel_only=PARALLEL_ONLY)


def mixer_shapes(kind, m, D, p, rank=5):
    """name -> (shape, kind) of one mixer's tensors under prefix p; D is the mixer's input width, rank the inner size of the
    decay's product."""
    H, d, e = m["heads"], m["dim"], m["vdim"]
    if kind == "left":
        G = m["kv_heads"]
        return {f"{p}.q": ((H * d, D), "matrix"), f"{p}.k": ((G * d, D), "matrix"), f"{p}.v": ((G * e, D), "matrix"),
                f"{p}.q.norm": ((H * d,), "gain"), f"{p}.k.norm": ((G * d,), "gain"), f"{p}.o": ((D, H * e), "matrix")}
    out = {f"{p}.q": ((H * d, D), "matrix"), f"{p}.k": ((H * d, D), "matrix"), f"{p}.v": ((H * e, D), "matrix"),
           f"{p}.g": ((H * e, D), "matrix"), f"{p}.o": ((D, H * e), "matrix")}
    if kind == "right":
        out.update({f"{p}.norm": ((e,), "gain"), f"{p}.a1": ((rank, D), "matrix"), f"{p}.a2": ((H * d, rank), "matrix"),
                    f"{p}.a2.b": ((H * d,), "decay_bias")})
    elif kind != "retention":
        raise ValueError(kind)
    return out


def tensor_shapes(cfg):
    """name -> (shape, kind)."""
    D = cfg["width"]
    out = {"embed": ((cfg["vocab"], D), "table"), "final.norm": ((D,), "offset_gain")}
    if cfg.get("loop"):
        out["loop.step"] = ((cfg["loop"]["times"], D), "vector")
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}"
        out[f"{p}.norm1"] = ((D,), "offset_gain")
        if L["type"] == "parallel":
            out.update(mixer_shapes("left", m["left"], D, f"{p}.mix.left"))
            out.update(mixer_shapes("right", m["right"], D, f"{p}.mix.right", rank=(5, 16, 1)[i % 3]))
        else:
            out.update(mixer_shapes("retention", m, D, f"{p}.mix"))
        out.update({f"{p}.shift": ((D,), "share"), f"{p}.rg1": ((D, D), "matrix"), f"{p}.rg1.b": ((D,), "bias")})
        if L.get("mlp") is not None:
            ff, q = L["mlp"]["ff"], f"{p}.mlp"
            out.update({f"{p}.norm2": ((D,), "offset_gain"), f"{q}.up": ((ff, D), "matrix"), f"{q}.down": ((D, ff), "matrix"),
                        f"{q}.act": ((4,), "coefficients"), f"{p}.rg2": ((D, D), "matrix"), f"{p}.rg2.b": ((D,), "bias")})
    return out


def draw(shapes, seed):
    """bfloat16 tensors (what a model file holds) for name -> (shape, kind)."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, (shape, kind) in shapes.items():
        r = lambda: torch.randn(shape, generator=g)
        if kind == "gain":
            t = 1.0 + 0.2 * r()
        elif kind == "offset_gain":
            t = 0.2 * r()
        elif kind == "bias":
            t = 0.5 * r()
        elif kind == "decay_bias":
            t = 3.0 + 1.5 * r()                   # decays from nearly one down to a fraction a token
        elif kind == "share":
            t = torch.rand(shape, generator=g)    # how much of the token before is mixed in
        elif kind == "coefficients":
            t = torch.tensor([0.8, -0.5, 0.4, 0.2]) + 0.2 * r()
        elif kind in ("table", "vector"):
            t = r()
        else:
            t = 1.3 * r() / shape[-1] ** 0.5
        w[name] = t.to(torch.bfloat16)
    return w


def random_weights(cfg, seed):
    return draw(tensor_shapes(cfg), seed)


def write_model(folder, name, seed=0, cfg=None, weights=None):
    """A model folder for configuration ``name``; returns (folder, config dict, float64 weights for the plain implementation)."""
    from paged_llm_rs_b200.weights.safetensors_io import write_safetensors

    cfg = cfg or CONFIGS[name]
    w = weights or random_weights(cfg, seed)
    d = os.path.join(str(folder), f"reperax_{name}_{seed}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), w)
    return d, cfg, {k: v.double() for k, v in w.items()}
