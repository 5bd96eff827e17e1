"""Small Tubevik configurations for the tests, and random weights for them.

Sizes differ between the configurations and between the layers of one: heads that share kv heads and heads that do not, key
and value sizes that differ, sizes that are no multiple of a 16-byte vector and sizes the tensor-core attention takes; whole,
partial and no rotation, with and without YaRN's scaling; windows and chunks inside a page, on page borders and over many, and
none; layers that borrow keys and values from one whose window is wider, narrower or absent; one tap and many; one inner size of
the products in two factors after another; layers without a feed-forward, limits that clamp much and little; a residual constant
of one, below and above it; no cap on the logits; models of one mixer kind.  Weights are drawn so that scores, caps, decays,
gates and clamps all decide something.
"""

import json
import os

import torch

YARN = dict(factor=8.0, original=64, fast=16.0, slow=1.0)


def rotation(dims, base=10000.0, scaling=None):
    if not dims:
        return None
    r = dict(dims=dims, base=base)
    if scaling:
        r["scaling"] = dict(scaling)
    return r


def _attention(heads, kv_heads, dim, vdim, scale, mask, rot):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else 1.5 / dim ** 0.5)
    if mask:
        m["mask"] = dict(size=mask)
    if rot:
        m["rot"] = rot
    return m


def attention(heads, kv_heads, dim, vdim, window=20, rot=None, softcap=4.0, kv_from=None, scale=None):
    m = _attention(heads, kv_heads, dim, vdim, scale, window, rot)
    if softcap:
        m["softcap"] = softcap
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m)


def left(heads, kv_heads, dim, vdim, chunk=24, rot=None, scale=None):
    return _attention(heads, kv_heads, dim, vdim, scale, chunk, rot)


def right(heads, kv_heads, dim, vdim, conv=4):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def parallel(l, r, left_scale=1.0, right_scale=1.0):
    return dict(type="parallel", mixer=dict(left=l, right=r, left_scale=left_scale, right_scale=right_scale))


def dense(ff, limit=1.2):
    return dict(kind="dense", ff=ff, limit=limit)


def layer(mix, mlp):
    return dict(mix, mlp=mlp)


def model(vocab, width, layers, eps=1e-5, cap=20.0, mult=0.6):
    c = dict(architecture="Tubevik", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, layers=layers)
    if cap:
        c["logit_softcap"] = cap
    return c


# S: both mixers in turn, a layer that borrows from a layer two before it with a narrower window of its own, one without feed-forward
SMALL = model(200, 64, [
    layer(attention(4, 2, 16, 8, window=21, rot=rotation(8, 100.0, YARN), softcap=3.0), dense(96)),
    layer(parallel(left(4, 2, 16, 24, chunk=21, rot=rotation(8, 50.0)), right(4, 2, 16, 8, conv=3), 0.7, 1.3), dense(80, 0.7)),
    layer(attention(4, 2, 16, 8, window=9, rot=rotation(16, 300.0), softcap=None, kv_from=0), None),
    layer(parallel(left(2, 2, 8, 16, chunk=32), right(3, 3, 8, 16, conv=1), 1.1, 0.6), dense(48, 3.0))])

# O: sizes that are no multiple of eight, a window shorter than a page, two borrowers (one wider than its lender, one that sees all),
# a convolution longer than most portions, no cap
ODD = model(333, 90, [
    layer(parallel(left(5, 5, 12, 20, chunk=7, rot=rotation(12, 1000.0)), right(5, 1, 20, 12, conv=9), 1.5, 0.25), None),
    layer(attention(6, 3, 20, 12, window=5, rot=rotation(20, 1000.0, dict(factor=2.0, original=48, fast=8.0, slow=2.0)), softcap=1.5), dense(50)),
    layer(attention(6, 3, 20, 12, window=33, rot=rotation(20, 1000.0, dict(factor=2.0, original=48, fast=8.0, slow=2.0)), kv_from=1), dense(70, 0.4)),
    layer(attention(6, 3, 20, 12, window=0, rot=rotation(6, 30.0), kv_from=1, softcap=8.0), None),
    layer(parallel(left(6, 1, 24, 24, chunk=0, scale=0.5), right(2, 2, 12, 37, conv=2), 0.3, 2.0), dense(70))], eps=1e-6, cap=None, mult=1.0)

# W: sizes the tensor-core attention takes, more query heads than one tile's rows, wide states, a lender that is borrowed from twice
WIDE = model(512, 128, [
    layer(attention(20, 1, 32, 64, window=48, rot=rotation(32, 1e4, YARN), softcap=6.0), dense(192, 2.0)),
    layer(attention(20, 1, 32, 64, window=100, rot=rotation(32, 1e4, YARN), softcap=6.0, kv_from=0), dense(256)),
    layer(parallel(left(8, 2, 64, 32, chunk=100, rot=rotation(64, 1e6)), right(4, 4, 64, 64), 0.5, 2.0), dense(64)),
    layer(parallel(left(16, 4, 32, 32, chunk=64, rot=rotation(16, 1e4)), right(2, 1, 128, 32, conv=4), 1.2, 0.8), None),
    layer(attention(20, 1, 32, 64, window=16, rot=rotation(32, 1e4), kv_from=0), dense(128, 1.0))], cap=30.0, mult=0.4)

# only windowed layers; only side-by-side layers
WINDOW_ONLY = model(128, 48, [layer(attention(3, 3, 16, 16, window=16, rot=rotation(2, 3.0), softcap=2.0), dense(64)),
                              layer(attention(8, 2, 8, 24, window=40, softcap=None), None)], mult=1.5)
PARALLEL_ONLY = model(128, 48, [layer(parallel(left(3, 3, 16, 16, chunk=16), right(1, 1, 16, 16)), dense(64)),
                                layer(parallel(left(8, 2, 8, 8, chunk=40, rot=rotation(8)), right(6, 3, 8, 24, conv=5), 0.4, 0.9), dense(32))], cap=5.0)

CONFIGS = dict(small=SMALL, odd=ODD, wide=WIDE, window_only=WINDOW_ONLY, parallel_only=PARALLEL_ONLY)


def mixer_shapes(kind, m, D, p, ranks=(5, 3)):
    """name -> (shape, kind) of one mixer's tensors under prefix p; D is the mixer's input width, ranks the inner sizes of the
    decays' and the gate's product in two factors."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    if kind == "right":
        C = {f"{p}.q": G * d, f"{p}.k": G * d, f"{p}.v": H * e}
        out = {n: ((c, D), "matrix") for n, c in C.items()}
        out.update({f"{n}.conv": ((c, m["conv"]), "taps") for n, c in C.items()})
        out.update({f"{p}.b": ((H, D), "matrix"), f"{p}.A_log": ((H,), "rate"), f"{p}.norm": ((e,), "gain"), f"{p}.a1": ((ranks[0], D), "matrix"),
                    f"{p}.a2": ((H * d, ranks[0]), "matrix"), f"{p}.dt_bias": ((H * d,), "bias"), f"{p}.g1": ((ranks[1], D), "matrix"),
                    f"{p}.g2": ((H * e, ranks[1]), "matrix"), f"{p}.o": ((D, H * e), "matrix")})
        return out
    out = {f"{p}.q": ((H * d, D), "matrix"), f"{p}.o": ((D, H * e), "matrix")}
    if m.get("kv_from") is None:
        out.update({f"{p}.k": ((G * d, D), "matrix"), f"{p}.v": ((G * e, D), "matrix")})
    if kind == "attention":
        out.update({f"{p}.g": ((H, D), "matrix"), f"{p}.q.b": ((H * d,), "bias"), f"{p}.q.norm": ((H * d,), "gain")})
        if m.get("kv_from") is None:
            out.update({f"{p}.k.b": ((G * d,), "bias"), f"{p}.v.b": ((G * e,), "bias"), f"{p}.k.norm": ((G * d,), "gain")})
    elif kind != "left":
        raise ValueError(kind)
    return out


def tensor_shapes(cfg):
    """name -> (shape, kind)."""
    D = cfg["width"]
    norm = lambda n: {n: ((D,), "gain"), f"{n}.b": ((D,), "bias")}
    out = {"embed": ((cfg["vocab"], D), "table"), "head": ((cfg["vocab"], D), "matrix"), **norm("embed.norm"), **norm("final.norm")}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}"
        out.update(norm(f"{p}.norm1"))
        if L["type"] == "parallel":
            out.update(mixer_shapes("left", m["left"], D, f"{p}.mix.left"))
            out.update(mixer_shapes("right", m["right"], D, f"{p}.mix.right", ranks=[(5, 3), (16, 24), (1, 8), (33, 1), (8, 16)][i % 5]))
        else:
            out.update(mixer_shapes("attention", m, D, f"{p}.mix"))
        if L.get("mlp") is not None:
            ff, q = L["mlp"]["ff"], f"{p}.mlp"
            out.update({f"{q}.gate": ((ff, D), "matrix"), f"{q}.up": ((ff, D), "matrix"), f"{q}.down": ((D, ff), "matrix")})
    return out


def draw(shapes, seed):
    """bfloat16 tensors (what a model file holds) for name -> (shape, kind)."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, (shape, kind) in shapes.items():
        r = lambda: torch.randn(shape, generator=g)
        if kind == "gain":
            t = 1.0 + 0.2 * r()
        elif kind == "bias":
            t = 0.5 * r()
        elif kind == "rate":
            t = -2.0 + 1.5 * r()                  # decays from nearly one down to a fraction a token
        elif kind == "taps":
            t = r() / shape[-1] ** 0.5
        elif kind == "table":
            t = 0.3 + r()                         # (a mean that the layer norm takes off)
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
    d = os.path.join(str(folder), f"tubevik_{name}_{seed}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), w)
    return d, cfg, {k: v.double() for k, v in w.items()}
