"""Tubevik without a GPU: the configuration reader, the description as parts and what layers that borrow keys and values make of
it, the tensors it asks for, what a layer asks of the cache manager (pages kept as long as any borrower reads them, pages of
finished chunks, state slots), the rotation's frequencies, and the plain implementation against itself."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_tubevik as P
from tubevik_models import CONFIGS, ODD, SMALL, WIDE, YARN, attention, dense, layer, model, random_weights, rotation, tensor_shapes

from paged_llm_rs_b200.cache.manager import CacheManager
from paged_llm_rs_b200.config.registry import resolve_architecture
from paged_llm_rs_b200.errors import ConfigError, UnsupportedModelError, WeightError
from paged_llm_rs_b200.parts.base import CompositeNeed, JoinedKVNeed, StateNeed, stack_rows
from paged_llm_rs_b200.parts.decoder import DecoderModel, Runtime, tensor_specs_of
from paged_llm_rs_b200.parts.position import rotary_frequencies
from paged_llm_rs_b200.weights.loader import check_tensors


def describe(cfg):
    arch = resolve_architecture(cfg)
    return arch, arch.describe(arch.parse(cfg))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_parts_ask_for_the_files_tensors(name):
    cfg = CONFIGS[name]
    arch, spec = describe(cfg)
    assert arch.name == "Tubevik"
    spec.validate()
    specs = tensor_specs_of(spec)
    shapes = {n: tuple(shape) for n, (shape, _) in tensor_shapes(cfg).items()}
    assert {s.name for s in specs} == set(shapes) and not any(s.optional for s in specs)
    check_tensors(specs, shapes)


def test_inner_sizes_come_from_the_file():
    _, spec = describe(SMALL)
    specs = {s.name: s for s in tensor_specs_of(spec)}
    for one, two, rows in (("a1", "a2", 64), ("g1", "g2", 32)):
        assert specs[f"l1.mix.right.{one}"].fits((7, 64)) and specs[f"l1.mix.right.{two}"].fits((rows, 7))
        assert not specs[f"l1.mix.right.{one}"].fits((7, 65)) and not specs[f"l1.mix.right.{two}"].fits((rows + 1, 7))
        model_ = DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32))
        w = {k: v.float() for k, v in random_weights(SMALL, 0).items()}
        w[f"l1.mix.right.{one}"] = torch.zeros(9, 64)
        with pytest.raises(WeightError):
            model_.bind(w)                                   # the two factors do not meet


def test_every_constant_comes_from_the_configuration():
    cfg = copy.deepcopy(SMALL)
    cfg["norm"]["eps"], cfg["logit_softcap"], cfg["residual_mult"] = 1e-3, 3.5, 0.25
    a = cfg["layers"][0]["mixer"]
    a.update(scale=0.9, softcap=7.0, mask=dict(size=13), rot=dict(dims=4, base=77.0, scaling=dict(factor=3.0, original=11, fast=5.0, slow=2.0)))
    par = cfg["layers"][1]["mixer"]
    par.update(left_scale=0.11, right_scale=9.0)
    par["left"].update(scale=0.8, mask=dict(size=17), rot=dict(dims=2, base=5.0))
    par["right"]["conv"] = 6
    cfg["layers"][1]["mlp"]["limit"] = 0.125
    _, spec = describe(cfg)
    p = spec.layers[0].mixer.params
    assert (p["scale"], p["softcap"], p["window"], p["rot_dims"], p["rot_base"], p["eps"]) == (0.9, 7.0, 13, 4, 77.0, 1e-3)
    assert p["rot_scaling"] == dict(factor=3.0, original=11.0, fast=5.0, slow=2.0) and p["rot_layout"] == "half" and p["biases"]
    assert (p["qk_norm"], p["gate"], p["gate_per"]) == ("projection", "sigmoid", "head")
    l, r = spec.layers[1].mixer.params["parts"]
    assert (l["scale"], r["scale"], l["under"], r["under"]) == (0.11, 9.0, "left", "right")
    q = l["params"]
    assert (q["scale"], q["chunk"], q["rot_dims"], q["rot_base"], q["rot_layout"], q["qk_norm"], q["sink_one"], q["eps"]) == \
        (0.8, 17, 2, 5.0, "pairs", "head_after_rotation", True, 1e-3)
    assert r["params"]["conv"] == 6 and r["params"]["eps"] == 1e-3
    f = spec.layers[1].feed_forward.params
    assert (f["activation"], f["limit"], f["intermediate_size"]) == ("clamped", 0.125, 80) and spec.layers[2].feed_forward is None
    assert spec.head.params["softcap"] == 3.5 and spec.head.prefix == "head"
    for n in [spec.final_norm] + [x.norms["mixer"] for x in spec.layers]:
        assert n.params["mult"] == 0.25 and n.params["centered"] and n.params["eps"] == 1e-3
    assert spec.embedding.params["centered"] and spec.embedding.params["eps"] == 1e-3


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="ring"), UnsupportedModelError),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), ConfigError),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), ConfigError),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=1.0), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), ConfigError),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), ConfigError),          # not an attention layer
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), ConfigError),          # itself
    (lambda c: c["layers"][2]["mixer"].update(kv_from=7), ConfigError),
    (lambda c: c["layers"][2]["mixer"].update(heads=2), ConfigError),            # other heads than its lender
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=3), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["right"].update(conv=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), ConfigError),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), UnsupportedModelError),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), ConfigError),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), ConfigError),
    (lambda c: c["norm"].update(eps=0.0), ConfigError),
    (lambda c: c.update(logit_softcap=-1.0), ConfigError),
    (lambda c: c.pop("layers"), ConfigError)])
def test_bad_configurations_are_refused(change, error):
    cfg = copy.deepcopy(SMALL)
    change(cfg)
    with pytest.raises(error):
        describe(cfg)


def test_a_borrower_has_a_lender_of_its_own_keys():
    cfg = copy.deepcopy(ODD)
    cfg["layers"][3]["mixer"]["kv_from"] = 2                    # layer 2 borrows itself
    with pytest.raises(ConfigError):
        describe(cfg)


def test_what_may_be_absent():
    cfg = copy.deepcopy(SMALL)
    cfg.pop("logit_softcap")
    for k in ("rot", "mask", "softcap"):
        cfg["layers"][0]["mixer"].pop(k)
    cfg["layers"][1]["mixer"]["left"].pop("mask")
    cfg["layers"][1]["mlp"] = None
    _, spec = describe(cfg)
    p = spec.layers[0].mixer.params
    assert p["rot_dims"] == 0 and p["window"] == 0 and p["softcap"] is None and spec.head.params["softcap"] is None
    assert spec.layers[1].mixer.params["parts"][0]["params"]["chunk"] == 0 and spec.layers[1].feed_forward is None


def test_keys_and_values_are_kept_as_long_as_any_borrower_reads_them():
    kept = lambda cfg: [(L.mixer.params.get("keeps"), L.mixer.params.get("window"), L.mixer.params.get("cache_window"), e.reads_cache_of)
                        for L, e in zip(describe(cfg)[1].layers, describe(cfg)[1].schedule)]
    assert kept(SMALL) == [("own", 21, 21, None), (None, None, None, None), ("nothing", 9, 9, 0), (None, None, None, None)]
    assert kept(ODD)[1:4] == [("own", 5, 0, None), ("nothing", 33, 33, 1), ("nothing", 0, 0, 1)]           # one borrower sees all
    assert kept(WIDE)[:2] == [("own", 48, 100, None), ("nothing", 100, 100, 0)]
    # two lenders of equal windows, one of which is read further back, do not share pages
    a = lambda **k: layer(attention(2, 1, 8, 8, rot=rotation(4), **k), dense(16))
    _, spec = describe(model(50, 16, [a(window=12), a(window=12), a(window=12, kv_from=0), a(window=30, kv_from=1)]))
    m = DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32))
    cm = CacheManager(m.cache_needs(), 4, 64, 2, torch.float32, "cpu")
    assert [(g.window, g.entries) for g in cm.groups] == [(12, [0]), (30, [1])]
    cm.open("r")
    for at in range(0, 60, 3):
        assert cm.reserve("r", 3)
        cm.commit("r", 3)
        for g, t in zip(cm.groups, cm.get("r").tables):
            first = max(0, at + 3 - g.window + 1)
            assert [b >= 0 for b in t.blocks] == [(i + 1) * 4 > first for i in range(len(t.blocks))]


def test_cache_needs_groups_and_slots():
    _, spec = describe(SMALL)
    m = DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32))
    needs = m.cache_needs()
    assert isinstance(needs[0], JoinedKVNeed) and (needs[0].kind, needs[0].window, needs[0].key_dim, needs[0].value_dim) == ("window", 21, 16, 8)
    assert needs[2] is None                                     # it reads layer 0's
    assert isinstance(needs[1], CompositeNeed)
    l, r = needs[1].parts
    assert (l.kind, l.chunk, l.num_kv_heads, l.key_dim, l.value_dim, l.group_size) == ("chunk", 21, 2, 16, 24, 2)
    # every head's matrix, and a ring of one row more of inputs than the convolution reaches back to
    assert isinstance(r, StateNeed) and r.dtype == torch.float32 and r.shape == (4 * 16 * 8 + 3 * (2 * 2 * 16 + 4 * 8),)
    assert needs[3].parts[1].shape == (3 * 8 * 16,)             # one tap: nothing is kept of the inputs
    cm = CacheManager(needs, 8, 16, 4, torch.float32, "cpu")
    assert [g.cells for g in cm.groups] == [[0], [(1, 0)], [(3, 0)]] and cm.prefix_cache is False
    caches = cm.layer_caches()
    assert caches[2] is None and tuple(caches[0][0].shape) == (16, 2, 8, 24)
    cm.open("a")
    s = cm.get("a").state_slot
    caches[1][1][s] = 3.0
    cm.close("a")
    cm.open("b")
    assert cm.get("b").state_slot == s and float(caches[1][1][s].abs().max()) == 0.0


def test_stacked_rows_are_filled_up():
    a, b = torch.ones(3, 4), 2 * torch.ones(6, 4)
    w = stack_rows([a, b])
    assert w.shape == (16, 4) and w.sum(1).tolist() == [4.0] * 3 + [8.0] * 6 + [0.0] * 7
    assert stack_rows([torch.ones(8, 4)]).shape == (8, 4)


@pytest.mark.parametrize("dims,base,s", [(48, 5e5, dict(factor=6.0, original=2048, fast=24.0, slow=1.5)), (8, 100.0, YARN), (2, 50.0, YARN),
                                         (128, 1e4, dict(factor=40.0, original=4096, fast=32.0, slow=1.0)), (16, 10.0, dict(factor=2.0, original=7, fast=40.0, slow=9.0)),
                                         (20, 1e3, dict(factor=1.0, original=48, fast=8.0, slow=2.0)), (32, 1e4, dict(factor=5.0, original=1e9, fast=4.0, slow=3.9))])
def test_yarn_frequencies(dims, base, s):
    """The product's against the plain ones, and what they are for: pairs that turn often keep their frequency, pairs that turn
    less than once are slowed by the factor."""
    got, factor = rotary_frequencies(dims, base, s)
    want, wf = P.yarn_frequencies(dims, base, s)
    assert np.allclose(got, want, rtol=1e-12) and abs(factor - wf) < 1e-12 and abs(factor - (0.1 * math.log(s["factor"]) + 1)) < 1e-12
    plain, one = rotary_frequencies(dims, base)
    assert one == 1.0 and np.allclose(plain, P.plain_frequencies(dims, base))
    ratio = got / plain
    assert (ratio <= 1 + 1e-12).all() and (ratio >= 1 / s["factor"] - 1e-12).all() and (np.diff(ratio) <= 1e-12).all()
    turns = s["original"] * plain / (2 * math.pi)
    width = 2.0 * math.log(base) / dims                    # (the borders are rounded outward to whole pairs)
    assert np.allclose(ratio[turns > s["fast"] * math.exp(width)], 1.0)


def test_plain_token_by_token_equals_whole():
    """The plain implementation keeps nothing between calls: a prefix's logits are the whole's."""
    for cfg in (SMALL, ODD):
        w = {k: v.double() for k, v in random_weights(cfg, 3).items()}
        toks = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
        whole = P.forward(cfg, w, toks)
        assert torch.allclose(P.forward(cfg, w, toks[:17]), whole[:17], atol=1e-9)


def test_plain_mechanisms_alone():
    F = P.F64
    t = lambda *x: torch.tensor(x, dtype=F)
    # the mean is taken off and the squared deviations' mean divides
    got = P.layer_norm(t([1.0, 3.0, 5.0]), t(1.0, 2.0, 1.0), t(0.0, 0.5, -1.0), 0.0)
    assert torch.allclose(got, t([-2.0, 0.0, 2.0]) / math.sqrt(8 / 3) * t(1.0, 2.0, 1.0) + t(0.0, 0.5, -1.0))
    # a window of three: itself and two before it; chunks are counted from the sequence's start
    assert [P.in_window(i, 3) for i in (0, 2, 3, 9)] == [0, 0, 1, 7] and P.in_window(9, 0) == 0
    assert [P.in_chunk(i, 3) for i in (0, 2, 3, 5, 6)] == [0, 0, 3, 3, 6] and P.in_chunk(9, 0) == 0
    q, v = torch.zeros(4, 1, 2, dtype=F), t(1.0, 3.0, 100.0, 200.0).view(4, 1, 1)
    assert P.attention(q, q, v, 1.0, lambda i: P.in_window(i, 2)).flatten().tolist() == [1.0, 2.0, 51.5, 150.0]
    # one more in the denominator, with scores of zero: one of two, of three, ...
    assert torch.allclose(P.attention(q, q, v, 1.0, lambda i: 0, extra_one=True).flatten(), t(0.5, 4 / 3, 26.0, 60.8))
    # a cap bounds the score
    k = t([[[1.0]], [[-1.0]]]).view(2, 1, 1)
    o = P.attention(100 * k.abs(), 100 * k, t(1.0, 0.0).view(2, 1, 1), 1.0, lambda i: 0, cap=2.0)
    assert abs(float(o[1]) - 1 / (1 + math.exp(-4.0))) < 1e-9
    # both layouts of pairs; the factor scales what is turned and nothing else
    x = torch.arange(8, dtype=F).view(1, 1, 8)
    r = P.rotate(x, [3], (4, [1.0, 0.1], 1.0), "half")
    assert torch.equal(r[..., 4:], x[..., 4:]) and abs(float(r[0, 0, 0]) - (0 * math.cos(3.0) - 2 * math.sin(3.0))) < 1e-12
    r = P.rotate(x, [3], (4, [1.0, 0.1], 2.0), "pairs")
    assert torch.equal(r[..., 4:], x[..., 4:])
    assert abs(float(r[0, 0, 2]) - 2 * (2 * math.cos(0.3) - 3 * math.sin(0.3))) < 1e-12 and abs(float(r[0, 0, 3]) - 2 * (3 * math.cos(0.3) + 2 * math.sin(0.3))) < 1e-12
    # a decay acts on the rows that belong to key entries; the read-out sees the token's own write; a key written again replaces
    k = t([[[1.0, 0.0]], [[1.0, 0.0]]]).view(2, 1, 2)
    g = t([[[1.0, 1.0]], [[0.5, 0.0]]]).view(2, 1, 2)
    o = P.delta_rule(k, k, t(6.0, 1.0).view(2, 1, 1), torch.ones(2, 1, dtype=F), g)
    assert o.flatten().tolist() == [6.0, 1.0]
    o = P.delta_rule(k, k, t(6.0, 1.0).view(2, 1, 1), 0.5 * torch.ones(2, 1, dtype=F), g)
    assert o.flatten().tolist() == [3.0, 1.25]               # 0.5 * 3 = 1.5, then half of the way to 1
    z = P.channel_decay(t([0.0, 1.0, 0.0, 1.0]), t(0.0, math.log(2.0)), t(0.0, 0.0, 0.0, 0.0), 2)
    sp = lambda y: math.log1p(math.exp(y))
    assert torch.allclose(z.flatten(), torch.exp(-t(sp(0.0), sp(1.0), 2 * sp(0.0), 2 * sp(1.0))))
    # the last column of the taps meets the current token
    c = P.causal_conv_silu(t([[1.0], [10.0], [100.0]]).view(3, 1), t([[2.0, 1.0]]).view(1, 2))
    assert torch.allclose(c, P.silu(t([[1.0], [12.0], [120.0]]).view(3, 1)))
    # the gate is bounded from above only, the up product on both sides
    w = {"m.gate": t([1.0]), "m.up": t([1.0]), "m.down": t([1.0])}
    ff = lambda y: float(P.clamped_ff(t([[y]]).view(1, 1), w, "m", 2.0))
    sg = lambda y: y / (1 + math.exp(-1.702 * y))
    assert abs(ff(5.0) - sg(2.0) * 3.0) < 1e-12 and abs(ff(-5.0) - sg(-5.0) * -1.0) < 1e-12 and abs(ff(1.0) - sg(1.0) * 2.0) < 1e-12


def test_every_piece_of_the_plain_implementation_decides_something():
    """The random weights are such that leaving any one mechanism out moves the logits: what the engine is compared with
    would show it."""
    w = {k: v.double() for k, v in random_weights(SMALL, 3).items()}
    toks = torch.randint(0, SMALL["vocab"], (60,), generator=torch.Generator().manual_seed(2)).tolist()
    base = P.forward(SMALL, w, toks)

    def moved(cfg=SMALL, ends=()):
        ww = {k: torch.zeros_like(v) if any(k.endswith(z) for z in ends) else v for k, v in w.items()}
        d = P.forward(cfg, ww, toks) - base
        return float(d.pow(2).mean().sqrt() / base.pow(2).mean().sqrt())
    pieces = ("embed.norm.b", "norm1.b", "final.norm.b", "mix.q.b", "mix.k.b", "mix.v.b", "mix.g", "right.b", "A_log", "right.a2", "right.dt_bias",
              "right.g2", "left.o", "right.o", "mlp.down", "q.conv", "k.conv")
    assert all(moved(ends=[z]) > 0.01 for z in pieces), {z: moved(ends=[z]) for z in pieces}
    L = lambda c, i: c["layers"][i]["mixer"]
    for change in (lambda c: L(c, 0)["mask"].update(size=20), lambda c: L(c, 2)["mask"].update(size=8), lambda c: L(c, 0).update(softcap=2.0),
                   lambda c: L(c, 0)["rot"].pop("scaling"), lambda c: L(c, 0).pop("rot"), lambda c: L(c, 1)["left"]["mask"].update(size=20),
                   lambda c: L(c, 1)["left"].pop("rot"), lambda c: L(c, 1).update(left_scale=0.6), lambda c: c["layers"][0]["mlp"].update(limit=0.8),
                   lambda c: c.update(logit_softcap=15.0), lambda c: c.update(residual_mult=0.5)):
        cfg = copy.deepcopy(SMALL)
        change(cfg)
        assert moved(cfg) > 0.003, change
