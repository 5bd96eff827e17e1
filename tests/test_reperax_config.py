"""Reperax without a GPU: the configuration reader, the description as parts and the order layers run in, the tensors it asks
for, what a layer asks of the cache manager (pages that go back chunk by chunk, state slots, the shift's row, all under one
layer), where a chunk's attention begins, and the plain implementation against itself."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_reperax as P
from reperax_models import CONFIGS, ODD, SMALL, WIDE, random_weights, tensor_shapes, write_model

from paged_llm_rs_b200.cache.manager import CacheManager
from paged_llm_rs_b200.config.registry import resolve_architecture
from paged_llm_rs_b200.errors import ConfigError, UnsupportedModelError, WeightError
from paged_llm_rs_b200.kernels import attention_plan
from paged_llm_rs_b200.parts.base import CompositeNeed, JoinedKVNeed, StateNeed
from paged_llm_rs_b200.parts.decoder import DecoderModel, Runtime, tensor_specs_of
from paged_llm_rs_b200.weights.loader import check_tensors


def describe(cfg):
    arch = resolve_architecture(cfg)
    return arch, arch.describe(arch.parse(cfg))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_parts_ask_for_the_files_tensors(name):
    cfg = CONFIGS[name]
    arch, spec = describe(cfg)
    assert arch.name == "Reperax"
    specs = tensor_specs_of(spec)
    shapes = {n: tuple(shape) for n, (shape, _) in tensor_shapes(cfg).items()}
    assert {s.name for s in specs if not s.optional} == set(shapes)
    assert all(s.fits(shapes[s.name]) for s in specs if s.name in shapes)
    check_tensors(specs, shapes)
    # a layer without feed-forward: that sublayer's norm and gate may lie in the file
    assert all(s.name.split(".")[1] in ("norm2", "rg2") for s in specs if s.optional)


def test_the_inner_size_of_the_decays_product_comes_from_the_file():
    _, spec = describe(SMALL)
    specs = {s.name: s for s in tensor_specs_of(spec)}
    assert specs["l1.mix.right.a1"].fits((7, 64)) and specs["l1.mix.right.a2"].fits((24, 7))
    assert not specs["l1.mix.right.a1"].fits((7, 65)) and not specs["l1.mix.right.a2"].fits((24, 7, 1))
    shapes = {n: tuple(shape) for n, (shape, _) in tensor_shapes(SMALL).items()}
    with pytest.raises(WeightError):
        check_tensors(specs.values(), dict(shapes, **{"l1.mix.right.a1": (7, 63)}))
    model = DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32))
    w = {k: v.float() for k, v in random_weights(SMALL, 0).items()}
    w["l1.mix.right.a1"] = torch.zeros(9, 64)
    with pytest.raises(WeightError):
        model.bind(w)                                   # the two factors do not meet


def test_every_constant_comes_from_the_configuration():
    cfg = copy.deepcopy(SMALL)
    cfg["norm"]["eps"], cfg["logit_softcap"] = 1e-3, 3.5
    cfg["layers"][0]["mixer"].update(decay=[0.25, 0.75])
    cfg["layers"][0]["mixer"]["rot"] = dict(dims=4, base=77.0)
    par = cfg["layers"][1]["mixer"]
    par.update(left_scale=0.11, right_scale=9.0)
    par["left"].update(scale=0.9, mask=dict(size=13))
    par["right"]["tau"] = 2.25
    cfg["loop"] = dict(start=0, stop=2, times=3)
    _, spec = describe(cfg)
    r = spec.layers[0].mixer.params
    assert (r["decay"], r["rot_dims"], r["rot_base"], r["eps"]) == ([0.25, 0.75], 4, 77.0, 1e-3)
    l, g = spec.layers[1].mixer.params["parts"]
    assert (l["scale"], g["scale"], l["under"], g["under"]) == (0.11, 9.0, "left", "right")
    assert (l["params"]["scale"], l["params"]["chunk"], l["params"]["qk_norm"], l["params"]["eps"]) == (0.9, 13, "projection", 1e-3)
    assert g["params"]["tau"] == 2.25 and g["params"]["eps"] == 1e-3
    assert spec.head.params["softcap"] == 3.5 and spec.final_norm.params["eps"] == 1e-3 and spec.final_norm.params["one_plus"]
    assert spec.layers[2].feed_forward is None and spec.layers[0].feed_forward.params["eps"] == 1e-3
    assert [(e.layer, e.add_embedding, e.add_pass) for e in spec.schedule] == \
        [(0, False, 0), (1, False, None), (0, True, 1), (1, False, None), (0, True, 2), (1, False, None), (2, False, None), (3, False, None)]
    assert spec.pass_vectors.params == dict(width=64, times=3)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_layers_run_in_the_plain_implementations_order(name):
    cfg = CONFIGS[name]
    _, spec = describe(cfg)
    spec.validate()
    assert [(e.layer, e.add_pass) for e in spec.schedule] == P.runs(cfg)
    assert all(e.add_embedding == bool(e.add_pass) for e in spec.schedule)
    assert all(e.reads_cache_of is None for e in spec.schedule)           # every pass keeps a cache or state of its own


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="ring"), UnsupportedModelError),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), ConfigError),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5]), ConfigError),
    (lambda c: c["layers"][0]["mixer"].pop("decay"), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["right"].update(tau=0.0), ConfigError),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), ConfigError),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), UnsupportedModelError),
    (lambda c: c["norm"].update(eps=0.0), ConfigError),
    (lambda c: c.update(logit_softcap=-1.0), ConfigError),
    (lambda c: c["loop"].update(stop=5), ConfigError),
    (lambda c: c["loop"].update(start=3), ConfigError),
    (lambda c: c["loop"].update(times=0), ConfigError),
    (lambda c: c.pop("layers"), ConfigError)])
def test_bad_configurations_are_refused(change, error):
    cfg = copy.deepcopy(SMALL)
    change(cfg)
    with pytest.raises(error):
        describe(cfg)


def test_what_may_be_absent():
    cfg = copy.deepcopy(SMALL)
    cfg.pop("loop"), cfg.pop("logit_softcap")
    cfg["layers"][0]["mixer"].pop("rot")
    cfg["layers"][1]["mixer"]["left"].pop("mask")
    cfg["layers"][1]["mlp"] = None
    _, spec = describe(cfg)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3] and spec.pass_vectors is None and spec.head.params["softcap"] is None
    assert spec.layers[0].mixer.params["rot_dims"] == 0 and spec.layers[1].mixer.params["parts"][0]["params"]["chunk"] == 0
    assert spec.layers[1].feed_forward is None


def test_cache_needs_groups_and_slots():
    _, spec = describe(SMALL)
    model = DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32))
    needs = model.cache_needs()
    assert len(needs) == 6 and all(isinstance(n, CompositeNeed) for n in needs)          # two layers run twice
    kept, shift = needs[0].parts
    assert isinstance(kept, StateNeed) and kept.shape == (2 * 16 * 24,) and shift == StateNeed((64,), torch.float32)
    (l, r), shift = needs[1].parts[0].parts, needs[1].parts[1]
    assert isinstance(l, JoinedKVNeed) and (l.kind, l.chunk, l.num_kv_heads, l.key_dim, l.value_dim, l.group_size) == ("chunk", 21, 2, 16, 8, 2)
    assert r.shape == (3 * 8 * 16,) and shift.shape == (64,)
    cm = CacheManager(needs, 8, 16, 4, torch.float32, "cpu")
    # the layer that runs twice has two caches in one group; the layer with another chunk has pages of its own
    assert [g.cells for g in cm.groups] == [[(1, 0, 0), (3, 0, 0)], [(5, 0, 0)]] and [g.chunk for g in cm.groups] == [21, 32]
    assert cm.prefix_cache is False
    caches = cm.layer_caches()
    (pool, gi), slots = caches[3][0]
    assert gi == 0 and tuple(pool.shape) == (16, 2, 8, 16 + 8) and pool.data_ptr() != caches[1][0][0][0].data_ptr()
    assert tuple(slots.shape) == (4, 3 * 8 * 16) and tuple(caches[3][1].shape) == (4, 64)
    assert tuple(caches[2][0].shape) == (4, 3 * 8 * 8) and tuple(caches[2][1].shape) == (4, 64)
    # the owner of each cell: the mixer that its group's attention is cut for
    blk = model.blocks[spec.schedule[1].layer]
    assert blk.owner((0, 0)) is blk.mixer.parts[0] and blk.owner((0, 1)) is blk.mixer.parts[1] and blk.owner((1,)) is blk.shift
    # a slot is zeroed when it is taken again
    cm.open("a")
    s = cm.get("a").state_slot
    for t in (slots, caches[3][1], caches[2][0], caches[0][1]):
        t[s] = 3.0
    cm.close("a")
    cm.open("b")
    assert cm.get("b").state_slot == s and all(float(t[s].abs().max()) == 0.0 for t in (slots, caches[3][1], caches[2][0], caches[0][1]))


@pytest.mark.parametrize("chunk,page", [(24, 8), (21, 8), (5, 8), (40, 16), (16, 16), (100, 4)])
def test_pages_of_finished_chunks_go_back(chunk, page):
    """Whatever the steps: after each, exactly the pages from the one with the current chunk's first position on are held, and
    the next chunk's first query still finds its own page."""
    need = JoinedKVNeed("chunk", 1, 8, 8, None, 0, chunk=chunk)
    most = -(-(chunk + 9) // page) + 1
    cm = CacheManager([need], page, most, 2, torch.float32, "cpu", allocate_device=False)
    cm.open("r")
    at, rng = 0, np.random.default_rng(chunk)
    while at < 5 * chunk:
        n = int(rng.integers(1, 10))
        assert cm.reserve("r", n), (at, n)
        cm.commit("r", n)
        at += n
        t = cm.get("r").tables[0]
        first = at // chunk * chunk                    # the first position that the next query sees
        assert [b >= 0 for b in t.blocks] == [(i + 1) * page > first for i in range(len(t.blocks))]
        cm.check_invariants()
    assert cm.pages_for(10 ** 6, 9) <= most
    cm.close("r")
    assert cm.available() == most


def test_attention_items_begin_where_their_chunk_begins():
    for chunk in (7, 64, 120):
        work, red, parts = attention_plan.plan_attention([(0, 50, 130), (50, 1, 119), (51, 1, 120), (52, 3, 0)], 8, None, 2, 1, chunk=chunk)
        for seg, q0, qn, p0, begin, end, part, split in work.tolist():
            assert begin == p0 // chunk * chunk and end == p0 + qn and part == -1
    # decoded tokens whose key range is cut in parts: together they cover the chunk and nothing before it
    work, red, parts = attention_plan.plan_attention([(0, 1, 999)], 8, None, 1, 64, chunk=500)
    assert len(work) > 1 and work[0][4] == 500 and work[-1][5] == 1000 and all(a[5] == b[4] for a, b in zip(work, work[1:]))


def test_native_packer_agrees_on_chunks():
    from test_step_pack import setup

    from paged_llm_rs_b200.engine.step import GroupPlanConfig, StepEntry
    needs = [JoinedKVNeed("chunk", 2, 16, 16, None, 0, chunk=90), JoinedKVNeed("full", 1, 16, 16)]
    plans = [GroupPlanConfig(8, 2, None, chunk=90), GroupPlanConfig(16, 1, None)]
    for target in (1, 296):
        cache, packer, caps, work_caps, native, out = setup(needs, plans, 700, 16, 8, 64, target)
        rng = np.random.default_rng(3)
        for i, ctx in enumerate([0, 1, 89, 90, 91, 179, 180, 500]):
            cache.open(i)
            assert cache.reserve(i, ctx + 1)
            cache.commit(i, ctx)
        entries = [StepEntry(i, [int(rng.integers(0, 1000))], [0]) for i in range(8)]
        want, _, _ = packer.pack(entries, caps, work_caps)
        native.pack(entries, None, None)
        assert np.array_equal(out, want)


def test_random_weights_have_an_inner_size(tmp_path):
    from paged_llm_rs_b200.weights.random_init import random_tensors
    _, spec = describe(SMALL)
    t = random_tensors(spec, 1)
    assert t["l1.mix.right.a1"].shape[0] == t["l1.mix.right.a2"].shape[1] > 0
    check_tensors(tensor_specs_of(spec), {n: tuple(x.shape) for n, x in t.items() if not n.startswith(("l2.norm2", "l2.rg2"))})


def test_plain_token_by_token_equals_whole():
    """The plain implementation keeps nothing between calls: a prefix's logits are the whole's."""
    for cfg in (SMALL, ODD, WIDE):
        w = {k: v.double() for k, v in random_weights(cfg, 3).items()}
        toks = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
        whole = P.forward(cfg, w, toks)
        assert torch.allclose(P.forward(cfg, w, toks[:17]), whole[:17], atol=1e-9)


def test_plain_mechanisms_alone():
    F = P.F64
    # the norm whose file holds gain - 1
    x = torch.tensor([[3.0, 4.0]], dtype=F)
    assert torch.allclose(P.norm_one_plus(x, torch.tensor([0.0, 1.0], dtype=F), 0.0), torch.tensor([[3.0, 8.0]], dtype=F) / math.sqrt(12.5))
    # the shift mixes in the token before; the first token has a zero before it
    h = torch.tensor([[2.0, 4.0], [10.0, 20.0]], dtype=F)
    assert P.token_shift(h, torch.tensor([0.25, 1.0], dtype=F)).tolist() == [[1.5, 0.0], [8.0, 4.0]]
    # chunks are counted from the sequence's start
    assert [list(P.visible_keys(t, 3)) for t in (0, 2, 3, 5, 6)] == [[0], [0, 1, 2], [3], [3, 4, 5], [6]]
    assert list(P.visible_keys(4, 0)) == [0, 1, 2, 3, 4]
    q = torch.zeros(4, 1, 2, dtype=F)
    v = torch.tensor([1.0, 3.0, 100.0, 200.0], dtype=F).view(4, 1, 1)
    assert P.chunked_attention(q, q, v, 1.0, 2).flatten().tolist() == [1.0, 2.0, 100.0, 150.0]
    # a decay acts on the rows that belong to key entries
    k = torch.tensor([[[1.0, 1.0]], [[0.0, 0.0]]], dtype=F)
    alpha = torch.tensor([[[1.0, 1.0]], [[0.5, 0.0]]], dtype=F)
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 10.0]]], dtype=F)
    assert P.linear_recurrence(q, k, torch.tensor([[[6.0]], [[1.0]]], dtype=F), alpha).flatten().tolist() == [6.0, 3.0]
    # sigmoid(z)^(1 / tau)
    w = {"r.a1": torch.tensor([[1.0, 1.0]], dtype=F), "r.a2": torch.tensor([[2.0], [0.0]], dtype=F), "r.a2.b": torch.tensor([0.0, 0.5], dtype=F)}
    got = P.channel_decay(torch.tensor([[0.25, 0.5]], dtype=F), w, "r", 2.0)
    assert torch.allclose(got, torch.sigmoid(torch.tensor([[1.5, 0.5]], dtype=F)).sqrt())
    # the polynomial of normed powers: each power over its own root mean square
    u = torch.tensor([[1.0, -2.0]], dtype=F)
    got = P.poly_norm(u, torch.tensor([1.0, 10.0, 100.0, 7.0], dtype=F), 0.0)
    want = u / math.sqrt(2.5) + 10 * u ** 2 / math.sqrt(8.5) + 100 * u ** 3 / math.sqrt(32.5) + 7
    assert torch.allclose(got, want)
    # rotation turns pairs (i, i + dims / 2) and leaves the rest
    x = torch.arange(8, dtype=F).view(1, 1, 8)
    r = P.rotate_half(x, [3], 4, 10.0)
    assert torch.equal(r[..., 4:], x[..., 4:])
    assert abs(float(r[0, 0, 0]) - (0 * math.cos(3.0) - 2 * math.sin(3.0))) < 1e-12 and abs(float(r[0, 0, 2]) - (2 * math.cos(3.0) + 0 * math.sin(3.0))) < 1e-12


def test_every_piece_of_the_plain_implementation_decides_something():
    """The random weights are such that leaving any one mechanism out moves the logits: what the engine is compared with
    would show it."""
    w = {k: v.double() for k, v in random_weights(SMALL, 3).items()}
    toks = torch.randint(0, SMALL["vocab"], (60,), generator=torch.Generator().manual_seed(2)).tolist()
    base = P.forward(SMALL, w, toks)

    def moved(cfg=SMALL, **zeroed):
        ww = {k: torch.zeros_like(v) if any(k.endswith(z) for z in zeroed.get("ends", [])) else v for k, v in w.items()}
        d = P.forward(cfg, ww, toks) - base
        return float(d.pow(2).mean().sqrt() / base.pow(2).mean().sqrt())
    assert all(moved(ends=[z]) > 0.03 for z in (".shift", ".rg1", ".rg2", "loop.step", ".a2", ".a2.b", ".act", "left.o", "right.o"))
    for change in (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=20), lambda c: c["layers"][1]["mixer"]["left"].pop("mask"),
                   lambda c: c["layers"][0]["mixer"].pop("rot"), lambda c: c["layers"][0]["mixer"].update(decay=[0.9, 0.9]),
                   lambda c: c["layers"][3]["mixer"]["right"].update(tau=2.0), lambda c: c.update(logit_softcap=10.0)):
        cfg = copy.deepcopy(SMALL)
        change(cfg)
        assert moved(cfg) > 0.005, change
