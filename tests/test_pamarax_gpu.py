"""Pamarax on the GPU against the plain implementation (tests/plain_pamarax.py): each kernel and each mixer alone (through
the cache manager and the step packer, with inputs made so that one far key, a missing extra one in the softmax, a
temperature that steps a token early or a lost state would show), then whole models through the engine's step function,
cache manager, state slots and scheduler."""

import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_pamarax as P
from pamarax_models import (CONFIGS, attention, dense, draw, layer, left, mixer_shapes, mlstm, model, parallel, right,
                            write_model)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
NAMES = {torch.float32: "float32", torch.bfloat16: "bfloat16"}
EPS = 1e-5


def ops_():
    from paged_llm_rs_b200.kernels import ops
    return ops


def close(got, want, dtype, what="", f32=2e-5, bf16=2e-2):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max()) / max(1e-9, float(want.abs().max()))
    assert err < (f32 if dtype == torch.float32 else bf16), f"{what}: relative error {err}"


def close_recurrent(got, want, dtype, what=""):
    """A recurrent mixer's output.  Each head's read-out is divided by its own root mean square, so a read-out that nearly
    cancels leaves at full size whatever it was, and rounding q, k and v to bfloat16 decides its direction: float32 is
    compared entry by entry, bfloat16 over all entries together, with no entry far out."""
    if dtype == torch.float32:
        return close(got, want, dtype, what, f32=1e-4)
    got, want = got.double().cpu(), want.double().cpu()
    rms = float((got - want).pow(2).mean().sqrt()) / max(1e-9, float(want.pow(2).mean().sqrt()))
    worst = float((got - want).abs().max()) / max(1e-9, float(want.abs().max()))
    assert rms < 3e-2 and worst < 0.3, f"{what}: root mean square of the error {rms}, largest {worst}, relative"


def status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def gen(seed):
    return torch.Generator().manual_seed(seed)


# ------------------------------------------------------------------------ each kernel alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 90), (300, 1024), (3, 4100), (2, 9000)])
def test_output_norm_sum_and_input_norm_in_one_pass(dtype, rows, width):
    ops = ops_()
    g = gen(0)
    x0 = torch.randn(rows, width, generator=g)
    a = (torch.randn(rows, width, generator=g) * 3).to(dtype)
    bias = torch.randn(width, generator=g)
    ga, gb = 1 + 0.2 * torch.randn(width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
    for b in (None, bias):
        ad = a.double() + (b.double() if b is not None else 0)
        summed = x0.double() + P.unit_rms(ad, EPS) * ga.double()
        normed = P.unit_rms(summed, EPS) * gb.double()
        bd = b.to(DEV) if b is not None else None
        # every row: the stream takes the sum
        x = x0.clone().to(DEV)
        y = torch.empty(rows, width, dtype=dtype, device=DEV)
        ops.sandwich_norm32(x, a.to(DEV), bd, ga.to(DEV), gb.to(DEV), y, EPS)
        close(x, summed, torch.float32, "stream", f32=1e-5)
        close(y, normed, dtype, "norm", bf16=8e-3)
        # some rows only: the sum is formed for them and not stored
        idx = torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
        x = x0.clone().to(DEV)
        y2 = torch.empty(2, width, dtype=dtype, device=DEV)
        ops.sandwich_norm32(x, a.to(DEV), bd, ga.to(DEV), gb.to(DEV), y2, EPS, rows=idx)
        assert torch.equal(x.cpu(), x0)
        close(y2, normed[[rows - 1, 0]], dtype, "norm of gathered rows", bf16=8e-3)
        # the sum alone, with no norm behind it
        x = x0.clone().to(DEV)
        ops.sandwich_norm32(x, a.to(DEV), bd, ga.to(DEV), None, None, EPS)
        close(x, summed, torch.float32, "sum alone", f32=1e-5)
    # nothing pending: the norm of the stream as it is
    y = torch.empty(rows, width, dtype=dtype, device=DEV)
    ops.sandwich_norm32(x0.to(DEV), None, None, None, gb.to(DEV), y, EPS)
    close(y, P.unit_rms(x0.double(), EPS) * gb.double(), dtype, "norm alone", bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,inter", [(3, 64), (70, 128), (5, 37), (300, 256)])
def test_gated_activation_with_biases_and_the_weighted_sum(dtype, rows, inter):
    ops = ops_()
    g = gen(1)
    gu = torch.randn(rows, 2 * inter, generator=g).to(dtype)
    bias = torch.randn(2 * inter, generator=g)
    out = torch.empty(rows, inter, dtype=dtype, device=DEV)
    ops.swiglu_bias(gu.to(DEV), bias.to(DEV), out)
    z = gu.double() + bias.double()
    close(out, P.silu(z[:, :inter]) * z[:, inter:], dtype, "activation with biases", bf16=1e-2)
    x, y = torch.randn(rows, inter, generator=g).to(dtype), torch.randn(rows, inter, generator=g).to(dtype)
    s = ops.scaled_sum2(x.to(DEV), y.to(DEV), 1.25, -0.4)
    close(s, 1.25 * x.double() - 0.4 * y.double(), dtype, "weighted sum", bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,nh,nkv,dk,dv,norm,rot,every,keys_as_values,page", [
    (9, 4, 2, 16, 16, "projection", 8, 0, True, 16), (40, 5, 5, 12, 20, "head", 0, 1, False, 8), (3, 8, 2, 64, 64, "projection", 64, 0, True, 16),
    (17, 20, 1, 32, 64, "head", 0, 4, False, 4), (6, 3, 3, 24, 8, None, 6, 3, False, 8), (5, 2, 1, 128, 128, "projection", 2, 0, True, 16)])
def test_qk_norm_temperature_rotation_and_the_cache_write(dtype, T, nh, nkv, dk, dv, norm, rot, every, keys_as_values, page):
    ops = ops_()
    g = gen(2)
    k_off, v_off = nh * dk, nh * dk + nkv * dk
    extra = 7                                                    # columns behind q | k | v that the kernel must not touch
    width = v_off + (0 if keys_as_values else nkv * dv) + extra
    proj = torch.randn(T, width, generator=g).to(dtype)
    sizes = {"projection": (nh * dk, nkv * dk), "head": (dk, dk), None: (0, 0)}[norm]
    qg, kg = 1 + 0.3 * torch.randn(sizes[0], generator=g), 1 + 0.3 * torch.randn(sizes[1], generator=g)
    base, coef = 77.0, 0.8
    inv_freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64).float() if rot else None
    pos = torch.arange(30, 30 + T, dtype=torch.int32)
    n_pages = 8 + T // page
    slots = torch.randperm(n_pages * page, generator=g)[:T].to(torch.int32)
    slots[0] = -1                                                # a token whose row is not written
    pool = torch.full((n_pages, nkv, page, dk + dv), 7.0, dtype=dtype, device=DEV)
    q = torch.empty(T, nh * dk, dtype=dtype, device=DEV)
    st = status()
    ops.normed_qk_kv_write(proj.to(DEV), k_off, v_off, q, qg.to(DEV) if norm else None, kg.to(DEV) if norm else None, norm, EPS, coef, every,
                           inv_freq.to(DEV) if rot else None, rot, pos.to(DEV), slots.to(DEV), pool, nh, nkv, dk, dv, keys_as_values, st)
    assert st.item() == 0
    pd = proj.double()
    qq, kk = pd[:, :k_off], pd[:, k_off:v_off]
    vv = kk.view(T, nkv, dk) if keys_as_values else pd[:, v_off:v_off + nkv * dv].view(T, nkv, dv)
    if norm == "projection":
        qq, kk = P.unit_rms(qq, EPS) * qg.double(), P.unit_rms(kk, EPS) * kg.double()
    qq, kk = qq.view(T, nh, dk), kk.view(T, nkv, dk)
    if norm == "head":
        qq, kk = P.unit_rms(qq, EPS) * qg.double(), P.unit_rms(kk, EPS) * kg.double()
    if every:
        qq = qq * torch.tensor([1.0 + coef * np.log((int(p) + 1) // every + 1) for p in pos], dtype=torch.float64)[:, None, None]
    qq, kk = P.rotate_half(qq, pos.tolist(), rot, base), P.rotate_half(kk, pos.tolist(), rot, base)
    # the angle is a float32 product: at position p its error is about p * 6e-8
    close(q.view(T, nh, dk), qq, dtype, "q", f32=1e-4, bf16=2e-2)
    rows = pool.double().cpu().permute(0, 2, 1, 3).reshape(n_pages * page, nkv, dk + dv)
    for t in range(1, T):
        close(rows[slots[t], :, :dk], kk[t], dtype, "cached key", f32=1e-4, bf16=2e-2)
        assert torch.equal(rows[slots[t], :, dk:], vv[t]), "a value is stored as it was projected"
    untouched = torch.ones(n_pages * page, dtype=torch.bool)
    untouched[slots[1:].long()] = False
    assert bool((rows[untouched] == 7.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["sigmoid", "silu"])
def test_gate_on_a_strided_view(dtype, kind):
    ops = ops_()
    g = gen(3)
    wide = torch.randn(33, 200, generator=g).to(dtype)
    y = torch.randn(33, 90, generator=g).to(dtype)
    got = ops.gate_mul(y.clone().to(DEV), wide.to(DEV)[:, 50:140], kind)
    z = wide.double()[:, 50:140]
    close(got, y.double() * (torch.sigmoid(z) if kind == "sigmoid" else P.silu(z)), dtype, "gate", bf16=1e-2)


# ------------------------------------------------------------------------ each mixer alone, through the cache manager

class MixerRig:
    """One mixer of a registered kind with the cache manager and the step packer the engine gives it: steps of
    (request, input rows [n, width]), several requests side by side; returns each request's output rows."""

    def __init__(self, kind, params, tensors, dtype, page=16, pages=64, max_requests=4):
        from paged_llm_rs_b200.cache.manager import CacheManager
        from paged_llm_rs_b200.engine.runner import group_plans
        from paged_llm_rs_b200.engine.step import StepPacker
        from paged_llm_rs_b200.parts import base, decoder  # noqa: F401  (registers the parts)
        from paged_llm_rs_b200.parts.spec import PartSpec
        self.dtype = dtype
        self.rt = base.Runtime(torch.device(DEV), dtype)
        self.mixer = base.make(base.MIXERS, "mixer", PartSpec(kind, params, "m"), self.rt)
        bound = {}
        for s in self.mixer.tensors():
            t = tensors[s.name]
            assert s.fits(tuple(t.shape)), s.name
            bound[s.name] = (t.to(dtype) if s.role == "matrix" else t.float()).to(DEV)
        self.mixer.bind(bound)
        self.cache = CacheManager([self.mixer.cache_need()], page, pages, max_requests, dtype, DEV, prefix_cache=False)
        of = lambda cell: self.mixer if not isinstance(cell, tuple) else self.mixer.parts[cell[1]]
        self.packer = StepPacker(self.cache, group_plans(self.cache, of, page), 296, 1000, 1 << 24, DEV)

    def step(self, entries):
        from paged_llm_rs_b200.engine.step import StepEntry
        es = []
        for rid, x in entries:
            if not self.cache.has(rid):
                self.cache.open(rid)
            assert self.cache.reserve(rid, x.shape[0]), "no pages left"
            es.append(StepEntry(rid, [0] * x.shape[0], []))
        host, layout, sizes = self.packer.pack(es)
        state = self.packer.to_state(torch.from_numpy(host).to(DEV), layout, sizes)
        x = torch.cat([x for _, x in entries]).to(self.dtype).to(DEV).contiguous()
        out = self.mixer.forward(x, state, self.cache.layer_caches()[0]).double().cpu()
        assert self.rt.status.item() == 0
        res, at = [], 0
        for rid, xi in entries:
            self.cache.commit(rid, xi.shape[0], None)
            res.append(out[at:at + xi.shape[0]])
            at += xi.shape[0]
        return res

    def end(self, rid):
        self.cache.close(rid)

    def cut(self, rid, x, cuts):
        """One request alone, its rows in portions."""
        assert sum(cuts) == x.shape[0]
        outs, at = [], 0
        for c in cuts:
            outs.append(self.step([(rid, x[at:at + c])])[0])
            at += c
        return torch.cat(outs)


def rounded(t, dtype):
    """What the engine is given: the compute dtype's rounding of t, as float64."""
    return t.to(dtype).double()


def attention_rig(dtype, m, W, seed, page=16, pages=64, craft=None):
    w = draw(mixer_shapes("attention", m, W, "m"), seed)
    if craft:
        craft(w)
    rot = m.get("rot") or {}
    params = dict(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["dim"], scale=m["scale"],
                  eps=EPS, qk_norm="projection", values_are_keys=True, rot_dims=rot.get("dims", 0), rot_base=rot.get("base", 1.0), gate="sigmoid")
    plain = {k.replace("m.", "L.mix.", 1): v.double() for k, v in w.items()}
    return MixerRig("normed_qk_attention", params, w, dtype, page, pages), lambda h: P.gated_attention_mixer(h, plain, "L", m, EPS)


def left_rig(dtype, m, W, seed, page=16, pages=64, craft=None):
    w = draw(mixer_shapes("left", m, W, "m"), seed)
    if craft:
        craft(w)
    qt = m.get("q_temp") or {}
    params = dict(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"],
                  eps=EPS, qk_norm="head", temp_coef=qt.get("coef", 0.0), temp_every=qt.get("every", 0), sink_one=True)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("normed_qk_attention", params, w, dtype, page, pages), lambda h: P.sink_attention_mixer(h, plain, "m", m, EPS)


def mlstm_rig(dtype, m, W, seed, max_requests=4):
    w = draw(mixer_shapes("mlstm", m, W, "m"), seed)
    params = dict(hidden_size=W, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], gate_cap=m["gate_cap"], eps=EPS)
    plain = {k.replace("m.", "L.mix.", 1): v.double() for k, v in w.items()}
    return MixerRig("matrix_lstm", params, w, dtype, max_requests=max_requests), lambda h: P.mlstm_mixer(h, plain, "L", m, EPS)


def delta_rig(dtype, m, W, seed, max_requests=4):
    w = draw(mixer_shapes("right", m, W, "m"), seed)
    params = dict(hidden_size=W, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"], eps=EPS)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("gated_delta_rule", params, w, dtype, max_requests=max_requests), lambda h: P.delta_mixer(h, plain, "m", m, EPS)


CUTS = [[75], [2] * 5 + [1, 1, 3, 17, 16, 20, 2, 1, 1, 1, 1, 1], [1] * 75, [40, 35], [64, 2, 9]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,rot,base,W,page", [(4, 2, 16, 8, 100.0, 64, 16), (6, 1, 24, 0, 1.0, 90, 8), (3, 3, 12, 12, 50.0, 40, 4),
                                                           (8, 2, 64, 32, 1e4, 128, 16), (2, 1, 128, 64, 5e5, 96, 16)])
def test_gated_attention_whole_in_portions_and_token_by_token(dtype, heads, kv, dim, rot, base, W, page):
    m = attention(heads, kv, dim, rot=rot, base=base)["mixer"]
    x = rounded(torch.randn(75, W, generator=gen(10)), dtype)
    for cuts in CUTS:
        rig, plain = attention_rig(dtype, m, W, 11, page=page)
        close(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}", f32=1e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,coef,every,W,page", [(4, 2, 16, 8, 0.3, 7, 64, 16), (5, 5, 12, 20, 1.0, 1, 90, 8), (20, 1, 32, 64, 0.0, 0, 128, 16),
                                                                  (8, 2, 64, 32, 2.0, 16, 128, 16), (3, 1, 24, 24, 4.0, 5, 48, 4)])
def test_attention_with_one_more_in_the_softmax_and_a_temperature(dtype, heads, kv, dim, vdim, coef, every, W, page):
    """The temperature steps at positions every - 1, 2 every - 1, ...: with a large coefficient a step taken one token early
    or late moves the output far beyond rounding, in a prompt's portion and in a decoded token, also on a page's border."""
    m = left(heads, kv, dim, vdim, coef=coef, every=every)
    x = rounded(torch.randn(75, W, generator=gen(12)), dtype)
    for cuts in CUTS:
        rig, plain = left_rig(dtype, m, W, 13, page=page)
        close(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}", f32=1e-4, bf16=3e-2)


def same_direction(w, heads, kv, dim, sign=1.0):
    """W_q of every head becomes sign * W_k of its kv head (plain gains): a token's query then points along (or against)
    the key of any token with the same input."""
    k = w["m.k"].view(kv, dim, -1)
    w["m.q"] = (sign * k.repeat_interleave(heads // kv, 0)).reshape(heads * dim, -1).contiguous()
    w["m.q.norm"], w["m.k.norm"] = torch.ones_like(w["m.q.norm"]), torch.ones_like(w["m.k.norm"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gated", "extra_one"])
def test_one_far_key_decides(dtype, kind):
    """The last token's input is a third of that of ONE earlier token, and queries point along keys: after the q/k norm that
    key scores like the token's own, and its value is three times as large, so it decides the output wherever it lies: the first token, a page's last and first row, hundreds of tokens back, the token before
    and the token itself; in a decoded token, at the end of a portion and beside other requests."""
    W, heads, kv, dim, ctx = 64, 4, 2, 32, 420
    g = gen(14)
    base_x = torch.randn(ctx + 1, W, generator=g)
    for at in (0, 15, 16, 255, 256, ctx - 1, ctx):
        x = base_x.clone()
        x[at] = 3.0 * x[ctx]
        x = rounded(x, dtype)
        if kind == "gated":
            m = attention(heads, kv, dim, scale=1.0)["mixer"]       # (no rotation: it would turn the far key away from the query)
            make = lambda: attention_rig(dtype, m, W, 15, pages=90, craft=lambda w: same_direction(w, heads, kv, dim))
        else:
            m = left(heads, kv, dim, 24, every=0, scale=1.0)
            make = lambda: left_rig(dtype, m, W, 15, pages=90, craft=lambda w: same_direction(w, heads, kv, dim))
        rig, plain = make()
        want = plain(x)
        # the reference itself: leaving the key out would change the last row by far more than the tolerance
        without = plain(torch.cat([x[:at], x[at + 1:]]))[-1] if at < ctx else None
        if without is not None:
            assert float((without - want[-1]).abs().max()) > 0.2 * float(want[-1].abs().max())
        got = rig.cut("a", x, [ctx, 1])
        close(got[-1:], want[-1:], dtype, f"decoded, key {at}", f32=1e-4, bf16=3e-2)
        rig, _ = make()
        got = rig.cut("b", x, [ctx - 20, 21])
        close(got[-1:], want[-1:], dtype, f"portion, key {at}", f32=1e-4, bf16=3e-2)
        rig, _ = make()
        other = rounded(torch.randn(40, W, generator=g), dtype)
        rig.step([("c", x[:ctx - 2]), ("d", other[:5])])
        res = rig.step([("d", other[5:6]), ("c", x[ctx - 2:]), ("e", other[6:])])
        close(res[1][-1:], want[-1:], dtype, f"batch, key {at}", f32=1e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_extra_one_takes_the_weight_when_every_score_is_low(dtype):
    """Queries point against every key: all scores are far below zero, the one in the denominator takes the weight and the
    output vanishes.  Without it the softmax would hand out all the weight and the output would be of the values' size."""
    W, heads, kv, dim, vdim = 48, 4, 2, 16, 8
    m = left(heads, kv, dim, vdim, every=0, scale=2.0)
    x = rounded(torch.randn(1, W, generator=gen(16)).repeat(30, 1), dtype)
    rig, plain = left_rig(dtype, m, W, 17, craft=lambda w: same_direction(w, heads, kv, dim, sign=-1.0))
    got, want = rig.cut("r", x, [13, 2, 14, 1]), plain(x)
    assert float(want.abs().max()) < 1e-6 and float(got.abs().max()) < 1e-4
    rig, plain = left_rig(dtype, m, W, 17, craft=lambda w: same_direction(w, heads, kv, dim, sign=1.0))
    got, want = rig.cut("r", x, [13, 2, 14, 1]), plain(x)
    assert float(want.abs().max()) > 0.1
    close(got, want, dtype, "scores far above zero", f32=1e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,cap,W", [(2, 8, 16, 10.0, 64), (3, 20, 12, 5.0, 90), (4, 64, 64, 15.0, 128), (1, 96, 8, 20.0, 48),
                                                   (6, 8, 24, 15.0, 48), (1, 256, 40, 15.0, 64), (2, 48, 48, 2.0, 72)])
def test_matrix_lstm_whole_in_portions_and_token_by_token(dtype, heads, dim, vdim, cap, W):
    m = mlstm(heads, dim, vdim, cap)["mixer"]
    x = rounded(torch.randn(75, W, generator=gen(18)) * 1.5, dtype)
    for cuts in CUTS:
        rig, plain = mlstm_rig(dtype, m, W, 19)
        close_recurrent(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,conv,W", [(4, 2, 8, 16, 3, 64), (3, 3, 20, 12, 2, 90), (4, 2, 64, 32, 4, 128), (2, 1, 128, 64, 5, 96),
                                                       (6, 1, 16, 24, 1, 48), (2, 2, 256, 16, 4, 64), (2, 1, 48, 40, 4, 72)])
def test_gated_delta_rule_whole_in_portions_and_token_by_token(dtype, heads, kv, dim, vdim, conv, W):
    m = right(heads, kv, dim, vdim, conv)
    x = rounded(torch.randn(75, W, generator=gen(20)) * 1.5, dtype)
    for cuts in CUTS:
        rig, plain = delta_rig(dtype, m, W, 21)
        close_recurrent(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["mlstm", "delta"])
def test_recurrent_mixers_in_batches_with_slots_used_again_and_long_decoding(dtype, kind):
    """Three slots for five requests: requests of unequal length side by side, a finished request's slot taken by the next
    (whose state must start at zero), a request left out of a step, and one request decoded for 300 tokens."""
    W = 64
    if kind == "mlstm":
        rig, plain = mlstm_rig(dtype, mlstm(3, 16, 24, 8.0)["mixer"], W, 23, max_requests=3)
    else:
        rig, plain = delta_rig(dtype, right(4, 2, 16, 8, 3), W, 23, max_requests=3)
    g = gen(22)
    lengths = dict(a=330, b=33, c=7, d=64, e=21)
    xs = {k: rounded(torch.randn(n, W, generator=g) * 1.5, dtype) for k, n in lengths.items()}
    want = {k: plain(x) for k, x in xs.items()}
    got, at = {k: [] for k in xs}, {k: 0 for k in xs}

    def run(step):
        res = rig.step([(k, xs[k][at[k]:at[k] + n]) for k, n in step])
        for (k, n), r in zip(step, res):
            got[k].append(r); at[k] += n
            if at[k] == lengths[k]:
                rig.end(k)
    run([("a", 20), ("b", 2), ("c", 1)])
    run([("a", 1), ("b", 31), ("c", 6)])              # b and c end: two slots are free again
    run([("d", 17), ("a", 1)])
    run([("e", 2), ("d", 47)])                        # a is left out of this step
    run([("a", 8), ("e", 19)])
    for _ in range(300):
        run([("a", 1)])
    for k in xs:
        assert at[k] == lengths[k]
        close_recurrent(torch.cat(got[k]), want[k], dtype, k)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_side_by_side_alone(dtype):
    """The two halves through one mixer: pages for the left, a slot for the right, the constants on the sum."""
    from paged_llm_rs_b200.parts import decoder  # noqa: F401
    W = 72
    l, r = left(6, 3, 16, 8, coef=0.7, every=9), right(4, 2, 8, 16, conv=3)
    w = dict(draw(mixer_shapes("left", l, W, "m.left"), 30), **draw(mixer_shapes("right", r, W, "m.right"), 31))
    lp = dict(hidden_size=W, num_heads=6, num_kv_heads=3, key_dim=16, value_dim=8, scale=l["scale"], eps=EPS, qk_norm="head",
              temp_coef=0.7, temp_every=9, sink_one=True)
    rp = dict(hidden_size=W, heads=4, kv_heads=2, dim=8, vdim=16, conv=3, eps=EPS)
    params = dict(parts=[dict(kind="normed_qk_attention", params=lp, under="left", scale=0.6),
                         dict(kind="gated_delta_rule", params=rp, under="right", scale=1.7)])
    plain = {k: v.double() for k, v in w.items()}
    x = rounded(torch.randn(75, W, generator=gen(32)), dtype)
    want = 0.6 * P.sink_attention_mixer(x, plain, "m.left", l, EPS) + 1.7 * P.delta_mixer(x, plain, "m.right", r, EPS)
    for cuts in CUTS:
        rig = MixerRig("parallel_mixers", params, w, dtype, page=8)
        close_recurrent(rig.cut("r", x, cuts), want, dtype, f"{cuts}")


# ------------------------------------------------------------------------ whole models through the engine

class Served:
    """A model on the engine's runner with its cache manager: steps of (request, tokens, wanted places)."""

    def __init__(self, folder, dtype, page=16, pages=64, max_requests=4):
        from paged_llm_rs_b200.engine.runner import ModelRunner
        self.runner = ModelRunner(folder, dtype=NAMES[dtype], page_size=page, num_pages=pages, max_requests=max_requests,
                                  prefix_cache=False, use_graphs=False)

    def step(self, entries, trace=None):
        from paged_llm_rs_b200.engine.step import StepEntry
        cache = self.runner.cache
        es = []
        for rid, toks, want in entries:
            if not cache.has(rid):
                cache.open(rid)
            assert cache.reserve(rid, len(toks)), "no pages left"
            es.append(StepEntry(rid, list(toks), list(want)))
        out = self.runner.step(es, trace=trace).double().cpu()
        for rid, toks, _ in entries:
            cache.commit(rid, len(toks), None)
        return out

    def end(self, rid):
        self.runner.cache.close(rid)


def errors(got, want):
    """Per position: difference of logits with its mean taken off, root mean square over the vocabulary, over the logits' own."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}


def rounding_alone(cfg, w, toks, want):
    """Per position, the error of the plain implementation itself when it runs in float32: what rounding alone does there."""
    P.F64 = torch.float32
    try:
        return errors(P.forward(cfg, w, toks).double(), want)
    finally:
        P.F64 = torch.float64


def agrees(got, want, dtype, rounding=None):
    """float32: every position within rounding (the fixed bound, or three times what rounding alone does at that position
    where that is more).  bfloat16: the typical position well within and nine in ten not far: where a
    recurrent head's read-out nearly cancels (the first tokens above all, when the state holds one or two keys), its norm
    makes rounding decide the head's direction, and such a position differs by a large part of its logits."""
    e = errors(got, want)
    if dtype == torch.float32:
        bound = torch.full_like(e, TOL[dtype]) if rounding is None else torch.clamp(3 * rounding.to(e), min=TOL[dtype])
        ok = bool((e < bound).all())
    else:
        ok = float(e.median()) < TOL[dtype] and float(e.quantile(0.9)) < 0.3
    if not ok:
        print(f"errors: median {float(e.median()):.3g}, over {float((e > TOL[dtype]).double().mean()):.3g}, max {float(e.max()):.3g} at {int(e.argmax())}")
    return ok


_models = {}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("pamarax")

    def get(name):
        if name not in _models:
            _models[name] = write_model(root, name, seed=sorted(CONFIGS).index(name))
        return _models[name]
    return get


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_every_layer(models, dtype, name):
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 45, 1)
    want, streams = P.forward(cfg, w, toks, want_layers=True)
    s = Served(folder, dtype)
    trace = {}
    got = s.step([("a", toks, list(range(len(toks))))], trace=trace)
    assert agrees(got, want, dtype)
    for i in range(len(cfg["layers"])):
        x = trace[f"l{i}.out"]
        assert x.dtype == torch.float32, "the stream between layers is float32 whatever the compute dtype"
        if dtype == torch.float32:
            close(x, streams[i], dtype, f"stream after layer {i}", f32=5e-5)
        else:
            per_token = (x.double().cpu() - streams[i]).pow(2).mean(-1).sqrt() / streams[i].pow(2).mean(-1).sqrt()
            assert float(per_token.median()) < TOL[dtype] and float(per_token.quantile(0.9)) < 0.3, f"stream after layer {i}: {per_token}"
    # the first tokens of a sequence, alone
    s2 = Served(folder, dtype)
    first = torch.cat([s2.step([("b", toks[:1], [0])]), s2.step([("b", toks[1:2], [0])]), s2.step([("b", toks[2:4], [0, 1])])])
    if dtype == torch.float32:
        assert agrees(first, want[:4], dtype)
    else:
        # (with one or two keys in a recurrent state a head's read-out is a value times q . k, and its norm keeps only the
        #  sign: rounding decides these positions, however the prompt is cut.  They may be as far off as in the whole prompt.)
        assert float(errors(first, want[:4]).max()) < max(0.3, 1.5 * float(errors(got[:4], want[:4]).max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("small", 16), ("odd", 8), ("wide", 32), ("recurrent_only", 16), ("attention_only", 4)])
def test_prefill_against_token_by_token_decoding(models, dtype, name, page):
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 70, 2)
    want = P.forward(cfg, w, toks)
    s = Served(folder, dtype, page=page, pages=40)
    whole = s.step([("w", toks, list(range(70)))])
    one = torch.cat([s.step([("d", toks[i:i + 1], [0])]) for i in range(70)])
    assert agrees(whole, want, dtype) and agrees(one, want, dtype)
    if dtype == torch.float32:
        assert float(errors(one, whole).max()) < 3e-5          # cutting changes nothing beyond rounding


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small", "odd", "wide"])
def test_portions_of_every_size(models, dtype, name):
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 150, 3)
    want = P.forward(cfg, w, toks)
    for cuts in ([2] * 10 + [3, 5, 16, 17, 31, 33, 25], [64, 64, 22], [1, 2, 13, 48, 1, 1, 84], [149, 1]):
        assert sum(cuts) == 150
        s = Served(folder, dtype, page=16, pages=12)
        at, outs = 0, []
        for c in cuts:
            outs.append(s.step([("p", toks[at:at + c], list(range(c)))]))
            at += c
        assert agrees(torch.cat(outs), want, dtype), cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small", "odd", "wide"])
def test_batches_of_unequal_requests_pages_and_slots_used_again(models, dtype, name):
    """Four live requests, portions beside single tokens, in a pool and with state slots that only hold them if those
    of finished requests are used again; every row against the plain implementation of its request alone."""
    folder, cfg, w = models(name)
    lengths = dict(a=90, b=33, c=7, d=64, e=50, f=21)
    toks = {k: tokens_for(cfg, n, 10 + i) for i, (k, n) in enumerate(lengths.items())}
    want = {k: P.forward(cfg, w, t) for k, t in toks.items()}
    s = Served(folder, dtype, page=16, pages=14, max_requests=4)
    at = {k: 0 for k in toks}
    got = {k: [] for k in toks}
    plan = [[("a", 40), ("b", 2), ("c", 1)], [("a", 1), ("b", 30), ("c", 3), ("d", 17)], [("a", 1), ("c", 3), ("d", 47), ("b", 1)],
            [("a", 48), ("e", 2)], [("e", 47), ("f", 1)], [("e", 1), ("f", 20)]]
    for step in plan:
        out = s.step([(k, toks[k][at[k]:at[k] + n], list(range(n))) for k, n in step])
        row = 0
        for k, n in step:
            got[k].append(out[row:row + n]); row += n; at[k] += n
            if at[k] == lengths[k]:
                s.end(k)
    for k in toks:
        assert at[k] == lengths[k]
        assert agrees(torch.cat(got[k]), want[k], dtype), k
    s.runner.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("small", 8), ("odd", 4)])
def test_long_decoding(models, dtype, name, page):
    """330 tokens, all but ten decoded one by one: the temperature steps many times, the recurrent states run long, and
    the attention reads dozens of pages."""
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 330, 5)
    want = P.forward(cfg, w, toks)
    s = Served(folder, dtype, page=page, pages=-(-330 // page) + 1)
    s.step([("x", toks[:10], [])])
    outs = torch.cat([s.step([("x", toks[i:i + 1], [0])]) for i in range(10, 330)])
    assert agrees(outs, want[10:], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_request_left_out_of_steps_goes_on_later(models, dtype):
    folder, cfg, w = models("small")
    ta, tb = tokens_for(cfg, 60, 8), tokens_for(cfg, 40, 9)
    wa, wb = P.forward(cfg, w, ta), P.forward(cfg, w, tb)
    s = Served(folder, dtype)
    a1 = s.step([("a", ta[:25], list(range(25)))])
    b1 = s.step([("b", tb[:39], list(range(39)))])
    both = s.step([("a", ta[25:], list(range(35))), ("b", tb[39:], [0])])
    assert agrees(torch.cat([a1, both[:35]]), wa, dtype) and agrees(torch.cat([b1, both[35:]]), wb, dtype)


# ------------------------------------------------------------------------ generation, replay, command line

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small", "wide"])
def test_greedy_generation_through_the_scheduler(models, dtype, name):
    """Engine.generate: chunked prompts, captured decode steps, several requests at once; every produced token
    against the plain implementation on the same history."""
    from paged_llm_rs_b200 import Engine
    folder, cfg, w = models(name)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (3, 41, 18, 70, 1)]
    eng = Engine(folder, dtype=NAMES[dtype], block_size=16, blocks=64, max_batch=4, chunk=32, prefix_cache=False)
    outs = eng.generate(prompts, max_tokens=12)
    decided = total = out_of_noise = 0
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        seq = list(p)
        for tok in o:
            logits = P.forward(cfg, w, seq)[-1]
            best = P.greedy(logits)
            top2 = torch.topk(logits, 2).values
            noise = (1e-4 if dtype == torch.float32 else 0.05) * max(1.0, float(logits.abs().max()))
            out_of_noise += float(logits[best] - logits[tok]) >= noise
            decided += float(top2[0] - top2[1]) >= noise
            total += 1
            seq.append(tok)
    assert out_of_noise <= (0 if dtype == torch.float32 else 0.05 * total), (out_of_noise, total)
    assert decided >= 0.5 * total


def test_trace_replay_and_command_line(models, tmp_path):
    folder, cfg, w = models("small")
    from trace_tools import TraceBuilder, replay
    toks = tokens_for(cfg, 60, 7)
    tb = TraceBuilder()
    tb.step([("r", toks[:33], [0, 32])])
    tb.step([("r", toks[33:59], [25]), ("q", toks[:5], [4])], end=["q"])
    tb.step([("r", toks[59:], [0])], end=["r"])
    got = tb.collect(replay(folder, "float32", tb.steps, 128, cfg["vocab"]))
    want = P.forward(cfg, w, toks)
    for pos, row in got["r"].items():
        assert float(errors(torch.from_numpy(row).double()[None], want[pos:pos + 1]).max()) < 2e-4
    # the captured and replayed steps of generation give the same logits
    got2 = tb.collect(replay(folder, "float32", tb.steps, 128, cfg["vocab"], graphs=True, step_tokens=48))
    for pos, row in got2["r"].items():
        assert float(errors(torch.from_numpy(row).double()[None], want[pos:pos + 1]).max()) < 2e-4
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "paged_llm_rs_b200", "generate", "--model", folder, "--dtype", "f32",
                        "--prompt-ids", ",".join(map(str, toks[:9])), "--max-tokens", "4", "--blocks", "32"],
                       cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    out = [int(t) for t in r.stdout.strip().splitlines()[-1].split(",")]
    seq = toks[:9]
    for tok in out:
        assert tok == P.greedy(P.forward(cfg, w, seq)[-1])
        seq = seq + [tok]


# ------------------------------------------------------------------------ configurations drawn at random

def random_configuration(seed):
    """Sizes, counts, layer order and constants drawn from a seed."""
    rnd = random.Random(seed)
    width = rnd.choice([48, 64, 96, 128, 192])

    def an_attention():
        kv = rnd.choice([1, 2, 3])
        dim = rnd.choice([8, 16, 24, 32, 64, 128])
        rot = rnd.choice([0, 2, dim // 2, dim])
        return attention(kv * rnd.choice([1, 2, 4, 5]), kv, dim, rot=rot - rot % 2, base=rnd.choice([100.0, 10000.0, 5e5]),
                         scale=rnd.choice([0.4, 1.2, 4.0]) / dim ** 0.5)

    def an_mlstm():
        return mlstm(rnd.choice([1, 2, 3, 6]), rnd.choice([8, 24, 48, 64, 128]), rnd.choice([8, 12, 32, 64]), cap=rnd.choice([2.0, 15.0, 30.0]))

    def a_parallel():
        kv = rnd.choice([1, 2, 3])
        dim = rnd.choice([8, 16, 24, 64])
        l = left(kv * rnd.choice([1, 2, 4]), kv, dim, rnd.choice([8, 12, 32, 64]), coef=rnd.choice([0.1, 0.5, 2.0]),
                 every=rnd.choice([0, 1, 3, 16, 50, 1000]), scale=rnd.choice([0.4, 1.2, 4.0]) / dim ** 0.5)
        g = rnd.choice([1, 2, 3])
        r = right(g * rnd.choice([1, 2, 3]), g, rnd.choice([8, 20, 64, 128]), rnd.choice([8, 12, 32, 64]), conv=rnd.choice([1, 2, 3, 4, 6]))
        return parallel(l, r, rnd.choice([0.5, 1.0, 1.2]), rnd.choice([0.25, 1.0, 2.0]))

    def a_mlp():
        return dense(rnd.choice([32, 72, 128, 192])) if rnd.random() < 0.75 else None
    layers = [layer(rnd.choice([an_attention, an_mlstm, a_parallel])(), a_mlp()) for _ in range(rnd.randint(2, 6))]
    return model(rnd.choice([97, 256, 640]), width, layers, eps=rnd.choice([1e-5, 1e-6]), embedding_scale=rnd.choice([0.5, 1.0, 3.0, 8.0]))


@pytest.mark.parametrize("seed", list(range(1, 13)))
def test_configurations_drawn_at_random(tmp_path, seed):
    cfg = random_configuration(seed)
    toks = tokens_for(cfg, 130, seed)
    folder, cfg, w = write_model(tmp_path, f"random{seed}", seed=seed, cfg=cfg)
    want = P.forward(cfg, w, toks)
    rounding = rounding_alone(cfg, w, toks, want)
    for dtype in DTYPES:
        s = Served(folder, dtype, page=16, pages=24)
        whole = s.step([("w", toks, list(range(130)))])
        s.end("w")
        outs, at = [], 0
        for c in [50, 2, 47, 1, 1, 19, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1]:
            outs.append(s.step([("c", toks[at:at + c], list(range(c)))]))
            at += c
        assert at == 130
        assert agrees(whole, want, dtype, rounding), (seed, dtype, cfg)
        assert agrees(torch.cat(outs), want, dtype, rounding), (seed, dtype, cfg)


FAR_SIZES = {
    # keys of 256 and 512 entries, a value of 4, a delta rule without convolution (one tap), six heads over two q/k heads
    "long_keys": lambda: model(300, 256, [
        layer(mlstm(2, 256, 128, cap=10.0), dense(64)),
        layer(parallel(left(4, 2, 128, 96, coef=0.7, every=5, scale=0.1), right(6, 2, 256, 64, conv=1), 0.9, 1.1), None),
        layer(attention(6, 3, 96, rot=32, base=1000.0, scale=0.2), dense(96)),
        layer(mlstm(1, 512, 4, cap=3.0), None)], eps=1e-6, embedding_scale=2.0),
    # keys of 4 entries beside values of 200 and 300, sixteen taps, sizes that are no multiple of eight
    "short_keys": lambda: model(130, 72, [
        layer(parallel(left(3, 1, 40, 4, coef=0.2, every=2, scale=0.3), right(2, 1, 4, 200, conv=7), 1.0, 0.5), dense(40)),
        layer(mlstm(5, 4, 300, cap=20.0), dense(24)),
        layer(mlstm(3, 36, 20, cap=1.0), None),
        layer(parallel(left(2, 2, 8, 8, coef=0.0, every=0, scale=0.5), right(3, 3, 100, 36, conv=16), 0.3, 2.0), None)],
        eps=1e-5, embedding_scale=1.0),
}


@pytest.mark.parametrize("name", sorted(FAR_SIZES))
def test_sizes_far_from_the_usual(tmp_path, name):
    """State matrices much longer than wide and much wider than long, whole and in portions with decoded tokens behind."""
    cfg = FAR_SIZES[name]()
    toks = tokens_for(cfg, 150, 5)
    folder, cfg, w = write_model(tmp_path, name, seed=7, cfg=cfg)
    want = P.forward(cfg, w, toks)
    rounding = rounding_alone(cfg, w, toks, want)
    for dtype in DTYPES:
        s = Served(folder, dtype, page=16, pages=40)
        whole = s.step([("w", toks, list(range(150)))])
        s.end("w")
        outs, at = [], 0
        for c in [37, 2, 64, 33] + [1] * 14:
            outs.append(s.step([("c", toks[at:at + c], list(range(c)))]))
            at += c
        assert at == 150
        assert agrees(whole, want, dtype, rounding), (name, dtype)
        assert agrees(torch.cat(outs), want, dtype, rounding), (name, dtype)
