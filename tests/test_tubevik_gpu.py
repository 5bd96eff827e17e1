"""Tubevik on the GPU against the plain implementation (tests/plain_tubevik.py): each kernel and each mixer alone (through the
cache manager and the step packer, with inputs made so that one key just inside or just outside a window or a chunk, a missing
one in the softmax, one far token in a recurrent state, a lost state or input of the convolution would show), then whole models
through the engine's step function, cache manager, state slots and scheduler."""

import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tubevik as P
from test_pamarax_gpu import CUTS, NAMES, MixerRig, Served, close, close_recurrent, errors, gen, rounded, status
from tubevik_models import (CONFIGS, YARN, attention, dense, draw, layer, left, mixer_shapes, model, parallel, random_weights, right, rotation,
                            write_model)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5


def ops_():
    from paged_llm_rs_b200.kernels import ops
    return ops


# ------------------------------------------------------------------------ each kernel alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 90), (300, 1024), (3, 4100), (2, 9000), (4, 8), (70, 192)])
def test_terms_sum_and_norm_in_one_pass(dtype, rows, width):
    ops = ops_()
    g = gen(width)
    x0 = 3.0 + torch.randn(rows, width, generator=g)             # a mean that a layer norm takes off
    a, b = (torch.randn(rows, width, generator=g).to(dtype) for _ in range(2))
    wide = torch.randn(rows, width + 24, generator=g).to(dtype)
    gain, bias = 1 + 0.3 * torch.randn(width, generator=g), torch.randn(width, generator=g)
    strided = wide.to(DEV)[:, 8:8 + width]
    cases = [[], [(a, 0.7)], [(a, 0.7), (b, -1.3)], [(a, 0.7), (b, -1.3), ("wide", 0.4)]]
    for terms in cases:
        want = x0.double()
        for t, c in terms:
            want = want + c * (wide[:, 8:8 + width] if isinstance(t, str) else t).double()
        dev = [(strided if isinstance(t, str) else t.to(DEV), c) for t, c in terms]
        for centered in (True, False):
            normed = P.layer_norm(want, gain.double(), bias.double(), EPS) if centered else P.unit_rms(want, EPS) * gain.double()
            args = dict(bias=bias.to(DEV) if centered else None, centered=centered)
            x, y = x0.clone().to(DEV), torch.empty(rows, width, dtype=dtype, device=DEV)
            ops.add_terms_norm32(x, dev, gain.to(DEV), EPS, y, **args)
            close(x, want, torch.float32, "stream", f32=1e-6)
            close(y, normed, dtype, "norm", f32=1e-5, bf16=8e-3)
            idx = torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
            x, y = x0.clone().to(DEV), torch.empty(2, width, dtype=dtype, device=DEV)
            ops.add_terms_norm32(x, dev, gain.to(DEV), EPS, y, rows=idx, **args)
            assert torch.equal(x.cpu(), x0), "with rows the stream stays as it is"
            close(y, normed[[rows - 1, 0]], dtype, "norm of gathered rows", f32=1e-5, bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_norm_behind_the_embedding(dtype):
    ops = ops_()
    g = gen(3)
    table = (2.0 + torch.randn(50, 90, generator=g)).to(dtype)
    gain, bias = 1 + 0.3 * torch.randn(90, generator=g), torch.randn(90, generator=g)
    toks = torch.randint(0, 50, (33,), generator=g).to(torch.int32)
    out = torch.empty(33, 90, dtype=torch.float32, device=DEV)
    ops.embed_norm32(toks.to(DEV), table.to(DEV), gain.to(DEV), EPS, out, status(), bias=bias.to(DEV), centered=True)
    close(out, P.layer_norm(table.double()[toks.long()], gain.double(), bias.double(), EPS), torch.float32, "layer norm", f32=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,nh,nkv,dk,dv,norm,rot,layout,scaled,biases,page", [
    (9, 4, 2, 16, 8, "projection", 8, "half", True, True, 16), (40, 5, 5, 12, 20, "head_after_rotation", 12, "pairs", False, False, 8),
    (3, 8, 2, 64, 64, "projection", 64, "half", True, True, 16), (17, 20, 1, 32, 64, "head_after_rotation", 16, "pairs", True, True, 4),
    (6, 3, 3, 21, 7, "head", 6, "pairs", False, True, 8), (5, 2, 1, 128, 128, "head_after_rotation", 0, "pairs", False, False, 16),
    (4, 3, 1, 10, 9, "projection", 2, "half", False, True, 16), (7, 2, 2, 16, 16, None, 16, "pairs", True, True, 4)])
def test_biases_norms_both_rotations_and_the_cache_write(dtype, T, nh, nkv, dk, dv, norm, rot, layout, scaled, biases, page):
    ops = ops_()
    g = gen(2)
    k_off, v_off = nh * dk, nh * dk + nkv * dk
    width = v_off + nkv * dv + 7                                 # columns behind q | k | v that the kernel must not touch
    proj = torch.randn(T, width, generator=g).to(dtype)
    sizes = {"projection": (nh * dk, nkv * dk), "head": (dk, dk)}.get(norm)
    qg, kg = (1 + 0.3 * torch.randn(n, generator=g) for n in sizes) if sizes else (None, None)
    qb, kb, vb = (torch.randn(n, generator=g) for n in (nh * dk, nkv * dk, nkv * dv)) if biases else (None, None, None)
    turn = P.rotation(rotation(rot, 77.0, YARN if scaled else None))
    inv_freq = torch.tensor(turn[1], dtype=torch.float64).float() if rot else None
    pos = torch.arange(30, 30 + T, dtype=torch.int32)
    n_pages = 8 + T // page
    slots = torch.randperm(n_pages * page, generator=g)[:T].to(torch.int32)
    slots[0] = -1                                                # a token whose row is not written
    dv_ = lambda t: None if t is None else t.to(DEV)
    pd = proj.double()
    qq, kk, vv = pd[:, :k_off], pd[:, k_off:v_off], pd[:, v_off:v_off + nkv * dv]
    if biases:
        qq, kk, vv = qq + qb.double(), kk + kb.double(), vv + vb.double()
    if norm == "projection":
        qq, kk = P.unit_rms(qq, EPS) * qg.double(), P.unit_rms(kk, EPS) * kg.double()
    qq, kk, vv = qq.view(T, nh, dk), kk.view(T, nkv, dk), vv.view(T, nkv, dv)
    if norm == "head":
        qq, kk = P.unit_rms(qq, EPS) * qg.double(), P.unit_rms(kk, EPS) * kg.double()
    qq, kk = P.rotate(qq, pos.tolist(), turn, layout), P.rotate(kk, pos.tolist(), turn, layout)
    if norm == "head_after_rotation":
        qq, kk = P.unit_rms(qq, EPS), P.unit_rms(kk, EPS)
    for queries_only in (False, True):
        pool = torch.full((n_pages, nkv, page, dk + dv), 7.0, dtype=dtype, device=DEV)
        q = torch.empty(T, nh * dk, dtype=dtype, device=DEV)
        st = status()
        p = proj[:, :k_off].contiguous() if queries_only else proj
        ops.normed_qk_kv_write(p.to(DEV), -1 if queries_only else k_off, v_off, q, dv_(qg), None if queries_only else dv_(kg), norm, EPS, 0.0, 0,
                               dv_(inv_freq), rot, pos.to(DEV), slots.to(DEV), None if queries_only else pool, nh, nkv, dk, dv, False, st,
                               q_bias=dv_(qb), k_bias=dv_(kb), v_bias=dv_(vb), rot_pairs=layout == "pairs", rot_factor=turn[2])
        assert st.item() == 0
        close(q.view(T, nh, dk), qq, dtype, "q", f32=1e-4, bf16=2e-2)
        if queries_only:
            assert bool((pool == 7.0).all())
            continue
        rows = pool.double().cpu().permute(0, 2, 1, 3).reshape(n_pages * page, nkv, dk + dv)
        for t in range(1, T):
            close(rows[slots[t], :, :dk], kk[t], dtype, "cached key", f32=1e-4, bf16=2e-2)
            close(rows[slots[t], :, dk:], vv[t], dtype, "cached value", f32=1e-6, bf16=8e-3)
        untouched = torch.ones(n_pages * page, dtype=torch.bool)
        untouched[slots[1:].long()] = False
        assert bool((rows[untouched] == 7.0).all())


def segments_of(cuts, pad=0):
    """(tokens, tokens before) a request -> the step's segment list, request i in slot i + 1; then ``pad`` empty ones."""
    rows, at = [], 0
    for i, (n, before) in enumerate(cuts):
        rows.append((at, n, before, i + 1))
        at += n
    return torch.tensor(rows + [(0, 0, 0, 0)] * pad, dtype=torch.int32), at


def kernel_delta(dtype, H, G, d, e, taps, cuts, pad, seed, ranks=(6, 4), rate=-2.0, longest=None):
    """channel_delta_mix on random inputs, slots and earlier inputs against the plain rule, request by request:
    (got, want, slots, their want)."""
    ops = ops_()
    g = gen(seed)
    segs, T = segments_of(cuts, pad)
    channels = 2 * G * d + H * e
    r = lambda *s: torch.randn(*s, generator=g)
    u = r(T, channels + ranks[1] + 3).to(dtype)
    small = r(T, H + ranks[0])
    conv = (r(channels, taps) / taps ** 0.5).to(dtype)
    a2, g2 = (r(H * d, ranks[0]) / ranks[0] ** 0.5).to(dtype), r(H * e, ranks[1]).to(dtype)
    a_log, dt, gain = rate + r(H), r(H * d), 1 + 0.3 * r(e)
    floats = ops.channel_delta_state_floats(H, G, d, e, taps)
    slots = r(len(cuts) + 2, floats)
    st, out = slots.clone().to(DEV), torch.empty(T, H * e, dtype=dtype, device=DEV)
    longest = max(n for n, _ in cuts) if longest is None else longest
    gate = (u.double()[:, channels:channels + ranks[1]] @ g2.double().T).to(dtype)
    dv = lambda t: t.to(DEV)
    ops.channel_delta_mix(dv(u), dv(conv), dv(small), H, dv(a2), dv(a_log), dv(dt), channels, dv(g2), dv(gain), dv(segs), longest, st, out,
                          H, G, d, e, taps, EPS, gate=None if longest == 1 else dv(gate))
    ud = u.double()
    want, left_behind = torch.zeros(T, H * e, dtype=torch.float64), slots.double().clone()
    for t0, n, before, slot in segs.tolist():
        if not n:
            continue
        ring = left_behind[slot][H * d * e:].view(taps, channels) if taps > 1 else None
        past = torch.stack([ring[p % taps] if p >= 0 else torch.zeros(channels, dtype=torch.float64)
                            for p in range(before - taps + 1, before)]) if taps > 1 else torch.zeros(0, channels, dtype=torch.float64)
        x = torch.cat([past, ud[t0:t0 + n, :channels]])
        c = P.silu(sum(x[j:j + n] * conv.double()[:, j] for j in range(taps)))
        q, k = P.unit_vector(c[:, :G * d].view(n, G, d)) * d ** -0.5, P.unit_vector(c[:, G * d:2 * G * d].view(n, G, d))
        v = c[:, 2 * G * d:].view(n, H, e)
        s = small.double()[t0:t0 + n]
        beta = torch.sigmoid(s[:, :H])
        alpha = P.channel_decay(s[:, H:] @ a2.double().T, a_log.double(), dt.double(), H)
        o = torch.zeros(n, H, e, dtype=torch.float64)
        for h in range(H):
            kh = h // (H // G)
            S = left_behind[slot][:H * d * e].view(H, d, e)[h].clone() if before else torch.zeros(d, e, dtype=torch.float64)
            for t in range(n):
                S = alpha[t, h][:, None] * S
                S = S + torch.outer(k[t, kh], beta[t, h] * (v[t, h] - S.T @ k[t, kh]))
                o[t, h] = S.T @ q[t, kh]
            left_behind[slot][:H * d * e].view(H, d, e)[h] = S
        if taps > 1:
            for t in range(max(0, n - taps + 1), n):
                ring[(before + t) % taps] = ud[t0 + t, :channels]
        o = (P.unit_rms(o, EPS) * gain.double()).reshape(n, H * e)
        logits = gate.double()[t0:t0 + n] if longest != 1 else ud[t0:t0 + n, channels:channels + ranks[1]] @ g2.double().T
        want[t0:t0 + n] = o * torch.sigmoid(logits)
    return out, want, st, left_behind


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e,taps,ranks,cuts,pad", [
    (4, 2, 16, 24, 3, (6, 4), [(1, 0), (1, 5), (1, 300)], 2),                                 # decoded tokens
    (3, 3, 20, 12, 1, (1, 9), [(1, 9), (1, 0)], 0), (2, 1, 20, 37, 16, (24, 8), [(1, 3), (1, 40)], 1),
    (1, 1, 256, 256, 4, (16, 32), [(1, 77)], 0), (2, 2, 512, 24, 2, (8, 1), [(1, 7)], 0), (4, 1, 4, 300, 5, (3, 3), [(1, 3), (1, 1)], 0),
    (2, 1, 1, 1, 2, (1, 1), [(1, 4), (1, 0)], 0), (5, 5, 32, 28, 4, (20, 12), [(1, i) for i in range(40)], 24),
    (1, 1, 384, 512, 2, (4, 4), [(1, 5)], 0), (8, 4, 128, 128, 4, (128, 128), [(1, 9)] * 3, 1),
    (4, 2, 16, 24, 3, (6, 4), [(5, 0), (1, 5), (33, 2), (2, 0)], 3),                          # portions beside decoded tokens
    (1, 1, 32, 32, 4, (16, 8), [(70, 0), (1, 6), (19, 40), (16, 0), (17, 3), (4, 4), (3, 1)], 2),
    (3, 3, 20, 12, 1, (5, 5), [(30, 7)], 0), (2, 2, 96, 8, 9, (33, 2), [(20, 0), (3, 100), (2, 1)], 30), (1, 1, 512, 20, 2, (4, 4), [(15, 1)], 0),
    (2, 1, 8, 301, 5, (2, 2), [(9, 0), (3, 0)], 0), (2, 1, 2, 1, 16, (1, 1), [(40, 3)], 0), (4, 2, 128, 128, 4, (16, 16), [(40, 3), (1, 2)], 0),
    (2, 2, 256, 64, 4, (16, 16), [(21, 0)], 0), (20, 5, 64, 64, 2, (8, 8), [(18, 2)] * 9, 0)])
def test_delta_rule_kernels_alone(dtype, H, G, d, e, taps, ranks, cuts, pad):
    got, want, st, left_behind = kernel_delta(dtype, H, G, d, e, taps, cuts, pad, 40 + d, ranks)
    close_recurrent(got, want, dtype, "read-out")
    close(st, left_behind, torch.float32, "slots", f32=5e-5)


@pytest.mark.parametrize("cuts", [[(1, 4), (1, 0)], [(90, 3), (33, 0)]])
@pytest.mark.parametrize("rate", [-40.0, 6.0, 0.0])
def test_decays_of_one_and_of_zero(rate, cuts):
    """A rate of nearly nothing keeps all of the state, a large one drops it at every token; nothing overflows on the way."""
    got, want, st, left_behind = kernel_delta(torch.float32, 4, 2, 16, 16, 3, cuts, 0, 5, rate=rate)
    assert bool(torch.isfinite(got).all()) and bool(torch.isfinite(st).all())
    close_recurrent(got, want, torch.float32, f"rate {rate}")
    close(st, left_behind, torch.float32, "slots", f32=1e-4)


def test_a_captured_steps_bound_on_a_segments_tokens_changes_nothing():
    """The kernels get only a bound on how many tokens one request brings (a captured step's capacity)."""
    a = kernel_delta(torch.float32, 2, 1, 24, 16, 3, [(1, 4), (9, 0)], 5, 7, longest=9)
    b = kernel_delta(torch.float32, 2, 1, 24, 16, 3, [(1, 4), (9, 0)], 5, 7, longest=512)
    assert torch.equal(a[0], b[0]) and torch.equal(a[2], b[2])
    # one token through the form for portions and through the one for decoded tokens
    a = kernel_delta(torch.float32, 2, 1, 24, 16, 3, [(1, 4), (1, 0)], 5, 7, longest=1)
    b = kernel_delta(torch.float32, 2, 1, 24, 16, 3, [(1, 4), (1, 0)], 5, 7, longest=8)
    close(a[0], b[0], torch.float32, "forms", f32=1e-5)
    close(a[2], b[2], torch.float32, "slots", f32=1e-6)


# ------------------------------------------------------------------------ each mixer alone, through the cache manager

def rot_params(rot, layout):
    rot = rot or {}
    return dict(rot_dims=rot.get("dims", 0), rot_base=rot.get("base", 1.0), rot_scaling=rot.get("scaling"), rot_layout=layout)


def window_params(m, W, **more):
    window = (m.get("mask") or {}).get("size", 0)
    return dict(dict(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"], eps=EPS,
                     biases=True, qk_norm="projection", softcap=m.get("softcap"), window=window, cache_window=window, gate="sigmoid", gate_per="head",
                     **rot_params(m.get("rot"), "half")), **more)


def chunk_params(m, W):
    return dict(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"], eps=EPS,
                qk_norm="head_after_rotation", chunk=(m.get("mask") or {}).get("size", 0), sink_one=True, **rot_params(m.get("rot"), "pairs"))


def window_rig(dtype, m, W, seed, page=16, pages=64, craft=None):
    w = draw(mixer_shapes("attention", m, W, "m"), seed)
    if craft:
        craft(w)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("normed_qk_attention", window_params(m, W), w, dtype, page, pages), lambda h: P.window_mixer(h, plain, "m", m, EPS)[0]


def chunk_rig(dtype, m, W, seed, page=16, pages=64, craft=None):
    w = draw(mixer_shapes("left", m, W, "m"), seed)
    if craft:
        craft(w)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("normed_qk_attention", chunk_params(m, W), w, dtype, page, pages), lambda h: P.chunk_mixer(h, plain, "m", m, EPS)


def delta_rig(dtype, m, W, seed, max_requests=4, craft=None, ranks=(5, 3)):
    w = draw(mixer_shapes("right", m, W, "m", ranks), seed)
    if craft:
        craft(w)
    params = dict(hidden_size=W, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"], eps=EPS)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("channel_gated_delta_rule", params, w, dtype, max_requests=max_requests), lambda h: P.delta_mixer(h, plain, "m", m, EPS)


class LendingRig(MixerRig):
    """A layer and one that borrows its keys and values, on the same input; a step returns both layers' rows side by side."""

    def __init__(self, m, borrower, W, dtype, page=16, pages=64, seed=60, craft=None):
        w = draw(mixer_shapes("attention", m, W, "m"), seed)
        wb = draw(mixer_shapes("attention", dict(borrower, kv_from=0), W, "b"), seed + 1)
        if craft:
            craft(w, wb)
        a, b = ((x.get("mask") or {}).get("size", 0) for x in (m, borrower))
        super().__init__("normed_qk_attention", window_params(m, W, cache_window=0 if 0 in (a, b) else max(a, b)), w, dtype, page, pages)
        from paged_llm_rs_b200.parts import base
        from paged_llm_rs_b200.parts.spec import PartSpec
        second = base.make(base.MIXERS, "mixer", PartSpec("normed_qk_attention", window_params(borrower, W, keeps="nothing"), "b"), self.rt)
        second.bind({s.name: (wb[s.name].to(dtype) if s.role == "matrix" else wb[s.name].float()).to(DEV) for s in second.tensors()})
        first = self.mixer

        class Both:
            def forward(self, x, state, cache):
                return torch.cat([first.forward(x, state, cache), second.forward(x, state, cache, writes_cache=False)], 1)
        self.mixer = Both()
        plain, plain_b = {k: v.double() for k, v in w.items()}, {k: v.double() for k, v in wb.items()}

        def both(h):
            o, kept = P.window_mixer(h, plain, "m", m, EPS)
            return torch.cat([o, P.window_mixer(h, plain_b, "b", borrower, EPS, kept)[0]], 1)
        self.plain = both


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,window,rot,cap,W,page", [
    (4, 2, 16, 8, 21, rotation(8, 100.0, YARN), 3.0, 64, 16), (5, 5, 12, 20, 7, rotation(12, 50.0), 1.0, 90, 8), (20, 1, 32, 64, 48, rotation(32, 1e4, YARN), 6.0, 128, 16),
    (8, 2, 64, 32, 30, rotation(32, 1e4), None, 128, 16), (3, 1, 24, 24, 0, None, 2.0, 48, 4), (6, 2, 128, 64, 16, rotation(128, 1e6, YARN), 20.0, 64, 16),
    (6, 6, 10, 9, 1, rotation(2, 3.0), 4.0, 40, 8), (2, 1, 200, 136, 33, rotation(40, 1e4), 4.0, 96, 16)])
def test_window_attention_whole_in_portions_and_token_by_token(dtype, heads, kv, dim, vdim, window, rot, cap, W, page):
    m = attention(heads, kv, dim, vdim, window=window, rot=rot, softcap=cap, scale=3.0 / dim ** 0.5)["mixer"]
    x = rounded(torch.randn(75, W, generator=gen(12)), dtype)
    for cuts in CUTS:
        rig, plain = window_rig(dtype, m, W, 13, page=page)
        close(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}", f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,chunk,rot,W,page", [
    (4, 2, 16, 8, 21, rotation(8, 100.0), 64, 16), (5, 5, 12, 20, 7, rotation(12, 50.0), 90, 8), (20, 1, 32, 64, 48, rotation(16, 1e4), 128, 16),
    (8, 2, 64, 32, 30, rotation(64, 1e4, YARN), 128, 16), (3, 1, 24, 24, 0, None, 48, 4), (6, 2, 128, 64, 16, rotation(64, 1e6), 64, 16),
    (6, 6, 10, 9, 1, rotation(2, 3.0), 40, 8)])
def test_chunk_attention_whole_in_portions_and_token_by_token(dtype, heads, kv, dim, vdim, chunk, rot, W, page):
    m = left(heads, kv, dim, vdim, chunk=chunk, rot=rot, scale=2.0 / dim ** 0.5)
    x = rounded(torch.randn(75, W, generator=gen(12)), dtype)
    for cuts in CUTS:
        rig, plain = chunk_rig(dtype, m, W, 13, page=page)
        close(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}", f32=1e-4, bf16=4e-2)


def same_direction(heads, kv, dim, sign=1.0, names=("m", "m")):
    """W_q of every head becomes sign * W_k of its kv head, with no biases and gains of one: a token's query points along (or
    against) the key of any token with the same input."""
    def craft(w, wb=None):
        q, k = names
        wq = w if wb is None else wb
        wq[f"{q}.q"] = (sign * w[f"{k}.k"].view(kv, dim, -1).repeat_interleave(heads // kv, 0)).reshape(heads * dim, -1).contiguous()
        for d in (w, wq):
            for n in d:
                if n.endswith(".norm"):
                    d[n] = torch.ones_like(d[n])
                elif n.endswith(".b"):
                    d[n] = torch.zeros_like(d[n])
    return craft


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["window", "chunk"])
@pytest.mark.parametrize("size,page,dim,vdim", [(24, 8, 32, 64), (21, 16, 16, 24), (150, 16, 64, 64), (64, 16, 64, 32), (10, 16, 32, 32)])
def test_one_key_just_inside_and_just_outside(dtype, kind, size, page, dim, vdim):
    """ONE earlier token has three times the last token's input, and queries point along keys: after the norm it scores like the
    token's own key and its value is three times as large, so it decides the output where it is seen.  It lies at the first
    position the last token sees, the one before it (not seen), at page borders inside and outside; the query is decoded alone, at
    a portion's end, in a portion that begins inside what it sees, and beside other requests."""
    W, heads, kv = 64, 4, 2
    if kind == "chunk":
        m = left(heads, kv, dim, vdim, chunk=size, scale=4.0 / dim ** 0.5)
        make = lambda: chunk_rig(dtype, m, W, 15, page=page, pages=120, craft=same_direction(heads, kv, dim))
        n = 3 * size + size // 2 + 1                        # the last query lies in the middle of the fourth chunk
        start = 3 * size
    else:
        m = attention(heads, kv, dim, vdim, window=size, softcap=30.0, scale=4.0 / dim ** 0.5)["mixer"]
        make = lambda: window_rig(dtype, m, W, 15, page=page, pages=120, craft=same_direction(heads, kv, dim))
        n = 3 * size + size // 2 + 1
        start = n - size
    g = gen(14)
    base_x = torch.randn(n, W, generator=g)
    spots = sorted({start, start - 1, start + 1, start - size, start // page * page, start // page * page - 1, -(-start // page) * page, n - 2, 0})
    for at in [s for s in spots if 0 <= s < n - 1]:
        x = base_x.clone()
        x[at] = 3.0 * x[n - 1]
        x = rounded(x, dtype)
        _, plain = make()
        want = plain(x)
        other = x.clone()
        other[at] = base_x[at]
        changed = float((plain(rounded(other, dtype))[-1] - want[-1]).abs().max()) / float(want[-1].abs().max())
        assert (changed > 0.1) if at >= start else (changed == 0.0), (at, start, changed)
        for what, run in (("decoded", lambda r: r.cut("a", x, [n - 1, 1])), ("portion", lambda r: r.cut("b", x, [n - 3, 3])),
                          ("portion over the edge", lambda r: r.cut("c", x, [start - 2, n - start + 2]))):
            rig, _ = make()
            close(run(rig)[-1:], want[-1:], dtype, f"{what}, key {at}", f32=1e-4, bf16=4e-2)
        rig, _ = make()
        rig.step([("d", x[:start + 1]), ("e", rounded(torch.randn(5, W, generator=g), dtype))])
        res = rig.step([("e", rounded(torch.randn(1, W, generator=g), dtype)), ("d", x[start + 1:]), ("f", rounded(torch.randn(40, W, generator=g), dtype))])
        close(res[1][-1:], want[-1:], dtype, f"batch, key {at}", f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_extra_one_takes_the_weight_when_every_score_is_low(dtype):
    """Queries point against every key: all scores are far below zero, the one in the denominator takes the weight and the
    output vanishes; also for the first token of a sequence and of a chunk."""
    W, heads, kv, dim, vdim = 48, 4, 2, 16, 8
    m = left(heads, kv, dim, vdim, chunk=11, scale=2.0)
    x = rounded(torch.randn(1, W, generator=gen(16)).repeat(30, 1), dtype)
    rig, plain = chunk_rig(dtype, m, W, 17, craft=same_direction(heads, kv, dim, sign=-1.0))
    got, want = rig.cut("r", x, [13, 2, 14, 1]), plain(x)
    assert float(want.abs().max()) < 1e-6 and float(got.abs().max()) < 1e-4
    rig, plain = chunk_rig(dtype, m, W, 17, craft=same_direction(heads, kv, dim))
    got, want = rig.cut("r", x, [13, 2, 14, 1]), plain(x)
    assert float(want.abs().max()) > 0.1
    close(got, want, dtype, "scores far above zero", f32=1e-4, bf16=4e-2)
    # a lone key whose score is zero gets half the weight
    m = left(heads, kv, dim, vdim, chunk=1, scale=1e-9)
    rig, plain = chunk_rig(dtype, m, W, 17)
    close(rig.cut("r", x, [28, 1, 1]), plain(x), dtype, "chunks of one", f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,borrowed,heads,kv,dim,vdim,page", [(20, 20, 4, 2, 16, 8, 8), (9, 33, 4, 2, 32, 32, 16), (33, 9, 6, 3, 20, 12, 4), (12, 0, 4, 1, 64, 64, 16),
                                                                      (0, 12, 2, 2, 8, 8, 8), (16, 17, 3, 3, 32, 64, 16)])
def test_a_layer_that_borrows_keys_and_values(dtype, window, borrowed, heads, kv, dim, vdim, page):
    """Its own queries, scale, cap, rotation of the queries and window over the lender's cached rows, in a pool that holds no more
    than the wider of the two windows needs."""
    W = 64
    m = attention(heads, kv, dim, vdim, window=window, rot=rotation(8, 100.0, YARN), softcap=3.0)["mixer"]
    b = attention(heads, kv, dim, vdim, window=borrowed, rot=rotation(4, 30.0), softcap=None, scale=2.0 / dim ** 0.5)["mixer"]
    x = rounded(torch.randn(75, W, generator=gen(18)), dtype)
    widest = 75 if 0 in (window, borrowed) else max(window, borrowed)
    for cuts in CUTS:
        rig = LendingRig(m, b, W, dtype, page=page, pages=-(-(widest + max(cuts)) // page) + 2)
        close(rig.cut("r", x, cuts), rig.plain(x), dtype, f"{cuts}", f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_borrower_that_sees_further_back_than_its_lender(dtype):
    """ONE key that only the borrower's window still holds decides the borrower's output and leaves the lender's alone."""
    W, heads, kv, dim, n = 64, 4, 2, 32, 120
    m = attention(heads, kv, dim, 32, window=10, softcap=30.0, scale=4.0 / dim ** 0.5)["mixer"]
    b = attention(heads, kv, dim, 32, window=50, softcap=30.0, scale=4.0 / dim ** 0.5)["mixer"]
    craft = same_direction(heads, kv, dim, names=("b", "m"))
    base_x = torch.randn(n, W, generator=gen(19))
    for at in (n - 50, n - 51, n - 49, 79, 80, n - 11):
        x = base_x.clone()
        x[at] = 3.0 * x[n - 1]
        x = rounded(x, dtype)
        for cuts in ([n - 1, 1], [n - 30, 30], [40, 2, 60, 18]):
            rig = LendingRig(m, b, W, dtype, page=16, pages=20, craft=craft)
            want = rig.plain(x)
            y = x.clone()
            y[at] = rounded(base_x, dtype)[at]
            d = (rig.plain(y)[-1] - want[-1]).abs()
            assert float(d[:W].max()) == 0.0 and (float(d[W:].max()) > 0.1 * float(want[-1].abs().max())) == (at >= n - 50)
            close(rig.cut("r", x, cuts)[-1:], want[-1:], dtype, f"{at} {cuts}", f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["window", "chunk"])
def test_attention_in_a_pool_of_little_more_than_it_sees(dtype, kind):
    """Pages that a window or chunk has left are used again while the request goes on, and by a second one."""
    if kind == "window":
        m = attention(4, 2, 16, 16, window=24, rot=rotation(8, 100.0))["mixer"]
        rig, plain = window_rig(dtype, m, 48, 17, page=8, pages=2 * (24 // 8 + 2))
    else:
        m = left(4, 2, 16, 16, chunk=24, rot=rotation(8, 100.0))
        rig, plain = chunk_rig(dtype, m, 48, 17, page=8, pages=2 * (24 // 8 + 2))
    a, b = rounded(torch.randn(170, 48, generator=gen(3)), dtype), rounded(torch.randn(90, 48, generator=gen(4)), dtype)
    got = {"a": [], "b": []}
    for i in range(0, 170, 5):
        entries = [("a", a[i:i + 5])] + ([("b", b[i // 5 * 3:i // 5 * 3 + 3])] if i // 5 < 30 else [])
        for (k, _), r in zip(entries, rig.step(entries)):
            got[k].append(r)
    close(torch.cat(got["a"]), plain(a), dtype, "a", f32=1e-4, bf16=4e-2)
    close(torch.cat(got["b"]), plain(b), dtype, "b", f32=1e-4, bf16=4e-2)
    rig.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,conv,W,ranks", [(4, 2, 8, 16, 3, 64, (5, 3)), (3, 3, 20, 12, 2, 90, (1, 9)), (4, 2, 64, 32, 4, 128, (16, 24)),
                                                             (2, 1, 128, 64, 5, 96, (33, 8)), (6, 1, 16, 24, 1, 48, (7, 1)), (2, 2, 256, 16, 4, 64, (8, 8)),
                                                             (2, 1, 48, 37, 16, 72, (4, 4))])
def test_delta_rule_whole_in_portions_and_token_by_token(dtype, heads, kv, dim, vdim, conv, W, ranks):
    m = right(heads, kv, dim, vdim, conv)
    x = rounded(torch.randn(75, W, generator=gen(20)) * 1.5, dtype)
    for cuts in CUTS:
        rig, plain = delta_rig(dtype, m, W, 21, ranks=ranks)
        close_recurrent(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_token_decides_a_recurrent_state(dtype):
    """ONE token carries the only value that is not small, hardly anything decays and little is written over it: it stays in the
    state for hundreds of tokens and decides every later read-out, over a prompt's records, over portions and over decoded tokens."""
    W, heads, dim, vdim, n = 64, 2, 64, 16, 420
    m = right(heads, heads, dim, vdim, 3)

    def craft(w):
        w["m.A_log"] = torch.full_like(w["m.A_log"], -12.0)
        w["m.b"] = 0.2 * w["m.b"]
    make = lambda: delta_rig(dtype, m, W, 23, craft=craft)
    for at in (0, 15, 16, 200, n - 3):
        x = torch.randn(n, W, generator=gen(24))
        x[at] *= 20.0
        x = rounded(x, dtype)
        _, plain = make()
        want = plain(x)
        y = x.clone()
        y[at] = 0.0
        if n - at < 250:
            assert float((plain(y)[-1] - want[-1]).norm()) > 0.05 * float(want[-1].norm())
        for cuts in ([n], [n - 20] + [1] * 20, [at + 1, n - at - 2, 1], [100, 2, 218, 100]):
            rig, _ = make()
            close_recurrent(rig.cut("r", x, cuts)[-25:], want[-25:], dtype, f"{at} {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_in_batches_with_slots_used_again_and_long_decoding(dtype):
    """Three slots for five requests: requests of unequal length side by side, a finished request's slot taken by the next
    (whose state and inputs must start at zero), a request left out of a step, and one request decoded for 300 tokens."""
    W = 64
    rig, plain = delta_rig(dtype, right(4, 2, 16, 8, 4), W, 23, max_requests=3)
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
    W = 72
    l, r = left(6, 3, 16, 8, chunk=22, rot=rotation(8, 100.0)), right(4, 2, 8, 16, conv=3)
    w = dict(draw(mixer_shapes("left", l, W, "m.left"), 30), **draw(mixer_shapes("right", r, W, "m.right"), 31))
    rp = dict(hidden_size=W, heads=4, kv_heads=2, dim=8, vdim=16, conv=3, eps=EPS)
    params = dict(parts=[dict(kind="normed_qk_attention", params=chunk_params(l, W), under="left", scale=0.6),
                         dict(kind="channel_gated_delta_rule", params=rp, under="right", scale=1.7)])
    plain = {k: v.double() for k, v in w.items()}
    x = rounded(torch.randn(75, W, generator=gen(32)), dtype)
    want = P.parallel_mixer(x, plain, "m", dict(left=l, right=r, left_scale=0.6, right_scale=1.7), EPS)
    for cuts in CUTS:
        rig = MixerRig("parallel_mixers", params, w, dtype, page=8)
        close_recurrent(rig.cut("r", x, cuts), want, dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,inter,limit", [(3, 64, 96, 0.5), (70, 128, 192, 1.0), (9, 90, 50, 2.5), (300, 128, 256, 0.25)])
def test_clamped_feed_forward(dtype, rows, width, inter, limit):
    """Gates and up products far beyond the limit on both sides, for few rows and many."""
    from paged_llm_rs_b200.parts import base, decoder  # noqa: F401
    from paged_llm_rs_b200.parts.spec import PartSpec
    rt = base.Runtime(torch.device(DEV), dtype)
    ff = base.make(base.FEED_FORWARDS, "feed-forward", PartSpec("swiglu_mlp", dict(hidden_size=width, intermediate_size=inter, activation="clamped", limit=limit,
                                                                                     names=dict(gate="gate", up="up", down="down")), "m"), rt)
    w = draw({"m.gate": ((inter, width), "matrix"), "m.up": ((inter, width), "matrix"), "m.down": ((width, inter), "matrix")}, 5)
    ff.bind({k: v.to(dtype).to(DEV) for k, v in w.items()})
    x = rounded(torch.randn(rows, width, generator=gen(6)) * 1.5, dtype)
    close(ff.forward(x.to(dtype).to(DEV), None), P.clamped_ff(x, {k: v.double() for k, v in w.items()}, "m", limit), dtype, "feed-forward", bf16=2e-2)


# ------------------------------------------------------------------------ whole models through the engine

TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}


def rounding_alone(cfg, w, toks, want):
    """Per position, the error of the plain implementation itself when it runs in float32: what rounding alone does there."""
    P.F64 = torch.float32
    try:
        return errors(P.forward(cfg, w, toks).double(), want)
    finally:
        P.F64 = torch.float64


def agrees(got, want, dtype, rounding=None):
    """float32: every position within rounding (the fixed bound, or three times what rounding alone does at that position where
    that is more).  bfloat16: the typical position well within and nine in ten not far: where a recurrent head's read-out
    nearly cancels its norm makes rounding decide the head's direction."""
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
    root = tmp_path_factory.mktemp("tubevik")

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
        assert float(errors(first, want[:4]).max()) < max(0.3, 1.5 * float(errors(got[:4], want[:4]).max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("small", 16), ("odd", 8), ("wide", 32), ("window_only", 16), ("parallel_only", 4)])
def test_prefill_against_token_by_token_decoding(models, dtype, name, page):
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 110, 2)
    want = P.forward(cfg, w, toks)
    s = Served(folder, dtype, page=page, pages=64)
    whole = s.step([("w", toks, list(range(110)))])
    one = torch.cat([s.step([("d", toks[i:i + 1], [0])]) for i in range(110)])
    assert agrees(whole, want, dtype) and agrees(one, want, dtype)
    if dtype == torch.float32:
        assert float(errors(one, whole).max()) < 5e-5          # cutting changes nothing beyond rounding


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small", "odd", "wide"])
def test_portions_of_every_size(models, dtype, name):
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 150, 3)
    want = P.forward(cfg, w, toks)
    for cuts in ([2] * 10 + [3, 5, 16, 17, 31, 33, 25], [64, 64, 22], [1, 2, 13, 48, 1, 1, 84], [149, 1], [20, 1, 1, 40, 2, 86]):
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
    """Four live requests, portions beside single tokens, in a pool and with state slots that only hold them if those of
    finished requests (windows and chunks) are used again; every row against the plain implementation of its request alone."""
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
    assert at == lengths
    assert agrees(torch.cat([r for k in toks for r in got[k]]), torch.cat([want[k] for k in toks]), dtype)
    for k in toks if dtype == torch.float32 else ():       # (bfloat16: a request of seven tokens is too few for a typical position)
        assert agrees(torch.cat(got[k]), want[k], dtype), k
    s.runner.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("small", 8), ("odd", 4), ("wide", 16)])
def test_long_prompts_and_long_decoding(models, dtype, name, page):
    """330 tokens, first all but ten decoded one by one (windows and chunks pass under the decoded tokens and their pages go
    back), then in one prompt with the rest decoded."""
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 330, 5)
    want = P.forward(cfg, w, toks)
    sizes = [(L["mixer"].get("left") or L["mixer"]).get("mask", {}).get("size", 0) for L in cfg["layers"]]
    pages = -(-330 // page) + 1 if 0 in sizes else -(-(max(sizes) + 12) // page) + 2
    s = Served(folder, dtype, page=page, pages=pages)
    s.step([("x", toks[:10], [])])
    outs = torch.cat([s.step([("x", toks[i:i + 1], [0])]) for i in range(10, 330)])
    assert agrees(outs, want[10:], dtype)
    s = Served(folder, dtype, page=page, pages=-(-330 // page) + 1)
    outs = [s.step([("y", toks[:300], list(range(300)))])] + [s.step([("y", toks[i:i + 1], [0])]) for i in range(300, 330)]
    assert agrees(torch.cat(outs), want, dtype)


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
    """Engine.generate: chunked prompts, captured decode steps, several requests at once; every produced token against the
    plain implementation on the same history."""
    from paged_llm_rs_b200 import Engine
    folder, cfg, w = models(name)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (3, 41, 18, 70, 1)]
    eng = Engine(folder, dtype=NAMES[dtype], block_size=16, blocks=64, max_batch=4, chunk=32, prefix_cache=False)
    outs = eng.generate(prompts, max_tokens=12)
    decided = total = out_of_noise = 0
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits_all = P.forward(cfg, w, list(p) + list(o))
        for i, tok in enumerate(o):
            logits = logits_all[len(p) + i - 1]
            top2 = torch.topk(logits, 2).values
            noise = (1e-4 if dtype == torch.float32 else 0.05) * max(1.0, float(logits.abs().max()))
            out_of_noise += float(logits[P.greedy(logits)] - logits[tok]) >= noise
            decided += float(top2[0] - top2[1]) >= noise
            total += 1
    assert out_of_noise <= (0 if dtype == torch.float32 else 0.05 * total), (out_of_noise, total)
    assert decided >= 0.3 * total


def test_trace_replay_and_command_line(models, tmp_path):
    folder, cfg, w = models("small")
    from trace_tools import TraceBuilder, replay
    toks = tokens_for(cfg, 60, 7)
    tb = TraceBuilder()
    tb.step([("r", toks[:33], [0, 32])])
    tb.step([("r", toks[33:59], [25]), ("q", toks[:5], [4])], end=["q"])
    tb.step([("r", toks[59:], [0])], end=["r"])
    want = P.forward(cfg, w, toks)
    for graphs in (dict(), dict(graphs=True, step_tokens=48)):       # (plain launches; the captured and replayed steps of generation)
        got = tb.collect(replay(folder, "float32", tb.steps, 128, cfg["vocab"], **graphs))
        for rid, tk in (("r", toks), ("q", toks[:5])):
            for pos, row in got[rid].items():
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
    """Sizes, counts, layer order, lenders and borrowers, and constants drawn from a seed."""
    rnd = random.Random(seed)
    width = rnd.choice([48, 64, 96, 128, 192])
    masks = [0, 1, 5, 16, 40, 63, 64, 100, 1000]

    def a_rotation(dim):
        dims = rnd.choice([0, 2, dim // 2, dim])
        s = dict(factor=rnd.choice([2.0, 8.0, 32.0]), original=rnd.choice([32, 128, 1000]), fast=rnd.choice([8.0, 32.0]), slow=rnd.choice([1.0, 2.0]))
        return rotation(dims - dims % 2, rnd.choice([100.0, 10000.0, 5e5]), s if rnd.random() < 0.6 else None)

    def an_attention(layers):
        lenders = [i for i, L in enumerate(layers) if L["type"] == "attention" and L["mixer"].get("kv_from") is None]
        if lenders and rnd.random() < 0.6:
            j = rnd.choice(lenders)
            o = layers[j]["mixer"]
            return attention(o["heads"], o["kv_heads"], o["dim"], o["vdim"], window=rnd.choice(masks), rot=o.get("rot"), softcap=rnd.choice([None, 3.0, 50.0]),
                             kv_from=j, scale=rnd.choice([0.4, 1.2, 3.0]) / o["dim"] ** 0.5)
        kv, dim = rnd.choice([1, 2, 3]), rnd.choice([8, 16, 24, 32, 64, 128])
        return attention(kv * rnd.choice([1, 2, 4, 5]), kv, dim, rnd.choice([8, 12, 32, 64]), window=rnd.choice(masks), rot=a_rotation(dim),
                         softcap=rnd.choice([None, 2.0, 20.0]), scale=rnd.choice([0.4, 1.2, 3.0]) / dim ** 0.5)

    def a_parallel(layers):
        kv, dim = rnd.choice([1, 2, 3]), rnd.choice([8, 16, 24, 32, 64, 128])
        rot = a_rotation(dim)
        if rot:
            rot.pop("scaling", None)
        l = left(kv * rnd.choice([1, 2, 4, 5]), kv, dim, rnd.choice([8, 12, 32, 64]), chunk=rnd.choice(masks), rot=rot, scale=rnd.choice([0.4, 1.2, 3.0]) / dim ** 0.5)
        G = rnd.choice([1, 2, 3])
        r = right(G * rnd.choice([1, 2, 3]), G, rnd.choice([8, 20, 64, 128]), rnd.choice([8, 12, 32, 64]), conv=rnd.choice([1, 2, 4, 7]))
        return parallel(l, r, rnd.choice([0.5, 1.0, 1.2]), rnd.choice([0.25, 1.0, 2.0]))

    layers = []
    for _ in range(rnd.randint(2, 5)):
        layers.append(layer(rnd.choice([an_attention, a_parallel])(layers), dense(rnd.choice([32, 72, 128, 192]), rnd.choice([0.5, 2.0, 7.0])) if rnd.random() < 0.75 else None))
    return model(rnd.choice([97, 256, 640]), width, layers, eps=rnd.choice([1e-5, 1e-6]), cap=rnd.choice([None, 5.0, 30.0]), mult=rnd.choice([0.2, 0.7, 1.0]))


@pytest.mark.parametrize("seed", list(range(1, 15)))
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
