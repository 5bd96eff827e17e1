"""Reperax on the GPU against the plain implementation (tests/plain_reperax.py): each kernel and each mixer alone (through the
cache manager and the step packer, with inputs made so that one key just inside or just outside a chunk, one far key in a
recurrent state, a lost state or a forgotten token before would show), then whole models through the engine's step function,
cache manager, state slots and scheduler."""

import copy
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_reperax as P
from reperax_models import (CONFIGS, dense, draw, layer, left, mixer_shapes, model, parallel, random_weights, retention, right,
                            write_model)
from test_pamarax_gpu import CUTS, NAMES, MixerRig, Served, close, close_recurrent, errors, gen, rounded, status

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5


def ops_():
    from paged_llm_rs_b200.kernels import ops
    return ops


# ------------------------------------------------------------------------ each kernel alone

def segments_of(cuts, pad=0):
    """(tokens, tokens before) a request -> the step's segment list, request i in slot i + 1; then ``pad`` empty ones."""
    rows, at = [], 0
    for i, (n, before) in enumerate(cuts):
        rows.append((at, n, before, i + 1))
        at += n
    return torch.tensor(rows + [(0, 0, 0, 0)] * pad, dtype=torch.int32), at


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,cuts,pad,padding_rows", [
    (64, [(1, 0), (1, 7), (5, 0), (2, 3), (1, 1)], 3, 4), (90, [(7, 2), (1, 0), (40, 0)], 0, 0), (1024, [(1500, 0), (1, 4), (1499, 12)], 1, 0),
    (4104, [(3, 0), (2, 9)], 0, 0), (1024, [(2, 0)] * 40, 24, 0), (200, [(17, 5)], 0, 1)])
def test_gated_sum_two_norms_and_the_shift_in_one_pass(dtype, width, cuts, pad, padding_rows):
    ops = ops_()
    g = gen(width)
    segs, T = segments_of(cuts, pad)
    n = T + padding_rows                                     # (a captured step's rows of no segment)
    x0 = torch.randn(n, width, generator=g)
    wide = torch.randn(n, 3 * width + 8, generator=g).to(dtype)
    a1, a2, f = (torch.randn(n, width, generator=g).to(dtype) for _ in range(3))
    ba, bf, vec, mix = (torch.randn(width, generator=g) for _ in range(4))
    g1, g2 = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    emb = torch.randn(n, width, generator=g)
    state0 = torch.randn(len(cuts) + 2, width, generator=g)
    # the gates are column ranges of a wider product
    ga, gf = wide[:, 8:8 + width], wide[:, 8 + width:8 + 2 * width]
    sg = lambda z, b: torch.sigmoid(z.double() + b.double())
    cases = [dict(), dict(mixed=a1, mixed_scale=0.7), dict(mixed=a1, mixed_gate=ga, mixed_bias=ba), dict(vector=vec), dict(embedded=emb, vector=vec),
             dict(mixed=a1, mixed_scale=0.6, mixed2=a2, mixed2_scale=-1.4, mixed_gate=ga, mixed_bias=ba, fed=f, fed_gate=gf, fed_bias=bf,
                  embedded=emb, vector=vec)]
    for case in cases:
        want = x0.double()
        if "mixed" in case:
            m = case.get("mixed_scale", 1.0) * a1.double() + (case["mixed2_scale"] * a2.double() if "mixed2" in case else 0)
            want = want + (m * sg(ga, ba) if "mixed_gate" in case else m)
        if "fed" in case:
            want = want + f.double() * sg(gf, bf)
        want = want + (emb.double() if "embedded" in case else 0) + (vec.double() if "vector" in case else 0)
        h = P.unit_rms(want, EPS) * g1.double()
        h2 = P.unit_rms(want, EPS) * g2.double()
        before = torch.zeros(n, width, dtype=torch.float64)
        state = state0.double().clone()
        for t0, c, b, slot in segs.tolist():
            if c:
                before[t0] = state0[slot].double() if b else 0.0
                before[t0 + 1:t0 + c] = h[t0:t0 + c - 1]
                state[slot] = h[t0 + c - 1]
        shifted = h + (before - h) * mix.double()
        dev = {}
        for k, v in case.items():
            if v is ga or v is gf:
                o = 8 if v is ga else 8 + width
                dev[k] = wide.to(DEV)[:, o:o + width]
            else:
                dev[k] = v.to(DEV) if isinstance(v, torch.Tensor) else v
        x, st = x0.to(DEV), state0.clone().to(DEV)
        new = lambda: torch.empty(n, width, dtype=dtype, device=DEV)
        y1, ys, y2, xo = new(), new(), new(), torch.empty(n, width, device=DEV)
        ops.gated_sum_norm32(x, g1.to(DEV), y1, EPS, x_out=xo, shift=mix.to(DEV), shifted=ys, segments=segs.to(DEV), state=st, gain2=g2.to(DEV),
                             out2=y2, **dev)
        assert torch.equal(x.cpu(), x0), "the stream it is given stays as it is"
        close(xo, want, torch.float32, "sum", f32=1e-5)
        for got, w, what in ((y1, h, "norm"), (ys[:T], shifted[:T], "shifted"), (y2, h2, "second norm")):
            close(got, w, dtype, what, f32=1e-5, bf16=8e-3)
        close(st, state, torch.float32, "state", f32=1e-5)
        assert torch.equal(st.cpu()[0], state0[0]) and torch.equal(st.cpu()[-1], state0[-1]), "nobody else's slot is touched"
        # some rows only, normed once
        idx = torch.tensor([n - 1, 0, n // 2], dtype=torch.int32)
        y = torch.empty(3, width, dtype=dtype, device=DEV)
        ops.gated_sum_norm32(x, g1.to(DEV), y, EPS, rows=idx.to(DEV), **dev)
        close(y, h[idx.long()], dtype, "norm of gathered rows", f32=1e-5, bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,wider", [(3, 64, 0), (70, 37, 11), (300, 1536, 1024), (2, 9000, 8), (1, 1, 0)])
def test_polynomial_of_normed_powers(dtype, rows, width, wider):
    ops = ops_()
    g = gen(rows)
    u = (torch.randn(rows, width + wider, generator=g) * 1.7).to(dtype)
    c = torch.tensor([0.9, -0.7, 0.5, 0.3])
    out = torch.empty(rows, width, dtype=dtype, device=DEV)
    ops.poly_norm(u.to(DEV)[:, :width], c.to(DEV), EPS, out)
    close(out, P.poly_norm(u.double()[:, :width], c.double(), EPS), dtype, "polynomial", f32=1e-5, bf16=8e-3)


def test_logit_cap():
    ops = ops_()
    x = torch.randn(7, 333, generator=gen(1)) * 40
    got = ops.softcap32(x.clone().to(DEV), 15.0)
    close(got, 15.0 * torch.tanh(x.double() / 15.0), torch.float32, "cap", f32=1e-6)


def kernel_recurrence(dtype, H, d, e, cuts, pad, rot, channel, seed, decay=None, longest=None, state=None, bias=3.0):
    """linear_attention_mix on random inputs against the plain recurrence, request by request: (got, want, slots, their want)."""
    ops = ops_()
    g = gen(seed)
    segs, T = segments_of(cuts, pad)
    width = H * (2 * d + 2 * e) + 5
    u = torch.randn(T, width, generator=g).to(dtype)
    rank, tau = 6, 4.0
    gain = 1 + 0.3 * torch.randn(e, generator=g) if channel else None
    a1, a2, ab = torch.randn(T, rank, generator=g), (torch.randn(H * d, rank, generator=g) / rank ** 0.5).to(dtype), bias + torch.randn(H * d, generator=g)
    decay = decay or [1.0 - 2.0 ** -(2 + i) for i in range(H)]
    base = 40.0
    inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64).float() if rot else None
    slots = torch.randn(len(cuts) + 2, H * d * e, generator=g) if state is None else state
    st, out = slots.clone().to(DEV), torch.empty(T, H * e, dtype=dtype, device=DEV)
    dv = lambda t: None if t is None else t.to(DEV)
    qs, ks = (d ** -0.5, 1.0) if channel else (1.0, d ** -0.5)
    positions = torch.zeros(T, dtype=torch.int32)
    for t0, n, before, _ in segs.tolist():
        positions[t0:t0 + n] = torch.arange(before, before + n, dtype=torch.int32)
    rope = ops.rope_table(positions.to(DEV), dv(inv)) if rot else None
    ops.linear_attention_mix(u.to(DEV), 0, H * d, 2 * H * d, 2 * H * d + H * e, qs, ks, rot, dv(inv), None if channel else torch.tensor(decay, device=DEV),
                             dv(a1) if channel else None, dv(a2) if channel else None, dv(ab) if channel else None, tau, dv(gain), segs.to(DEV),
                             max(n for n, _ in cuts) if longest is None else longest, st, out, H, d, e, EPS, rope=rope)
    ud = u.double()
    want, left_behind = torch.zeros(T, H * e, dtype=torch.float64), slots.double().clone()
    for t0, n, before, slot in segs.tolist():
        if not n:
            continue
        r = ud[t0:t0 + n]
        turn = lambda z: P.rotate_half(z, list(range(before, before + n)), rot, base)
        q, k = turn(r[:, :H * d].view(n, H, d)) * qs, turn(r[:, H * d:2 * H * d].view(n, H, d)) * ks
        v, gate = r[:, 2 * H * d:2 * H * d + H * e].view(n, H, e), r[:, 2 * H * d + H * e:2 * H * d + 2 * H * e]
        if channel:
            alpha = (torch.sigmoid(a1[t0:t0 + n].double() @ a2.double().T + ab.double()) ** (1.0 / tau)).view(n, H, d)
        else:
            alpha = torch.tensor(decay, dtype=torch.float32).double()[None, :, None].expand(n, H, d)
        o = torch.zeros(n, H, e, dtype=torch.float64)
        for h in range(H):
            S = left_behind[slot].view(H, d, e)[h].clone() if before else torch.zeros(d, e, dtype=torch.float64)
            for t in range(n):
                S = alpha[t, h][:, None] * S + torch.outer(k[t, h], v[t, h])
                o[t, h] = S.T @ q[t, h]
            left_behind[slot].view(H, d, e)[h] = S
        o = P.unit_rms(o, EPS) * (gain.double() if channel else 1.0)
        want[t0:t0 + n] = o.reshape(n, H * e) * P.silu(gate)
    return out, want, st, left_behind


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("H,d,e,rot,cuts,pad", [
    (2, 16, 24, 8, [(1, 0), (1, 5), (1, 300)], 2),                                # decoded tokens
    (3, 20, 12, 20, [(1, 9), (1, 0)], 0),                                         # ... of sizes that are no multiple of eight
    (1, 256, 512, 64, [(1, 77)], 0), (4, 4, 300, 0, [(1, 3), (1, 1)], 0),         # ... a state shared out among SMs
    (2, 1, 1, 0, [(1, 4), (3, 2)], 0),
    (2, 16, 24, 8, [(5, 0), (1, 5), (33, 2), (2, 0)], 3),                         # portions beside decoded tokens
    (1, 32, 32, 32, [(700, 0), (1, 6), (129, 40), (64, 0), (65, 3)], 2),          # several blocks of tokens side by side
    (3, 20, 12, 0, [(300, 7)], 0), (2, 96, 8, 2, [(200, 0), (200, 100)], 30), (1, 600, 20, 0, [(150, 1)], 0), (1, 8, 300, 8, [(90, 0), (3, 0)], 0)])
def test_linear_recurrence_alone(dtype, channel, H, d, e, rot, cuts, pad):
    got, want, st, left_behind = kernel_recurrence(dtype, H, d, e, cuts, pad, rot, channel, 40 + d)
    close_recurrent(got, want, torch.float32 if dtype == torch.float32 else dtype, "read-out")
    close(st, left_behind, torch.float32, "slots", f32=5e-5)


@pytest.mark.parametrize("channel", [False, True])
def test_blocks_of_tokens_with_strong_and_no_decay(channel):
    """A prompt cut into blocks that run at the same time: decays of one carry everything over every block's edge, decays of
    (almost) zero carry nothing, and nothing overflows on the way."""
    H, d, e = 4, 16, 16
    if channel:
        for bias in (60.0, -400.0, 0.0):
            got, want, st, left_behind = kernel_recurrence(torch.float32, H, d, e, [(500, 3), (200, 0)], 0, 0, True, 5, bias=bias)
            assert bool(torch.isfinite(got).all())
            close_recurrent(got, want, torch.float32, f"bias {bias}")
            close(st, left_behind, torch.float32, "slots", f32=1e-4)
    else:
        got, want, st, left_behind = kernel_recurrence(torch.float32, H, d, e, [(500, 3), (200, 0)], 0, 8, False, 6, decay=[1.0, 0.0, 1e-30, 0.999])
        close_recurrent(got, want, torch.float32, "read-out")
        close(st, left_behind, torch.float32, "slots", f32=1e-4)


@pytest.mark.parametrize("channel", [False, True])
def test_a_captured_steps_bound_on_a_segments_tokens_changes_nothing(channel):
    """The kernels get only a bound on how many tokens one request brings (a captured step's capacity)."""
    a = kernel_recurrence(torch.float32, 2, 24, 16, [(1, 4), (9, 0)], 5, 8, channel, 7, longest=9)
    b = kernel_recurrence(torch.float32, 2, 24, 16, [(1, 4), (9, 0)], 5, 8, channel, 7, longest=512)
    assert torch.equal(a[0], b[0]) and torch.equal(a[2], b[2])
    close_recurrent(a[0], a[1], torch.float32)


# ------------------------------------------------------------------------ each mixer alone, through the cache manager

def left_rig(dtype, m, W, seed, page=16, pages=64, craft=None):
    w = draw(mixer_shapes("left", m, W, "m"), seed)
    if craft:
        craft(w)
    params = dict(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"],
                  eps=EPS, qk_norm="projection", chunk=(m.get("mask") or {}).get("size", 0))
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("normed_qk_attention", params, w, dtype, page, pages), lambda h: P.attention_mixer(h, plain, "m", m, EPS)


def retention_rig(dtype, m, W, seed, max_requests=4, craft=None):
    w = draw(mixer_shapes("retention", m, W, "m"), seed)
    if craft:
        craft(w)
    rot = m.get("rot") or {}
    params = dict(hidden_size=W, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=m["decay"], rot_dims=rot.get("dims", 0),
                  rot_base=rot.get("base", 1.0), eps=EPS)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("retention", params, w, dtype, max_requests=max_requests), lambda h: P.retention_mixer(h, plain, "m", m, EPS)


def gla_rig(dtype, m, W, seed, max_requests=4, craft=None, rank=5):
    w = draw(mixer_shapes("right", m, W, "m", rank), seed)
    if craft:
        craft(w)
    params = dict(hidden_size=W, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=m["tau"], eps=EPS)
    plain = {k: v.double() for k, v in w.items()}
    return MixerRig("gated_linear_attention", params, w, dtype, max_requests=max_requests), lambda h: P.gla_mixer(h, plain, "m", m, EPS)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,chunk,W,page", [(4, 2, 16, 8, 21, 64, 16), (5, 5, 12, 20, 7, 90, 8), (20, 1, 32, 64, 48, 128, 16),
                                                             (8, 2, 64, 32, 30, 128, 16), (3, 1, 24, 24, 0, 48, 4), (6, 2, 128, 64, 16, 64, 16)])
def test_chunked_attention_whole_in_portions_and_token_by_token(dtype, heads, kv, dim, vdim, chunk, W, page):
    m = left(heads, kv, dim, vdim, chunk=chunk)
    x = rounded(torch.randn(75, W, generator=gen(12)), dtype)
    for cuts in CUTS:
        rig, plain = left_rig(dtype, m, W, 13, page=page)
        close(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}", f32=1e-4, bf16=3e-2)


def same_direction(w, heads, kv, dim):
    """W_q of every head becomes W_k of its kv head (plain gains): a token's query points along the key of any token with the
    same input."""
    w["m.q"] = w["m.k"].view(kv, dim, -1).repeat_interleave(heads // kv, 0).reshape(heads * dim, -1).contiguous()
    w["m.q.norm"], w["m.k.norm"] = torch.ones_like(w["m.q.norm"]), torch.ones_like(w["m.k.norm"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk,page,dim,vdim", [(24, 8, 32, 64), (21, 16, 16, 24), (150, 16, 64, 64), (64, 16, 64, 32), (10, 16, 32, 32)])
def test_one_key_just_inside_and_just_outside_a_chunk(dtype, chunk, page, dim, vdim):
    """ONE earlier token has three times the last token's input, and queries point along keys: after the norm it
    scores like the token's own key and its value is three times as large, so it decides the output where it is seen.  It lies at
    the chunk's first position, the one before it (in the chunk before: not seen), at page borders inside and outside; the
    query is decoded alone, at a portion's end, in a portion that begins inside a chunk, and beside other requests."""
    W, heads, kv = 64, 4, 2
    m = left(heads, kv, dim, vdim, chunk=chunk, scale=4.0 / dim ** 0.5)
    make = lambda: left_rig(dtype, m, W, 15, page=page, pages=120, craft=lambda w: same_direction(w, heads, kv, dim))
    g = gen(14)
    n = 3 * chunk + chunk // 2 + 1                          # the last query lies in the middle of the fourth chunk
    start = 3 * chunk
    base_x = torch.randn(n, W, generator=g)
    spots = sorted({start, start - 1, start + 1, start - chunk, start // page * page, start // page * page - 1, -(-start // page) * page, n - 2, 0})
    for at in [s for s in spots if s < n - 1]:
        x = base_x.clone()
        x[at] = 3.0 * x[n - 1]
        x = rounded(x, dtype)
        _, plain = make()
        want = plain(x)
        other = x.clone()
        other[at] = base_x[at]
        changed = float((plain(rounded(other, dtype))[-1] - want[-1]).abs().max()) / float(want[-1].abs().max())
        assert (changed > 0.1) if at >= start else (changed == 0.0), (at, start, changed)
        rig, _ = make()
        close(rig.cut("a", x, [n - 1, 1])[-1:], want[-1:], dtype, f"decoded, key {at}", f32=1e-4, bf16=3e-2)
        rig, _ = make()
        close(rig.cut("b", x, [n - 3, 3])[-1:], want[-1:], dtype, f"portion, key {at}", f32=1e-4, bf16=3e-2)
        rig, _ = make()
        close(rig.cut("c", x, [start - 2, n - start + 2])[-1:], want[-1:], dtype, f"portion over the edge, key {at}", f32=1e-4, bf16=3e-2)
        rig, _ = make()
        rig.step([("d", x[:start + 1]), ("e", rounded(torch.randn(5, W, generator=g), dtype))])
        res = rig.step([("e", rounded(torch.randn(1, W, generator=g), dtype)), ("d", x[start + 1:]), ("f", rounded(torch.randn(40, W, generator=g), dtype))])
        close(res[1][-1:], want[-1:], dtype, f"batch, key {at}", f32=1e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_chunked_attention_in_a_pool_of_little_more_than_a_chunk(dtype):
    """Pages of finished chunks are used again while the request goes on, and by a second one."""
    m = left(4, 2, 16, 16, chunk=24)
    rig, plain = left_rig(dtype, m, 48, 17, page=8, pages=2 * (24 // 8 + 2))
    a, b = rounded(torch.randn(170, 48, generator=gen(3)), dtype), rounded(torch.randn(90, 48, generator=gen(4)), dtype)
    got = {"a": [], "b": []}
    for i in range(0, 170, 5):
        entries = [("a", a[i:i + 5])] + ([("b", b[i // 5 * 3:i // 5 * 3 + 3])] if i // 5 < 30 else [])
        for (k, _), r in zip(entries, rig.step(entries)):
            got[k].append(r)
    close(torch.cat(got["a"]), plain(a), dtype, "a", f32=1e-4, bf16=3e-2)
    close(torch.cat(got["b"]), plain(b), dtype, "b", f32=1e-4, bf16=3e-2)
    rig.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,rot,base,W", [(2, 16, 24, 8, 100.0, 64), (3, 20, 12, 20, 50.0, 90), (4, 64, 64, 64, 1e6, 128), (1, 96, 8, 0, 1.0, 48),
                                                        (6, 8, 24, 2, 3.0, 48), (1, 256, 40, 128, 1e4, 64)])
def test_retention_whole_in_portions_and_token_by_token(dtype, heads, dim, vdim, rot, base, W):
    m = retention(heads, dim, vdim, rot=rot, base=base)["mixer"]
    x = rounded(torch.randn(75, W, generator=gen(18)) * 1.5, dtype)
    for cuts in CUTS:
        rig, plain = retention_rig(dtype, m, W, 19)
        close_recurrent(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,tau,W,rank", [(2, 16, 24, 4.0, 64, 5), (3, 20, 12, 1.0, 90, 1), (4, 64, 32, 16.0, 128, 16), (1, 96, 8, 8.0, 48, 33),
                                                        (6, 8, 24, 2.5, 48, 7), (2, 128, 64, 16.0, 64, 16)])
def test_gated_linear_attention_whole_in_portions_and_token_by_token(dtype, heads, dim, vdim, tau, W, rank):
    m = right(heads, dim, vdim, tau)
    x = rounded(torch.randn(75, W, generator=gen(20)) * 1.5, dtype)
    for cuts in CUTS:
        rig, plain = gla_rig(dtype, m, W, 21, rank=rank)
        close_recurrent(rig.cut("r", x, cuts), plain(x), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["retention", "gated"])
def test_one_far_token_decides_a_recurrent_state(dtype, kind):
    """ONE token's input is twenty times the others', and hardly anything decays: its key and value stay in the state for
    hundreds of tokens and decide every later read-out, over blocks of a prompt that run side by side, over portions and over
    decoded tokens.  Without it the output points elsewhere."""
    W, heads, dim, vdim, n = 64, 2, 16, 16, 520
    if kind == "retention":
        m = retention(heads, dim, vdim, decay=[1.0, 0.9999])["mixer"]
        make = lambda: retention_rig(dtype, m, W, 23)
    else:
        m = right(heads, dim, vdim, tau=16.0)

        def craft(w):
            w["m.a2.b"] = torch.full_like(w["m.a2.b"], 12.0)
            w["m.a2"] = 0.1 * w["m.a2"]
        make = lambda: gla_rig(dtype, m, W, 23, craft=craft)
    for at in (0, 63, 64, 200, n - 3):
        x = torch.randn(n, W, generator=gen(24))
        x[at] *= 20.0
        x = rounded(x, dtype)
        _, plain = make()
        want = plain(x)
        y = x.clone()
        y[at] = 0.0
        d = plain(y)[-1] - want[-1]
        assert float(d.norm()) > 0.3 * float(want[-1].norm())
        for cuts in ([n], [n - 20] + [1] * 20, [at + 1, n - at - 2, 1], [100, 2, 318, 100]):
            rig, _ = make()
            got = rig.cut("r", x, cuts)
            close_recurrent(got[-25:], want[-25:], dtype, f"{at} {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["retention", "gated"])
def test_recurrent_mixers_in_batches_with_slots_used_again_and_long_decoding(dtype, kind):
    """Three slots for five requests: requests of unequal length side by side, a finished request's slot taken by the next
    (whose state must start at zero), a request left out of a step, and one request decoded for 300 tokens."""
    W = 64
    if kind == "retention":
        rig, plain = retention_rig(dtype, retention(3, 16, 24, rot=16)["mixer"], W, 23, max_requests=3)
    else:
        rig, plain = gla_rig(dtype, right(4, 16, 8, 4.0), W, 23, max_requests=3)
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
    l, r = left(6, 3, 16, 8, chunk=22), right(4, 8, 16, tau=4.0)
    w = dict(draw(mixer_shapes("left", l, W, "m.left"), 30), **draw(mixer_shapes("right", r, W, "m.right"), 31))
    lp = dict(hidden_size=W, num_heads=6, num_kv_heads=3, key_dim=16, value_dim=8, scale=l["scale"], eps=EPS, qk_norm="projection", chunk=22)
    rp = dict(hidden_size=W, heads=4, dim=8, vdim=16, tau=4.0, eps=EPS)
    params = dict(parts=[dict(kind="normed_qk_attention", params=lp, under="left", scale=0.6),
                         dict(kind="gated_linear_attention", params=rp, under="right", scale=1.7)])
    plain = {k: v.double() for k, v in w.items()}
    x = rounded(torch.randn(75, W, generator=gen(32)), dtype)
    want = P.parallel_mixer(x, plain, "m", dict(left=l, right=r, left_scale=0.6, right_scale=1.7), EPS)
    for cuts in CUTS:
        rig = MixerRig("parallel_mixers", params, w, dtype, page=8)
        close_recurrent(rig.cut("r", x, cuts), want, dtype, f"{cuts}")


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
    root = tmp_path_factory.mktemp("reperax")

    def get(name):
        if name not in _models:
            _models[name] = write_model(root, name, seed=sorted(CONFIGS).index(name))
        return _models[name]
    return get


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_every_layer_run(models, dtype, name):
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 45, 1)
    want, streams = P.forward(cfg, w, toks, want_layers=True)
    s = Served(folder, dtype)
    trace = {}
    got = s.step([("a", toks, list(range(len(toks))))], trace=trace)
    assert agrees(got, want, dtype)
    for j, (i, _) in enumerate(P.runs(cfg)):
        x = trace.get(f"run{j}.out", trace[f"l{i}.out"])
        assert x.dtype == torch.float32, "the stream between layers is float32 whatever the compute dtype"
        if dtype == torch.float32:
            close(x, streams[j], dtype, f"stream after layer run {j}", f32=5e-5)
        else:
            per_token = (x.double().cpu() - streams[j]).pow(2).mean(-1).sqrt() / streams[j].pow(2).mean(-1).sqrt()
            assert float(per_token.median()) < TOL[dtype] and float(per_token.quantile(0.9)) < 0.3, f"stream after layer run {j}: {per_token}"
    # the first tokens of a sequence, alone: nothing before them for the shift, a state of zeros, a chunk of one
    s2 = Served(folder, dtype)
    first = torch.cat([s2.step([("b", toks[:1], [0])]), s2.step([("b", toks[1:2], [0])]), s2.step([("b", toks[2:4], [0, 1])])])
    if dtype == torch.float32:
        assert agrees(first, want[:4], dtype)
    else:
        assert float(errors(first, want[:4]).max()) < max(0.3, 1.5 * float(errors(got[:4], want[:4]).max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("small", 16), ("odd", 8), ("wide", 32), ("retention_only", 16), ("parallel_only", 4)])
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
    finished requests (and finished chunks) are used again; every row against the plain implementation of its request alone."""
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
    together = (torch.cat([r for k in toks for r in got[k]]), torch.cat([want[k] for k in toks]))
    assert agrees(*together, dtype)
    for k in toks if dtype == torch.float32 else ():       # (bfloat16: a request of seven tokens is too few for a typical position)
        assert agrees(torch.cat(got[k]), want[k], dtype), k
    s.runner.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("small", 8), ("odd", 4), ("wide", 16)])
def test_long_prompts_and_long_decoding(models, dtype, name, page):
    """330 tokens, first all but ten decoded one by one (chunk after chunk ends under the decoded tokens and its pages go back),
    then in one prompt of several blocks with the rest decoded."""
    folder, cfg, w = models(name)
    toks = tokens_for(cfg, 330, 5)
    want = P.forward(cfg, w, toks)
    chunks = [L["mixer"]["left"].get("mask", {}).get("size", 0) for L in cfg["layers"] if L["type"] == "parallel"]
    pages = -(-330 // page) + 1 if 0 in chunks else -(-(max(chunks) + 12) // page) + 2
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_token_before_alone_decides(tmp_path, dtype):
    """With a shift of one the mixer reads nothing but the token before, in every layer and pass: a row kept wrong at a portion's
    edge, handed to another request, or left from a slot's last owner would change the next token's logits altogether."""
    cfg = copy.deepcopy(CONFIGS["wide"])
    weights = random_weights(cfg, 40)
    for k in weights:
        if k.endswith(".shift"):
            weights[k] = torch.ones_like(weights[k])
    folder, cfg, w = write_model(tmp_path, "shifted", seed=40, cfg=cfg, weights=weights)
    toks = {k: tokens_for(cfg, n, 50 + n) for k, n in dict(a=40, b=31, c=12).items()}
    want = {k: P.forward(cfg, w, t) for k, t in toks.items()}
    s = Served(folder, dtype, max_requests=2)
    got, at = {k: [] for k in toks}, {k: 0 for k in toks}
    for step in ([("a", 7)], [("b", 1), ("a", 1)], [("a", 2), ("b", 29)], [("b", 1), ("a", 9)], [("c", 1), ("a", 1)], [("a", 20), ("c", 11)]):
        out, row = s.step([(k, toks[k][at[k]:at[k] + n], list(range(n))) for k, n in step]), 0
        for k, n in step:
            got[k].append(out[row:row + n]); row += n; at[k] += n
            if at[k] == len(toks[k]):
                s.end(k)
    assert agrees(torch.cat([r for k in toks for r in got[k]]), torch.cat([want[k] for k in toks]), dtype)
    # what forgetting it would do
    lost = P.forward(cfg, dict(w, **{k: torch.zeros_like(v) for k, v in w.items() if k.endswith(".shift")}), toks["a"])
    assert float(errors(lost, want["a"]).median()) > 0.3


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
    """Sizes, counts, layer order, loop and constants drawn from a seed."""
    rnd = random.Random(seed)
    width = rnd.choice([48, 64, 96, 128, 192])

    def a_retention():
        heads, dim = rnd.choice([1, 2, 3, 6]), rnd.choice([8, 16, 24, 64, 128])
        rot = rnd.choice([0, 2, dim // 2, dim])
        return retention(heads, dim, rnd.choice([8, 12, 32, 64]), decay=[rnd.choice([0.5, 0.9, 0.99, 0.999, 1.0]) for _ in range(heads)],
                         rot=rot - rot % 2, base=rnd.choice([100.0, 10000.0, 5e5]))

    def a_parallel():
        kv, dim = rnd.choice([1, 2, 3]), rnd.choice([8, 16, 24, 32, 64, 128])
        l = left(kv * rnd.choice([1, 2, 4, 5]), kv, dim, rnd.choice([8, 12, 32, 64]), chunk=rnd.choice([0, 1, 5, 16, 40, 63, 64, 100, 1000]),
                 scale=rnd.choice([0.4, 1.2, 4.0]) / dim ** 0.5)
        r = right(rnd.choice([1, 2, 3]), rnd.choice([8, 20, 64, 128]), rnd.choice([8, 12, 32, 64]), tau=rnd.choice([1.0, 2.0, 16.0]))
        return parallel(l, r, rnd.choice([0.5, 1.0, 1.2]), rnd.choice([0.25, 1.0, 2.0]))

    layers = [layer(rnd.choice([a_retention, a_parallel])(), dense(rnd.choice([32, 72, 128, 192])) if rnd.random() < 0.75 else None)
              for _ in range(rnd.randint(2, 5))]
    start = rnd.randrange(len(layers))
    loop = (start, rnd.randint(start + 1, len(layers)), rnd.choice([1, 2, 3])) if rnd.random() < 0.8 else None
    return model(rnd.choice([97, 256, 640]), width, layers, eps=rnd.choice([1e-5, 1e-6]), cap=rnd.choice([None, 5.0, 30.0]), loop=loop)


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
