#!/usr/bin/env python3
"""Decode and prefill throughput of the engine on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

The default run has the layer sizes of the Qwen3-0.6B shape with random weights
(N(0, 0.02), norm gains 1 + N(0, 0.1)), a batch of 8 and a context of 4096
tokens, in bfloat16.  A "step" is one decode step: every live request gets its
next token.  One JSON line is printed:

  value        decoded tokens a second, K replays of the captured decode step
               timed on the device with CUDA events
  e2e          the same through the Python entry point (Engine.submit / Engine.step):
               host token ids in, host token ids out, every step with its copy of
               the packed step from pinned memory and its copy of the tokens back; five
               timed rounds of K steps, the last of which (the K positions before the
               context) is the one reported and the others its spread
  prefill      one prompt of 2048 tokens through the step function (frac: of the library product's burst rate;
               frac_sustained: of its rate in a seconds-long loop under the power cap)
  roofline     bytes the decode step has to read (every weight once and the live
               requests' cache) over its time, against the measured copy bandwidth
  points       decode tokens a second at batch 1 and 64 at the same context, and at batch 1, 8 and 64
               at context 512 (right after the baseline's 512-token prompts), each with its fraction
               of the HBM roofline
  generate     whole generations through Engine.generate by the wall clock: 64 prompts of 512 tokens,
               128 new tokens each, steps of at most 2048 tokens (the first call, which captures its
               steps, is not counted)
  repeats      the spread of the timed region: it is repeated ten times (median, min, max)
  shapes       the same figures at the baseline's 8B shape (36 of 36 layers; with its mixed step: 64
               requests decoding at context 4096 beside a 512-token portion) and at the 32B shape's
               layer sizes (16 of 64 layers, named)
  reference_kernel   the reference's own CUDA kernel (paged_attention.cu, compiled unchanged for
               sm_100a) against this engine's decode attention on the same keys and values

The engine runs on one GPU: for --gpus above 1 a line says so and the exit code is 2.
"""

from __future__ import annotations

import argparse
import json
import os
import shutil
import statistics
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

SHAPE_0_6B = dict(
    architectures=["Qwen3ForCausalLM"], model_type="qwen3", hidden_act="silu", attention_bias=False,
    hidden_size=1024, intermediate_size=3072, num_hidden_layers=28, num_attention_heads=16, num_key_value_heads=8,
    head_dim=128, rms_norm_eps=1e-6, vocab_size=151936, max_position_embeddings=40960, tie_word_embeddings=True,
    rope_theta=1000000.0, sliding_window=None, use_sliding_window=False,
)
# the other two shapes the baseline names, for --shape: the default run and its JSON contract stay the 0.6B one
SHAPE_8B = dict(SHAPE_0_6B, hidden_size=4096, intermediate_size=12288, num_hidden_layers=36, num_attention_heads=32,
                num_key_value_heads=8, tie_word_embeddings=False)
SHAPE_32B = dict(SHAPE_0_6B, hidden_size=5120, intermediate_size=25600, num_hidden_layers=64, num_attention_heads=64,
                 num_key_value_heads=8, tie_word_embeddings=False)
SHAPES = {"0.6b": ("Qwen3-0.6B", SHAPE_0_6B), "8b": ("Qwen3-8B", SHAPE_8B), "32b": ("Qwen3-32B", SHAPE_32B)}
PAGE = 16
PREFILL_TOKENS = 2048


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            d = json.load(f)
        return dict(hbm_gbs=float(d["hbm_gbs"]), bf16_tflops=float(d["bf16_tflops"]),
                    bf16_tflops_sustained=float(d.get("bf16_tflops_sustained", d["bf16_tflops"])), source="measured")
    return dict(hbm_gbs=6650.0, bf16_tflops=1590.0, bf16_tflops_sustained=1400.0, source="fallback")


class ClockSampler:
    """nvidia-smi clocks and throttle reasons every 200 ms while the timed regions run."""

    FIELDS = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
              "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc, self.marks = [], None, []

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                                          "-lms", "200"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None
            return
        threading.Thread(target=self._read, daemon=True).start()

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append((time.time(), [c.strip() for c in line.split(",")]))

    def region(self, t0, t1):
        self.marks.append((t0, t1))

    def stop(self):
        if self.proc is not None:
            time.sleep(0.25)
            self.proc.terminate()
        inside = [r for t, r in self.rows if any(a - 0.1 <= t <= b + 0.1 for a, b in self.marks)] or [r for _, r in self.rows]
        if not inside:
            return dict(sm_mhz=None, sm_max_mhz=None, reasons=["nvidia-smi gave no samples"])
        sm = [float(r[0]) for r in inside if r[0].replace(".", "").isdigit()]
        mx = [float(r[1]) for r in inside if r[1].replace(".", "").isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) > 4 + i and r[4 + i].lower().startswith("active") for r in inside)]
        return dict(sm_mhz=statistics.median(sm) if sm else None, sm_max_mhz=max(mx) if mx else None,
                    reasons=reasons, samples=len(inside))


REF_KERNEL = os.path.join(ROOT, "baseline", "_ref", "crates", "pagedllm", "src", "kernels", "paged_attention.cu")


def reference_kernel_points(clocks, reps=10):
    """The reference's one CUDA kernel (crates/pagedllm/src/kernels/paged_attention.cu, compiled unchanged for
    sm_100a with -DELEM=__nv_bfloat16 and launched as crates/pagedllm/src/kernels/paged_attention.rs:626-634,
    684-688 launches it: grid (heads, rows), 128 threads, (blocks x block size + 128) floats of shared memory)
    against this engine's decode attention (the bulk-copy kernel and the reduction of its splits) on the same
    random keys, values and queries, each in its own cache layout.  Microseconds a launch, median of ``reps``."""
    import ctypes
    import subprocess as sp
    import numpy as np
    import torch
    from paged_llm_rs_b200.kernels import attention_plan, ops
    from paged_llm_rs_b200.parts.base import AttentionWork

    if not os.path.exists(REF_KERNEL):
        return {"unavailable": "baseline/_ref holds no copy of the reference's paged_attention.cu"}
    try:
        from cuda.bindings import driver
    except Exception as e:     # noqa: BLE001
        return {"unavailable": f"cuda-python is not importable: {e}"}
    tmp = tempfile.mkdtemp(prefix="pllm_ref_kernel_")
    try:
        cubin = os.path.join(tmp, "paged_attention.cubin")
        r = sp.run(["nvcc", "-cubin", "-arch=sm_100a", "-DELEM=__nv_bfloat16", REF_KERNEL, "-o", cubin],
                   capture_output=True, text=True)
        if r.returncode != 0:
            return {"unavailable": "nvcc failed on the reference's kernel: " + r.stderr.strip()[-200:]}
        torch.zeros(1, device="cuda")                      # the primary context, current
        err, module = driver.cuModuleLoadData(open(cubin, "rb").read())
        if int(err) != 0:
            return {"unavailable": f"cuModuleLoadData: {err}"}
        err, fn = driver.cuModuleGetFunction(module, b"paged_attention_decode")
        if int(err) != 0:
            return {"unavailable": f"cuModuleGetFunction: {err}"}
    finally:
        shutil.rmtree(tmp, ignore_errors=True)

    dev, page = "cuda", PAGE
    out = {}
    g = torch.Generator(device=dev).manual_seed(0)
    sm2 = 2 * torch.cuda.get_device_properties(0).multi_processor_count

    def timed(fn_):
        for _ in range(3):
            fn_()
        torch.cuda.synchronize()
        ts = []
        for _ in range(reps):
            flush_l2()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(); fn_(); b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b) * 1e3)
        return statistics.median(ts)

    worst = 0.0
    for nh, nkv, hd, tag in ((16, 8, 128, "h16"), (32, 8, 128, "h32")):
        for ctx in (512, 4096):
            for B in (1, 8, 64):
                n_blocks = ctx // page
                tokens = B * ctx
                k = torch.randn(tokens, nkv, hd, device=dev, generator=g).bfloat16()
                v = torch.randn(tokens, nkv, hd, device=dev, generator=g).bfloat16()
                q = torch.randn(B, nh * hd, device=dev, generator=g).bfloat16()
                # pages in a shuffled order, the same order in both layouts
                perm = torch.randperm(B * n_blocks, device=dev, generator=g).to(torch.int32).view(B, n_blocks)
                # the reference's layout: [slots, kv_heads * head_dim], slot = block * block_size + offset
                slot_of = (perm.long()[:, :, None] * page + torch.arange(page, device=dev)[None, None]).view(-1)
                rk = torch.empty(tokens, nkv * hd, device=dev, dtype=torch.bfloat16)
                rv = torch.empty_like(rk)
                rk[slot_of] = k.view(tokens, -1); rv[slot_of] = v.view(tokens, -1)
                table_u32 = perm.contiguous()
                lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
                r_out = torch.zeros(B, nh * hd, device=dev, dtype=torch.bfloat16)
                shared = (n_blocks * page + 128) * 4
                assert shared <= 48 << 10
                stream = torch.cuda.current_stream().cuda_stream
                vals = (q.data_ptr(), rk.data_ptr(), rv.data_ptr(), table_u32.data_ptr(), lens.data_ptr(), r_out.data_ptr(),
                        page, hd, nh, nkv, n_blocks, 128, 4, float(hd ** -0.5))
                types = (ctypes.c_void_p,) * 6 + (ctypes.c_uint,) * 7 + (ctypes.c_float,)

                def ref():
                    (e,) = driver.cuLaunchKernel(fn, nh, B, 1, 128, 1, 1, shared, stream, (vals, types), 0)
                    assert int(e) == 0, e
                # this engine's layout: [pages, kv_heads, page, head_dim], rows swizzled
                kp = k.view(B * n_blocks, page, nkv, hd).transpose(1, 2).contiguous()
                vp = v.view(B * n_blocks, page, nkv, hd).transpose(1, 2).contiguous()
                ok = torch.empty_like(kp); ov = torch.empty_like(vp)
                ok[perm.view(-1).long()] = kp; ov[perm.view(-1).long()] = vp
                ops.swizzle_pool_(ok); ops.swizzle_pool_(ov)
                work, red, parts = attention_plan.plan_attention([(i, 1, ctx - 1) for i in range(B)], 1, None, nkv, sm2)
                wd = torch.from_numpy(np.ascontiguousarray(work)).to(dev)
                rd = torch.from_numpy(np.ascontiguousarray(red)).to(dev) if len(red) else torch.zeros(1, 4, dtype=torch.int32, device=dev)
                nw = torch.tensor([len(work)], dtype=torch.int32, device=dev)
                nr = torch.tensor([len(red)], dtype=torch.int32, device=dev)
                po = torch.zeros(max(parts, 1), nh, hd, device=dev)
                pm = torch.zeros(max(parts, 1), nh, 2, device=dev)
                o_out = torch.zeros_like(r_out)
                st = torch.zeros(1, dtype=torch.int32, device=dev)

                plan = AttentionWork(wd, nw, len(work), rd, nr, len(red), po, pm, kinds=1,
                                     many_splits=attention_plan.many_splits(B, nkv, sm2))

                def ours():
                    ops.paged_attention(q, ok, ov, perm, plan, o_out, nh, nkv, hd, 0, hd ** -0.5, st, swizzled=True)
                t0 = time.time()
                t_ref, t_ours = timed(ref), timed(ours)
                clocks.region(t0, time.time())
                assert int(st.item()) == 0
                worst = max(worst, float((r_out.float() - o_out.float()).abs().max()))
                key = f"{tag}_b{B}_ctx{ctx}"
                out[key + "_ref_us"] = round(t_ref, 1)
                out[key + "_ours_us"] = round(t_ours, 1)
                del k, v, rk, rv, kp, vp, ok, ov
    out["max_abs_diff"] = round(worst, 5)
    out["what"] = ("decode attention alone, microseconds a launch (ours: attention + reduction of splits), cold L2; "
                   "h16 = 16 query heads over 8 kv heads of 128 (0.6B), h32 = 32 over 8 (8B)")
    return out


_FLUSH = None


def flush_l2():
    """Write a buffer larger than the 126 MB L2."""
    import torch
    global _FLUSH
    if _FLUSH is None:
        _FLUSH = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    _FLUSH.fill_(1)


def time_on_device(fn, steps, warmup, repeats=0):
    """``warmup`` untimed calls, then exactly ``steps`` calls between two events (the contract's timed
    region); then, for the spread, ``repeats`` more such regions.  Returns (ms a call in the first
    region, (wall start, wall end), {"n", "median_ms", "min_ms", "max_ms"} over all regions)."""
    import torch
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    per = []
    t0 = time.time()
    for _ in range(1 + repeats):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(steps):
            fn()
        b.record()
        torch.cuda.synchronize()
        per.append(a.elapsed_time(b) / steps)
    spread = dict(n=len(per), median_ms=round(statistics.median(per), 4), min_ms=round(min(per), 4), max_ms=round(max(per), 4))
    return per[0], (t0, time.time()), spread


def decode_point(runner, batch, context, steps, warmup, clocks, repeats=9):
    """Device time of the captured decode step at ``batch`` requests of ``context`` tokens."""
    import numpy as np
    from paged_llm_rs_b200.engine.step import StepEntry

    cache = runner.cache
    ids = [f"bench{b}" for b in range(batch)]
    for r in ids:
        cache.open(r)
        assert cache.reserve(r, context), "the cache pool is too small for this point"
        cache.commit(r, context - 1)   # the cache holds context-1 tokens (random contents); the step adds one
    entries = [StepEntry(r, [1 + i], [0]) for i, r in enumerate(ids)]
    temp = np.zeros(batch, dtype=np.float32)
    uni = np.zeros(batch, dtype=np.float32)
    runner.step_and_sample(entries, temp, uni)          # packs the step, captures the graph on first use
    graph = runner._decode_graph(entries)
    ms, span, spread = time_on_device(graph.replay, steps, warmup, repeats)
    clocks.region(*span)
    launches = graph.launches
    for r in ids:
        cache.close(r)
    return ms, launches, spread


def mixed_point(runner, decoding, context, portion, behind, vocab, steps, warmup, clocks, repeats=9):
    """Device time of one captured mixed step: ``decoding`` requests at ``context`` tokens take their next
    token beside a portion of ``portion`` prompt tokens that has ``behind`` tokens of its prompt before it."""
    import numpy as np
    from paged_llm_rs_b200.engine.step import StepEntry

    cache = runner.cache
    ids = [f"mix{b}" for b in range(decoding)]
    for r in ids:
        cache.open(r)
        assert cache.reserve(r, context)
        cache.commit(r, context - 1)
    cache.open("mixp")
    assert cache.reserve("mixp", behind + portion)
    cache.commit("mixp", behind)
    prompt = np.random.default_rng(0).integers(0, vocab, portion).tolist()
    entries = [StepEntry(r, [1 + i], [0]) for i, r in enumerate(ids)] + [StepEntry("mixp", prompt, [])]
    zeros = np.zeros(decoding, dtype=np.float32)
    was = runner.graph_step_tokens
    runner.graph_step_tokens = decoding + portion
    try:
        runner.step_and_sample(entries, zeros, zeros)
        graph = runner._portion_graph(entries)
        assert graph is not None, "the mixed step does not run as a captured step"
        ms, span, spread = time_on_device(graph.replay, steps, warmup, repeats)
    finally:
        runner.graph_step_tokens = was
    clocks.region(*span)
    for r in ids + ["mixp"]:
        cache.close(r)
    return ms, spread


def prefill_point(runner, vocab, clocks, repeats=9):
    """One prompt of PREFILL_TOKENS tokens through the step function, as the engine runs a prompt's portion:
    the step and its greedy sample, captured and replayed, host packing included."""
    import numpy as np
    from paged_llm_rs_b200.engine.step import StepEntry

    prompt = np.random.default_rng(0).integers(0, vocab, PREFILL_TOKENS).tolist()
    one_zero = np.zeros(1, dtype=np.float32)

    def prefill():
        runner.cache.open("prefill")
        runner.cache.reserve("prefill", PREFILL_TOKENS)
        runner.step_and_sample([StepEntry("prefill", prompt, [PREFILL_TOKENS - 1])], one_zero, one_zero)
        runner.cache.close("prefill")

    # five prompts to a timed region: the host packs the next step while the GPU runs this one
    ms, span, spread = time_on_device(prefill, 5, 3, repeats)
    clocks.region(*span)
    return spread["median_ms"], spread


def generate_point(model_dir, vocab, clocks, requests=64, prompt=512, new=128, repeats=3):
    """Whole generations through ``Engine.generate``: ``requests`` random prompts of ``prompt`` tokens, ``new``
    tokens each, greedy, no stop token; host token lists in and out, by the wall clock.  The first call
    captures the steps it needs and is not counted.  What the scheduler, the portions under the token
    budget, the step packing and the copies cost shows as the gap to the device-timed points."""
    import numpy as np
    import torch
    from paged_llm_rs_b200 import Engine
    eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=requests * ((prompt + new) // PAGE + 2) + 64,
                 max_batch=requests, chunk=PREFILL_TOKENS, prefix_cache=False,
                 max_prefill_seqs=max(1, PREFILL_TOKENS // prompt))    # (the token budget decides, not the count)
    rng = np.random.default_rng(2)
    prompts = [rng.integers(0, vocab, prompt).tolist() for _ in range(requests)]
    eng.generate(prompts, max_tokens=new, stop_tokens=())
    torch.cuda.synchronize()
    per = []
    for _ in range(repeats):
        t0 = time.time()
        outs = eng.generate(prompts, max_tokens=new, stop_tokens=())
        torch.cuda.synchronize()
        t1 = time.time()
        clocks.region(t0, t1)
        assert all(len(o) == new for o in outs)
        per.append((t1 - t0) * 1e3)
    ms = statistics.median(per)
    m = eng.scheduler.metrics
    return dict(requests=requests, prompt_tokens=prompt, new_tokens=new, ms=round(ms, 1), min_ms=round(min(per), 1),
                max_ms=round(max(per), 1), generated_tokens_s=round(requests * new / (ms / 1e3), 1),
                all_tokens_s=round(requests * (prompt + new) / (ms / 1e3), 1), step_token_budget=PREFILL_TOKENS,
                steps_per_call=m.steps // (repeats + 1))


def long_prompt_points(runner, sizes, total, clocks):
    """A prompt of ``total`` tokens through the step function in portions of 2048: each portion's device time, and
    the fraction of the tensor peak its flops make (the products of 2048 rows, and the attention over everything
    before the portion and half of itself)."""
    import numpy as np
    import torch
    from paged_llm_rs_b200.engine.step import StepEntry
    T, cache, pk = PREFILL_TOKENS, runner.cache, peaks()
    L, nh, hd, V, H = sizes["L"], sizes["nh"], sizes["hd"], sizes["V"], sizes["H"]
    products = sizes["prefill_flops"] - 2 * V * H - 2 * T * T * nh * hd * L        # of a portion's 2048 rows
    prompt = np.random.default_rng(0).integers(0, V, total).tolist()
    zero = np.zeros(1, dtype=np.float32)
    out = {}
    for rep in range(2):                         # (the first pass captures the steps)
        cache.open("long")
        events = []
        t0 = time.time()
        for c in range(0, total, T):
            assert cache.reserve("long", T)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            runner.step_and_sample([StepEntry("long", prompt[c:c + T], [T - 1])], zero, zero)
            b.record()
            events.append((c, a, b))
            cache.commit("long", T)
        torch.cuda.synchronize()
        clocks.region(t0, time.time())
        cache.close("long")
    for c, a, b in events:
        if c % 8192 == 0 or c == total - T:
            ms = a.elapsed_time(b)
            attention = 4 * T * (c + T / 2) * nh * hd * L
            flops = products + attention + 2 * V * H
            out[f"portion_at_{c}"] = dict(ms=round(ms, 3), tokens_s=round(T / ms * 1e3, 1), attention_share_of_flops=round(attention / flops, 3),
                                          bf16_frac=round(flops / (ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4))
    out["whole_prompt_ms"] = round(sum(a.elapsed_time(b) for _, a, b in events), 1)
    out["tokens"] = total
    return out


def shape_sizes(shape):
    L, H, I = shape["num_hidden_layers"], shape["hidden_size"], shape["intermediate_size"]
    nh, nkv, hd, V = shape["num_attention_heads"], shape["num_key_value_heads"], shape["head_dim"], shape["vocab_size"]
    layer_params = H * (nh + 2 * nkv) * hd + nh * hd * H + 3 * H * I
    return dict(L=L, H=H, I=I, nh=nh, nkv=nkv, hd=hd, V=V, layer_params=layer_params,
                weight_bytes=2 * (L * layer_params + V * H),          # a tied table is read once, as the head
                kv_token_bytes=2 * L * nkv * hd * 2,
                prefill_flops=2 * PREFILL_TOKENS * L * layer_params + 2 * PREFILL_TOKENS ** 2 * nh * hd * L + 2 * V * H)


def scratch_dir():
    """Where the random model folder is written: memory-backed when there is room (a 16 GB file is written
    and read back once), else the temporary folder."""
    try:
        if shutil.disk_usage("/dev/shm").free > (40 << 30):
            return "/dev/shm"
    except OSError:
        pass
    return None


def other_shape(key, layers, pk, clocks, steps, warmup):
    """Decode at batch 1, 8 and 64 (contexts 4096 and 512), the 2048-token prefill and, for the 8B shape, the
    baseline's mixed step, at another of the baseline's shapes: flat figures with their roofline fractions."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    name, shape = SHAPES[key][0], dict(SHAPES[key][1])
    full = shape["num_hidden_layers"]
    shape["num_hidden_layers"] = layers or full
    z = shape_sizes(shape)
    out = {f"{key}_layers": z["L"], f"{key}_layers_of_shape": full}
    tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
    try:
        model_dir = write_random_model(os.path.join(tmp, "model"), shape, 0, device="cuda")
        ctx = 4096
        pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
        eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                     prefix_cache=False)
        shutil.rmtree(tmp, ignore_errors=True)
        runner = eng.runner
        for g in runner.cache.groups:
            g.pool.normal_(0.0, 1.0)
        for c in (4096, 512):
            for b in (1, 8, 64):
                ms, _, spread = decode_point(runner, b, c, max(5, steps // 2), warmup, clocks, repeats=4)
                ms = spread["median_ms"]
                gbs = (z["weight_bytes"] + b * c * z["kv_token_bytes"]) / (ms / 1e3) / 1e9
                tag = f"{key}_decode_b{b}" + ("" if c == 4096 else f"_ctx{c}")
                out[tag] = round(b / (ms / 1e3), 1)
                out[tag + "_hbm_frac"] = round(gbs / pk["hbm_gbs"], 4)
        pms, _ = prefill_point(runner, z["V"], clocks, repeats=4)
        out[f"{key}_prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
        out[f"{key}_prefill_ms"] = round(pms, 3)
        out[f"{key}_prefill_bf16_frac"] = round(z["prefill_flops"] / (pms / 1e3) / (pk["bf16_tflops"] * 1e12), 4)
        # (against the library product's rate in a seconds-long loop under the power cap: these steps of 26 ms and more,
        #  five to a timed region, run at those clocks)
        out[f"{key}_prefill_bf16_frac_sustained"] = round(z["prefill_flops"] / (pms / 1e3) / (pk["bf16_tflops_sustained"] * 1e12), 4)
        if key == "8b":
            # the baseline's workload for this shape: 64 requests decoding at context 4096 beside a 512-token
            # portion of a 2048-token prompt (its third portion: 1024 tokens behind it)
            mms, spread = mixed_point(runner, 64, ctx, 512, 1024, z["V"], max(3, steps // 4), warmup, clocks, repeats=4)
            mms = spread["median_ms"]
            out["8b_mixed_64_decodes_512_portion_ms"] = round(mms, 3)
            out["8b_mixed_tok_s"] = round(576 / (mms / 1e3), 1)
            read = z["weight_bytes"] + (64 * ctx + 1024 + 512) * z["kv_token_bytes"]
            flops = 2 * 576 * z["L"] * z["layer_params"] + 2 * 64 * z["V"] * z["H"]
            bound = max(read / (pk["hbm_gbs"] * 1e9), flops / (pk["bf16_tflops"] * 1e12))
            out["8b_mixed_frac_of_slower_bound"] = round(bound / (mms / 1e3), 4)
            # (both bounds: the decoded tokens' attention streams the cache while the tensor cores idle, the products
            # of 576 rows keep the tensor cores busy while little streams, and a layer runs them one after the other)
            out["8b_mixed_hbm_bound_ms"] = round(read / (pk["hbm_gbs"] * 1e9) * 1e3, 3)
            out["8b_mixed_flop_bound_ms"] = round(flops / (pk["bf16_tflops"] * 1e12) * 1e3, 3)
        del eng, runner
    finally:
        shutil.rmtree(tmp, ignore_errors=True)
        gc.collect()
        torch.cuda.empty_cache()
    return out


# ---- the latent-attention / mixture-of-experts decoder beside the grouped-query dense one at equal size ------------
# Sizes that resemble real layers: the widths of the 0.6B and of a 2B-class shape, sixteen heads of 128, a cached
# latent of 256 values a token (against 8 kv heads x 128 x 2 = 2048), layers that alternate a dense gated
# feed-forward with a routed one whose chosen experts together are as wide as the dense one.
LATENT_SIZES = {
    "1024": dict(width=1024, heads=16, dim=128, vdim=128, q_rank=512, kv_rank=256, ff=3072, experts=16, top=4, expert_ff=768,
                 shared_ff=768, groups=(4, 2)),
    "2048": dict(width=2048, heads=16, dim=128, vdim=128, q_rank=768, kv_rank=256, ff=6144, experts=32, top=4, expert_ff=1536,
                 shared_ff=1536, groups=(8, 4)),
}
LATENT_VOCAB = 32768


def latent_config(z, layers):
    mix = dict(heads=z["heads"], dim=z["dim"], vdim=z["vdim"], q_rank=z["q_rank"], kv_rank=z["kv_rank"], scale=z["dim"] ** -0.5)
    dense = dict(kind="dense", ff=z["ff"])
    moe = dict(kind="moe", expert=dict(ff=z["expert_ff"]), shared=dict(ff=z["shared_ff"]),
               router=dict(experts=z["experts"], identity=0, top=z["top"], groups=dict(count=z["groups"][0], keep=z["groups"][1])))
    return dict(architecture="Surelorn", vocab=LATENT_VOCAB, width=z["width"], embedding=dict(scale=1.0), norm=dict(eps=1e-6),
                layers=[dict(type="latent_attention", mixer=mix, mlp=dense if i % 2 == 0 else moe) for i in range(layers)])


def latent_beside_dense(size, layers, pk, clocks, steps, warmup, prefill_only=False, decode_only=False, which="both"):
    """Decode (batch 1, 8, 64 at context 4096) and the 2048-token prefill of the Surelorn shape ``size`` and of the Qwen3
    shape of the same width, heads, feed-forward width, layers and vocabulary: tokens a second, side by side."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    z = LATENT_SIZES[size]
    qwen = dict(SHAPE_0_6B, hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=layers,
                num_attention_heads=z["heads"], num_key_value_heads=8, head_dim=z["dim"], vocab_size=LATENT_VOCAB,
                tie_word_embeddings=False)
    out = dict(size=size, layers=layers, vocab=LATENT_VOCAB, latent=dict(z))
    for name, cfg in (("surelorn", latent_config(z, layers)), ("qwen3", qwen)):
        if which not in ("both", name):
            continue
        tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
        try:
            model_dir = write_random_model(os.path.join(tmp, "model"), cfg, 0, device="cuda")
            ctx = 4096
            pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
            eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                         prefix_cache=False)
            shutil.rmtree(tmp, ignore_errors=True)
            runner = eng.runner
            for g in runner.cache.groups:
                g.pool.normal_(0.0, 1.0)
            res = dict(weight_bytes=runner.weight_bytes(), cache_bytes_a_token=runner.cache.bytes_per_token())
            if not prefill_only:
                for b in (1, 8, 64):
                    ms, launches, spread = decode_point(runner, b, ctx, max(5, steps // 2), warmup, clocks, repeats=4)
                    res[f"decode_b{b}_tok_s"] = round(b / (spread["median_ms"] / 1e3), 1)
                    res[f"decode_b{b}_ms"] = spread["median_ms"]
                    res[f"decode_b{b}_launches"] = launches
            if not decode_only:
                pms, _ = prefill_point(runner, LATENT_VOCAB, clocks, repeats=4)
                res["prefill_ms"] = round(pms, 3)
                res["prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
            out[name] = res
            del eng, runner
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
            gc.collect()
            torch.cuda.empty_cache()
    return out


# ---- the windowed-attention / state-space / clamped-experts decoder (Bumisun) beside the grouped-query dense one ------
# Sizes that resemble real layers: the widths of the 0.6B and of a 2B-class shape; attention of sixteen heads over eight
# kv heads, keys of 128 and values of 64 entries, a window of 1024 tokens that keeps the first eight, half of each head
# rotated; Mamba-2 layers of width / 32 heads of 64 with a state of 128 rows; layers alternate a state-space mixer with
# a dense gated feed-forward and an attention mixer with routed experts that together are as wide as the dense one.
HYBRID_SIZES = {
    "1024": dict(width=1024, heads=16, kv_heads=8, dim=128, vdim=64, window=1024, keep_first=8, rot=64, m_heads=32, m_vdim=64,
                 m_state=128, m_groups=1, conv=4, ff=3072, experts=16, top=4, expert_ff=768, shared_ff=768),
    "2048": dict(width=2048, heads=16, kv_heads=8, dim=128, vdim=64, window=1024, keep_first=8, rot=64, m_heads=64, m_vdim=64,
                 m_state=128, m_groups=1, conv=4, ff=6144, experts=32, top=4, expert_ff=1536, shared_ff=1536),
}


def hybrid_config(z, layers):
    att = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["vdim"], scale=z["dim"] ** -0.5, softcap=50.0,
               mask=dict(size=z["window"], keep_first=z["keep_first"]), rot=dict(dims=z["rot"], base=10000.0), v_mix=True)
    ssm = dict(heads=z["m_heads"], vdim=z["m_vdim"], state=z["m_state"], groups=z["m_groups"], conv=z["conv"], norm_groups=1)
    dense = dict(kind="dense", ff=z["ff"])
    moe = dict(kind="moe", expert=dict(ff=z["expert_ff"], limit=7.0), shared=dict(ff=z["shared_ff"], limit=7.0),
               router=dict(experts=z["experts"], top=z["top"]))
    return dict(architecture="Bumisun", vocab=LATENT_VOCAB, width=z["width"], norm=dict(eps=1e-6), residual_mult=0.5, logit_scale=1.0,
                layers=[dict(type="mamba2", mixer=ssm, mlp=dense) if i % 2 == 0 else dict(type="attention", mixer=att, mlp=moe)
                        for i in range(layers)])


def hybrid_beside_dense(size, layers, pk, clocks, steps, warmup, which="both"):
    """Decode (batch 1, 8, 64 at context 4096) and the 2048-token prefill of the Bumisun shape ``size`` and of the Qwen3
    shape of the same width, heads, kv heads, feed-forward width, layers and vocabulary: tokens a second, side by side."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    z = HYBRID_SIZES[size]
    qwen = dict(SHAPE_0_6B, hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=layers,
                num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"], vocab_size=LATENT_VOCAB,
                tie_word_embeddings=False)
    out = dict(size=size, layers=layers, vocab=LATENT_VOCAB, hybrid=dict(z))
    for name, cfg in (("bumisun", hybrid_config(z, layers)), ("qwen3", qwen)):
        if which not in ("both", name):
            continue
        tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
        try:
            model_dir = write_random_model(os.path.join(tmp, "model"), cfg, 0, device="cuda")
            ctx = 4096
            pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
            eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                         prefix_cache=False)
            shutil.rmtree(tmp, ignore_errors=True)
            runner = eng.runner
            for g in runner.cache.groups:
                g.pool.normal_(0.0, 1.0)
            res = dict(weight_bytes=runner.weight_bytes(), cache_bytes_a_token=runner.cache.bytes_per_token())
            for b in (1, 8, 64):
                ms, launches, spread = decode_point(runner, b, ctx, max(5, steps // 2), warmup, clocks, repeats=4)
                res[f"decode_b{b}_tok_s"] = round(b / (spread["median_ms"] / 1e3), 1)
                res[f"decode_b{b}_ms"] = spread["median_ms"]
                res[f"decode_b{b}_launches"] = launches
            pms, _ = prefill_point(runner, LATENT_VOCAB, clocks, repeats=4)
            res["prefill_ms"] = round(pms, 3)
            res["prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
            out[name] = res
            del eng, runner
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
            gc.collect()
            torch.cuda.empty_cache()
    out["kernels"] = hybrid_kernels(HYBRID_SIZES[size], pk)
    return out


def hybrid_kernels(z, pk):
    """Bumisun's own kernels alone, at the sizes of ``z``, beside the like kernels of the grouped-query dense model:
    device time (CUDA events, the median of nine after three warm-ups, the cache pools larger than L2), the algorithmic
    bytes and FLOPs, and the fraction of the measured copy bandwidth or bfloat16 product rate they come to."""
    import numpy as np
    import torch
    from paged_llm_rs_b200.kernels import attention_plan, ops
    from paged_llm_rs_b200.parts.base import AttentionWork

    dev, bf = "cuda", torch.bfloat16
    nh, nkv, dk, dv, W, keep = z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["window"], z["keep_first"]
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    target = 2 * ops.sm_count()
    out = {}

    def timed(fn):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(9):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(); fn(); b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return statistics.median(ts)

    def note(name, ms, nbytes, flops):
        r = dict(us=round(ms * 1e3, 2), mbytes=round(nbytes / 1e6, 2), gflop=round(flops / 1e9, 3),
                 hbm_frac=round(nbytes / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4),
                 bf16_frac=round(flops / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4))
        r["frac_of_slower_bound"] = round(max(r["hbm_frac"], r["bf16_frac"]), 4)
        out[name] = r

    def plan(segs, tile, ctas, window):
        work, red, parts = attention_plan.plan_attention(segs, tile, window, ctas, target)
        wd = torch.from_numpy(np.ascontiguousarray(work)).reshape(-1, 8).to(dev) if len(work) else torch.zeros(1, 8, dtype=torch.int32, device=dev)
        rd = torch.from_numpy(np.ascontiguousarray(red)).reshape(-1, 4).to(dev) if len(red) else torch.zeros(1, 4, dtype=torch.int32, device=dev)
        singles = all(n == 1 for _, n, _ in segs)
        return lambda heads, hd: AttentionWork(wd, torch.tensor([len(work)], dtype=torch.int32, device=dev), max(len(work), 1), rd,
                                                torch.tensor([len(red)], dtype=torch.int32, device=dev), len(red),
                                                torch.zeros(max(parts, 1), heads, hd, device=dev), torch.zeros(max(parts, 1), heads, 2, device=dev),
                                                kinds=1 if singles else 2, many_splits=attention_plan.many_splits(len(segs), ctas, target))

    ctx, B, T = 4096, 64, PREFILL_TOKENS
    n_pages = B * ctx // PAGE
    tables = torch.randperm(n_pages, dtype=torch.int32).view(B, ctx // PAGE).to(dev)
    cases = {"decode_b64_ctx4096": [(i, 1, ctx - 1) for i in range(B)], "prefill_2048": [(0, T, 0)]}
    # -- attention: capped, windowed, with sinks, joined rows (this design) and plain grouped-query with the same window (Qwen3's)
    pool = torch.randn(n_pages, nkv, PAGE, dk + dv, device=dev).to(bf)
    kp, vp = (torch.randn(n_pages, nkv, PAGE, dk, device=dev).to(bf) for _ in range(2))
    swz = ops.pool_is_swizzled(bf, nh, nkv, dk)
    sinks = torch.zeros(nh, device=dev)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        keys = sum(min(p + i + 1, W) + min(keep, max(0, p + i + 1 - W)) for _, c, p in segs for i in range(c))
        q, o = torch.randn(n, nh * dk, device=dev).to(bf), torch.empty(n, nh * dv, dtype=bf, device=dev)
        w = plan(segs, ops.attention_sink_tile_tokens(nh, nkv, bf, dk, dv), ops.attention_sink_ctas_per_item(nh, nkv, bf, dk, dv), W)(nh, dv)
        ms = timed(lambda: ops.attention_sink(q, pool, tables, w, o, sinks, nh, nkv, dk, dv, W, keep, dk ** -0.5, 50.0, status))
        seg_keys = sum(min(p + c, W + c) for _, c, p in segs)            # cache rows a segment's queries read, once
        note(f"attention_sink_{case}", ms, seg_keys * nkv * (dk + dv) * 2 + n * nh * (dk + dv) * 2, 2 * nh * (dk + dv) * keys)
        o2 = torch.empty(n, nh * dk, dtype=bf, device=dev)
        w2 = plan(segs, ops.attention_tile_tokens(nh, nkv, bf, dk, PAGE, W), nkv * -(-(nh // nkv) // 16), W)(nh, dk)
        keys2 = sum(min(p + i + 1, W) for _, c, p in segs for i in range(c))
        ms = timed(lambda: ops.paged_attention(q, kp, vp, tables, w2, o2, nh, nkv, dk, W, dk ** -0.5, status, swizzled=swz))
        note(f"qwen3_attention_window_{case}", ms, seg_keys * nkv * 2 * dk * 2 + n * nh * 2 * dk * 2, 2 * nh * 2 * dk * keys2)
    # -- rotation and the cache write
    for case, n in (("decode_b64", B), ("prefill_2048", T)):
        pos = torch.arange(n, dtype=torch.int32, device=dev)
        slots = torch.randperm(n_pages * PAGE, dtype=torch.int32)[:n].to(dev)
        qkv = torch.randn(n, nh * dk + nkv * (dk + dv), device=dev).to(bf)
        q = torch.empty(n, nh * dk, dtype=bf, device=dev)
        inv = torch.rand(z["rot"] // 2, device=dev)
        vf, lam = torch.randn(n, nkv * dv, device=dev).to(bf), torch.tensor([0.5], device=dev)
        ms = timed(lambda: ops.rope_mix_kv_write(qkv, q, inv, z["rot"], pos, slots, pool, vf, lam, nh, nkv, dk, dv, status))
        note(f"rope_mix_kv_write_{case}", ms, 2 * qkv.numel() * 2 + vf.numel() * 2, 0)
        qkv2 = torch.randn(n, (nh + 2 * nkv) * dk, device=dev).to(bf)
        g1 = torch.ones(dk, device=dev)
        cos, sin = torch.rand(ctx, dk // 2, device=dev), torch.rand(ctx, dk // 2, device=dev)
        ms = timed(lambda: ops.qk_norm_rope_kv(qkv2, q, g1, g1, 1e-6, cos, sin, dk, pos, slots, kp, vp, nh, nkv, dk, status, swizzled=swz))
        note(f"qwen3_qk_norm_rope_kv_{case}", ms, 2 * qkv2.numel() * 2, 0)
    # -- the add before a norm, on a float32 stream and on a bfloat16 one
    for case, n in (("decode_b64", B), ("prefill_2048", T)):
        x32, d = torch.randn(n, z["width"], device=dev), torch.randn(n, z["width"], device=dev).to(bf)
        g1, y = torch.ones(z["width"], device=dev), torch.empty(n, z["width"], dtype=bf, device=dev)
        ms = timed(lambda: ops.add_scaled_norm32(x32, d, 0.5, g1, 1e-6, y))
        note(f"add_scaled_norm32_{case}", ms, n * z["width"] * (4 + 4 + 2 + 2), 0)
        x16 = x32.to(bf)
        ms = timed(lambda: ops.rmsnorm(x16, g1, 1e-6, y, delta=d, residual_out=x16))
        note(f"qwen3_add_rmsnorm_{case}", ms, n * z["width"] * (2 + 2 + 2 + 2), 0)
    # -- the state-space mixer between its projections (no like kernel in the other models)
    H, P_, N, G, taps = z["m_heads"], z["m_vdim"], z["m_state"], z["m_groups"], z["conv"]
    inner, ch = H * P_, H * P_ + 2 * G * N
    floats = ops.mamba2_state_floats(H, G, P_, N, taps)
    state = torch.zeros(B + 1, floats, device=dev)
    cw, cb = torch.randn(ch, taps, device=dev).to(bf), torch.randn(ch, device=dev).to(bf)
    hb, gain = torch.zeros(H, device=dev), torch.ones(inner, device=dev)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        u = torch.randn(n, inner + ch + H, device=dev).to(bf)
        sg = torch.tensor([(t0, c, p, i + 1) for i, (t0, c, p) in enumerate(segs)], dtype=torch.int32, device=dev)
        if len(segs) > 1:
            sg[:, 0] = torch.arange(len(segs), dtype=torch.int32, device=dev)
        y = torch.empty(n, inner, dtype=bf, device=dev)
        longest = max(c for _, c, _ in segs)
        ms = timed(lambda: ops.mamba2_mix(u, cw, cb, hb, hb, hb, gain, sg, longest, state, y, H, G, P_, N, taps, 1, 1e-6))
        nbytes = u.numel() * 2 * 2 + n * ch * 4 * 2 + n * inner * 4 * 2 + y.numel() * 2 + len(segs) * floats * 4 * 2
        note(f"mamba2_mix_{case}", ms, nbytes, 6 * n * H * N * P_)
    return out


# ---- the matrix-memory decoder (Pamarax) beside the windowed-attention / state-space one (Bumisun) --------------------
# Sizes that resemble real layers, at the widths of the 0.6B and of a 2B-class shape: attention of sixteen heads over
# eight kv heads with keys of 128 entries that are also the values, half of each head rotated; a matrix LSTM of
# width / 256 heads with keys of 128 and values of 256 entries; beside an attention with values of 64 entries, a gated
# delta rule of width / 128 heads of 128 by 128 over half as many q/k heads, behind convolutions of four taps.  Layers
# go attention, matrix LSTM, the two side by side, matrix LSTM; every layer has a dense gated feed-forward.  The other
# model has the same width, layers, feed-forward and vocabulary: Mamba-2 layers and windowed attention in turn.
MATRIX_SIZES = {
    "1024": dict(width=1024, heads=16, kv_heads=8, dim=128, rot=64, left_vdim=64, temp_every=256, m_heads=4, m_dim=128, m_vdim=256,
                 d_heads=8, d_kv_heads=4, d_dim=128, d_vdim=128, conv=4, ff=3072),
    "2048": dict(width=2048, heads=16, kv_heads=8, dim=128, rot=64, left_vdim=64, temp_every=256, m_heads=8, m_dim=128, m_vdim=256,
                 d_heads=16, d_kv_heads=8, d_dim=128, d_vdim=128, conv=4, ff=6144),
}


def matrix_config(z, layers):
    att = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["dim"], scale=z["dim"] ** -0.5,
               rot=dict(dims=z["rot"], base=10000.0))
    lstm = dict(heads=z["m_heads"], dim=z["m_dim"], vdim=z["m_vdim"], gate_cap=15.0)
    left = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["left_vdim"], scale=z["dim"] ** -0.5,
                q_temp=dict(coef=0.5, every=z["temp_every"]))
    right = dict(heads=z["d_heads"], kv_heads=z["d_kv_heads"], dim=z["d_dim"], vdim=z["d_vdim"], conv=z["conv"])
    cycle = [dict(type="attention", mixer=att), dict(type="mlstm", mixer=lstm),
             dict(type="parallel", mixer=dict(left=left, right=right, left_scale=1.0, right_scale=1.0)), dict(type="mlstm", mixer=lstm)]
    return dict(architecture="Pamarax", vocab=LATENT_VOCAB, width=z["width"], norm=dict(eps=1e-6), embedding=dict(scale=1.0),
                layers=[dict(cycle[i % 4], mlp=dict(kind="dense", ff=z["ff"])) for i in range(layers)])


def matrix_beside_hybrid(size, layers, pk, clocks, steps, warmup, which="both"):
    """Decode (batch 1, 8, 64 at context 4096) and the 2048-token prefill of the Pamarax shape ``size`` and of the Bumisun
    shape of the same width, layers, dense feed-forward and vocabulary: tokens a second, side by side; then Pamarax's own
    kernels alone beside the like kernels of Bumisun."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    z = MATRIX_SIZES[size]
    hz = dict(HYBRID_SIZES[size], ff=z["ff"])
    hybrid = hybrid_config(hz, layers)
    for L in hybrid["layers"]:
        L["mlp"] = dict(kind="dense", ff=z["ff"])
    out = dict(size=size, layers=layers, vocab=LATENT_VOCAB, matrix=dict(z))
    for name, cfg in (("pamarax", matrix_config(z, layers)), ("bumisun", hybrid)):
        if which not in ("both", name):
            continue
        tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
        try:
            model_dir = write_random_model(os.path.join(tmp, "model"), cfg, 0, device="cuda")
            ctx = 4096
            pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
            eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                         prefix_cache=False)
            shutil.rmtree(tmp, ignore_errors=True)
            runner = eng.runner
            for g in runner.cache.groups:
                if g.pool is not None:
                    g.pool.normal_(0.0, 1.0)
            res = dict(weight_bytes=runner.weight_bytes(), cache_bytes_a_token=runner.cache.bytes_per_token())
            for b in (1, 8, 64):
                ms, launches, spread = decode_point(runner, b, ctx, max(5, steps // 2), warmup, clocks, repeats=4)
                res[f"decode_b{b}_tok_s"] = round(b / (spread["median_ms"] / 1e3), 1)
                res[f"decode_b{b}_ms"] = spread["median_ms"]
                res[f"decode_b{b}_launches"] = launches
            pms, _ = prefill_point(runner, LATENT_VOCAB, clocks, repeats=4)
            res["prefill_ms"] = round(pms, 3)
            res["prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
            out[name] = res
            del eng, runner
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
            gc.collect()
            torch.cuda.empty_cache()
    out["kernels"] = matrix_kernels(z, pk)
    like = hybrid_kernels(HYBRID_SIZES[size], pk)
    out["kernels"].update({f"bumisun_{k}": v for k, v in like.items() if not k.startswith("qwen3_")})
    return out


def matrix_kernels(z, pk):
    """Pamarax's own kernels alone, at the sizes of ``z``: device time (CUDA events, the median of nine after three
    warm-ups, the cache pools and state slots larger than L2 where a model's would be), the algorithmic bytes and FLOPs,
    and the fraction of the measured copy bandwidth or bfloat16 product rate they come to."""
    import numpy as np
    import torch
    from paged_llm_rs_b200.kernels import attention_plan, ops
    from paged_llm_rs_b200.parts.base import AttentionWork

    dev, bf = "cuda", torch.bfloat16
    nh, nkv, dk = z["heads"], z["kv_heads"], z["dim"]
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    target = 2 * ops.sm_count()
    out = {}

    def timed(fn):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(9):
            flush_l2()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(); fn(); b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return statistics.median(ts)

    def note(name, ms, nbytes, flops):
        r = dict(us=round(ms * 1e3, 2), mbytes=round(nbytes / 1e6, 2), gflop=round(flops / 1e9, 3),
                 hbm_frac=round(nbytes / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4),
                 bf16_frac=round(flops / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4))
        r["frac_of_slower_bound"] = round(max(r["hbm_frac"], r["bf16_frac"]), 4)
        out[name] = r

    def plan(segs, tile, ctas):
        work, red, parts = attention_plan.plan_attention(segs, tile, 0, ctas, target)
        wd = torch.from_numpy(np.ascontiguousarray(work)).reshape(-1, 8).to(dev) if len(work) else torch.zeros(1, 8, dtype=torch.int32, device=dev)
        rd = torch.from_numpy(np.ascontiguousarray(red)).reshape(-1, 4).to(dev) if len(red) else torch.zeros(1, 4, dtype=torch.int32, device=dev)
        singles = all(n == 1 for _, n, _ in segs)
        return lambda heads, hd: AttentionWork(wd, torch.tensor([len(work)], dtype=torch.int32, device=dev), max(len(work), 1), rd,
                                                torch.tensor([len(red)], dtype=torch.int32, device=dev), len(red),
                                                torch.zeros(max(parts, 1), heads, hd, device=dev), torch.zeros(max(parts, 1), heads, 2, device=dev),
                                                kinds=1 if singles else 2, many_splits=attention_plan.many_splits(len(segs), ctas, target))

    ctx, B, T = 4096, 64, PREFILL_TOKENS
    n_pages = B * ctx // PAGE
    tables = torch.randperm(n_pages, dtype=torch.int32).view(B, ctx // PAGE).to(dev)
    cases = {"decode_b64_ctx4096": [(i, 1, ctx - 1) for i in range(B)], "prefill_2048": [(0, T, 0)]}
    # -- attention over the whole context: keys that are the values (one more in no denominator), and the half beside the delta rule
    for label, dv, sink in (("keys_are_values", dk, None), ("extra_one", z["left_vdim"], torch.zeros(nh, device=dev))):
        pool = torch.randn(n_pages, nkv, PAGE, dk + dv, device=dev).to(bf)
        for case, segs in cases.items():
            n = sum(c for _, c, _ in segs)
            keys = sum(p + i + 1 for _, c, p in segs for i in range(c))
            q, o = torch.randn(n, nh * dk, device=dev).to(bf), torch.empty(n, nh * dv, dtype=bf, device=dev)
            w = plan(segs, ops.attention_sink_tile_tokens(nh, nkv, bf, dk, dv), ops.attention_sink_ctas_per_item(nh, nkv, bf, dk, dv))(nh, dv)
            ms = timed(lambda: ops.attention_sink(q, pool, tables, w, o, sink, nh, nkv, dk, dv, 0, 0, dk ** -0.5, 0.0, status))
            seg_keys = sum(p + c for _, c, p in segs)
            note(f"attention_{label}_{case}", ms, seg_keys * nkv * (dk + dv) * 2 + n * nh * (dk + dv) * 2, 2 * nh * (dk + dv) * keys)
        del pool
    # -- q/k norm, temperature, rotation and the cache write
    pool = torch.randn(n_pages, nkv, PAGE, 2 * dk, device=dev).to(bf)
    pool_l = torch.randn(n_pages, nkv, PAGE, dk + z["left_vdim"], device=dev).to(bf)
    for case, n in (("decode_b64", B), ("prefill_2048", T)):
        pos = torch.arange(n, dtype=torch.int32, device=dev)
        slots = torch.randperm(n_pages * PAGE, dtype=torch.int32)[:n].to(dev)
        q = torch.empty(n, nh * dk, dtype=bf, device=dev)
        inv = torch.rand(z["rot"] // 2, device=dev)
        k_off, v_off = nh * dk, (nh + nkv) * dk
        proj = torch.randn(n, (2 * nh + nkv) * dk, device=dev).to(bf)                  # q | k | gate
        gq, gk = torch.ones(nh * dk, device=dev), torch.ones(nkv * dk, device=dev)
        ms = timed(lambda: ops.normed_qk_kv_write(proj, k_off, v_off, q, gq, gk, "projection", 1e-6, 0.0, 0, inv, z["rot"], pos, slots, pool,
                                                  nh, nkv, dk, dk, True, status))
        note(f"normed_qk_kv_write_projection_{case}", ms, n * (nh + nkv) * dk * 2 + n * nh * dk * 2 + n * nkv * 2 * dk * 2, 0)
        dv = z["left_vdim"]
        proj2 = torch.randn(n, (nh + nkv) * dk + nkv * dv, device=dev).to(bf)
        g1 = torch.ones(dk, device=dev)
        ms = timed(lambda: ops.normed_qk_kv_write(proj2, k_off, v_off, q, g1, g1, "head", 1e-6, 0.5, z["temp_every"], None, 0, pos, slots, pool_l,
                                                  nh, nkv, dk, dv, False, status))
        note(f"normed_qk_kv_write_head_{case}", ms, 2 * proj2.numel() * 2, 0)
    del pool, pool_l
    # -- a sublayer's output normed and added, the next one's input normed: one pass over a float32 stream
    W = z["width"]
    for case, n in (("decode_b64", B), ("prefill_2048", T)):
        x32, a = torch.randn(n, W, device=dev), torch.randn(n, W, device=dev).to(bf)
        g1, y = torch.ones(W, device=dev), torch.empty(n, W, dtype=bf, device=dev)
        ms = timed(lambda: ops.sandwich_norm32(x32, a, None, g1, g1, y, 1e-6))
        note(f"sandwich_norm32_{case}", ms, n * W * (4 + 4 + 2 + 2), 0)
    # -- the recurrent mixers between their projections
    H, d, E = z["m_heads"], z["m_dim"], z["m_vdim"]
    floats = ops.mlstm_state_floats(H, d, E)
    state = torch.zeros(B + 1, floats, device=dev)
    gain, hb = torch.ones(H * E, device=dev), torch.zeros(H, device=dev)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        u = torch.randn(n, 2 * H * d + 2 * H * E, device=dev).to(bf)
        gates = torch.randn(n, 2 * H, device=dev)
        sg = torch.tensor([(t0, c, p, i + 1) for i, (t0, c, p) in enumerate(segs)], dtype=torch.int32, device=dev)
        if len(segs) > 1:
            sg[:, 0] = torch.arange(len(segs), dtype=torch.int32, device=dev)
        y = torch.empty(n, H * E, dtype=bf, device=dev)
        ms = timed(lambda: ops.mlstm_mix(u, gates, hb, hb, 15.0, gain, sg, state, y, H, d, E, 1e-6, max(c for _, c, _ in segs)))
        nbytes = u.numel() * 2 + gates.numel() * 4 + n * H * E * 4 * 2 + y.numel() * 2 + len(segs) * floats * 4 * 2
        note(f"mlstm_mix_{case}", ms, nbytes, 6 * n * H * d * E)
    del state
    H, G, d, E, taps = z["d_heads"], z["d_kv_heads"], z["d_dim"], z["d_vdim"], z["conv"]
    ch = 2 * G * d + H * E
    floats = ops.delta_state_floats(H, G, d, E, taps)
    state = torch.zeros(B + 1, floats, device=dev)
    cw, gain, hb = torch.randn(ch, taps, device=dev).to(bf), torch.ones(E, device=dev), torch.zeros(H, device=dev)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        u = torch.randn(n, ch + H * E, device=dev).to(bf)
        ba = torch.randn(n, 2 * H, device=dev)
        sg = torch.tensor([(t0, c, p, i + 1) for i, (t0, c, p) in enumerate(segs)], dtype=torch.int32, device=dev)
        if len(segs) > 1:
            sg[:, 0] = torch.arange(len(segs), dtype=torch.int32, device=dev)
        y = torch.empty(n, H * E, dtype=bf, device=dev)
        longest = max(c for _, c, _ in segs)
        ms = timed(lambda: ops.delta_mix(u, cw, ba, hb, hb, gain, sg, longest, state, y, H, G, d, E, taps, 1e-6))
        nbytes = u.numel() * 2 * 2 + n * ch * 4 * 2 + ba.numel() * 4 + n * H * E * 4 * 2 + y.numel() * 2 + len(segs) * floats * 4 * 2
        note(f"delta_mix_{case}", ms, nbytes, 8 * n * H * d * E)
    return out


# ---- the differential-attention / matrix-LSTM / latent-attention decoder with squared-relu experts (Tebozen) ------------
# Sizes that resemble real layers, at the widths of the 0.6B and of a 2B-class shape: differential attention of eight or
# sixteen heads over half as many kv heads, two maps of 64 key entries a head over values of 128, behind convolutions of
# four taps, in a window of 1024 tokens, every map wholly rotated; a matrix LSTM of width / 256 heads with keys of 128 and
# values of 256 entries; latent attention of sixteen heads with 64 unrotated and 64 rotated key entries over a cached row of
# 192 + 64 values; every layer has sixteen or thirty-two experts without gates, four a token, and a shared expert.  Layers
# go attention, matrix LSTM, latent attention, matrix LSTM; the second latent layer attends over the first one's cache.
# The other model is the Bumisun shape of the same width, layers, experts and vocabulary.
TEBOZEN_SIZES = {
    "1024": dict(width=1024, heads=8, kv_heads=4, dim=64, vdim=128, conv=4, window=1024, rot=64, m_heads=4, m_dim=128, m_vdim=256,
                 l_heads=16, l_dim=64, l_rot=64, l_vdim=64, kv_rank=192, experts=16, top=4, expert_ff=768, shared_ff=768),
    "2048": dict(width=2048, heads=16, kv_heads=8, dim=64, vdim=128, conv=4, window=1024, rot=64, m_heads=8, m_dim=128, m_vdim=256,
                 l_heads=16, l_dim=64, l_rot=64, l_vdim=64, kv_rank=192, experts=32, top=4, expert_ff=1536, shared_ff=1536),
}


def tebozen_config(z, layers):
    att = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["vdim"], conv=z["conv"], diff=0.3, scale=z["dim"] ** -0.5,
               mask=dict(size=z["window"]), rot=dict(dims=z["rot"], base=10000.0))
    lstm = dict(heads=z["m_heads"], dim=z["m_dim"], vdim=z["m_vdim"], gate_cap=15.0)
    lat = dict(heads=z["l_heads"], dim=z["l_dim"], rot_dim=z["l_rot"], vdim=z["l_vdim"], kv_rank=z["kv_rank"],
               scale=(z["l_dim"] + z["l_rot"]) ** -0.5, rot=dict(dims=z["l_rot"], base=10000.0))
    moe = dict(kind="moe", expert=dict(ff=z["expert_ff"]), shared=dict(ff=z["shared_ff"]), router=dict(experts=z["experts"], top=z["top"]))
    out, first_latent = [], None
    for i in range(layers):
        kind = ("attention", "mlstm", "latent_attention", "mlstm")[i % 4]
        mixer = dict(att if kind == "attention" else lstm if kind == "mlstm" else lat)
        if kind == "latent_attention":
            if first_latent is None:
                first_latent = i
            else:
                mixer["kv_from"] = first_latent
        out.append(dict(type=kind, mixer=mixer, mlp=moe))
    return dict(architecture="Tebozen", vocab=LATENT_VOCAB, width=z["width"], norm=dict(eps=1e-6), embedding=dict(scale=1.0), layers=out)


def tebozen_beside_hybrid(size, layers, pk, clocks, steps, warmup, which="both"):
    """Decode (batch 1, 8, 64 at context 4096) and the 2048-token prefill of the Tebozen shape ``size`` and of the Bumisun
    shape of the same width, layers, experts and vocabulary (a routed feed-forward in every layer): tokens a second, side by
    side; then Tebozen's own kernels alone beside their like kernels."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    z = TEBOZEN_SIZES[size]
    hz = dict(HYBRID_SIZES[size], experts=z["experts"], top=z["top"], expert_ff=z["expert_ff"], shared_ff=z["shared_ff"])
    hybrid = hybrid_config(hz, layers)
    routed = next(L["mlp"] for L in hybrid["layers"] if L["mlp"]["kind"] == "moe")
    for L in hybrid["layers"]:
        L["mlp"] = routed
    out = dict(size=size, layers=layers, vocab=LATENT_VOCAB, tebozen=dict(z))
    for name, cfg in (("tebozen", tebozen_config(z, layers)), ("bumisun", hybrid)):
        if which not in ("both", name):
            continue
        tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
        try:
            model_dir = write_random_model(os.path.join(tmp, "model"), cfg, 0, device="cuda")
            ctx = 4096
            pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
            eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                         prefix_cache=False)
            shutil.rmtree(tmp, ignore_errors=True)
            runner = eng.runner
            for g in runner.cache.groups:
                if g.pool is not None:
                    g.pool.normal_(0.0, 1.0)
            res = dict(weight_bytes=runner.weight_bytes(), cache_bytes_a_token=runner.cache.bytes_per_token())
            for b in (1, 8, 64):
                ms, launches, spread = decode_point(runner, b, ctx, max(5, steps // 2), warmup, clocks, repeats=4)
                res[f"decode_b{b}_tok_s"] = round(b / (spread["median_ms"] / 1e3), 1)
                res[f"decode_b{b}_ms"] = spread["median_ms"]
                res[f"decode_b{b}_launches"] = launches
            pms, _ = prefill_point(runner, LATENT_VOCAB, clocks, repeats=4)
            res["prefill_ms"] = round(pms, 3)
            res["prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
            out[name] = res
            del eng, runner
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
            gc.collect()
            torch.cuda.empty_cache()
    out["kernels"] = tebozen_kernels(z, pk)
    like = hybrid_kernels(HYBRID_SIZES[size], pk)
    out["kernels"].update({f"bumisun_{k}": v for k, v in like.items() if not k.startswith("qwen3_")})
    return out


def tebozen_kernels(z, pk):
    """Tebozen's own kernels alone, at the sizes of ``z``, each beside its like kernel of another design where that is not
    among Bumisun's: device time (CUDA events, the median of nine after three warm-ups, an L2 flush before each, the cache
    pools larger than L2 where a model's would be), the algorithmic bytes and FLOPs, and the fraction of the measured copy
    bandwidth or bfloat16 product rate they come to."""
    import numpy as np
    import torch
    from paged_llm_rs_b200.kernels import attention_plan, ops
    from paged_llm_rs_b200.parts.base import AttentionWork

    dev, bf = "cuda", torch.bfloat16
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    target = 2 * ops.sm_count()
    out = {}

    def timed(fn):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(9):
            flush_l2()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(); fn(); b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return statistics.median(ts)

    def note(name, ms, nbytes, flops):
        r = dict(us=round(ms * 1e3, 2), mbytes=round(nbytes / 1e6, 2), gflop=round(flops / 1e9, 3),
                 hbm_frac=round(nbytes / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4),
                 bf16_frac=round(flops / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4))
        r["frac_of_slower_bound"] = round(max(r["hbm_frac"], r["bf16_frac"]), 4)
        out[name] = r

    def plan(segs, tile, ctas, window):
        work, red, parts = attention_plan.plan_attention(segs, tile, window, ctas, target)
        wd = torch.from_numpy(np.ascontiguousarray(work)).reshape(-1, 8).to(dev) if len(work) else torch.zeros(1, 8, dtype=torch.int32, device=dev)
        rd = torch.from_numpy(np.ascontiguousarray(red)).reshape(-1, 4).to(dev) if len(red) else torch.zeros(1, 4, dtype=torch.int32, device=dev)
        singles = all(n == 1 for _, n, _ in segs)
        return lambda heads, hd: AttentionWork(wd, torch.tensor([len(work)], dtype=torch.int32, device=dev), max(len(work), 1), rd,
                                                torch.tensor([len(red)], dtype=torch.int32, device=dev), len(red),
                                                torch.zeros(max(parts, 1), heads, hd, device=dev), torch.zeros(max(parts, 1), heads, 2, device=dev),
                                                kinds=1 if singles else 2, many_splits=attention_plan.many_splits(len(segs), ctas, target))

    def segments(segs):
        sg = torch.tensor([(t0, c, p, i + 1) for i, (t0, c, p) in enumerate(segs)], dtype=torch.int32, device=dev)
        if len(segs) > 1:
            sg[:, 0] = torch.arange(len(segs), dtype=torch.int32, device=dev)
        return sg

    ctx, B, T = 4096, 64, PREFILL_TOKENS
    n_pages = B * ctx // PAGE
    tables = torch.randperm(n_pages, dtype=torch.int32).view(B, ctx // PAGE).to(dev)
    cases = {"decode_b64_ctx4096": [(i, 1, ctx - 1) for i in range(B)], "prefill_2048": [(0, T, 0)]}
    W = z["width"]
    # -- differential attention: the two maps as heads of their own over doubled kv heads, in the window
    H, G, dk, dv, win, taps = z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["window"], z["conv"]
    nh, nkv = 2 * H, 2 * G
    pool = torch.randn(n_pages, nkv, PAGE, dk + dv, device=dev).to(bf)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        keys = sum(min(p + i + 1, win) for _, c, p in segs for i in range(c))
        q, a = torch.randn(n, nh * dk, device=dev).to(bf), torch.empty(n, nh * dv, dtype=bf, device=dev)
        w = plan(segs, ops.attention_sink_tile_tokens(nh, nkv, bf, dk, dv), ops.attention_sink_ctas_per_item(nh, nkv, bf, dk, dv), win)(nh, dv)
        ms = timed(lambda: ops.attention_sink(q, pool, tables, w, a, None, nh, nkv, dk, dv, win, 0, dk ** -0.5, 0.0, status))
        seg_keys = sum(min(p + c, win + c - 1) for _, c, p in segs)
        note(f"attention_maps_{case}", ms, seg_keys * nkv * (dk + dv) * 2 + n * nh * (dk + dv) * 2, 2 * nh * (dk + dv) * keys)
        # the maps' difference, its norm and the gate a head
        gate, o = torch.randn(n, H, device=dev).to(bf), torch.empty(n, H * dv, dtype=bf, device=dev)
        ms = timed(lambda: ops.diff_combine(a, gate, o, H, H // G, dv, 0.4, 0.7, 1e-6))
        note(f"diff_combine_{case}", ms, (a.numel() + o.numel() + gate.numel()) * 2, 0)
        # bias, convolution, rotation and the cache write
        ch = (nh + nkv) * dk + G * dv
        proj = torch.randn(n, ch + H, device=dev).to(bf)
        bias, cw = torch.randn(ch, device=dev), torch.randn(ch, taps, device=dev)
        state = torch.zeros(B + 1, ops.conv_state_floats(ch, taps), device=dev)
        inv = torch.rand(z["rot"] // 2, device=dev)
        pos = torch.arange(n, dtype=torch.int32, device=dev)
        slots = torch.randperm(n_pages * PAGE, dtype=torch.int32)[:n].to(dev)
        sg = segments(segs)
        ms = timed(lambda: ops.conv_rope_kv_write(proj, bias, cw, sg, max(c for _, c, _ in segs), state, inv, z["rot"], pos, slots, q, pool,
                                                  nh, nkv, 2, dk, dv, status))
        note(f"conv_rope_kv_write_{case}", ms, n * ch * 2 + n * nh * dk * 2 + n * nkv * (dk + dv) * 2 + len(segs) * state.shape[1] * 4 * 2, 0)
    del pool
    # -- latent attention over rows [latent | rotated key part], and the kernel that makes the rows
    LH, ld, lr, R = z["l_heads"], z["l_dim"], z["l_rot"], z["kv_rank"]
    width = R + lr
    rows = torch.randn(n_pages, PAGE, width, device=dev).to(bf)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        keys = sum(p + i + 1 for _, c, p in segs for i in range(c))
        q_rows, o_rows = torch.randn(n, LH, width, device=dev).to(bf), torch.empty(n, LH, width, dtype=bf, device=dev)
        w = plan(segs, ops.latent_attention_tile_tokens(LH, width, bf), ops.latent_attention_ctas_per_item(LH, width, bf), 0)(LH, width)
        ms = timed(lambda: ops.latent_attention(q_rows, rows, tables, w, o_rows, 0.1, status))
        seg_keys = sum(p + c for _, c, p in segs)
        note(f"latent_attention_{case}", ms, seg_keys * width * 2 + 2 * n * LH * width * 2, 2 * LH * 2 * width * keys)
        proj = torch.randn(n, LH * (ld + lr) + LH + width, device=dev).to(bf)
        gain, inv = torch.ones(R, device=dev), torch.rand(lr // 2, device=dev)
        pos = torch.arange(n, dtype=torch.int32, device=dev)
        slots = torch.randperm(n_pages * PAGE, dtype=torch.int32)[:n].to(dev)
        ms = timed(lambda: ops.latent_rope_write(proj[:, LH * (ld + lr) + LH:], gain, 1e-6, proj[:, :LH * (ld + lr)], q_rows, rows, slots, pos, inv,
                                                 LH, ld, lr, lr, R, status))
        note(f"latent_rope_write_{case}", ms, n * (width + LH * lr) * 2 * 2, 0)
        # its like: both latents normed and the cache row written (a q latent as wide as the rotated parts of all heads)
        qa, cq = torch.randn(n, LH * lr + width, device=dev).to(bf), torch.empty(n, LH * lr, dtype=bf, device=dev)
        ms = timed(lambda: ops.latent_norm_write(qa, torch.ones(LH * lr, device=dev), torch.ones(width, device=dev), 1e-6, cq, rows, slots,
                                                 LH * lr, width, status))
        note(f"like_latent_norm_write_{case}", ms, n * (width + LH * lr) * 2 * 2, 0)
    del rows
    # -- the experts: without gates, the token times its score (both forms), beside the gated ones of equal width
    E, top, ff = z["experts"], z["top"], z["expert_ff"]
    w_up, w_gu, w_d = (torch.randn(E, ff, W, device=dev) * 0.02).to(bf), (torch.randn(E, 2 * ff, W, device=dev) * 0.02).to(bf), \
        (torch.randn(E, W, ff, device=dev) * 0.02).to(bf)
    wr = torch.randn(E, W, device=dev)
    ws_up, ws_gu = (torch.randn(z["shared_ff"], W, device=dev) * 0.02).to(bf), (torch.randn(2 * z["shared_ff"], W, device=dev) * 0.02).to(bf)
    for case, n in (("decode_b8", 8), ("decode_b64", B), ("prefill_2048", T)):
        h = torch.randn(n, W, device=dev).to(bf)
        ms = timed(lambda: ops.moe_route(h, wr, None, top, 1, 1, scoring="sigmoid", renormalize=False))
        note(f"router_sigmoid_{case}", ms, n * W * 2 + E * W * 4, 2 * n * E * W)
        ms = timed(lambda: ops.moe_route(h, wr, None, top, 1, 1))
        note(f"like_router_softmax_{case}", ms, n * W * 2 + E * W * 4, 2 * n * E * W)
        ids, weights = ops.moe_route(h, wr, None, top, 1, 1, scoring="sigmoid", renormalize=False)
        used = min(E, n * top)
        ms = timed(lambda: ops.moe_experts(h, ids, weights, w_up, w_d, None, status, act="squared_relu", gated=False, weight_input=True))
        note(f"experts_ungated_{case}", ms, used * 2 * ff * W * 2 + n * W * 2 * 2, 2 * n * top * 2 * ff * W)
        ms = timed(lambda: ops.moe_experts(h, ids, weights, w_gu, w_d, None, status, act="silu"))
        note(f"like_experts_gated_{case}", ms, used * 3 * ff * W * 2 + n * W * 2 * 2, 2 * n * top * 3 * ff * W)
        ms = timed(lambda: ops.linear_act(h, ws_up, "squared_relu", status=status))
        note(f"shared_up_squared_relu_{case}", ms, ws_up.numel() * 2 + n * (W + z["shared_ff"]) * 2, 2 * n * z["shared_ff"] * W)
        ms = timed(lambda: ops.linear_glu(h, ws_gu, status=status))
        note(f"like_shared_gate_up_silu_{case}", ms, ws_gu.numel() * 2 + n * (W + z["shared_ff"]) * 2, 2 * n * 2 * z["shared_ff"] * W)
    return out


# ---- the retention / chunked-attention-beside-gated-linear-attention decoder (Reperax) ----------------------------------
# Sizes that resemble real layers, at the widths of the 0.6B and of a 2B-class shape: retention of width / 256 heads with
# keys of 128 (all rotated) and values of 256 entries; chunked attention of sixteen heads over eight kv heads of 128 with
# values of 64, in chunks of 1024, beside gated linear attention of width / 128 heads of 128 x 128 with a decay of inner
# size 16; a feed-forward without a gate.  Layers alternate and are run once, ahead of them the pass's vector.  The other
# model is Pamarax at the same width, depth, head sizes, feed-forward and vocabulary, its matrix LSTM layers in the place of
# retention, its side-by-side layers (attention over the whole context, gated delta rule) in the place of the side-by-side ones.
REPERAX_SIZES = {
    "1024": dict(width=1024, heads=16, kv_heads=8, dim=128, vdim=64, chunk=1024, r_heads=4, r_dim=128, r_vdim=256, g_heads=8, g_dim=128,
                 g_vdim=128, rank=16, ff=3072),
    "2048": dict(width=2048, heads=16, kv_heads=8, dim=128, vdim=64, chunk=1024, r_heads=8, r_dim=128, r_vdim=256, g_heads=16, g_dim=128,
                 g_vdim=128, rank=16, ff=6144),
}


def reperax_config(z, layers):
    ret = dict(heads=z["r_heads"], dim=z["r_dim"], vdim=z["r_vdim"], rot=dict(dims=z["r_dim"], base=10000.0),
               decay=[1.0 - 2.0 ** -(5 + i * 5 / max(1, z["r_heads"] - 1)) for i in range(z["r_heads"])])
    left = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["vdim"], scale=z["dim"] ** -0.5, mask=dict(size=z["chunk"]))
    right = dict(heads=z["g_heads"], dim=z["g_dim"], vdim=z["g_vdim"], tau=16.0)
    cycle = [dict(type="retention", mixer=ret), dict(type="parallel", mixer=dict(left=left, right=right, left_scale=0.8, right_scale=0.6))]
    return dict(architecture="Reperax", vocab=LATENT_VOCAB, width=z["width"], norm=dict(eps=1e-6), logit_softcap=30.0,
                loop=dict(start=0, stop=layers, times=1), layers=[dict(cycle[i % 2], mlp=dict(kind="dense", ff=z["ff"])) for i in range(layers)])


def reperax_beside_matrix(size, layers, pk, clocks, steps, warmup, which="both"):
    """Decode (batch 1, 8, 64 at context 4096) and the 2048-token prefill of the Reperax shape ``size`` and of the Pamarax shape
    of the same width, layers, head sizes, feed-forward and vocabulary: tokens a second, side by side; then Reperax's own
    kernels alone beside the like kernels of Pamarax."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    z = REPERAX_SIZES[size]
    mz = MATRIX_SIZES[size]
    matrix = matrix_config(mz, 4)
    matrix["layers"] = [matrix["layers"][1 + i % 2] for i in range(layers)]        # matrix LSTM, side by side, ...
    out = dict(size=size, layers=layers, vocab=LATENT_VOCAB, reperax=dict(z))
    for name, cfg in (("reperax", reperax_config(z, layers)), ("pamarax", matrix)):
        if which not in ("both", name):
            continue
        tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
        try:
            model_dir = write_random_model(os.path.join(tmp, "model"), cfg, 0, device="cuda")
            ctx = 4096
            pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
            eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                         prefix_cache=False)
            shutil.rmtree(tmp, ignore_errors=True)
            runner = eng.runner
            for g in runner.cache.groups:
                if g.pool is not None:
                    g.pool.normal_(0.0, 1.0)
            res = dict(weight_bytes=runner.weight_bytes(), cache_bytes_a_token=runner.cache.bytes_per_token())
            for b in (1, 8, 64):
                ms, launches, spread = decode_point(runner, b, ctx, max(5, steps // 2), warmup, clocks, repeats=4)
                res[f"decode_b{b}_tok_s"] = round(b / (spread["median_ms"] / 1e3), 1)
                res[f"decode_b{b}_ms"] = spread["median_ms"]
                res[f"decode_b{b}_launches"] = launches
            pms, _ = prefill_point(runner, LATENT_VOCAB, clocks, repeats=4)
            res["prefill_ms"] = round(pms, 3)
            res["prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
            out[name] = res
            del eng, runner
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
            gc.collect()
            torch.cuda.empty_cache()
    out["kernels"] = reperax_kernels(z, pk)
    like = matrix_kernels(mz, pk)
    out["kernels"].update({f"pamarax_{k}": v for k, v in like.items()})
    return out


def reperax_kernels(z, pk):
    """Reperax's own kernels alone, at the sizes of ``z``, each beside its like kernel of another design where that is not among
    Pamarax's: device time (CUDA events, the median of nine after three warm-ups, an L2 flush before each), the algorithmic
    bytes and FLOPs, and the fraction of the measured copy bandwidth or bfloat16 product rate they come to."""
    import numpy as np
    import torch
    from paged_llm_rs_b200.kernels import attention_plan, ops
    from paged_llm_rs_b200.parts.base import AttentionWork

    dev, bf = "cuda", torch.bfloat16
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    target = 2 * ops.sm_count()
    out = {}

    def timed(fn):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(9):
            flush_l2()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(); fn(); b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return statistics.median(ts)

    def note(name, ms, nbytes, flops):
        r = dict(us=round(ms * 1e3, 2), mbytes=round(nbytes / 1e6, 2), gflop=round(flops / 1e9, 3),
                 hbm_frac=round(nbytes / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4),
                 bf16_frac=round(flops / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4))
        r["frac_of_slower_bound"] = round(max(r["hbm_frac"], r["bf16_frac"]), 4)
        out[name] = r

    def plan(segs, tile, ctas, window=0, chunk=0):
        work, red, parts = attention_plan.plan_attention(segs, tile, window, ctas, target, chunk=chunk)
        wd = torch.from_numpy(np.ascontiguousarray(work)).reshape(-1, 8).to(dev)
        rd = torch.from_numpy(np.ascontiguousarray(red)).reshape(-1, 4).to(dev) if len(red) else torch.zeros(1, 4, dtype=torch.int32, device=dev)
        singles = all(n == 1 for _, n, _ in segs)
        return lambda heads, hd: AttentionWork(wd, torch.tensor([len(work)], dtype=torch.int32, device=dev), len(work), rd,
                                                torch.tensor([len(red)], dtype=torch.int32, device=dev), len(red),
                                                torch.zeros(max(parts, 1), heads, hd, device=dev), torch.zeros(max(parts, 1), heads, 2, device=dev),
                                                kinds=1 if singles else 2, many_splits=attention_plan.many_splits(len(segs), ctas, target))

    ctx, B, T, W = 4096, 64, PREFILL_TOKENS, z["width"]
    n_pages = B * ctx // PAGE
    tables = torch.randperm(n_pages, dtype=torch.int32).view(B, ctx // PAGE).to(dev)
    cases = {"decode_b64_ctx4096": [(i, 1, ctx - 1) for i in range(B)], "prefill_2048": [(0, T, 0)]}
    # -- attention in chunks, beside the same kernel with a window of the chunk's size
    nh, nkv, dk, dv, chunk = z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["chunk"]
    pool = torch.randn(n_pages, nkv, PAGE, dk + dv, device=dev).to(bf)
    tile, ctas = ops.attention_sink_tile_tokens(nh, nkv, bf, dk, dv), ops.attention_sink_ctas_per_item(nh, nkv, bf, dk, dv)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        q, o = torch.randn(n, nh * dk, device=dev).to(bf), torch.empty(n, nh * dv, dtype=bf, device=dev)
        for label, win, ch in (("attention_chunked", 0, chunk), ("like_attention_window", chunk, 0)):
            seen = lambda p: p % chunk + 1 if ch else min(p + 1, chunk)
            keys = sum(seen(p + i) for _, c, p in segs for i in range(c))
            seg_keys = sum((p + c) - (p - p % chunk if ch else max(0, p - chunk + 1)) for _, c, p in segs)
            w = plan(segs, tile, ctas, win, ch)(nh, dv)
            ms = timed(lambda: ops.attention_sink(q, pool, tables, w, o, None, nh, nkv, dk, dv, win, 0, dk ** -0.5, 0.0, status, chunk=ch))
            note(f"{label}_{case}", ms, seg_keys * nkv * (dk + dv) * 2 + n * nh * (dk + dv) * 2, 2 * nh * (dk + dv) * keys)
        # q/k norm over the projection and the cache write
        k_off, v_off = nh * dk, (nh + nkv) * dk
        proj = torch.randn(n, v_off + nkv * dv, device=dev).to(bf)
        gq, gk = torch.ones(nh * dk, device=dev), torch.ones(nkv * dk, device=dev)
        pos = torch.arange(n, dtype=torch.int32, device=dev)
        slots = torch.randperm(n_pages * PAGE, dtype=torch.int32)[:n].to(dev)
        ms = timed(lambda: ops.normed_qk_kv_write(proj, k_off, v_off, q, gq, gk, "projection", 1e-6, 0.0, 0, None, 0, pos, slots, pool,
                                                  nh, nkv, dk, dv, False, status))
        note(f"normed_qk_kv_write_{case}", ms, 2 * proj.numel() * 2, 0)
    del pool
    # -- the recurrences between their projections
    for label, H, d, E, channel in (("retention", z["r_heads"], z["r_dim"], z["r_vdim"], False), ("gated_linear", z["g_heads"], z["g_dim"], z["g_vdim"], True)):
        floats = ops.linear_attention_state_floats(H, d, E)
        state = torch.zeros(B + 1, floats, device=dev)
        inv = torch.rand(d // 2, device=dev)
        decay = torch.full((H,), 0.99, device=dev)
        a2, ab, gain = torch.randn(H * d, z["rank"], device=dev).to(bf), torch.full((H * d,), 3.0, device=dev), torch.ones(E, device=dev)
        for case, segs in cases.items():
            n = sum(c for _, c, _ in segs)
            u = torch.randn(n, 2 * H * d + 2 * H * E, device=dev).to(bf)
            a1 = torch.randn(n, z["rank"], device=dev)
            sg = torch.tensor([(t0, c, p, i + 1) for i, (t0, c, p) in enumerate(segs)], dtype=torch.int32, device=dev)
            y = torch.empty(n, H * E, dtype=bf, device=dev)
            longest = max(c for _, c, _ in segs)
            args = (u, 0, H * d, 2 * H * d, 2 * H * d + H * E)
            rope = ops.rope_table(torch.arange(n, dtype=torch.int32, device=dev), inv)          # (once a step, for all layers)
            if channel:
                run = lambda: ops.linear_attention_mix(*args, d ** -0.5, 1.0, 0, None, None, a1, a2, ab, 16.0, gain, sg, longest, state, y, H, d, E, 1e-6)
            else:
                run = lambda: ops.linear_attention_mix(*args, 1.0, d ** -0.5, d, inv, decay, None, None, None, 1.0, None, sg, longest, state, y, H, d, E, 1e-6, rope=rope)
            ms = timed(run)
            # (counted as for the like recurrences: the read-out in float written and read once, the state read and written)
            note(f"{label}_mix_{case}", ms, u.numel() * 2 + (a1.numel() * 4 if channel else 0) + n * H * E * 4 * 2 + y.numel() * 2 + len(segs) * floats * 4 * 2,
                 6 * n * H * d * E)
        del state
    # -- the gated sum, two norms and the shift; the polynomial activation beside silu(gate + b) * (up + b); the logits' cap
    ff = z["ff"]
    for case, n in (("decode_b64", B), ("prefill_2048", T)):
        x, xo = torch.randn(n, W, device=dev), torch.empty(n, W, device=dev)
        new = lambda: torch.randn(n, W, device=dev).to(bf)
        a1, a2, f, gate, y1, ys, y2 = new(), new(), new(), new(), new(), new(), new()
        wide = torch.randn(n, ff + W, device=dev).to(bf)
        vec = torch.ones(W, device=dev)
        sg = torch.tensor([(i, 1, 9, i + 1) for i in range(B)] if n == B else [(0, n, 0, 1)], dtype=torch.int32, device=dev)
        st = torch.zeros(B + 1, W, device=dev)
        ms = timed(lambda: ops.gated_sum_norm32(x, vec, y1, 1e-6, mixed=a1, mixed_scale=0.8, mixed2=a2, mixed2_scale=0.6, mixed_gate=gate, mixed_bias=vec,
                                                fed=f, fed_gate=wide[:, ff:], fed_bias=vec, x_out=xo, shift=vec, shifted=ys, segments=sg, state=st,
                                                gain2=vec, out2=y2))
        note(f"gated_sum_norm32_{case}", ms, n * W * (4 + 4 + 5 * 2 + 3 * 2) + sg.shape[0] * W * 8, 0)
        act = torch.empty(n, ff, dtype=bf, device=dev)
        ms = timed(lambda: ops.poly_norm(wide[:, :ff], vec[:4].contiguous(), 1e-6, act))
        note(f"poly_norm_{case}", ms, 2 * n * ff * 2, 0)
        gu, bias = torch.randn(n, 2 * ff, device=dev).to(bf), torch.zeros(2 * ff, device=dev)
        ms = timed(lambda: ops.swiglu_bias(gu, bias, act))
        note(f"like_swiglu_bias_{case}", ms, 3 * n * ff * 2, 0)
    logits = torch.randn(B, LATENT_VOCAB, device=dev)
    note("softcap32_decode_b64", timed(lambda: ops.softcap32(logits, 30.0)), logits.numel() * 8, 0)
    note("like_scale32_decode_b64", timed(lambda: ops.scale32(logits, 1.0)), logits.numel() * 8, 0)
    return out


# ---- the windowed-attention / chunked-attention-beside-delta-rule decoder (Tubevik) ----------------------------------------
# Sizes that resemble real layers, at the widths of the 0.6B and of a 2B-class shape: windowed attention (1024 tokens, capped
# scores, a gate a head, YaRN rotation of half of each head) of sixteen heads over eight kv heads of 128, every second such layer
# borrowing the keys and values of the one before; beside chunked attention (1024) with values of 64, the delta rule of width / 128
# heads of 128 x 128 over half as many q/k heads with a decay of inner size 64 (a random model's) behind convolutions of four taps; a clamped gated
# feed-forward.  The other model is Pamarax at the same width, depth, head sizes, feed-forward and vocabulary: its attention layers
# and its side-by-side layers (attention over the whole context, gated delta rule) in turn.
TUBEVIK_SIZES = {
    "1024": dict(width=1024, heads=16, kv_heads=8, dim=128, vdim=128, window=1024, rot=64, left_vdim=64, chunk=1024, d_heads=8, d_kv_heads=4,
                 d_dim=128, d_vdim=128, conv=4, rank=64, ff=3072),
    "2048": dict(width=2048, heads=16, kv_heads=8, dim=128, vdim=128, window=1024, rot=64, left_vdim=64, chunk=1024, d_heads=16, d_kv_heads=8,
                 d_dim=128, d_vdim=128, conv=4, rank=64, ff=6144),
}


def tubevik_config(z, layers):
    att = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["vdim"], scale=z["dim"] ** -0.5, softcap=30.0, mask=dict(size=z["window"]),
               rot=dict(dims=z["rot"], base=500000.0, scaling=dict(factor=8.0, original=8192, fast=32.0, slow=1.0)))
    left = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["dim"], vdim=z["left_vdim"], scale=z["dim"] ** -0.5, mask=dict(size=z["chunk"]),
                rot=dict(dims=z["rot"], base=10000.0))
    right = dict(heads=z["d_heads"], kv_heads=z["d_kv_heads"], dim=z["d_dim"], vdim=z["d_vdim"], conv=z["conv"])
    par = dict(type="parallel", mixer=dict(left=left, right=right, left_scale=0.8, right_scale=0.6))
    out = []
    for i in range(layers):
        mixer = par if i % 2 else dict(type="attention", mixer=dict(att, kv_from=i - 2) if i % 4 == 2 else att)
        out.append(dict(mixer, mlp=dict(kind="dense", ff=z["ff"], limit=7.0)))
    return dict(architecture="Tubevik", vocab=LATENT_VOCAB, width=z["width"], norm=dict(eps=1e-6), residual_mult=0.5, logit_softcap=30.0, layers=out)


def tubevik_beside_matrix(size, layers, pk, clocks, steps, warmup, which="both", kernels_only=False):
    """Decode (batch 1, 8, 64 at context 4096) and the 2048-token prefill of the Tubevik shape ``size`` and of the Pamarax shape
    of the same width, layers, head sizes, feed-forward and vocabulary: tokens a second, side by side; then Tubevik's own
    kernels alone beside the like kernels of Pamarax."""
    import gc
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    z = TUBEVIK_SIZES[size]
    mz = MATRIX_SIZES[size]
    matrix = matrix_config(mz, 4)
    matrix["layers"] = [matrix["layers"][2 * (i % 2)] for i in range(layers)]        # attention, side by side, ...
    out = dict(size=size, layers=layers, vocab=LATENT_VOCAB, tubevik=dict(z))
    for name, cfg in () if kernels_only else (("tubevik", tubevik_config(z, layers)), ("pamarax", matrix)):
        if which not in ("both", name):
            continue
        tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
        try:
            model_dir = write_random_model(os.path.join(tmp, "model"), cfg, 0, device="cuda")
            ctx = 4096
            pages = 64 * (ctx // PAGE + 4) + (PREFILL_TOKENS + 1024) // PAGE + 64
            eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=64, chunk=PREFILL_TOKENS,
                         prefix_cache=False)
            shutil.rmtree(tmp, ignore_errors=True)
            runner = eng.runner
            for g in runner.cache.groups:
                if g.pool is not None:
                    g.pool.normal_(0.0, 1.0)
            res = dict(weight_bytes=runner.weight_bytes(), cache_bytes_a_token=runner.cache.bytes_per_token())
            for b in (1, 8, 64):
                ms, launches, spread = decode_point(runner, b, ctx, max(5, steps // 2), warmup, clocks, repeats=4)
                res[f"decode_b{b}_tok_s"] = round(b / (spread["median_ms"] / 1e3), 1)
                res[f"decode_b{b}_ms"] = spread["median_ms"]
                res[f"decode_b{b}_launches"] = launches
            pms, _ = prefill_point(runner, LATENT_VOCAB, clocks, repeats=4)
            res["prefill_ms"] = round(pms, 3)
            res["prefill_tok_s"] = round(PREFILL_TOKENS / (pms / 1e3), 1)
            out[name] = res
            del eng, runner
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
            gc.collect()
            torch.cuda.empty_cache()
    out["kernels"] = tubevik_kernels(z, pk)
    like = matrix_kernels(mz, pk)
    out["kernels"].update({f"pamarax_{k}": v for k, v in like.items() if not k.startswith("mlstm")})
    return out


def tubevik_kernels(z, pk):
    """Tubevik's own kernels alone, at the sizes of ``z``, each beside its like kernel of another design where that is not among
    Pamarax's: device time (CUDA events, the median of nine after three warm-ups, an L2 flush before each), the algorithmic
    bytes and FLOPs, and the fraction of the measured copy bandwidth or bfloat16 product rate they come to."""
    import numpy as np
    import torch
    from paged_llm_rs_b200.kernels import attention_plan, ops
    from paged_llm_rs_b200.parts.base import AttentionWork

    dev, bf = "cuda", torch.bfloat16
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    target = 2 * ops.sm_count()
    out = {}

    def timed(fn):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(9):
            flush_l2()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(); fn(); b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return statistics.median(ts)

    def note(name, ms, nbytes, flops):
        r = dict(us=round(ms * 1e3, 2), mbytes=round(nbytes / 1e6, 2), gflop=round(flops / 1e9, 3),
                 hbm_frac=round(nbytes / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4),
                 bf16_frac=round(flops / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4))
        r["frac_of_slower_bound"] = round(max(r["hbm_frac"], r["bf16_frac"]), 4)
        out[name] = r

    def plan(segs, tile, ctas, window=0, chunk=0):
        work, red, parts = attention_plan.plan_attention(segs, tile, window, ctas, target, chunk=chunk)
        wd = torch.from_numpy(np.ascontiguousarray(work)).reshape(-1, 8).to(dev)
        rd = torch.from_numpy(np.ascontiguousarray(red)).reshape(-1, 4).to(dev) if len(red) else torch.zeros(1, 4, dtype=torch.int32, device=dev)
        singles = all(n == 1 for _, n, _ in segs)
        return lambda heads, hd: AttentionWork(wd, torch.tensor([len(work)], dtype=torch.int32, device=dev), len(work), rd,
                                                torch.tensor([len(red)], dtype=torch.int32, device=dev), len(red),
                                                torch.zeros(max(parts, 1), heads, hd, device=dev), torch.zeros(max(parts, 1), heads, 2, device=dev),
                                                kinds=1 if singles else 2, many_splits=attention_plan.many_splits(len(segs), ctas, target))

    ctx, B, T, W = 4096, 64, PREFILL_TOKENS, z["width"]
    n_pages = B * ctx // PAGE
    tables = torch.randperm(n_pages, dtype=torch.int32).view(B, ctx // PAGE).to(dev)
    cases = {"decode_b64_ctx4096": [(i, 1, ctx - 1) for i in range(B)], "prefill_2048": [(0, T, 0)]}
    nh, nkv, dk = z["heads"], z["kv_heads"], z["dim"]
    inv = torch.rand(z["rot"] // 2, device=dev)
    # -- the two attentions, each beside the same kernel without what it adds (cap; the one more, chunks instead of a window)
    for label, dv, variants in (("window", z["vdim"], [("attention_window_capped", z["window"], 0, 30.0, False), ("like_attention_window", z["window"], 0, 0.0, False)]),
                                ("chunk", z["left_vdim"], [("attention_chunk_extra_one", 0, z["chunk"], 0.0, True), ("like_attention_window_64", z["chunk"], 0, 0.0, False)])):
        pool = torch.randn(n_pages, nkv, PAGE, dk + dv, device=dev).to(bf)
        tile, ctas = ops.attention_sink_tile_tokens(nh, nkv, bf, dk, dv), ops.attention_sink_ctas_per_item(nh, nkv, bf, dk, dv)
        for case, segs in cases.items():
            n = sum(c for _, c, _ in segs)
            q, o = torch.randn(n, nh * dk, device=dev).to(bf), torch.empty(n, nh * dv, dtype=bf, device=dev)
            for name, win, ch, cap, one in variants:
                seen = lambda p: p % ch + 1 if ch else min(p + 1, win)
                keys = sum(seen(p + i) for _, c, p in segs for i in range(c))
                seg_keys = sum((p + c) - (p - p % ch if ch else max(0, p - win + 1)) for _, c, p in segs)
                w = plan(segs, tile, ctas, win, ch)(nh, dv)
                sinks = torch.zeros(nh, device=dev) if one else None
                ms = timed(lambda: ops.attention_sink(q, pool, tables, w, o, sinks, nh, nkv, dk, dv, win, 0, dk ** -0.5, cap, status, chunk=ch))
                note(f"{name}_{case}", ms, seg_keys * nkv * (dk + dv) * 2 + n * nh * (dk + dv) * 2, 2 * nh * (dk + dv) * keys)
            # what stands between the projection and the attention
            k_off, v_off = nh * dk, (nh + nkv) * dk
            width = v_off + nkv * dv + (nh if label == "window" else 0)
            proj = torch.randn(n, width, device=dev).to(bf)
            pos = torch.arange(n, dtype=torch.int32, device=dev)
            slots = torch.randperm(n_pages * PAGE, dtype=torch.int32)[:n].to(dev)
            ones = lambda k: torch.ones(k, device=dev)
            if label == "window":
                gq, gk, bq, bk, bv = ones(nh * dk), ones(nkv * dk), ones(nh * dk), ones(nkv * dk), ones(nkv * dv)
                run = lambda: ops.normed_qk_kv_write(proj, k_off, v_off, q, gq, gk, "projection", 1e-6, 0.0, 0, inv, z["rot"], pos, slots, pool, nh, nkv,
                                                     dk, dv, False, status, q_bias=bq, k_bias=bk, v_bias=bv, rot_factor=1.2)
                note(f"normed_qk_kv_write_biases_projection_{case}", timed(run), 2 * (v_off + nkv * dv) * n * 2, 0)
                wq, zero = proj[:, :nh * dk].contiguous(), None
                run = lambda: ops.normed_qk_kv_write(wq, -1, 0, q, gq, zero, "projection", 1e-6, 0.0, 0, inv, z["rot"], pos, slots, zero, nh, nkv,
                                                     dk, dv, False, status, q_bias=bq, rot_factor=1.2)
                note(f"normed_qk_queries_only_{case}", timed(run), 2 * nh * dk * n * 2, 0)
                note(f"gate_mul_a_head_{case}", timed(lambda: ops.gate_mul(o, proj[:, v_off + nkv * dv:], "sigmoid", per=dv)), n * nh * (2 * dv + 1) * 2, 0)
                wide = torch.randn(n, nh * dv, device=dev).to(bf)
                note(f"like_gate_mul_an_entry_{case}", timed(lambda: ops.gate_mul(o, wide, "sigmoid")), n * nh * 3 * dv * 2, 0)
            else:
                run = lambda: ops.normed_qk_kv_write(proj, k_off, v_off, q, None, None, "head_after_rotation", 1e-6, 0.0, 0, inv, z["rot"], pos, slots, pool,
                                                     nh, nkv, dk, dv, False, status, rot_pairs=True)
                note(f"normed_qk_kv_write_pairs_then_norm_{case}", timed(run), 2 * proj.numel() * 2, 0)
        del pool
    # -- the delta rule between its projections
    H, G, d, E, taps, R = z["d_heads"], z["d_kv_heads"], z["d_dim"], z["d_vdim"], z["conv"], z["rank"]
    ch = 2 * G * d + H * E
    floats = ops.channel_delta_state_floats(H, G, d, E, taps)
    state = torch.zeros(B + 1, floats, device=dev)
    cw, gain = torch.randn(ch, taps, device=dev).to(bf), torch.ones(E, device=dev)
    a2, g2 = (torch.randn(H * d, R, device=dev) * 0.1).to(bf), (torch.randn(H * E, R, device=dev) * 0.1).to(bf)
    a_log, dt = torch.zeros(H, device=dev), torch.zeros(H * d, device=dev)
    for case, segs in cases.items():
        n = sum(c for _, c, _ in segs)
        u = torch.randn(n, ch + R, device=dev).to(bf)
        small = torch.randn(n, H + R, device=dev)
        sg = torch.tensor([(t0, c, p, i + 1) for i, (t0, c, p) in enumerate(segs)], dtype=torch.int32, device=dev)
        y = torch.empty(n, H * E, dtype=bf, device=dev)
        longest = max(c for _, c, _ in segs)
        gate = torch.randn(n, H * E, device=dev).to(bf) if longest != 1 else None
        ms = timed(lambda: ops.channel_delta_mix(u, cw, small, H, a2, a_log, dt, ch, g2, gain, sg, longest, state, y, H, G, d, E, taps, 1e-6, gate=gate))
        # (counted as for the like recurrence: projection read twice, convolved channels and read-out in float written and read once, gate, state)
        note(f"channel_delta_mix_{case}", ms, n * (ch + H * E) * 2 * 2 + n * ch * 4 * 2 + small.numel() * 4 + n * H * E * 4 * 2 + y.numel() * 2 + len(segs) * floats * 4 * 2,
             8 * n * H * d * E)
    del state
    # -- the sum of three terms with the layer norm; the layer norm behind the embedding; the clamped activation; the logits' cap
    ff = z["ff"]
    table = torch.randn(LATENT_VOCAB, W, device=dev).to(bf)
    w_gu = (torch.randn(2 * ff, W, device=dev) * 0.02).to(bf)
    for case, n in (("decode_b64", B), ("prefill_2048", T)):
        x, vec = torch.randn(n, W, device=dev), torch.ones(W, device=dev)
        a1, a2_, f, y = (torch.randn(n, W, device=dev).to(bf) for _ in range(4))
        note(f"add_terms_norm32_{case}", timed(lambda: ops.add_terms_norm32(x, [(a1, 0.4), (a2_, 0.3), (f, 0.5)], vec, 1e-6, y, bias=vec, centered=True)),
             n * W * (4 + 4 + 3 * 2 + 2), 0)
        toks = torch.randint(0, LATENT_VOCAB, (n,), device=dev, dtype=torch.int32)
        note(f"embed_norm32_centered_{case}", timed(lambda: ops.embed_norm32(toks, table, vec, 1e-6, x, status, bias=vec, centered=True)), n * W * (2 + 4), 0)
        note(f"like_embed_norm32_{case}", timed(lambda: ops.embed_norm32(toks, table, vec, 1e-6, x, status)), n * W * (2 + 4), 0)
        h = torch.randn(n, W, device=dev).to(bf)
        nbytes, flops = w_gu.numel() * 2 + n * (W + ff) * 2, 2 * n * 2 * ff * W
        note(f"gate_up_clamped_{case}", timed(lambda: ops.linear_glu(h, w_gu, status=status, act="clamped", limit=7.0)), nbytes, flops)
        note(f"like_gate_up_silu_{case}", timed(lambda: ops.linear_glu(h, w_gu, status=status)), nbytes, flops)
    logits = torch.randn(B, LATENT_VOCAB, device=dev)
    note("softcap32_decode_b64", timed(lambda: ops.softcap32(logits, 30.0)), logits.numel() * 8, 0)
    note("like_scale32_decode_b64", timed(lambda: ops.scale32(logits, 1.0)), logits.numel() * 8, 0)
    return out


TRACE_KERNELS = {0: "(tcgen05 kernel)", 1: "embed", 2: "rmsnorm", 3: "swiglu", 4: "qk_norm_rope_kv", 5: "attention_generic", 6: "attention_reduce",
                 7: "attention_mma", 8: "attention_tma", 9: "skinny_gemm", 10: "sample_partial", 11: "sample_final", 12: "gemm_tcgen05", 13: "attention_tcgen05"}
TRACE_FILES = ["elementwise", "qk_norm_rope_kv", "attention_generic", "attention_mma", "attention_decode_tma", "sampling",
               "skinny_gemm", "gemm_tcgen05", "attention_prefill_tcgen05"]


def timeline(runner, batch, context, layers, prefill_tokens=0, vocab=1000, mixed_tokens=0) -> int:
    """One replay of the captured decode step, clocked by the kernels themselves (thread 0 of
    each kernel's first CTA reads the global timer before and after its wait for the kernel
    before it).  "to next" is the time from a kernel's wait ending to the next kernel's wait
    ending: what the kernel costs in the chain.  "in place" is how long its first CTA sat on an
    SM before its wait ended.  Library kernels (the output head) carry no stamps: their time
    shows in the "to next" of the kernel before them."""
    import ctypes
    import numpy as np
    import torch
    from paged_llm_rs_b200.engine.step import StepEntry
    from paged_llm_rs_b200.kernels import ops

    lib = ops.lib()
    buf = (ctypes.c_ulonglong * (8192 * 3))()

    def read():
        recs = []
        for f in TRACE_FILES:
            fn = getattr(lib, f"pllm_trace_read_{f}")
            fn.restype = ctypes.c_int
            n = fn(buf, 8192)
            recs += [(buf[3 * i + 2], buf[3 * i + 1], int(buf[3 * i])) for i in range(n)]
        return sorted(recs)

    cache = runner.cache
    if mixed_tokens:
        # a mixed step: the decoding requests beside one portion of a prompt that has 1024 tokens behind it
        ids = [f"t{b}" for b in range(batch)]
        for r in ids:
            cache.open(r)
            assert cache.reserve(r, context)
            cache.commit(r, context - 1)
        cache.open("tp")
        assert cache.reserve("tp", 1024 + mixed_tokens)
        cache.commit("tp", 1024)
        prompt = np.random.default_rng(0).integers(0, vocab, mixed_tokens).tolist()
        entries = [StepEntry(r, [1 + i], [0]) for i, r in enumerate(ids)] + [StepEntry("tp", prompt, [])]
        zeros = np.zeros(batch, dtype=np.float32)
        runner.graph_step_tokens = batch + mixed_tokens
        runner.step_and_sample(entries, zeros, zeros)
        graph = runner._portion_graph(entries)
        assert graph is not None, "the mixed step does not run as a captured step"
    elif prefill_tokens:
        prompt = np.random.default_rng(0).integers(0, vocab, prefill_tokens).tolist()
        cache.open("tp")
        assert cache.reserve("tp", prefill_tokens)
        entries = [StepEntry("tp", prompt, [prefill_tokens - 1])]
        zeros = np.zeros(1, dtype=np.float32)
        runner.step_and_sample(entries, zeros, zeros)
        graph = runner._portion_graph(entries)
        assert graph is not None, "the portion does not run as a captured step"
    else:
        ids = [f"t{b}" for b in range(batch)]
        for r in ids:
            cache.open(r)
            assert cache.reserve(r, context)
            cache.commit(r, context - 1)
        entries = [StepEntry(r, [1 + i], [0]) for i, r in enumerate(ids)]
        zeros = np.zeros(batch, dtype=np.float32)
        runner.step_and_sample(entries, zeros, zeros)
        graph = runner._decode_graph(entries)
    for _ in range(5):
        graph.replay()
    torch.cuda.synchronize()
    read()
    graph.replay()
    torch.cuda.synchronize()
    recs = read()
    rows = []
    for i, (after, before, kid) in enumerate(recs):
        nxt = recs[i + 1][0] if i + 1 < len(recs) else after
        rows.append((TRACE_KERNELS.get(kid, str(kid)), (after - recs[0][0]) / 1e3, (nxt - after) / 1e3, (after - before) / 1e3))
    per_layer = max(1, (len(rows) - 4) // max(1, layers))
    start = min(len(rows), 2 + per_layer * (layers // 2))
    what = f"prefill step, {prefill_tokens} tokens" if prefill_tokens else f"decode step, batch {batch}, context {context}"
    if mixed_tokens:
        what = f"mixed step, {batch} decoding at context {context} beside a portion of {mixed_tokens} tokens"
    print(f"{what}, {layers} layers: {len(rows)} kernels stamped, "
          f"{(recs[-1][0] - recs[0][0]) / 1e3:.1f} us from first to last")
    print(f"one layer from the middle:\n{'kernel':18s} {'at us':>9s} {'to next':>8s} {'in place':>8s}")
    for name, t, d, w in rows[start:start + per_layer]:
        print(f"{name:18s} {t:9.2f} {d:8.2f} {w:8.2f}")
    tot = {}
    for name, t, d, w in rows:
        a = tot.setdefault(name, [0, 0.0, 0.0])
        a[0] += 1; a[1] += d; a[2] += w
    print(f"whole step by kernel:\n{'kernel':18s} {'count':>5s} {'sum us':>9s} {'mean':>7s} {'in place':>8s}")
    for k, (n, d, w) in sorted(tot.items(), key=lambda kv: -kv[1][1]):
        print(f"{k:18s} {n:5d} {d:9.1f} {d / n:7.2f} {w / n:8.2f}")
    return 0


def plain_cpu_baseline() -> int:
    """Seconds the plain float32 implementation under tests/ takes on the CPU for one whole-sequence forward
    pass of 64 tokens (it has no cache: every generated token costs such a pass): the timed CPU baseline of
    the tiny configurations and of the 0.6B shape."""
    import numpy as np
    import torch
    sys.path.insert(0, os.path.join(ROOT, "tests"))
    import plain_qwen3 as P
    from tiny_configs import TINY_A, TINY_B
    from paged_llm_rs_b200 import write_random_model

    out = {"what": "plain float32 implementation on the CPU, one forward pass of 64 tokens, best of 3",
           "threads": torch.get_num_threads()}
    tmp = tempfile.mkdtemp(prefix="pllm_plain_")
    try:
        for name, cfg in (("tiny_a", TINY_A), ("tiny_b", TINY_B), ("qwen3_0.6b_shape", SHAPE_0_6B)):
            d = write_random_model(os.path.join(tmp, name), cfg, 0)
            c, w = P.load_model(d, torch.float32)
            toks = np.random.default_rng(0).integers(0, cfg["vocab_size"], 64).tolist()
            best = 1e9
            for _ in range(3):
                t0 = time.time()
                with torch.no_grad():
                    P.forward(c, w, toks, rows=[63])
                best = min(best, time.time() - t0)
            out[name + "_s"] = round(best, 4)
            out[name + "_tok_s_prefill"] = round(64 / best, 1)
            out[name + "_tok_s_decode"] = round(1 / best, 2)
            del w
    finally:
        shutil.rmtree(tmp, ignore_errors=True)
    print(json.dumps(out))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=50)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--shape", choices=sorted(SHAPES), default="0.6b", help="layer sizes: the baseline's 0.6B (default), 8B or 32B shape")
    ap.add_argument("--layers", type=int, default=None, help="run fewer layers than the shape has (named in config)")
    ap.add_argument("--no-points", action="store_true", help="skip batch 1 and 64")
    ap.add_argument("--no-shapes", action="store_true", help="skip the 8B and 32B shapes and the reference's kernel")
    ap.add_argument("--timeline-prefill", action="store_true",
                    help="with --only timeline: the captured step of a 2048-token prompt portion instead of the decode step")
    ap.add_argument("--timeline-mixed", type=int, default=0, metavar="TOKENS",
                    help="with --only timeline: the decoding requests beside one prompt portion of this many tokens")
    ap.add_argument("--latent-size", choices=sorted(LATENT_SIZES), default="1024",
                    help="with --only latent: the width of the latent-attention / mixture-of-experts shape")
    ap.add_argument("--latent-part", choices=["all", "decode", "prefill"], default="all", help="with --only latent: one part alone")
    ap.add_argument("--latent-model", choices=["both", "surelorn", "qwen3"], default="both", help="with --only latent: one model alone")
    ap.add_argument("--hybrid-size", choices=sorted(HYBRID_SIZES), default="1024",
                    help="with --only hybrid: the width of the windowed-attention / state-space / clamped-experts decoder")
    ap.add_argument("--hybrid-model", choices=["both", "bumisun", "qwen3"], default="both", help="with --only hybrid: one model alone")
    ap.add_argument("--matrix-size", choices=sorted(MATRIX_SIZES), default="1024",
                    help="with --only matrix: the width of the matrix-memory decoder (Pamarax)")
    ap.add_argument("--matrix-model", choices=["both", "pamarax", "bumisun"], default="both", help="with --only matrix: one model alone")
    ap.add_argument("--tebozen-size", choices=sorted(TEBOZEN_SIZES), default="1024",
                    help="with --only tebozen: the width of the differential-attention / matrix-LSTM / latent-attention decoder (Tebozen)")
    ap.add_argument("--tebozen-model", choices=["both", "tebozen", "bumisun"], default="both", help="with --only tebozen: one model alone")
    ap.add_argument("--reperax-size", choices=sorted(REPERAX_SIZES), default="1024",
                    help="with --only reperax: the width of the retention / chunked-attention-beside-gated-linear-attention decoder (Reperax)")
    ap.add_argument("--reperax-model", choices=["both", "reperax", "pamarax"], default="both", help="with --only reperax: one model alone")
    ap.add_argument("--tubevik-size", choices=sorted(TUBEVIK_SIZES), default="1024",
                    help="with --only tubevik: the width of the windowed-attention / chunked-attention-beside-delta-rule decoder (Tubevik)")
    ap.add_argument("--tubevik-model", choices=["both", "tubevik", "pamarax", "kernels"], default="both",
                    help="with --only tubevik: one model alone, or the kernels alone")
    ap.add_argument("--only", choices=["decode", "prefill", "long-prompt", "timeline", "reference-kernel", "plain-cpu", "latent", "hybrid", "matrix",
                                       "tebozen", "reperax", "tubevik"],
                    default=None,
                    help="run one part alone and print a short line (for profiling; not a bench record); "
                         "long-prompt: a prompt of --context tokens in portions of 2048, each portion timed; "
                         "timeline: one captured decode step as the kernels themselves clocked it; reference-kernel: "
                         "the reference's CUDA kernel against this engine's decode attention; plain-cpu: the plain "
                         "float32 implementation timed on the CPU (needs no GPU); latent: decode and prefill of the "
                         "latent-attention / mixture-of-experts decoder (Surelorn) beside the Qwen3 shape of equal size "
                         "(--latent-size, --layers, default 8); hybrid: the same for the windowed-attention / state-space / "
                         "clamped-experts decoder (Bumisun), with its own kernels timed alone beside the like kernels of the "
                         "Qwen3 shape (--hybrid-size, --layers, default 8); matrix: decode and prefill of the matrix-memory decoder "
                         "(Pamarax: gated attention, matrix LSTM, attention beside a gated delta rule) beside the Bumisun shape of "
                         "equal size, with its own kernels timed alone beside Bumisun's like ones (--matrix-size, --layers, default 8); "
                         "tebozen: the same for the decoder of differential attention, matrix LSTM and latent attention layers with "
                         "squared-relu experts (Tebozen) beside the Bumisun shape of equal size (--tebozen-size, --layers, default 8); "
                         "reperax: the same for the decoder of retention layers and chunked attention beside gated linear attention "
                         "(Reperax) beside the Pamarax shape of equal size (--reperax-size, --layers, default 8); "
                         "tubevik: the same for the decoder of windowed attention over lent keys and chunked attention beside a delta "
                         "rule with a decay a key entry (Tubevik) beside the Pamarax shape of equal size (--tubevik-size, --layers, default 8)")
    args = ap.parse_args(argv)

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "nicoNaeg/paged-llm-rs is a Rust workspace (cargo, candle): pip cannot install it "
                          "('neither setup.py nor pyproject.toml found') and this image has no cargo or rustc"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.only == "plain-cpu":
        return plain_cpu_baseline()
    steps, warmup = args.steps, max(3, args.warmup)
    if args.only == "timeline":
        # a build of the kernels that stamps the global timer around each kernel's wait for its predecessor
        os.environ["PAGED_LLM_NVCC_DEFINES"] = (os.environ.get("PAGED_LLM_NVCC_DEFINES", "") + " PLLM_TRACE=1").strip()

    import gc
    import numpy as np
    import torch
    from paged_llm_rs_b200 import Engine, write_random_model

    pk = peaks()
    clocks = ClockSampler()
    if args.only == "latent":
        clocks.start()
        out = latent_beside_dense(args.latent_size, args.layers or 8, pk, clocks, steps, warmup,
                                  prefill_only=args.latent_part == "prefill", decode_only=args.latent_part == "decode",
                                  which=args.latent_model)
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    if args.only == "hybrid":
        clocks.start()
        out = hybrid_beside_dense(args.hybrid_size, args.layers or 8, pk, clocks, steps, warmup, which=args.hybrid_model)
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    if args.only == "matrix":
        clocks.start()
        out = matrix_beside_hybrid(args.matrix_size, args.layers or 8, pk, clocks, steps, warmup, which=args.matrix_model)
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    if args.only == "tebozen":
        clocks.start()
        out = tebozen_beside_hybrid(args.tebozen_size, args.layers or 8, pk, clocks, steps, warmup, which=args.tebozen_model)
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    if args.only == "reperax":
        clocks.start()
        out = reperax_beside_matrix(args.reperax_size, args.layers or 8, pk, clocks, steps, warmup, which=args.reperax_model)
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    if args.only == "tubevik":
        clocks.start()
        out = tubevik_beside_matrix(args.tubevik_size, args.layers or 8, pk, clocks, steps, warmup, which=args.tubevik_model,
                                    kernels_only=args.tubevik_model == "kernels")
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    if args.only == "reference-kernel":
        clocks.start()
        out = reference_kernel_points(clocks)
        out["clocks"] = clocks.stop()
        print(json.dumps(out))
        return 0
    shape_name, shape = SHAPES[args.shape][0], dict(SHAPES[args.shape][1])
    layers_full = shape["num_hidden_layers"]
    if args.layers:
        shape["num_hidden_layers"] = args.layers
    B, ctx = args.batch, args.context
    tmp = tempfile.mkdtemp(prefix="pllm_bench_", dir=scratch_dir())
    try:
        model_dir = write_random_model(os.path.join(tmp, "model"), shape, 0, device="cuda")
        most = 1 if (args.no_points or args.only) else 64
        pages = max(most, B) * (ctx // PAGE + 4) + PREFILL_TOKENS // PAGE + 64
        if args.only == "long-prompt":
            pages = ctx // PAGE + 64
        eng = Engine(model_dir, dtype="bfloat16", block_size=PAGE, blocks=pages, max_batch=max(most, B),
                     chunk=PREFILL_TOKENS, prefix_cache=False)
        runner = eng.runner
        for g in runner.cache.groups:       # cache contents for the device-timed points: random, not zeros
            g.pool.normal_(0.0, 1.0)
        z = shape_sizes(shape)
        L, H, I, nh, nkv, hd, V = z["L"], z["H"], z["I"], z["nh"], z["nkv"], z["hd"], z["V"]
        weight_bytes, kv_token_bytes = z["weight_bytes"], runner.cache.bytes_per_token()
        assert kv_token_bytes == z["kv_token_bytes"]
        clocks.start()

        if args.only == "prefill":
            from paged_llm_rs_b200.engine.step import StepEntry
            prompt = np.random.default_rng(0).integers(0, V, PREFILL_TOKENS).tolist()
            one_zero = np.zeros(1, dtype=np.float32)
            for _ in range(warmup + steps):
                runner.cache.open("prefill")
                runner.cache.reserve("prefill", PREFILL_TOKENS)
                runner.step_and_sample([StepEntry("prefill", prompt, [PREFILL_TOKENS - 1])], one_zero, one_zero)
                runner.cache.close("prefill")
            torch.cuda.synchronize()
            print(json.dumps({"only": "prefill", "tokens": PREFILL_TOKENS, "steps": steps}))
            return 0

        if args.only == "long-prompt":
            out = long_prompt_points(runner, z, max(PREFILL_TOKENS, ctx // PREFILL_TOKENS * PREFILL_TOKENS), clocks)
            out.update(only="long-prompt", shape=shape_name, layers=L, clocks=clocks.stop())
            print(json.dumps(out))
            return 0

        if args.only == "timeline":
            return timeline(runner, B, ctx, L, PREFILL_TOKENS if args.timeline_prefill else 0, V, args.timeline_mixed)

        # -- decode, on the device -------------------------------------------------------
        ms, launches, spread = decode_point(runner, B, ctx, steps, warmup, clocks)
        if args.only == "decode":
            print(json.dumps({"only": "decode", "batch": B, "context": ctx, "ms_per_step": round(ms, 4),
                              "launches_per_step": launches, "repeats": spread}))
            return 0
        value = B / (ms / 1e3)
        step_bytes = weight_bytes + B * ctx * kv_token_bytes
        achieved = step_bytes / (ms / 1e3) / 1e9
        points = {}
        if not args.no_points:
            for c in (ctx, 512):                 # the bench context, and right after the baseline's 512-token prompts
                for b in (1, 8, 64):
                    if c == ctx and b == B:
                        continue
                    _, _, sp = decode_point(runner, b, c, max(10, steps // 2), warmup, clocks, repeats=4)
                    tag = f"decode_b{b}" + ("" if c == ctx else f"_ctx{c}")
                    points[tag] = round(b / (sp["median_ms"] / 1e3), 1)
                    points[tag + "_hbm_frac"] = round((weight_bytes + b * c * kv_token_bytes) / (sp["median_ms"] / 1e3) / 1e9
                                                      / pk["hbm_gbs"], 4)

        # -- prefill of 2048 tokens ---------------------------------------------------------
        pms, pspread = prefill_point(runner, V, clocks)
        prefill_out = dict(value=round(PREFILL_TOKENS / (pms / 1e3), 1), tokens=PREFILL_TOKENS, ms=round(pms, 3),
                           frac=round(z["prefill_flops"] / (pms / 1e3) / (pk["bf16_tflops"] * 1e12), 4),
                           frac_sustained=round(z["prefill_flops"] / (pms / 1e3) / (pk["bf16_tflops_sustained"] * 1e12), 4),
                           min_ms=pspread["min_ms"], max_ms=pspread["max_ms"], n=pspread["n"])

        # -- end to end through the entry point ---------------------------------------------
        rng = np.random.default_rng(1)
        rounds = 5
        budget = warmup + rounds * steps + 2
        for _ in range(B):
            eng.submit(rng.integers(0, V, ctx - budget - 16).tolist(), max_tokens=100000)
        while eng.scheduler.waiting or any(s.prompt_left for s in eng.scheduler.running):
            eng.step()                               # the prompts, untimed
        for _ in range(warmup):
            eng.step()
        torch.cuda.synchronize()
        per = []
        # (the prompts end so that the LAST round's steps run at the last positions before the bench's context, and
        #  that round is the one reported: the rounds before it, a little shorter in context, give the spread; a
        #  round past the context would need wider block tables and a capture of its own)
        for k in range(rounds):
            h2d = d2h = 0
            t0 = time.time()
            for _ in range(steps):
                out = eng.step()
                h2d += runner.bytes_h2d
                d2h += eng.bytes_d2h
                assert out is not None and len(out.tokens) == B
            torch.cuda.synchronize()
            t1 = time.time()
            clocks.region(t0, t1)
            per.append((t1 - t0) / steps * 1e3)
            if k == rounds - 1:
                e2e = dict(value=round(B * steps / (t1 - t0), 1), unit="tokens/s", h2d_bytes_per_step=h2d // steps,
                           d2h_bytes_per_step=d2h // steps, ms_per_step=round((t1 - t0) / steps * 1e3, 4))
        e2e.update(n=rounds, median_ms=round(statistics.median(per), 4), min_ms=round(min(per), 4), max_ms=round(max(per), 4))
        del eng, runner
        gc.collect()
        torch.cuda.empty_cache()

        # -- whole generations: 64 requests from their prompts to their last token ---------------
        generate_out = {}
        if not args.no_points:
            try:
                generate_out = generate_point(model_dir, V, clocks)
            except Exception as e:     # noqa: BLE001
                generate_out = {"error": f"{type(e).__name__}: {e}"[:200]}
            gc.collect()
            torch.cuda.empty_cache()
        shutil.rmtree(tmp, ignore_errors=True)

        # -- the baseline's other shapes, and the reference's own kernel -------------------------------
        shapes, ref_kernel = {}, {}
        if not args.no_shapes and args.shape == "0.6b" and not args.layers:
            # (what fails here is written into its own block: the headline above is measured already)
            for key, layers_of in (("8b", None), ("32b", 16)):
                # 16 of the 32B shape's 64 layers: the whole model's 65 GB of random weights take minutes to draw
                # and load; the layers are the shape's own size
                try:
                    shapes.update(other_shape(key, layers_of, pk, clocks, steps, warmup))
                except Exception as e:     # noqa: BLE001
                    shapes[f"{key}_error"] = f"{type(e).__name__}: {e}"[:200]
                    gc.collect()
                    torch.cuda.empty_cache()
            try:
                ref_kernel = reference_kernel_points(clocks, reps=5)
            except Exception as e:     # noqa: BLE001
                ref_kernel = {"error": f"{type(e).__name__}: {e}"[:200]}
        clk = clocks.stop()
    finally:
        shutil.rmtree(tmp, ignore_errors=True)

    line = {
        "metric": f"decode tokens/s ({shape_name} shape, batch {B}, context {ctx})", "value": round(value, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": round(ms, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {
            "model": f"{shape_name} shape, random weights N(0,0.02) seed 0", "layers": L, "layers_of_shape": layers_full,
            "hidden": H, "heads": nh, "kv_heads": nkv, "head_dim": hd, "intermediate": I, "vocab": V,
            "tie_word_embeddings": bool(shape["tie_word_embeddings"]), "global_batch": B, "seq_len": ctx, "page_size": PAGE,
            "prefill_tokens": PREFILL_TOKENS, "parallelism": "one GPU",
            "l2": f"inputs larger than L2: a step reads {step_bytes / 1e6:.0f} MB",
            "peaks": pk["source"], "hbm_gbs_peak": pk["hbm_gbs"], "bf16_tflops_peak": pk["bf16_tflops"],
            "bf16_tflops_sustained": pk["bf16_tflops_sustained"],
        },
        "repeats": spread,
        "e2e": e2e, "gpu_launches": launches * steps, "clocks": clk, "prefill": prefill_out,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
    }
    if generate_out:
        line["generate"] = generate_out
    if shapes:
        line["shapes"] = shapes
    if ref_kernel:
        line["reference_kernel"] = ref_kernel
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
