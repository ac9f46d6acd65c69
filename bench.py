#!/usr/bin/env python3
"""Decode and prefill throughput of the Gemma 2 engine on one B200, as one JSON line.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]
                    [--size 2b|9b|27b] [--layers L] [--batch B] [--context C] [--only-headline]
    python bench.py --micro attention|prompt-attention|gemm|products|reference|memory
                    (kernels alone, JSON lines; for the summaries in profiles/)
    python bench.py --compare bolonex
    python bench.py --compare petanex
    python bench.py --compare pimodra
    python bench.py --compare nukelix
    python bench.py --compare lurisun
    python bench.py --compare fovosun
                    (Bolonex beside Gemma 2, Petanex beside Bolonex, and so on, at equal layer sizes: prefill and decode throughput
                    and, per operation, the time of one step against the time its bytes, or its multiply-adds, take at the
                    measured rates; one JSON line)

A "step" is one decode step: every live request gets one token.  Default: the layer sizes of Gemma 2 2B, random
bfloat16 weights, 8 requests at a context of 8192 tokens.  `value` is decoded tokens per second timed with CUDA events
around K steps of the step function (the mean of `reps` such runs, `sd` beside it); `e2e` is the same through the
Python entry point (`Engine.step()`: host scheduling, the step's integers copied from pinned host memory, tokens drawn
on the device and read back).  `prefill` is one step of 2,048 prompt tokens; `roofline` is the bytes a decode step must
read (every weight once, the cache of the live requests) over its time; `points` holds decode at batch 1 and 64.
Beyond the headline the line carries: `mixed` (a step of 8 decode rows beside a 512-token prompt portion at context
8192, and that portion alone: GPU time by events and wall time through `Engine.step()`), `fp32` (the true 32-bit path at
the same sizes) and `sizes` (the same figures at Gemma 2 9B and 27B layer sizes; where 64 requests of 8192 tokens do not
fit beside the weights the context of that point is named).
Method after the reference's `kungfu bench` (crates/kungfu/src/main.rs:544-608): synthetic token ids, every shape run
before timing, mean and standard deviation over repetitions.  Caches are filled with random keys and values instead of
running the long prompts.
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import statistics
import subprocess
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

SIZES = {
    # the layer sizes of Gemma 2 2B, 9B and 27B
    "2b": dict(num_hidden_layers=26, hidden_size=2304, num_attention_heads=8, num_key_value_heads=4, head_dim=256,
               intermediate_size=9216, query_pre_attn_scalar=256),
    "9b": dict(num_hidden_layers=42, hidden_size=3584, num_attention_heads=16, num_key_value_heads=8, head_dim=256,
               intermediate_size=14336, query_pre_attn_scalar=256),
    "27b": dict(num_hidden_layers=46, hidden_size=4608, num_attention_heads=32, num_key_value_heads=16, head_dim=128,
                intermediate_size=36864, query_pre_attn_scalar=144),
}
COMMON = dict(architectures=["Gemma2ForCausalLM"], vocab_size=256000, rope_theta=10000.0, sliding_window=4096,
              attn_logit_softcapping=50.0, final_logit_softcapping=30.0, rms_norm_eps=1e-6, tie_word_embeddings=True,
              max_position_embeddings=8192 + 512, hidden_activation="gelu_pytorch_tanh")
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks() -> tuple[dict, str]:
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    try:
        with open(p) as f:
            raw = json.load(f)
        out = dict(FALLBACK_PEAKS)
        for k in out:
            if isinstance(raw.get(k), (int, float)):
                out[k] = float(raw[k])
        return out, "measured"
    except (OSError, ValueError):
        return dict(FALLBACK_PEAKS), "fallback"


class ClockSampler:
    QUERY = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.proc = None
        self.index = index

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "100", "-i", str(self.index)], stdout=subprocess.PIPE,
                                         stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            out, _ = self.proc.communicate(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
            out, _ = self.proc.communicate()
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in out.strip().split("\n"):
            f = [x.strip() for x in line.split(",")]
            if len(f) < 9:
                continue
            try:
                sm.append(float(f[1]))
                mx.append(float(f[2]))
            except ValueError:
                continue
            for name, v in zip(names, f[5:9]):
                if v.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(sm)}


def model_numbers(cfg, n_layers: int):
    """Weight bytes a decode step reads (bf16) and matrix parameters per token for the flop count."""
    H, I, V = cfg.hidden_size, cfg.intermediate_size, cfg.vocab_size
    per_layer = (cfg.q_size + 2 * cfg.kv_size) * H + H * cfg.q_size + 3 * H * I
    norms = 4 * H * n_layers + H
    weight_bytes = 2 * (per_layer * n_layers + V * H + norms)
    return per_layer, weight_bytes


def kv_bytes_read(cfg, n_layers: int, length: int) -> int:
    """Bytes of keys and values one decode step reads for one request at `length` tokens (bf16)."""
    n = 0
    for l in range(n_layers):
        w = cfg.window_of(l)
        n += 2 * cfg.kv_size * 2 * (min(length, w) if w else length)
    return n


def prefill_flops(cfg, n_layers: int, T: int) -> float:
    per_layer, _ = model_numbers(cfg, n_layers)
    gemm = 2.0 * T * per_layer * n_layers + 2.0 * cfg.vocab_size * cfg.hidden_size
    attn = 0.0
    for l in range(n_layers):
        w = cfg.window_of(l)
        pairs = sum(min(p + 1, w) if w else p + 1 for p in range(T))
        attn += 4.0 * cfg.num_attention_heads * cfg.head_dim * pairs
    return gemm + attn


def fill_cache(runner, rid, n_tokens: int) -> None:
    """Make request `rid` hold `n_tokens` tokens (of whatever the pages contain) without running them; in portions, so
    that a windowed group gives pages back as it would while a prompt is fed."""
    runner.cache.add_request(rid)
    at = 0
    while at < n_tokens:
        n = min(512, n_tokens - at)
        runner.cache.reserve(rid, n)
        runner.cache.commit(rid, n)
        at += n


def randomize_pages(runner, torch) -> None:
    g = torch.Generator(device=runner.device)
    g.manual_seed(1)
    stores = [t for v in runner.cache.storage.values() for t in (v if isinstance(v, list) else [v])]
    for t in stores:
        if t.dim() == 5:
            flat = t.view(-1)
            step = 1 << 28
            for i in range(0, flat.numel(), step):
                flat[i:i + step].normal_(0.0, 0.5, generator=g)


def mean_sd(xs) -> tuple[float, float]:
    xs = list(xs)
    return statistics.fmean(xs), (statistics.stdev(xs) if len(xs) > 1 else 0.0)


def time_decode(torch, runner, rids, steps: int, warmup: int, vocab: int, reps: int):
    """`reps` timed runs of `steps` decode steps each (CUDA events around each run, a synchronize on both sides), after
    `warmup` steps.  Returns the ms per step of every run and the kernels launched in the last one."""
    from kungfu_b200 import ops
    from kungfu_b200.engine import StepEntry
    tok = 17
    i = 0

    def one():
        nonlocal i
        entries = [StepEntry(r, [(tok + 31 * i + 7 * k) % vocab], [0]) for k, r in enumerate(rids)]
        i += 1
        return runner.step(entries)

    for _ in range(warmup):
        one()
    out, launches = [], 0
    for _ in range(reps):
        torch.cuda.synchronize()
        l0 = ops.launch_count()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(steps):
            one()
        e1.record()
        torch.cuda.synchronize()
        out.append(e0.elapsed_time(e1) / steps)
        launches = ops.launch_count() - l0
    return out, launches


def build(torch, size: str, n_layers: int, dtype: str, *, parallel: int, ctx_len: int, margin: int):
    """Model with random weights, and a runner whose pools hold `parallel` requests of `ctx_len` tokens or what fits."""
    from kungfu_b200 import api
    raw = dict(COMMON, **SIZES[size])
    raw["num_hidden_layers"] = n_layers
    device = torch.device("cuda:0")
    cfg, model = api.random_model(raw, seed=0, dtype=dtype, device=device)
    free, total = torch.cuda.mem_get_info(device)
    budget = int(free) - max(6 << 30, int(total) // 16)
    runner = api.make_runner(cfg, model, dtype=dtype, device=device, page_size=api.DEFAULT_PAGE_SIZE,
                             max_requests=parallel, max_context=ctx_len + margin, batch=512, budget_bytes=budget)
    randomize_pages(runner, torch)
    return cfg, model, runner


def context_that_fits(runner, batch: int, ctx_len: int) -> int:
    """The longest context (a multiple of 1,024, at most `ctx_len`) at which `batch` requests fit the pools."""
    page = runner.cache.page_size
    c = ctx_len
    while c > 1024:
        ok = True
        for g in runner.cache.groups:
            per = c + 64 if g.window is None else min(c + 64, g.window + 512 + page)
            ok = ok and batch * -(-per // page) <= g.pool.n_pages
        if ok:
            return c
        c -= 1024
    return c


def measure_size(torch, args, size: str, dtype: str, pk: dict, *, headline: bool) -> dict:
    """Decode at batch 8 / 1 / 64 and a 2,048-token prompt at one model size and precision."""
    from kungfu_b200 import ops
    from kungfu_b200.engine import StepEntry
    full_layers = SIZES[size]["num_hidden_layers"]
    n_layers = args.layers if (headline and args.layers) else full_layers
    ctx_len = args.context
    reps = args.reps
    steps = args.steps if headline else min(args.steps, 32 if dtype == "bfloat16" else 8)
    warmup = args.warmup
    margin = (reps * steps + warmup) + 128
    batches = [args.batch] if (args.only_headline or dtype != "bfloat16") else sorted({args.batch, 1, 64})
    cfg, model, runner = build(torch, size, n_layers, dtype, parallel=max(batches) + 2, ctx_len=ctx_len, margin=margin)
    vocab = cfg.vocab_size
    elt = 2 if dtype == "bfloat16" else 4
    per_layer, weight_bytes = model_numbers(cfg, n_layers)
    weight_bytes = weight_bytes * elt // 2
    out = {"layers": n_layers, "layers_full": full_layers, "pool_pages": [g.pool.n_pages for g in runner.cache.groups]}

    # ---- a prompt of 2,048 tokens in one step ---------------------------------------------------------------------------
    T = args.prefill_tokens
    toks = [(i * 7919 + 13) % vocab for i in range(T)]
    pf_ms = []
    for rep in range(reps + 1):
        runner.cache.add_request("pf")
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        runner.step([StepEntry("pf", toks, [T - 1])])
        e1.record()
        torch.cuda.synchronize()
        pf_ms.append(e0.elapsed_time(e1))
        runner.cache.release("pf")
    m, sd = mean_sd(pf_ms[1:])
    flops = prefill_flops(cfg, n_layers, T)
    peak_flops = pk["bf16_tflops"] * 1e12
    out["prefill"] = {"value": round(T / m * 1e3, 1), "tokens": T, "ms": round(m, 3), "sd_ms": round(sd, 3),
                      "frac": round(flops / (m * 1e-3) / peak_flops, 4) if dtype == "bfloat16" else None}

    # ---- decode ------------------------------------------------------------------------------------------------------------
    out["decode"] = {}
    for b in batches:
        c_len = context_that_fits(runner, b, ctx_len)
        rids = [f"d{b}_{k}" for k in range(b)]
        for r in rids:
            fill_cache(runner, r, c_len - warmup)
        clocks = None
        sampler = ClockSampler()
        if headline and b == args.batch:
            sampler.start()
            time.sleep(0.3)
        ms_runs, launches = time_decode(torch, runner, rids, steps, warmup, vocab, reps)
        if headline and b == args.batch:
            clocks = sampler.stop()
        for r in rids:
            runner.cache.release(r)
        m, sd = mean_sd(ms_runs)
        tps = [b / x * 1e3 for x in ms_runs]
        bytes_step = weight_bytes + b * kv_bytes_read(cfg, n_layers, c_len) * elt // 2
        achieved = bytes_step / (m * 1e-3) / 1e9
        out["decode"][f"b{b}"] = {"value": round(mean_sd(tps)[0], 1), "sd": round(mean_sd(tps)[1], 1), "ms_per_step": round(m, 4),
                                  "sd_ms": round(sd, 4), "context": c_len, "hbm_gbs": round(achieved, 1),
                                  "frac": round(achieved / pk["hbm_gbs"], 4), "launches": int(launches), "clocks": clocks}
    out["_live"] = (cfg, model, runner)
    return out


def measure_mixed(torch, args, cfg, runner) -> dict:
    """A step of `batch` decode rows beside one 512-token prompt portion at the headline context, and that portion
    alone: GPU time by CUDA events around `Runner.step` (tokens drawn on the device) and wall time of `Engine.step()`
    (planning, the step's integers, the launch or graph replay, the tokens read back)."""
    import numpy as np
    from kungfu_b200.engine import StepEntry
    from kungfu_b200.engine.engine import Engine
    from kungfu_b200.engine.scheduler import Request
    from kungfu_b200.sampling import STATE_WORDS, Sampling, pack_state
    B, ctx_len, vocab = args.batch, args.context, cfg.vocab_size
    out = {}
    states = torch.zeros((runner.cache.max_requests, STATE_WORDS), dtype=torch.int32, device=runner.device)
    states[:] = torch.from_numpy(pack_state(Sampling(temperature=0.0), 1)).to(runner.device)
    # the scheduler's budget counts decode rows, so with a budget of 512 a mixed step has 512 rows in all (the second case:
    # two whole 256-token tiles); the first case is 520 rows, a third tile for eight of them
    for name, n_dec, portion in ((f"decode{B}_portion512", B, 512), (f"decode{B}_portion{512 - B}", B, 512 - B), ("portion512", 0, 512)):
        rids = [f"m{k}" for k in range(n_dec)]
        for r in rids:
            fill_cache(runner, r, ctx_len - 16)
        gpu_ms = []
        for rep in range(args.reps + 2):                       # the first runs eagerly, the second is captured
            fill_cache(runner, "mp", ctx_len - portion)
            entries = [StepEntry(r, [(5 + 3 * rep + k) % vocab], [0]) for k, r in enumerate(rids)]
            entries.append(StepEntry("mp", [(i * 31 + rep) % vocab for i in range(portion)], [portion - 1]))
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            runner.step(entries, sample=(states, False))
            e1.record()
            torch.cuda.synchronize()
            gpu_ms.append(e0.elapsed_time(e1))
            runner.cache.release("mp")
        for r in rids:
            runner.cache.release(r)
        # the same step through the engine: requests adopted at their long context, one Engine.step() each repetition
        eng = Engine(runner=runner, batch=portion + n_dec, parallel=n_dec + 1, pipeline=False)
        eng.cfg = cfg
        for k in range(n_dec):
            rid = f"e{k}"
            req = Request(rid, [(k * 131 + i) % vocab for i in range(ctx_len - 16)], Sampling(temperature=0.0), max_tokens=10 ** 9,
                          eos=(), ignore_eos=True)
            fill_cache(runner, rid, ctx_len - 17)
            req.n_cached = ctx_len - 17
            eng.requests[rid] = req
            eng.scheduler.adopt(req)
        if n_dec:
            eng.step()                                         # every decoding request has produced a token
        wall_ms = []
        for rep in range(args.reps + 2):
            rid = f"p{rep}"
            req = Request(rid, [(rep + i * 7) % vocab for i in range(ctx_len)], Sampling(temperature=0.0), max_tokens=1, eos=(),
                          ignore_eos=True)
            fill_cache(runner, rid, ctx_len - portion)
            req.n_cached = ctx_len - portion
            eng.requests[rid] = req
            eng.scheduler.adopt(req)
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            ev = eng.step()
            torch.cuda.synchronize()
            wall_ms.append((time.perf_counter() - t0) * 1e3)
            assert any(r == rid and reason == "length" for r, _t, reason in ev), ev
        for k in range(n_dec):
            eng.cancel(f"e{k}")
        g, gs = mean_sd(gpu_ms[2:])
        w, ws = mean_sd(wall_ms[2:])
        out[name] = {"gpu_ms": round(g, 3), "gpu_sd_ms": round(gs, 3), "engine_wall_ms": round(w, 3), "engine_wall_sd_ms": round(ws, 3),
                     "eager_first_ms": round(gpu_ms[0], 3), "rows": n_dec + portion, "context": ctx_len}
    return out


def measure_e2e(torch, args, cfg, runner) -> dict:
    """Decode through the Python entry point: `Engine.step()` with host token ids in and out."""
    from kungfu_b200.engine.engine import Engine
    from kungfu_b200.engine.scheduler import Request
    from kungfu_b200.sampling import Sampling
    B, ctx_len, vocab = args.batch, args.context, cfg.vocab_size
    eng = Engine(runner=runner, batch=max(512, B), parallel=B)
    eng.cfg = cfg
    start = ctx_len - args.warmup
    for k in range(B):
        rid = f"e{k}"
        prompt = [(k * 131 + i * 7919 + 13) % vocab for i in range(start)]
        req = Request(rid, prompt, Sampling(temperature=0.0), max_tokens=10 ** 9, eos=(), ignore_eos=True)
        fill_cache(runner, rid, start - 1)               # all but the last prompt token are "already run"
        req.n_cached = start - 1
        eng.requests[rid] = req
        eng.scheduler.adopt(req)
    for _ in range(args.warmup):
        eng.step()
    rates, per_step = [], []
    for _ in range(args.reps):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        n_tok = 0
        for _ in range(args.steps):
            n_tok += sum(1 for _id, tok, _r in eng.step() if tok is not None)
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        rates.append(n_tok / dt)
        per_step.append(dt / args.steps * 1e3)
    meta_ints = runner.last_meta_ints
    for k in range(B):
        eng.cancel(f"e{k}")
    return {"value": round(mean_sd(rates)[0], 1), "sd": round(mean_sd(rates)[1], 1), "unit": "tokens/s",
            "h2d_bytes_per_step": int(meta_ints * 4), "d2h_bytes_per_step": int(B * 4),
            "ms_per_step": round(mean_sd(per_step)[0], 3),
            "reads": "ids of step n read on the host while step n+1 runs" if eng.pipeline else "every step before the next"}


def run_ours(args) -> dict:
    import torch
    from kungfu_b200 import api, ops

    pk, pk_src = peaks()
    api.require_cuda("cuda:0")
    ops.library()
    head = measure_size(torch, args, args.size, "bfloat16", pk, headline=True)
    cfg, model, runner = head.pop("_live")
    B, ctx_len = args.batch, args.context
    hd = head["decode"][f"b{B}"]
    e2e = measure_e2e(torch, args, cfg, runner)
    mixed = None if args.only_headline else measure_mixed(torch, args, cfg, runner)
    n_layers, full_layers = head["layers"], head["layers_full"]
    config = {"model": f"gemma2-{args.size}", "layers": n_layers, "layers_full": full_layers,
              "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads,
              "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
              "sliding_window": cfg.sliding_window, "global_batch": B, "seq_len": ctx_len, "page_size": runner.cache.page_size,
              "parallelism": "single", "weights": "random bf16", "cache": "bf16 random fill", "l2": "inputs larger than L2",
              "cuda_graphs": bool(getattr(runner, "cuda_graphs", False)), "reps": args.reps}
    del model, runner
    gc.collect()
    torch.cuda.empty_cache()

    fp32, sizes = None, {}
    if not args.only_headline:
        r = measure_size(torch, args, args.size, "float32", pk, headline=False)
        r.pop("_live")
        gc.collect()
        torch.cuda.empty_cache()
        fp32 = {"decode": r["decode"], "prefill": r["prefill"], "layers": r["layers"]}
        for other in [s for s in ("9b", "27b") if s != args.size]:
            r = measure_size(torch, args, other, "bfloat16", pk, headline=False)
            r.pop("_live")
            gc.collect()
            torch.cuda.empty_cache()
            sizes[other] = r
    points = {k: v["value"] for k, v in head["decode"].items() if k != f"b{B}"}
    return {"metric": "decode tokens/s (batch 8, context 8192, Gemma 2 2B sizes, 1 B200)" if (args.size, B, ctx_len) == ("2b", 8, 8192)
            else f"decode tokens/s (batch {B}, context {ctx_len}, Gemma 2 {args.size} sizes, 1 B200)",
            "value": hd["value"], "sd": hd["sd"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": hd["ms_per_step"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": "bf16", "data": "synthetic token ids, random-init weights, random-filled cache",
            "config": config, "clocks": hd["clocks"], "e2e": e2e, "gpu_launches": hd["launches"], "prefill": head["prefill"],
            "roofline": {"bound": "hbm", "achieved": hd["hbm_gbs"], "peak": pk["hbm_gbs"], "unit": "GB/s", "frac": hd["frac"],
                         "peaks": pk_src},
            "points": {f"decode_{k}": v for k, v in points.items()},
            "decode": {k: {kk: vv for kk, vv in v.items() if kk != "clocks"} for k, v in head["decode"].items()},
            "mixed": mixed, "fp32": fp32, "sizes": sizes, "slow_kernel_fallbacks": ops.fallbacks(), "impl": "ours"}

# ---- Bolonex beside Gemma 2 at equal layer sizes (--compare bolonex) ---------------------------------------------------
# Layer sizes that resemble real models: eight layers, one attention layer to three state-space layers, the same width,
# heads, head size, feed-forward width and vocabulary in both models (the Gemma 2 feed-forward is gated, so it has three
# matrices of that width where Bolonex has two).
BOLONEX_SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, ff=8192, ssm_heads=64, ssm_vdim=64, state=128, groups=1, norm_groups=1),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, ff=14336, ssm_heads=128, ssm_vdim=64, state=128, groups=8, norm_groups=8),
}
COMPARE_VOCAB, COMPARE_LAYERS = 32000, 8


def bolonex_config(z: dict) -> dict:
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "conv": 4,
           "scale": z["dim"] ** -0.5, "softcap": 30.0,
           "rot": {"base": 500000.0, "dims": z["dim"], "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    ssm = {"heads": z["ssm_heads"], "vdim": z["ssm_vdim"], "state": z["state"], "groups": z["groups"],
           "norm_groups": z["norm_groups"], "conv": 4}
    mlp = {"kind": "dense", "ff": z["ff"]}
    layers = [{"type": "attention" if i % 4 == 0 else "mamba2", "mixer": att if i % 4 == 0 else ssm, "mlp": mlp}
              for i in range(COMPARE_LAYERS)]
    return {"architecture": "Bolonex", "width": z["width"], "vocab": COMPARE_VOCAB, "embedding": {"scale": 1.0},
            "norm": {"eps": 1e-5}, "layers": layers}


def gemma_twin_config(z: dict) -> dict:
    return dict(COMMON, vocab_size=COMPARE_VOCAB, num_hidden_layers=COMPARE_LAYERS, hidden_size=z["width"],
                num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"],
                intermediate_size=z["ff"], query_pre_attn_scalar=z["dim"], sliding_window=1 << 20,
                layer_types=["full_attention"] * COMPARE_LAYERS)


def bolonex_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    """Bytes each operation of one Bolonex step must move (bfloat16 activations, 32-bit projections and states), summed
    over the layers that run it; for the products, the weights once plus their rows."""
    W, H, G, d, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["ff"]
    sh, sp, N, sg = z["ssm_heads"], z["ssm_vdim"], z["state"], z["groups"]
    inner, cw = sh * sp, sh * sp + 2 * sg * N
    n_att = sum(1 for i in range(COMPARE_LAYERS) if i % 4 == 0)
    n_ssm = COMPARE_LAYERS - n_att
    cq = (H + 2 * G) * d
    return {
        "qkv_prepare": n_att * T * (4 * cq + 2 * cq + 4 * d),
        "head_gate": n_att * T * H * d * 4,
        "short_conv": n_ssm * T * cw * 8,
        "short_conv_commit": n_att * n_reqs * 3 * cq * 8 + n_ssm * n_reqs * 3 * cw * 8,
        "ssm_scan": n_ssm * (T * (cw + inner) * 4 + 2 * n_reqs * inner * N * 4),
        "gated_group_norm": n_ssm * T * inner * 10,
        "add2_rmsnorm": COMPARE_LAYERS * T * W * 18,
        "paged_attention": n_att * (n_reqs * keys * 2 * G * d * 2 + T * H * d * 4),
    }


def gemma_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    W, H, G, d = z["width"], z["heads"], z["kv_heads"], z["dim"]
    cq = (H + 2 * G) * d
    L = COMPARE_LAYERS
    return {
        "rope_kv_append": L * T * (4 * cq + 2 * cq + 4 * d),
        "add_rmsnorm": 2 * L * T * W * 14,
        "paged_attention": L * (n_reqs * keys * 2 * G * d * 2 + T * H * d * 4),
        "rope_append_attend": L * (n_reqs * keys * 2 * G * d * 2 + T * (4 * cq + H * d * 2)),
    }


def compare_bolonex(args) -> dict:
    return compare_models(args, "bolonex", BOLONEX_SIZES, lambda z: (("bolonex", bolonex_config(z), bolonex_op_bytes),
                                                                      ("gemma2", gemma_twin_config(z), gemma_op_bytes)))


def compare_models(args, label: str, size_table: dict, archs_of) -> dict:
    """Prefill (one prompt of --prefill-tokens tokens) and decode (--batch requests at --context tokens) of two
    architectures at equal sizes, and per operation the time of one eager step beside the time its bytes would take at the
    measured copy rate, or its multiply-adds at the measured bfloat16 rate if that is longer (`x_roofline`: 1.0 = at the
    roofline).  An operation's entry in the byte tables is a byte count, or (bytes, floating-point operations)."""
    import torch
    from kungfu_b200 import api, ops
    from kungfu_b200.engine import StepEntry
    pk, pk_src = peaks()
    device = api.require_cuda("cuda:0")
    ops.library()
    T, B, ctx_len = args.prefill_tokens, args.batch, min(args.context, 4096)
    out = {"impl": "ours", "compare": label, "peaks": pk_src, "prefill_tokens": T, "decode_batch": B, "decode_context": ctx_len,
           "layers": COMPARE_LAYERS, "vocab": COMPARE_VOCAB, "dtype": "bf16", "data": "synthetic token ids, random-init weights",
           "sizes": {}}
    for name, z in size_table.items():
        row = {}
        for arch, raw, op_bytes in archs_of(z):
            cfg, model = api.random_model(raw, seed=0, dtype="bfloat16", device=device)
            steps, warmup, reps = min(args.steps, 32), max(args.warmup, 3), args.reps
            runner = api.make_runner(cfg, model, dtype="bfloat16", device=device, page_size=api.DEFAULT_PAGE_SIZE,
                                     max_requests=B + 2, max_context=ctx_len + reps * steps + warmup + 192,
                                     max_tokens=(B + 1) * (ctx_len + reps * steps + warmup + 192))
            randomize_pages(runner, torch)
            vocab = cfg.vocab_size
            toks = [(i * 7919 + 13) % vocab for i in range(T)]
            pf = []
            for rep in range(reps + 1):
                runner.cache.add_request("pf")
                torch.cuda.synchronize()
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                runner.step([StepEntry("pf", toks, [T - 1])])
                e1.record()
                torch.cuda.synchronize()
                pf.append(e0.elapsed_time(e1))
                runner.cache.release("pf")
            rids = [f"d{k}" for k in range(B)]
            for r in rids:
                fill_cache(runner, r, ctx_len - warmup)
            ms_runs, launches = time_decode(torch, runner, rids, steps, warmup, vocab, reps)
            # one eager prompt step and one eager decode step with every operation timed
            traces = {}
            runner.cache.add_request("tr")
            ops.trace_begin()
            runner.step([StepEntry("tr", toks, [T - 1])])
            traces["prefill"] = (ops.trace_end(), op_bytes(z, T, 1, T))
            runner.cache.release("tr")
            ops.trace_begin()
            runner.step([StepEntry(r, [(5 + k) % vocab], [0]) for k, r in enumerate(rids)])
            traces["decode"] = (ops.trace_end(), op_bytes(z, B, B, ctx_len))
            for r in rids:
                runner.cache.release(r)
            per_op = {}
            for phase, (rec, nbytes) in traces.items():
                agg = {}
                for op, ms in rec:
                    n, t = agg.get(op, (0, 0.0))
                    agg[op] = (n + 1, t + ms)
                total = sum(t for _, t in agg.values())
                per_op[phase] = {"total_ms": round(total, 3), "ops": {}}
                for op, (n, t) in sorted(agg.items(), key=lambda kv: -kv[1][1]):
                    e = {"n": n, "us": round(t * 1e3, 1), "share": round(t / total, 3)}
                    nb, fl = nbytes.get(op, 0) if isinstance(nbytes.get(op, 0), tuple) else (nbytes.get(op, 0), 0)
                    if nb > 0:
                        ideal_us = max(nb / (pk["hbm_gbs"] * 1e3), fl / (pk["bf16_tflops"] * 1e6))
                        e["bytes"] = int(nb)
                        if fl:
                            e["flops"] = int(fl)
                        e["x_roofline"] = round(t * 1e3 / ideal_us, 2)
                    per_op[phase]["ops"][op] = e
            m, sd = mean_sd(pf[1:])
            d, dsd = mean_sd(ms_runs)
            row[arch] = {"prefill": {"tokens_per_s": round(T / m * 1e3, 1), "ms": round(m, 3), "sd_ms": round(sd, 3)},
                         "decode": {"tokens_per_s": round(B / d * 1e3, 1), "ms_per_step": round(d, 4), "sd_ms": round(dsd, 4),
                                    "launches": int(launches)},
                         "weight_bytes": int(model.weight_bytes()), "per_op": per_op}
            del model, runner
            gc.collect()
            torch.cuda.empty_cache()
        out["sizes"][name] = dict(row, shape=z)
    out["slow_kernel_fallbacks"] = ops.fallbacks()
    ops.raise_on_device_error()
    return out


# ---- Petanex beside Bolonex at equal layer sizes (--compare petanex) -------------------------------------------------
# Eight layers in both: attention over a latent, then a delta rule per key channel, then two delta rules per head (Bolonex:
# attention, then three state-space layers); feed-forwards alternate between dense and a mixture whose chosen experts and
# shared expert together have the dense width; every layer has a per-token side input.
PETANEX_SIZES = {
    "w2048": dict(BOLONEX_SIZES["w2048"], lat_heads=16, rank=256, d_heads=16, d_kv_heads=8, d_dim=128, d_vdim=128, low=64,
                  experts=32, top=3, e_groups=4, e_keep=2, side=64),
    "w4096": dict(BOLONEX_SIZES["w4096"], lat_heads=32, rank=256, d_heads=32, d_kv_heads=16, d_dim=128, d_vdim=128, low=128,
                  experts=64, top=7, e_groups=8, e_keep=4, side=64),
}


def petanex_config(z: dict) -> dict:
    lat = {"heads": z["lat_heads"], "dim": z["dim"], "vdim": z["dim"], "kv_rank": z["rank"], "scale": z["dim"] ** -0.5}
    dl = {"heads": z["d_heads"], "kv_heads": z["d_kv_heads"], "dim": z["d_dim"], "vdim": z["d_vdim"], "conv": 4}
    ch = dict(dl, decay_rank=z["low"], gate_rank=z["low"])
    eff = z["ff"] // (z["top"] + 1) // 64 * 64
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": eff, "limit": 7.0}, "shared": {"ff": eff, "limit": 7.0},
           "router": {"experts": z["experts"], "top": z["top"], "scale": 2.5, "groups": {"count": z["e_groups"], "keep": z["e_keep"]}}}
    kinds = ["latent_attention", "channel_delta", "delta", "delta"]
    layers = [{"type": kinds[i % 4], "mixer": (lat, ch, dl, dl)[i % 4], "mlp": dense if i % 2 == 0 else moe}
              for i in range(COMPARE_LAYERS)]
    return {"architecture": "Petanex", "width": z["width"], "vocab": COMPARE_VOCAB, "embedding": {"scale": 1.0},
            "norm": {"eps": 1e-5}, "token_side": {"dim": z["side"]}, "layers": layers}


def petanex_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    """Bytes (and, for the grouped products, floating-point operations) each operation of one Petanex step must move,
    summed over the layers that run it."""
    W, L = z["width"], COMPARE_LAYERS
    H, d, r = z["lat_heads"], z["dim"], z["rank"]
    dh, dk, dd, dv, low = z["d_heads"], z["d_kv_heads"], z["d_dim"], z["d_vdim"], z["low"]
    n_lat, n_ch, n_dl = L // 4, L // 4, L // 2
    n_rec, n_moe = n_ch + n_dl, L // 2
    cq = 2 * dk * dd + dh * dv
    eff = z["ff"] // (z["top"] + 1) // 64 * 64
    P = T * z["top"]
    used = min(z["experts"], P)                                   # experts whose weights a step touches, at most
    return {
        "latent_append": n_lat * T * (4 * r + 4 * r),
        "head_linear": (n_lat * (T * H * (4 * d + 2 * r + 2 * r + 2 * d) + 4 * H * d * r), n_lat * 4 * T * H * d * r),
        "paged_attention": n_lat * (n_reqs * keys * 2 * r * 2 + T * H * r * 4),
        "short_conv": n_rec * T * cq * 8,
        "short_conv_commit": n_rec * n_reqs * 3 * cq * 8,
        "linear_cols": (n_ch * (T * 4 * (2 * low + dh * dd + dh * dv) + 2 * low * (dh * dd + dh * dv)), n_ch * 2 * T * low * (dh * dd + dh * dv)),
        "delta_rule": n_rec * (T * (cq + dh * dv) * 4 + 2 * n_reqs * dh * dd * dv * 4) + n_ch * T * dh * dd * 4,
        "head_norm_gate": n_rec * T * dh * dv * 10,
        "scale_add_rmsnorm": 2 * L * T * W * 14,
        "add_rmsnorm": L * T * W * 14,
        "side_gate": L * T * z["side"] * 8,
        "moe_route": n_moe * T * (z["experts"] * 4 + z["top"] * 8),
        "moe_plan": n_moe * P * 12,
        "moe_linear": (n_moe * (used * 3 * eff * W * 2 + P * (2 * W + 4 * eff + 4 * W)), n_moe * 6 * P * eff * W),
        "moe_combine": n_moe * T * W * (4 * z["top"] + 8),
    }


def compare_petanex(args) -> dict:
    return compare_models(args, "petanex", PETANEX_SIZES, lambda z: (("petanex", petanex_config(z), petanex_op_bytes),
                                                                      ("bolonex", bolonex_config(z), bolonex_op_bytes)))


# ---- Pimodra beside Gemma 2 at equal layer sizes (--compare pimodra) -------------------------------------------------
# Eight layer runs in both: Pimodra has four layers (feed-forwards dense, mixture, dense, mixture) that run twice as one
# looped stretch; the same width, heads, head size, dense feed-forward width and vocabulary; the mixture's chosen experts
# together have the dense width.  Every layer's window is longer than the contexts measured, as the Gemma 2 twin's is, so
# both attend to the same keys.  (The Gemma 2 feed-forward is gated: three matrices where Pimodra's dense one has two.)
PIMODRA_SIZES = {
    "w2048": dict(BOLONEX_SIZES["w2048"], experts=32, top=4, e_groups=4, e_keep=2),
    "w4096": dict(BOLONEX_SIZES["w4096"], experts=64, top=8, e_groups=8, e_keep=4),
}


def pimodra_config(z: dict) -> dict:
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
           "mask": {"size": 1 << 20},
           "rot": {"base": 10000.0, "dims": z["dim"], "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    eff = z["ff"] // z["top"] // 64 * 64
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": eff},
           "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": z["e_groups"], "keep": z["e_keep"]}}}
    layers = [{"type": "attention", "mixer": att, "mlp": dense if i % 2 == 0 else moe} for i in range(COMPARE_LAYERS // 2)]
    return {"architecture": "Pimodra", "width": z["width"], "vocab": COMPARE_VOCAB, "norm": {"eps": 1e-5, "groups": 8},
            "loop": {"start": 0, "stop": COMPARE_LAYERS // 2, "times": 2}, "layers": layers}


def pimodra_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    """Bytes (and, for the grouped products, floating-point operations) each operation of one Pimodra step must move,
    summed over the layer runs that use it.  The attention's entry is the same as the Gemma 2 twin's: the keys and values
    once, the queries and the result."""
    W, H, G, d, ff, L = z["width"], z["heads"], z["kv_heads"], z["dim"], z["ff"], COMPARE_LAYERS
    cq = (H + 2 * G) * d
    n_moe = L // 2
    n_dense = L - n_moe
    eff = ff // z["top"] // 64 * 64
    P = T * z["top"]
    used = min(z["experts"], P)
    return {
        "rotate_norm_append": L * T * (4 * cq + 2 * cq + 4 * d),
        "paged_attention": L * (n_reqs * keys * 2 * G * d * 2 + T * H * d * 4),
        "head_mix_gate": L * T * H * d * (2 * G + 4 + 2),
        "add_group_rmsnorm": (2 * L + 2) * T * W * 14,
        "group_rmsnorm": T * W * 6,
        "poly_norm": n_dense * T * ff * 6,
        "moe_route": n_moe * T * (z["experts"] * 4 + z["top"] * 8),
        "moe_plan": n_moe * P * 12,
        "moe_linear": (n_moe * (used * 3 * eff * W * 2 + P * (2 * W + 4 * eff + 4 * W)), n_moe * 6 * P * eff * W),
        "moe_combine": n_moe * T * W * (4 * z["top"] + 8),
    }


def compare_pimodra(args) -> dict:
    return compare_models(args, "pimodra", PIMODRA_SIZES, lambda z: (("pimodra", pimodra_config(z), pimodra_op_bytes),
                                                                      ("gemma2", gemma_twin_config(z), gemma_op_bytes)))


# ---- Nukelix beside Petanex at equal layer sizes (--compare nukelix) ---------------------------------------------------
# Eight layers in both.  Nukelix: windowed attention with kept first tokens, two layers of attention beside a matrix
# memory, latent attention with a shared rotated key part, twice; every feed-forward a mixture whose chosen experts and
# shared expert together have the dense width.  Petanex (the closest existing model: attention over a latent, a 32-bit
# recurrence with a d x dv state per head, mixtures with a shared expert) as in --compare petanex.  Same width, heads,
# head size, state size per head, experts and vocabulary.
NUKELIX_SIZES = {
    "w2048": dict(PETANEX_SIZES["w2048"], q_rank=512, kv_rank=192, rot_dim=64, window=1024, keep_first=64),
    "w4096": dict(PETANEX_SIZES["w4096"], q_rank=1024, kv_rank=192, rot_dim=64, window=1024, keep_first=64),
}


def nukelix_config(z: dict) -> dict:
    d = z["dim"]
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "v_mix": True,
           "mask": {"size": z["window"], "keep_first": z["keep_first"]},
           "rot": {"base": 500000.0, "dims": d // 2, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    left = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5,
            "rot": {"base": 10000.0, "dims": d}}
    par = {"left": left, "left_scale": 0.7, "right_scale": 1.2,
           "right": {"heads": z["d_heads"], "dim": z["d_dim"], "vdim": z["d_vdim"], "gate_cap": 15.0}}
    lat = {"heads": z["lat_heads"], "dim": d, "rot_dim": z["rot_dim"], "vdim": d, "kv_rank": z["kv_rank"], "q_rank": z["q_rank"],
           "scale": (d + z["rot_dim"]) ** -0.5,
           "rot": {"base": 10000.0, "dims": z["rot_dim"], "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    eff = z["ff"] // (z["top"] + 1) // 64 * 64
    moe = {"kind": "moe", "expert": {"ff": eff}, "shared": {"ff": eff}, "router": {"experts": z["experts"], "top": z["top"]}}
    kinds = ["attention", "parallel", "parallel", "latent_attention"]
    layers = [{"type": kinds[i % 4], "mixer": (att, par, par, lat)[i % 4], "mlp": moe} for i in range(COMPARE_LAYERS)]
    return {"architecture": "Nukelix", "width": z["width"], "vocab": COMPARE_VOCAB, "norm": {"eps": 1e-6},
            "logit_softcap": 50.0, "layers": layers}


def nukelix_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    """Bytes (and, for the grouped products, floating-point operations) each operation of one Nukelix step must move,
    summed over the layers that use it."""
    W, H, G, d, L = z["width"], z["heads"], z["kv_heads"], z["dim"], COMPARE_LAYERS
    n_att, n_par, n_lat = L // 4, L // 2, L // 4
    cq = (H + 2 * G) * d
    mh, md, mv = z["d_heads"], z["d_dim"], z["d_vdim"]
    lh, rank, rd = z["lat_heads"], z["kv_rank"], z["rot_dim"]
    D = 256 if rank + rd > 128 else 128
    seen = min(keys, z["window"] + z["keep_first"])
    eff = z["ff"] // (z["top"] + 1) // 64 * 64
    P = T * z["top"]
    used = min(z["experts"], P)
    return {
        "rownorm_rope_append": (n_att + n_par) * T * (4 * cq + 2 * cq + 4 * d),
        "paged_attention": n_att * (n_reqs * seen * 2 * G * d * 2 + T * H * d * 4) + n_par * (n_reqs * keys * 2 * G * d * 2 + T * H * d * 4)
                           + n_lat * (n_reqs * keys * 2 * D * 2 + T * lh * D * 4),
        "head_gate": (n_att + n_par + n_lat) * T * H * d * 4,
        "mlstm": n_par * (T * mh * (2 * md + 2 * mv) * 4 + 2 * n_reqs * mh * md * mv * 4),
        "head_norm_gate": n_par * T * mh * mv * 10,
        "weighted_sum2": n_par * T * W * 12,
        "latent_rope_append": n_lat * T * ((rank + rd) * 4 + 4 * D + lh * rd * 8),
        "cols_rmsnorm": n_lat * T * z["q_rank"] * 6,
        "head_linear": (n_lat * T * lh * (4 * (d + rd) + 2 * D + 2 * D + 2 * d), n_lat * 2 * T * lh * (D * (d + rd) + d * D)),
        "add_rmsnorm": 2 * L * T * W * 14,
        "moe_route": L * T * (z["experts"] * 4 + z["top"] * 8),
        "moe_plan": L * P * 12,
        "moe_linear": (L * (used * 3 * eff * W * 2 + P * (2 * W + 4 * eff + 4 * W)), L * 6 * P * eff * W),
        "moe_combine": L * T * W * (4 * z["top"] + 8),
    }


def compare_nukelix(args) -> dict:
    return compare_models(args, "nukelix", NUKELIX_SIZES, lambda z: (("nukelix", nukelix_config(z), nukelix_op_bytes),
                                                                      ("petanex", petanex_config(z), petanex_op_bytes)))


# ---- Lurisun beside Nukelix at equal layer sizes (--compare lurisun) ---------------------------------------------------
# Eight layers in both.  Lurisun: latent attention, linear attention with fixed decays, sigmoid attention over chunks, linear
# attention, twice; every feed-forward dense.  Nukelix (the closest existing model: blocks that read the residual stream,
# row-normed attention, attention over a latent with queries through their own, a 32-bit memory with a d x dv state per
# head) as in --compare nukelix.  Same width, heads, head size, state size per head, latents, reach of the attention and
# vocabulary; Nukelix's chosen and shared experts together have the dense feed-forward's width.
LURISUN_SIZES = {name: dict(z) for name, z in NUKELIX_SIZES.items()}


def lurisun_config(z: dict) -> dict:
    d, h = z["dim"], z["d_heads"]
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": z["window"]},
           "rot": {"base": 500000.0, "dims": d // 2}}
    lig = {"heads": h, "dim": z["d_dim"], "vdim": z["d_vdim"], "decay": [1.0 - 2.0 ** -(2.0 + 6.0 * i / h) for i in range(h)]}
    lat = {"heads": z["lat_heads"], "dim": d, "vdim": d, "kv_rank": z["kv_rank"], "q_rank": z["q_rank"], "scale": d ** -0.5,
           "mask": {"size": z["window"]}}
    kinds = ["latent_attention", "lightning", "attention", "lightning"]
    layers = [{"type": kinds[i % 4], "mixer": (lat, lig, att, lig)[i % 4], "mlp": {"kind": "dense", "ff": z["ff"]}}
              for i in range(COMPARE_LAYERS)]
    return {"architecture": "Lurisun", "width": z["width"], "vocab": COMPARE_VOCAB, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "canon": {"taps": 4}, "embedding": {"bigram": {"mul_prev": 1009, "mul_cur": 1, "buckets": COMPARE_VOCAB}}, "layers": layers}


def lurisun_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    """Bytes (and, for the products, floating-point operations) each operation of one Lurisun step must move, summed over
    the layers that use it; a prompt's attention also has the multiply-adds of the keys its rows see."""
    W, H, G, d, L = z["width"], z["heads"], z["kv_heads"], z["dim"], COMPARE_LAYERS
    n_att, n_lat, n_lig = L // 4, L // 4, L // 2
    mh, md, mv = z["d_heads"], z["d_dim"], z["d_vdim"]
    lh, rank = z["lat_heads"], z["kv_rank"]
    D = 256 if rank > 128 else 128
    seen = min(keys, z["window"])
    single = T == n_reqs
    cq = (H + G) * d
    # query-key pairs of a prompt: chunks of `window`, and a sliding window
    pairs_c = sum(i % z["window"] + 1 for i in range(T)) if not single else n_reqs * seen
    pairs_w = sum(min(i + 1, z["window"]) for i in range(T)) if not single else n_reqs * seen
    return {
        "embed_pair": T * W * 8,
        "input_conv": L * T * W * 6,
        "add_rmsnorm_conv": L * T * W * 14,
        "rownorm_rope_append": n_att * T * (4 * cq + 2 * (cq + G * d) + 4 * d),
        "paged_attention": (n_att * (n_reqs * seen * 2 * G * d * 2 + T * H * d * 4) + n_lat * (n_reqs * seen * 2 * D * 2 + T * lh * D * 4),
                            n_att * 4 * H * d * pairs_c + n_lat * 4 * lh * D * pairs_w),
        "decay_memory": n_lig * (T * mh * (2 * md + mv) * (4 if single else 2) + T * mh * mv * 4 + 2 * n_reqs * mh * md * mv * 4),
        "head_norm_gate": n_lig * T * mh * mv * 10,
        "latent_norms_append": n_lat * T * (rank * 4 + 4 * D + z["q_rank"] * 6),
        "head_linear": (n_lat * T * lh * (4 * d + 2 * D + 2 * D + 2 * d), n_lat * 4 * T * lh * D * d),
        "element_gate": n_lat * T * lh * d * 8,
        "add_rmsnorm": (L if single else 2 * L) * T * W * 14,
        "linear_gated": (L * (2 * z["ff"] * W * 2 + T * (2 * W + 2 * z["ff"])), L * 4 * T * z["ff"] * W),
    }


def compare_lurisun(args) -> dict:
    return compare_models(args, "lurisun", LURISUN_SIZES, lambda z: (("lurisun", lurisun_config(z), lurisun_op_bytes),
                                                                      ("nukelix", nukelix_config(z), nukelix_op_bytes)))


# ---- Fovosun beside Petanex, Lurisun and Bolonex at equal layer sizes (--compare fovosun) ------------------------------
# Eight layers in all four.  Fovosun: differential attention with a convolution and a temperature, differential attention
# over a window, two retention layers, twice; feed-forwards alternate between dense and a mixture as in Petanex, the closest
# existing model as a whole; four residual streams.  A head's two maps of dim / 2 have the width of one ordinary head.
# Lurisun has the like of retention (the same memory with a d x dv state per head), Bolonex the like of the first attention
# (grouped-query attention behind a convolution over q, k and v).
FOVOSUN_SIZES = {name: dict(z, window=LURISUN_SIZES[name]["window"], q_rank=LURISUN_SIZES[name]["q_rank"],
                            kv_rank=LURISUN_SIZES[name]["kv_rank"], streams=4) for name, z in PETANEX_SIZES.items()}


def fovosun_config(z: dict) -> dict:
    d, h = z["dim"], z["d_heads"]
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": d // 2, "vdim": d, "scale": (d // 2) ** -0.5, "diff": 0.5,
           "conv": 4, "q_temp": {"coef": 0.1, "every": 1024}}
    win = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": d // 2, "vdim": d, "scale": (d // 2) ** -0.5, "diff": 0.5,
           "mask": {"size": z["window"]}, "rot": {"base": 10000.0, "dims": d // 2}}
    ret = {"heads": h, "dim": z["d_dim"], "vdim": z["d_vdim"], "decay": [1.0 - 2.0 ** -(2.0 + 6.0 * i / h) for i in range(h)],
           "rot": {"base": 10000.0, "dims": z["d_dim"]}}
    eff = z["ff"] // (z["top"] + 1) // 64 * 64
    dense = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": eff, "limit": 7.0}, "shared": {"ff": eff, "limit": 7.0},
           "router": {"experts": z["experts"], "top": z["top"]}}
    kinds = ["attention", "attention_2", "retention", "retention"]
    layers = [{"type": kinds[i % 4], "mixer": (att, win, ret, ret)[i % 4], "mlp": dense if i % 2 == 0 else moe}
              for i in range(COMPARE_LAYERS)]
    return {"architecture": "Fovosun", "width": z["width"], "vocab": COMPARE_VOCAB, "streams": z["streams"],
            "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "layers": layers}


def fovosun_op_bytes(z: dict, T: int, n_reqs: int, keys: int) -> dict:
    """Bytes (and, for the products, floating-point operations) each operation of one Fovosun step must move, summed over
    the layers that use it; a prompt's attention also has the multiply-adds of the keys its rows see, those of the zero
    halves of its query rows not counted."""
    W, H, G, dv, L, n = z["width"], z["heads"], z["kv_heads"], z["dim"], COMPARE_LAYERS, z["streams"]
    d = dv // 2
    n_full, n_win, n_ret, n_moe = L // 4, L // 4, L // 2, L // 2
    mh, md, mv = z["d_heads"], z["d_dim"], z["d_vdim"]
    single = T == n_reqs
    cq = 2 * (H + G) * d + G * dv
    seen = min(keys, z["window"])
    pairs = n_reqs * keys if single else T * (T + 1) // 2
    pairs_w = n_reqs * seen if single else sum(min(i + 1, z["window"]) for i in range(T))
    eff = z["ff"] // (z["top"] + 1) // 64 * 64
    P = T * z["top"]
    used = min(z["experts"], P)
    return {
        "embed": T * W * (2 + 4 * n),
        "streams_step": 2 * L * T * W * (8 * n + 6),
        "streams_norm": T * W * (4 * n + 2) + n_reqs * W * (4 * n + 2),
        "qkv_prepare": (n_full + n_win) * T * 6 * cq + n_win * T * 4 * d,
        "short_conv_commit": n_full * n_reqs * 3 * cq * 8,
        "paged_attention": ((n_full * keys + n_win * seen) * n_reqs * G * (2 * d + dv) * 2 + (n_full + n_win) * T * H * (2 * d + 2 * dv) * 2,
                            4 * H * (d + dv) * (n_full * pairs + n_win * pairs_w)),
        "diff_combine": (n_full + n_win) * T * H * dv * 6,
        "decay_rotate": n_ret * T * (mh * (2 * md + mv) * 6 + 4 * md),
        "decay_memory": n_ret * (T * mh * (2 * md + mv) * (4 if single else 2) + T * mh * mv * 4 + 2 * n_reqs * mh * md * mv * 4),
        "head_norm_gate": n_ret * T * mh * mv * 10,
        "linear_gated": ((L - n_moe) * (2 * z["ff"] * W * 2 + T * (2 * W + 2 * z["ff"])) + n_moe * (2 * eff * W * 2 + T * (2 * W + 2 * eff)),
                         4 * T * W * ((L - n_moe) * z["ff"] + n_moe * eff)),
        "moe_route": n_moe * T * (z["experts"] * 4 + z["top"] * 8),
        "moe_plan": n_moe * P * 12,
        "moe_linear": (n_moe * (used * 3 * eff * W * 2 + P * (2 * W + 4 * eff + 4 * W)), n_moe * 6 * P * eff * W),
        "moe_combine": n_moe * T * W * (4 * z["top"] + 8),
    }


def compare_fovosun(args) -> dict:
    return compare_models(args, "fovosun", FOVOSUN_SIZES, lambda z: (
        ("fovosun", fovosun_config(z), fovosun_op_bytes), ("petanex", petanex_config(z), petanex_op_bytes),
        ("lurisun", lurisun_config(z), lurisun_op_bytes), ("bolonex", bolonex_config(z), bolonex_op_bytes)))


def micro_attention() -> int:
    """Decode attention alone: eight launches over distinct pages replayed from a CUDA graph, per batch size; one JSON
    line each with microseconds per launch and bytes of keys and values over that time."""
    import torch
    from kungfu_b200 import api, ops

    class View:
        def __init__(self, pages, page_size):
            self.pages, self.page_size, self.group, self.writes = pages, page_size, 0, False

    class Ctx:
        pass

    device = api.require_cuda("cuda:0")
    ops.library()
    nh, nkv, d, page, ctx_len, launches = 8, 4, 256, 64, 8192, 8
    for batch in (1, 2, 4, 8, 16, 64):
        per_req = ctx_len // page
        pages = torch.randn(launches * batch * per_req + 1, 2, nkv, page, d, device=device, dtype=torch.bfloat16)
        ctxs = []
        for l in range(launches):
            c = Ctx()
            c.positions = torch.full((batch,), ctx_len - 1, dtype=torch.int32, device=device)
            c.row_req = torch.arange(batch, dtype=torch.int32, device=device)
            c.block_tables = [(torch.arange(batch * per_req, dtype=torch.int32, device=device) + l * batch * per_req)
                              .view(batch, per_req).contiguous()]
            c.n_rows = c.n_dec_rows = batch
            c.n_pre_rows = c.n_tiles = c.n_wide = 0
            c.dec_rows = c.pre_rows = None
            c.max_kv_len = ctx_len
            ctxs.append(c)
        q = torch.randn(batch, nh * d, device=device, dtype=torch.bfloat16)
        out = torch.empty_like(q)
        view = View(pages, page)
        for window in (None, 4096):
            def run():
                for c in ctxs:
                    ops.paged_attention(q, out, c, view, nh, nkv, d, 1.0 / 16.0, 50.0, window)
            run()
            torch.cuda.synchronize()
            graph, side = torch.cuda.CUDAGraph(), torch.cuda.Stream()
            with torch.cuda.stream(side):
                run()
                with torch.cuda.graph(graph, stream=side):
                    run()
            torch.cuda.synchronize()
            for _ in range(3):
                graph.replay()
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            for _ in range(10):
                graph.replay()
            e1.record()
            torch.cuda.synchronize()
            us = e0.elapsed_time(e1) / 10 / launches * 1e3
            n_bytes = batch * min(ctx_len, window or ctx_len) * nkv * d * 2 * 2
            print(json.dumps({"micro": "decode attention", "batch": batch, "keys": min(ctx_len, window or ctx_len),
                              "us_per_launch": round(us, 1), "gb_per_s": round(n_bytes / us / 1e3, 1)}))
        del pages
    return 0


def micro_prompt_attention() -> int:
    """Prompt attention alone (8 heads / 4 kv heads of 256, softcap 50, page 64): whole prompts of 512 to 4,096 rows and a
    512-row portion at context 8,192, each replayed from a CUDA graph of three launches over distinct pages; one JSON line
    each with microseconds per launch and TFLOP/s."""
    import math
    import torch
    from kungfu_b200 import api, ops

    class View:
        def __init__(self, pages, page_size):
            self.pages, self.page_size, self.group, self.writes = pages, page_size, 0, False

    class Ctx:
        pass

    device = api.require_cuda("cuda:0")
    ops.library()
    gen = torch.Generator(device=device)
    gen.manual_seed(0)
    nh, nkv, d, page, copies = 8, 4, 256, 64, 3
    scale = 1.0 / math.sqrt(d)
    for T, past in ((512, 0), (1024, 0), (2048, 0), (4096, 0), (512, 7680)):
        total = T + past
        per_req = total // page
        pages = torch.empty(copies * per_req, 2, nkv, page, d, device=device, dtype=torch.bfloat16).normal_(0.0, 0.5, generator=gen)
        ctxs = []
        for k in range(copies):
            c = Ctx()
            c.positions = torch.arange(past, total, dtype=torch.int32, device=device)
            c.row_req = torch.zeros(T, dtype=torch.int32, device=device)
            c.block_tables = [(torch.arange(per_req, dtype=torch.int32, device=device) + k * per_req).view(1, per_req).contiguous()]
            c.n_rows = c.n_pre_rows = T
            c.n_dec_rows = 0
            c.dec_rows = None
            c.pre_rows = torch.arange(T, dtype=torch.int32, device=device)
            c.n_tiles, c.n_wide = T // 64, T // 128
            c.tile_row0 = torch.arange(0, T, 64, dtype=torch.int32, device=device)
            c.tile_nrows = torch.full((T // 64,), 64, dtype=torch.int32, device=device)
            c.wide_row0 = torch.arange(0, T, 128, dtype=torch.int32, device=device)
            c.wide_nrows = torch.full((T // 128,), 128, dtype=torch.int32, device=device)
            c.max_kv_len = total
            ctxs.append(c)
        q = torch.randn(T, nh * d, device=device, generator=gen).to(torch.bfloat16)
        out = torch.empty_like(q)
        view = View(pages, page)
        us = _graph_us(torch, lambda: [ops.paged_attention(q, out, c, view, nh, nkv, d, scale, 50.0, None) for c in ctxs], copies)
        flops = 4.0 * nh * d * (T * (T + 1) / 2 + T * past)
        print(json.dumps({"micro": "prompt attention", "rows": T, "keys_before": past, "us_per_launch": round(us, 1),
                          "tflops": round(flops / us / 1e6, 1)}), flush=True)
        del pages
    ops.raise_on_device_error()
    return 0


def micro_memory() -> int:
    """The matrix memory's walk alone (gates and walk, `ops.mlstm`) over one prompt of 2,048 rows and over 8 single rows, at
    16 heads of 128 x 128, timed with CUDA events; one JSON line per case with microseconds and the bytes it must move."""
    import types
    import torch
    from kungfu_b200 import api, ops
    device = api.require_cuda("cuda:0")
    ops.library()
    H, d, dv = 16, 128, 128
    width = 2 * H * d + 2 * H * dv + 2 * H
    for rows, reqs in ((2048, 1), (8, 8)):
        per = rows // reqs
        proj = torch.randn(rows, width, device=device)
        bufs = {}
        ctx = types.SimpleNamespace(
            n_reqs=reqs, req_row_start=torch.arange(0, rows, per, dtype=torch.int32, device=device),
            req_n_rows=torch.full((reqs,), per, dtype=torch.int32, device=device),
            req_state_slot=torch.arange(reqs, dtype=torch.int32, device=device),
            buf=lambda tag, shape, dt: bufs.setdefault(tag, torch.empty(shape, dtype=dt, device=device)))
        memory = torch.zeros(reqs, H, d, dv, device=device)
        norm_state = torch.zeros(reqs, H, ops.mlstm_norm_width(d, dv), device=device)
        bias = torch.zeros(H, device=device, dtype=torch.bfloat16)
        out = torch.empty(rows, H * dv, device=device)
        run = lambda: ops.mlstm(proj, 0, H * d, 2 * H * d, 2 * H * d + 2 * H * dv, 2 * H * d + 2 * H * dv + H, bias, bias + 4.0, 15.0,
                                memory, norm_state, out, H, d, dv, ctx)
        for _ in range(3):
            run()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(5):
            run()
        e1.record()
        torch.cuda.synchronize()
        nbytes = rows * H * (2 * d + 2 * dv) * 4 + 2 * reqs * H * d * dv * 4
        print(json.dumps({"micro": "matrix memory", "rows": rows, "requests": reqs, "heads": H, "dim": d, "vdim": dv,
                          "us": round(e0.elapsed_time(e1) / 5 * 1e3, 1), "bytes": nbytes}), flush=True)
    ops.raise_on_device_error()
    return 0


def micro_gemm() -> int:
    """One square bfloat16 product (8192 cubed) on the tensor-core kernel, timed with CUDA events; one JSON line."""
    import torch
    from kungfu_b200 import api, ops
    device = api.require_cuda("cuda:0")
    n = 8192
    x = torch.randn(n, n, device=device).bfloat16()
    w = torch.randn(n, n, device=device).bfloat16()
    out = torch.empty(n, n, device=device)
    for _ in range(3):
        ops.linear(x, w, out)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(5):
        ops.linear(x, w, out)
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / 5
    ops.raise_on_device_error()
    print(json.dumps({"micro": "product 8192^3 bf16", "ms": round(ms, 4), "tflops": round(2.0 * n ** 3 / ms / 1e9, 1)}))
    return 0


def micro_products(size: str = "2b") -> int:
    """The four products of a Gemma 2 layer (`--size`) over 8 to 2,048 rows, each replayed from a CUDA graph of six
    launches over distinct weights; one JSON line per (rows, product) with microseconds per launch."""
    import torch
    from kungfu_b200 import api, ops
    device = api.require_cuda("cuda:0")
    ops.library()
    sz = SIZES[size]
    H, inner, n_w = sz["hidden_size"], sz["intermediate_size"], 6
    Q = sz["num_attention_heads"] * sz["head_dim"]
    qkv = Q + 2 * sz["num_key_value_heads"] * sz["head_dim"]
    gen = torch.Generator(device=device)
    gen.manual_seed(0)
    shapes = {"q,k,v": (qkv, H, False), "o": (H, Q, False), "gate+up": (inner, H, True), "down": (H, inner, False)}
    for rows in (8, 64, 128, 256, 384, 512, 768, 1024, 2048):
        for name, (n_out, k, gated) in shapes.items():
            ws = [(torch.randn(2 * n_out if gated else n_out, k, device=device, generator=gen) * 0.02).to(torch.bfloat16)
                  for _ in range(n_w)]
            x = torch.randn(rows, k, device=device).to(torch.bfloat16)
            out = torch.empty(rows, n_out, device=device, dtype=torch.bfloat16 if gated else torch.float32)

            def run():
                for w in ws:
                    if gated:
                        ops.linear_gated(x, w, out, "gelu_tanh", None)
                    else:
                        ops.linear(x, w, out)
            run()
            torch.cuda.synchronize()
            graph, side = torch.cuda.CUDAGraph(), torch.cuda.Stream()
            with torch.cuda.stream(side):
                run()
                with torch.cuda.graph(graph, stream=side):
                    run()
            torch.cuda.synchronize()
            for _ in range(3):
                graph.replay()
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            for _ in range(10):
                graph.replay()
            e1.record()
            torch.cuda.synchronize()
            us = e0.elapsed_time(e1) / 10 / n_w * 1e3
            flops = 2.0 * rows * n_out * k * (2 if gated else 1)
            print(json.dumps({"micro": "product", "size": size, "rows": rows, "product": name, "us": round(us, 1),
                              "tflops": round(flops / us / 1e6, 1)}))
            del ws
    ops.raise_on_device_error()
    return 0


def micro_qkv_rope(size: str = "2b") -> int:
    """The q,k,v product of a prompt with rotation and cache append: the product that files its own result
    (`ops.linear_rope_kv_append`) beside the product that leaves 32-bit rows plus the kernel that rotates and files them;
    four launches over distinct weights and pages replayed from a CUDA graph, one JSON line per row count."""
    import torch
    from kungfu_b200 import api, ops
    device = api.require_cuda("cuda:0")
    ops.library()
    sz = SIZES[size]
    nh, nkv, d, K, P, n_w = sz["num_attention_heads"], sz["num_key_value_heads"], sz["head_dim"], sz["hidden_size"], 64, 4
    N = (nh + 2 * nkv) * d

    class View:
        def __init__(self, pages):
            self.pages, self.page_size, self.group, self.writes = pages, P, 0, True

    class Ctx:
        pass
    for rows in (768, 1024, 2048, 4096):
        ws = [(torch.randn(N, K, device=device) * 0.02).to(torch.bfloat16) for _ in range(n_w)]
        x = torch.randn(rows, K, device=device).to(torch.bfloat16)
        n_pages = -(-rows // P)
        ctx = Ctx()
        ctx.positions = torch.arange(rows, dtype=torch.int32, device=device)
        ctx.row_req = torch.zeros(rows, dtype=torch.int32, device=device)
        ctx.block_tables = [torch.arange(n_pages, dtype=torch.int32, device=device)[None, :].contiguous()]
        views = [View(torch.zeros(n_pages, 2, nkv, P, d, dtype=torch.bfloat16, device=device)) for _ in range(n_w)]
        inv = (10000.0 ** (-2.0 * torch.arange(d // 2, dtype=torch.float64) / d)).float().to(device)
        ang = ctx.positions.float()[:, None] * inv[None, :]
        cos, sin = torch.cos(ang).contiguous(), torch.sin(ang).contiguous()
        q = torch.empty(rows, nh * d, dtype=torch.bfloat16, device=device)
        qkv = torch.empty(rows, N, device=device)
        line = {"micro": "qkv-rope", "size": size, "rows": rows}

        def two():
            for w, v in zip(ws, views):
                ops.linear(x, w, qkv)
                ops.rope_kv_append(qkv, cos, sin, d, nh, nkv, d, ctx, v, q)

        def fused():
            for w, v in zip(ws, views):
                if not ops.linear_rope_kv_append(x, w, cos, sin, d, nh, nkv, d, ctx, v, q):
                    raise RuntimeError("declined")
        line["two_kernels_us"] = round(_graph_us(torch, two, n_w), 1)
        try:
            line["fused_us"] = round(_graph_us(torch, fused, n_w), 1)
        except RuntimeError:
            line["fused_us"] = None                       # this shape keeps the two-kernel path (head size 128)
        print(json.dumps(line))
        del ws, views
    ops.raise_on_device_error()
    return 0


def _graph_us(torch, run, n_launches: int, reps: int = 10) -> float:
    """Microseconds per launch of `run()` (which issues `n_launches` kernels) replayed from a CUDA graph."""
    run()
    torch.cuda.synchronize()
    graph, side = torch.cuda.CUDAGraph(), torch.cuda.Stream()
    with torch.cuda.stream(side):
        run()
        with torch.cuda.graph(graph, stream=side):
            run()
    torch.cuda.synchronize()
    for _ in range(3):
        graph.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps / n_launches * 1e3


def micro_reference() -> int:
    """The reference's own kernels (compiled unchanged, kungfu_b200/measure/reference_kernels.py) beside this engine's
    kernels on the same device and shapes: prompt attention over 2,048 rows, decode attention over 8 x 8,192 keys, the
    products of a Gemma 2 2B layer at 8 and 2,048 rows, the norm with residual.  Every case is replayed from a CUDA graph
    over several copies of its operands (more than the L2 holds), timed with CUDA events; one JSON line per case with
    microseconds per launch for both and their ratio.  The reference's kernels read 32-bit activations and a
    half-precision ring cache; this engine's read bfloat16 activations and pages."""
    import math
    import torch
    from kungfu_b200 import api, ops
    from kungfu_b200.measure import reference_kernels as rk
    device = api.require_cuda("cuda:0")
    ops.library()
    ref = rk.Reference()
    gen = torch.Generator(device=device)
    gen.manual_seed(0)

    class View:
        def __init__(self, pages, page_size):
            self.pages, self.page_size, self.group, self.writes = pages, page_size, 0, False

    class Ctx:
        pass

    def emit(case, us_ref, us_ours, note=""):
        print(json.dumps({"micro": "reference", "case": case, "reference_us": round(us_ref, 1), "ours_us": round(us_ours, 1),
                          "speedup": round(us_ref / us_ours, 2), "note": note}), flush=True)

    # ---- products: one row block against n_w copies of the weight -------------------------------------------------------
    H, Q, inner = 2304, 2048, 9216
    for rows in (8, 2048):
        for name, n_out, k in (("q,k,v", 4096, H), ("o", H, Q), ("gate or up", inner, H), ("down", H, inner)):
            n_w = max(2, int(300e6 // (n_out * k * 2)))
            ws = [(torch.randn(n_out, k, device=device, generator=gen) * 0.02).to(torch.bfloat16) for _ in range(n_w)]
            x32 = torch.randn(rows, k, device=device, generator=gen).to(torch.bfloat16).float()
            x16 = x32.to(torch.bfloat16)
            out = torch.empty(rows, n_out, device=device)
            us_ref = _graph_us(torch, lambda: [ref.linear_bf16(w, x32) for w in ws], n_w, reps=3 if rows > 8 else 10)
            us_ours = _graph_us(torch, lambda: [ops.linear(x16, w, out) for w in ws], n_w)
            emit(f"product {name} [{n_out} x {k}] x {rows} rows", us_ref, us_ours,
                 "reference: matvec (one warp per output)" if rows <= 8 else "reference: 32 x 64 x 64 tiles of 32-bit FMA")
            del ws
    # ---- norm with residual ------------------------------------------------------------------------------------------------
    for rows in (8, 2048):
        n_c = 16 if rows > 8 else 2
        xs = [torch.randn(rows, H, device=device, generator=gen) for _ in range(n_c)]
        res = [torch.randn(rows, H, device=device, generator=gen) for _ in range(n_c)]
        w32 = torch.randn(H, device=device, generator=gen) * 0.1
        w16 = w32.to(torch.bfloat16)
        us_ref = _graph_us(torch, lambda: [ref.rms_norm_add(x, w32, r, 1e-6) for x, r in zip(xs, res)], n_c)
        us_ours = _graph_us(torch, lambda: [ops.add_rmsnorm(x, w16, 1e-6, True, r) for x, r in zip(xs, res)], n_c)
        emit(f"norm + residual, {rows} rows x {H}", us_ref, us_ours)
    # ---- decode attention: 8 requests x 8,192 keys, heads 8/4 x 256 (Gemma 2 2B) and 32/16 x 128 (27B) -----------------------
    for nh, nkv, d in ((8, 4, 256), (32, 16, 128)):
        batch, keys, page, copies = 8, 8192, 64, 3
        scale = 1.0 / math.sqrt(d)
        caches = [ref.make_cache(batch, keys, nkv * d, device) for _ in range(copies)]
        for kc, vc in caches:
            kc.normal_(0.0, 0.5, generator=gen)
            vc.normal_(0.0, 0.5, generator=gen)
        q32 = torch.randn(batch, nh * d, device=device, generator=gen)
        pos = torch.full((batch,), keys - 1, dtype=torch.int32, device=device)
        seq = torch.arange(batch, dtype=torch.int32, device=device)
        us_ref = _graph_us(torch, lambda: [ref.attention_decode(q32, kc, vc, pos, seq, nh, nkv, d, scale, None, 50.0) for kc, vc in caches], copies)
        per_req = keys // page
        pages = torch.empty(copies * batch * per_req, 2, nkv, page, d, device=device, dtype=torch.bfloat16).normal_(0.0, 0.5, generator=gen)
        ctxs = []
        for c_i in range(copies):
            c = Ctx()
            c.positions, c.row_req = pos, seq
            c.block_tables = [(torch.arange(batch * per_req, dtype=torch.int32, device=device) + c_i * batch * per_req).view(batch, per_req).contiguous()]
            c.n_rows = c.n_dec_rows = batch
            c.n_pre_rows = c.n_tiles = c.n_wide = 0
            c.dec_rows = c.pre_rows = None
            c.max_kv_len = keys
            ctxs.append(c)
        q16 = q32.to(torch.bfloat16)
        o16 = torch.empty_like(q16)
        view = View(pages, page)
        us_ours = _graph_us(torch, lambda: [ops.paged_attention(q16, o16, c, view, nh, nkv, d, scale, 50.0, None) for c in ctxs], copies)
        n_bytes = batch * keys * nkv * d * 2 * 2
        emit(f"decode attention, {batch} x {keys} keys, heads {nh}/{nkv} x {d}", us_ref, us_ours,
             f"keys and values {n_bytes / 1e6:.0f} MB: reference {n_bytes / us_ref / 1e3:.0f} GB/s, ours {n_bytes / us_ours / 1e3:.0f} GB/s")
        del caches, pages
    # ---- prompt attention: one prompt of 2,048 rows ---------------------------------------------------------------------------
    for nh, nkv, d in ((8, 4, 256), (32, 16, 128)):
        T, page, copies = 2048, 64, 4
        scale = 1.0 / math.sqrt(d)
        pos = torch.arange(T, dtype=torch.int32, device=device)
        seq0 = torch.zeros(T, dtype=torch.int32, device=device)
        caches = [ref.make_cache(1, T, nkv * d, device) for _ in range(copies)]
        for kc, vc in caches:
            kc.normal_(0.0, 0.5, generator=gen)
            vc.normal_(0.0, 0.5, generator=gen)
        q32 = torch.randn(T, nh * d, device=device, generator=gen)
        tiles = ref.flash_tiles(pos, [(0, 0, T)], device)
        us_ref = _graph_us(torch, lambda: [ref.flash_prefill(q32, kc, vc, pos, seq0, [(0, 0, T)], nh, nkv, d, scale, None, 50.0, tiles=tiles)
                                           for kc, vc in caches], copies, reps=5)
        per_req = T // page
        pages = torch.empty(copies * per_req, 2, nkv, page, d, device=device, dtype=torch.bfloat16).normal_(0.0, 0.5, generator=gen)
        ctxs = []
        for c_i in range(copies):
            c = Ctx()
            c.positions, c.row_req = pos, seq0
            c.block_tables = [(torch.arange(per_req, dtype=torch.int32, device=device) + c_i * per_req).view(1, per_req).contiguous()]
            c.n_rows = c.n_pre_rows = T
            c.n_dec_rows = 0
            c.dec_rows = None
            c.pre_rows = torch.arange(T, dtype=torch.int32, device=device)
            c.n_tiles, c.n_wide = T // 64, T // 128
            c.tile_row0 = torch.arange(0, T, 64, dtype=torch.int32, device=device)
            c.tile_nrows = torch.full((T // 64,), 64, dtype=torch.int32, device=device)
            c.wide_row0 = torch.arange(0, T, 128, dtype=torch.int32, device=device)
            c.wide_nrows = torch.full((T // 128,), 128, dtype=torch.int32, device=device)
            c.max_kv_len = T
            ctxs.append(c)
        q16 = q32.to(torch.bfloat16)
        o16 = torch.empty_like(q16)
        view = View(pages, page)
        us_ours = _graph_us(torch, lambda: [ops.paged_attention(q16, o16, c, view, nh, nkv, d, scale, 50.0, None) for c in ctxs], copies)
        flops = 4.0 * nh * d * T * (T + 1) / 2
        emit(f"prompt attention, {T} rows, heads {nh}/{nkv} x {d}", us_ref, us_ours,
             f"reference {flops / us_ref / 1e6:.0f} TFLOP/s, ours {flops / us_ours / 1e6:.0f} TFLOP/s")
        del caches, pages
    ops.raise_on_device_error()
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--reps", type=int, default=3, help="timed runs of --steps steps each; mean and sd are reported")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--size", default="2b", choices=sorted(SIZES))
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the size has (named in config)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=8192)
    ap.add_argument("--prefill-tokens", type=int, default=2048)
    ap.add_argument("--only-headline", action="store_true", help="skip the other batch sizes, the mixed steps, 32-bit and the other model sizes")
    ap.add_argument("--micro", choices=["attention", "prompt-attention", "gemm", "products", "qkv-rope", "reference", "memory"],
                    help="time kernels alone instead of the model step")
    ap.add_argument("--compare", choices=["bolonex", "petanex", "pimodra", "nukelix", "lurisun", "fovosun"],
                    help="another workload: Bolonex beside Gemma 2, Petanex beside Bolonex, Pimodra beside Gemma 2, Nukelix beside Petanex, Lurisun beside Nukelix, or "
                         "Fovosun beside Petanex, Lurisun and Bolonex, at equal "
                         "layer sizes (prefill, decode, per-operation rooflines)")
    args = ap.parse_args()
    if args.compare:
        args.warmup = max(args.warmup, 3)
        args.reps = max(args.reps, 1)
        print(json.dumps({"bolonex": compare_bolonex, "petanex": compare_petanex, "pimodra": compare_pimodra,
                          "nukelix": compare_nukelix, "lurisun": compare_lurisun, "fovosun": compare_fovosun}[args.compare](args)))
        return 0
    if args.micro:
        return {"attention": micro_attention, "prompt-attention": micro_prompt_attention, "gemm": micro_gemm,
                "products": lambda: micro_products(args.size), "qkv-rope": lambda: micro_qkv_rope(args.size),
                "reference": micro_reference, "memory": micro_memory}[args.micro]()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": "nickheyer/kungfu is a Rust workspace (no setup.py or "
                          "pyproject.toml; pip: 'not installable') and this image has no cargo/rustc and no network, so it cannot be built "
                          "(its CUDA kernels alone are timed by --micro reference)"}))
        return 0
    if args.gpus != 1 or int(os.environ.get("WORLD_SIZE", "1")) != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    args.warmup = max(args.warmup, 3)
    args.reps = max(args.reps, 1)
    print(json.dumps(run_ours(args)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
