"""Decode and prefill throughput of the engine at Qwen2.5-7B shape on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

One JSON line is printed.  A "step" is one decode step of the whole batch (forward,
sampling, the sampled tokens back on the host).  `value` is decoded tokens per second
at batch 8 and a context of 1,024 tokens, timed with CUDA events around exactly K
steps; `e2e` is the same measured through `LLMEngine.step()`, host token ids in and
out; `prefill` is one 2,048-token prompt in one step; `roofline` relates the bytes a
decode step must read (every weight once, the cache of the live requests) to its time;
`points` holds decoding at batch 1 and 64; `mixed` the scheduler end to end (64 requests of mixed
lengths at Qwen2.5-1.5B widths, `--workload mixed` alone).  Weights are random (seeded), token ids
uniform random: no checkpoint and no dataset is read.  Peaks come from
MEASURED_PEAKS.json beside this file when present, else from an earlier measurement
on the same GPU pool.  `--shape 14b --context 8192` (and the like) time the same
workload at other layer sizes and context lengths; the default line is the 7B one.
"""

from __future__ import annotations

import argparse
import json
import math
import os
import statistics
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

def _shapes() -> dict:
    """The layer sizes of the Qwen2.5 dense family, read from the package's shape files; the
    larger ones run with --layers (or in --case timeline)."""
    from shrike_b200.shapes import shape_config

    return {key: (f"Qwen2.5-{key.upper()} shape", shape_config(f"qwen2.5-{key}"))
            for key in ("0.5b", "1.5b", "3b", "7b", "14b", "32b", "72b")}


SHAPES = _shapes()
MODEL_7B = SHAPES["7b"][1]
MODEL_1_5B = SHAPES["1.5b"][1]
DEVICE_BYTES_LIMIT = 120e9   # weights and cache pool together stay under this, whatever the options
CONTEXT = 1024
PREFILL_TOKENS = 2048
BLOCK_SIZE = 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def load_peaks() -> dict:
    path = ROOT / "MEASURED_PEAKS.json"
    if path.is_file():
        try:
            raw = json.loads(path.read_text())
            flat = {}

            def walk(node):
                if isinstance(node, dict):
                    for key, value in node.items():
                        if isinstance(value, (int, float)) and key in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                            flat.setdefault(key, float(value))
                        else:
                            walk(value)
                elif isinstance(node, list):
                    for item in node:
                        walk(item)

            walk(raw)
            if "hbm_gbs" in flat and "bf16_tflops" in flat:
                flat["source"] = "measured"
                return flat
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self.process = None
        self.thread = None

    def start(self):
        try:
            self.process = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            return

        def read():
            for line in self.process.stdout:
                self.samples.append((time.perf_counter(), line.strip()))

        self.thread = threading.Thread(target=read, daemon=True)
        self.thread.start()

    def stop(self):
        if self.process is not None:
            self.process.terminate()
            try:
                self.process.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.process.kill()

    def summary(self, windows) -> dict:
        clocks, max_clock, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for stamp, line in self.samples:
            if not any(lo <= stamp <= hi for lo, hi in windows):
                continue
            fields = [f.strip() for f in line.split(",")]
            if len(fields) < 6:
                continue
            try:
                clocks.append(int(fields[0]))
                max_clock = max(max_clock, int(fields[1]))
            except ValueError:
                continue
            for name, flag in zip(names, fields[2:6]):
                if flag.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": int(statistics.median(clocks)) if clocks else None, "sm_max_mhz": max_clock or None,
                "reasons": sorted(reasons), "samples": len(clocks)}


def model_numbers(raw: dict, layers: int) -> dict:
    h, inter, v = raw["hidden_size"], raw["intermediate_size"], raw["vocab_size"]
    heads, kv, d = raw["num_attention_heads"], raw["num_key_value_heads"], raw["head_dim"]
    matrices = h * (heads + 2 * kv) * d + heads * d * h + 3 * h * inter
    vectors = (heads + 2 * kv) * d + 2 * h
    return dict(
        layer_matrix_params=matrices, layer_params=matrices + vectors, head_params=v * h,
        kv_bytes_per_token=layers * 2 * kv * d * 2,
        weight_bytes_per_step=2 * (layers * (matrices + vectors) + v * h + h),
    )


def decode_bytes(numbers: dict, batch: int, context: float) -> float:
    return numbers["weight_bytes_per_step"] + batch * context * numbers["kv_bytes_per_token"]


def prefill_flops(raw: dict, layers: int, tokens: int) -> float:
    numbers = model_numbers(raw, layers)
    heads, d = raw["num_attention_heads"], raw["head_dim"]
    linear = 2.0 * tokens * layers * numbers["layer_matrix_params"]
    attention = layers * 4.0 * heads * d * (tokens * (tokens + 1) / 2)
    head = 2.0 * raw["vocab_size"] * raw["hidden_size"]
    return linear + attention + head


def run_ours(args) -> dict:
    import numpy as np
    import torch

    import shrike_b200.models  # noqa: F401
    from shrike_b200 import SamplingParams
    from shrike_b200.config import parse_config
    from shrike_b200.engine.batch import StepEntry
    from shrike_b200.engine.llm_engine import LLMEngine
    from shrike_b200.weights.random_init import random_tensors

    torch.cuda.set_device(0)
    device = torch.device("cuda:0")
    shape_name, shape = SHAPES[args.shape]
    raw = dict(shape)
    context = args.context
    full_layers = raw["num_hidden_layers"]
    raw["num_hidden_layers"] = args.layers or full_layers
    layers = raw["num_hidden_layers"]
    config = parse_config(raw)
    numbers = model_numbers(raw, layers)
    if numbers["weight_bytes_per_step"] > 0.8 * DEVICE_BYTES_LIMIT:
        raise SystemExit(f"{shape_name} with {layers} layers holds {numbers['weight_bytes_per_step'] / 1e9:.0f} GB "
                         "of weights: give --layers")
    tensors = random_tensors(config, seed=0, device=device, dtype=torch.bfloat16)
    budget = 4096   # the engine's tokens per step: long prompts are cut, and finish their prefill steps apart
    spread = args.batch * -(-context // budget)   # steps from the first request's first token to the last one's
    pages_per_request = -(-(context + args.steps + args.warmup + 8 + spread) // BLOCK_SIZE)
    page_bytes = BLOCK_SIZE * numbers["kv_bytes_per_token"]
    large = 64   # the large batch of `points`: 64, or what the memory limit leaves at this shape and context
    while large > 1 and numbers["weight_bytes_per_step"] + large * pages_per_request * page_bytes > DEVICE_BYTES_LIMIT:
        large //= 2
    if args.batch > large:
        raise SystemExit(f"--batch {args.batch} at --context {context} needs more than {DEVICE_BYTES_LIMIT / 1e9:.0f} GB")
    pages = large * pages_per_request + -(-PREFILL_TOKENS // BLOCK_SIZE) + 64
    engine = LLMEngine(None, block_size=BLOCK_SIZE, num_blocks=pages, max_tokens_per_step=budget, max_running=64,
                       dtype="bfloat16", config=config, tensors=tensors)
    del tensors
    runner, ops = engine.runner, engine.ops
    rng = np.random.default_rng(0)
    vocab = raw["vocab_size"]
    peaks = load_peaks()
    sampler = ClockSampler()
    sampler.start()
    windows = []

    def fill(batch: int):
        """`batch` requests with context - 1 tokens in the cache (untimed)."""
        caches = []
        for _ in range(batch):
            cache = runner.cache.open()
            ids = rng.integers(0, vocab, context - 1).tolist()
            runner.cache.append(cache, 0, len(ids))
            runner.step([StepEntry(cache, ids, 0, [])])
            caches.append(cache)
        torch.cuda.synchronize()
        return caches

    def decode_run(batch: int, steps: int, warmup: int):
        """Device-timed decode through the step function and the sampling kernel."""
        caches = fill(batch)
        tokens = rng.integers(0, vocab, batch).tolist()
        fed = context - 1
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)

        def launch(fed, tokens=None):
            """Launches the step that feeds position `fed`.  Without tokens the step takes them on
            the device from what the step before it draws (id -1 - row), as the engine does in
            steady decoding: the host has not seen them yet."""
            entries = []
            for index, cache in enumerate(caches):
                runner.cache.append(cache, fed, 1)
                entries.append(StepEntry(cache, [tokens[index] if tokens else -1 - index], fed, [0], (0.0, 1.0, 0)))
            _logits, drawn = runner.step(entries, sample=True)
            return runner.fetch(drawn)

        def run(count, in_flight, fed):
            """`count` steps, one launched and one read back per round; the device never waits."""
            for _ in range(count):
                fed += 1
                following = launch(fed)
                runner.wait(in_flight)          # this step's tokens reach the host
                in_flight = following
            return in_flight, fed

        in_flight, fed = run(warmup - 1, launch(fed, tokens), fed)
        tokens = runner.wait(in_flight)
        torch.cuda.synchronize()
        launches_before = ops.launches
        t0 = time.perf_counter()
        start.record()
        fed += 1
        in_flight, fed = run(steps - 1, launch(fed, tokens), fed)   # `steps` launches ...
        runner.wait(in_flight)                                       # ... and `steps` read-backs
        stop.record()
        torch.cuda.synchronize()
        windows.append((t0, time.perf_counter()))
        ms = start.elapsed_time(stop) / steps
        launches = ops.launches - launches_before
        for cache in caches:
            runner.cache.free(cache)
        mean_context = context + warmup + (steps - 1) / 2.0
        return ms, launches, mean_context

    # ---- decode at the headline batch, device-timed -------------------------
    ms, launches, mean_context = decode_run(args.batch, args.steps, args.warmup)
    value = args.batch * 1000.0 / ms
    bytes_step = decode_bytes(numbers, args.batch, mean_context)
    achieved = bytes_step / (ms * 1e-3) / 1e9

    # ---- the same through the public entry point ------------------------------
    def e2e_run(batch: int, steps: int, warmup: int):
        prompts = [rng.integers(0, vocab, context - 1).tolist() for _ in range(batch)]
        # every request decodes through all timed steps, although the prompts finish their prefill steps apart
        params = SamplingParams(max_new_tokens=steps + warmup + 8 + spread, ignore_eos=True)
        for prompt in prompts:
            engine.add_request(prompt, params)
        while any(not r.prefill_done for r in engine.requests.values()) or engine.scheduler.waiting:
            engine.step()
        for _ in range(warmup):
            engine.step()
        torch.cuda.synchronize()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        copied = runner.builder.copied_bytes
        t0 = time.perf_counter()
        start.record()
        produced = 0
        for _ in range(steps):
            produced += len(engine.step())
        stop.record()
        torch.cuda.synchronize()
        windows.append((t0, time.perf_counter()))
        e2e_ms = start.elapsed_time(stop) / steps
        for req_id in list(engine.requests):
            engine.abort(req_id)
        assert engine.block_manager.whole()
        h2d = (runner.builder.copied_bytes - copied) // steps   # the packed metadata block of each step
        return produced / steps * 1000.0 / e2e_ms, h2d, 4 * batch

    e2e_value, h2d, d2h = e2e_run(args.batch, args.steps, args.warmup)

    # ---- prefill of 2,048 tokens in one step ----------------------------------
    def prefill_run(repeats: int, warmup: int):
        times = []
        for index in range(warmup + repeats):
            cache = runner.cache.open()
            ids = rng.integers(0, vocab, PREFILL_TOKENS).tolist()
            runner.cache.append(cache, 0, PREFILL_TOKENS)
            torch.cuda.synchronize()
            start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            t0 = time.perf_counter()
            start.record()
            logits = runner.step([StepEntry(cache, ids, 0, [PREFILL_TOKENS - 1])])
            stop.record()
            torch.cuda.synchronize()
            if index >= warmup:
                times.append(start.elapsed_time(stop))
                windows.append((t0, time.perf_counter()))
            runner.cache.free(cache)
        return statistics.median(times)

    # the step function replays a batch shape as a CUDA graph once it has come a few times (a long
    # prompt cut into equal portions does that; a benchmark's repeats too).  Both figures are given:
    # the first sightings, launched kernel by kernel, and the replayed sequence.
    use_graphs = runner.use_graphs
    runner.use_graphs = False
    prefill_uncaptured_ms = prefill_run(5, 3)
    runner.use_graphs = use_graphs
    prefill_ms = prefill_run(5, 6)   # warm-up long enough for the step's launch sequence to be captured
    flops = prefill_flops(raw, layers, PREFILL_TOKENS)
    peak_flops = peaks["bf16_tflops"] * 1e12

    def prefill_through_engine(budget: int, repeats: int, warmup: int):
        """One 2,048-token prompt through `LLMEngine.step()` under a token budget (four portions at
        the stock 512), host token ids in, the first generated token out: wall clock around it,
        as the reference arm's prefill figure is taken."""
        stock = engine.scheduler.max_tokens_per_step
        engine.scheduler.max_tokens_per_step = budget
        times, steps_taken = [], 0
        try:
            for index in range(warmup + repeats):
                prompt = rng.integers(0, vocab, PREFILL_TOKENS).tolist()
                torch.cuda.synchronize()
                t0 = time.perf_counter()
                engine.add_request(prompt, SamplingParams(max_new_tokens=1, ignore_eos=True))
                steps_taken = 0
                while engine.has_work:
                    engine.step()
                    steps_taken += 1
                torch.cuda.synchronize()
                t1 = time.perf_counter()
                if index >= warmup:
                    times.append((t1 - t0) * 1000.0)
                    windows.append((t0, t1))
        finally:
            engine.scheduler.max_tokens_per_step = stock
        return statistics.median(times), steps_taken

    budget512_ms, budget512_steps = prefill_through_engine(512, 5, 3)

    points = {}
    for batch in (1, large):
        point_ms, _, _ = decode_run(batch, max(10, args.steps // 2), 3)
        points[f"decode_b{batch}"] = round(batch * 1000.0 / point_ms, 1)

    kernels = dominant_kernels(ops, raw, args.batch, peaks, context) if not args.layers else {}
    sampler.stop()
    clocks = sampler.summary(windows)
    return {
        "metric": f"decode_tokens_per_second_qwen2.5-{args.shape}_b{args.batch}_ctx{context}",
        "value": round(value, 1), "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: seeded random weights and uniform random token ids",
        "impl": "ours",
        "config": {
            "model": shape_name, "layers": layers, "layers_full": full_layers, "hidden": raw["hidden_size"],
            "heads": raw["num_attention_heads"], "kv_heads": raw["num_key_value_heads"], "head_dim": raw["head_dim"],
            "intermediate": raw["intermediate_size"], "vocab": raw["vocab_size"], "global_batch": args.batch,
            "seq_len": context, "block_size": BLOCK_SIZE, "prefill_tokens": PREFILL_TOKENS,
            "parallelism": "single_gpu", "l2": f"inputs larger than L2 (weights read per step: {numbers['weight_bytes_per_step'] / 1e9:.1f} GB)",
            "peaks": peaks["source"],
        },
        "e2e": {"value": round(e2e_value, 1), "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h},
        "gpu_launches": launches,
        "prefill": {"value": round(PREFILL_TOKENS * 1000.0 / prefill_ms, 1), "tokens": PREFILL_TOKENS,
                    "ms": round(prefill_ms, 3), "frac": round(flops / (prefill_ms * 1e-3) / peak_flops, 4),
                    "uncaptured_ms": round(prefill_uncaptured_ms, 3),
                    "uncaptured_frac": round(flops / (prefill_uncaptured_ms * 1e-3) / peak_flops, 4),
                    "budget512": {"value": round(PREFILL_TOKENS * 1000.0 / budget512_ms, 1), "ms": round(budget512_ms, 3),
                                  "steps": budget512_steps,
                                  "note": "through LLMEngine.step() with a 512-token budget, wall clock"}},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / peaks["hbm_gbs"], 4)},
        "points": points,
        "kernels": kernels,
        "clocks": clocks,
    }


def dominant_kernels(ops, raw: dict, batch: int, peaks: dict, context: int = 0) -> dict:
    """Each dominant decode kernel at the headline batch, as a stream of back-to-back launches
    over rotated operands (so every launch reads HBM) in one captured graph: the time the
    stream takes divided by its launches, and the bandwidth that is.  Under programmatic
    dependent launch a launch streams its weights while the one before it drains, so this is
    the rate the kernel sustains in a chain, not the duration of one launch alone (those are
    in profiles/, from ncu: longer, since a lone launch has nothing to overlap with)."""
    import torch

    dev = "cuda"
    h, inter, vocab = raw["hidden_size"], raw["intermediate_size"], raw["vocab_size"]
    heads, kv, d = raw["num_attention_heads"], raw["num_key_value_heads"], raw["head_dim"]

    def graph_us(fn, reps):
        fn(0)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for i in range(reps):
                fn(i)
        graph.replay()
        torch.cuda.synchronize()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        for _ in range(5):
            graph.replay()
        stop.record()
        torch.cuda.synchronize()
        return start.elapsed_time(stop) * 1e3 / (5 * reps)

    out = {}
    shapes = {"qkv": ((heads + 2 * kv) * d, h, 8), "o": (h, heads * d, 8), "gate_up": (2 * inter, h, 4),
              "down": (h, inter, 4), "lm_head": (vocab, h, 2)}
    for name, (n, k, copies) in shapes.items():
        weights = [torch.randn(n, k, device=dev, dtype=torch.bfloat16) for _ in range(copies)]
        x = torch.randn(batch, k, device=dev, dtype=torch.bfloat16)
        result = torch.empty(batch, n, device=dev, dtype=torch.bfloat16 if name == "gate_up" else torch.float32)
        partial = name in ("qkv", "o", "down")
        us = graph_us(lambda i: ops.linear(x, weights[i % copies], result, allow_partials=partial), 2 * copies)
        gbs = n * k * 2 / us / 1e3
        out[name] = {"us": round(us, 1), "GBps": round(gbs, 0), "frac": round(gbs / peaks["hbm_gbs"], 3)}
        del weights
    context = context or CONTEXT
    blocks = -(-context // BLOCK_SIZE)
    sets = 4   # rotated key/value pools, so that a launch does not find its keys in L2
    pools = [(torch.randn(batch * blocks, BLOCK_SIZE, kv, d, device=dev, dtype=torch.bfloat16),
              torch.randn(batch * blocks, BLOCK_SIZE, kv, d, device=dev, dtype=torch.bfloat16)) for _ in range(sets)]
    q = torch.randn(batch, heads * d, device=dev, dtype=torch.bfloat16)
    width = max(8, 1 << (blocks - 1).bit_length())
    table = torch.full((batch, width), -1, dtype=torch.int32, device=dev)
    table[:, :blocks] = torch.arange(batch * blocks, dtype=torch.int32, device=dev).view(batch, blocks)
    q_start = torch.arange(batch + 1, dtype=torch.int32, device=dev)
    ctx = torch.full((batch,), context, dtype=torch.int32, device=dev)
    seq_of = torch.arange(batch, dtype=torch.int32, device=dev)
    attn = torch.empty_like(q)
    us = graph_us(lambda i: ops.paged_attention(q, pools[i % sets][0], pools[i % sets][1], table, q_start, ctx, seq_of,
                                                heads, kv, d, d ** -0.5, None, attn, max_q_len=1, min_q_len=1), 2 * sets)
    gbs = batch * context * 2 * kv * d * 2 / us / 1e3
    out["attention"] = {"us": round(us, 1), "GBps": round(gbs, 0), "frac": round(gbs / peaks["hbm_gbs"], 3)}
    out["note"] = "back-to-back launches in one graph, time per launch of the stream (launches overlap): a sustained rate, not one kernel's duration"
    return out


def run_mixed(args) -> dict:
    """The scheduler end to end at Qwen2.5-1.5B shape: 64 requests, random-id prompts of 32 to
    2,048 tokens, 32 to 256 output tokens each (lengths drawn as shrike's bench/workload.py:15-22
    does, `random.Random(20260718).randint`), greedy, fixed lengths, chunked-prefill budget 512,
    through `LLMEngine.generate`.  Wall-clock, as shrike's bench/bench_engine.py:54-62 measures."""
    import random

    import torch

    import shrike_b200.models  # noqa: F401
    from shrike_b200 import SamplingParams
    from shrike_b200.config import parse_config
    from shrike_b200.engine.llm_engine import LLMEngine
    from shrike_b200.weights.random_init import random_tensors

    torch.cuda.set_device(0)
    design = getattr(args, "arch", "qwen2")   # the same workload on another decoder at the same widths
    sadodra = design in ("sadodra", "vupitar", "kavedra", "setotar", "nulazen", "radilix")
    if sadodra:
        from shrike_b200.shapes import shape_config

        raw = dict(shape_config(f"{design}-1.5b"))
        if args.layers:
            raw["layers"] = raw["layers"][: args.layers]
        raw["vocab_size"], raw["num_hidden_layers"] = raw["vocab"], len(raw["layers"])
    else:
        raw = dict(MODEL_1_5B)
        if args.layers:
            raw["num_hidden_layers"] = args.layers
    config = parse_config(raw)
    tensors = random_tensors(config, seed=0, device="cuda", dtype=torch.bfloat16)
    engine = LLMEngine(None, block_size=BLOCK_SIZE, num_blocks=args.num_blocks or 12000, max_tokens_per_step=512,
                       max_running=256, dtype="bfloat16", config=config, tensors=tensors)
    del tensors
    rng = random.Random(20260718)
    outputs = [rng.randint(32, 256) for _ in range(64)]
    prompts = [[rng.randrange(raw["vocab_size"]) for _ in range(rng.randint(32, 2048))] for _ in range(64)]
    params = [SamplingParams(max_new_tokens=n, temperature=0.0, ignore_eos=True) for n in outputs]
    engine.generate(prompts[:4], params[:4])   # warm-up: builds, graphs for small batches
    torch.cuda.synchronize()
    steps_before = engine.stats.steps
    began = time.perf_counter()
    results = engine.generate(prompts, params)
    torch.cuda.synchronize()
    seconds = time.perf_counter() - began
    engine.ops.check_status()
    generated = sum(len(r) for r in results)
    assert [len(r) for r in results] == outputs and engine.block_manager.whole()
    return {
        "workload": "mixed", "model": f"{design.capitalize()} at Qwen2.5-1.5B widths" if sadodra else "Qwen2.5-1.5B shape",
        "layers": raw["num_hidden_layers"], "requests": 64,
        "prompt_tokens": sum(len(p) for p in prompts), "generated_tokens": generated, "seconds": round(seconds, 3),
        "value": round(generated / seconds, 1), "unit": "generated tok/s",
        "total_tokens_per_second": round((generated + sum(len(p) for p in prompts)) / seconds, 1),
        "steps": engine.stats.steps - steps_before, "preemptions": engine.scheduler.num_preemptions,
        "kv_blocks": engine.block_manager.total_pages, "budget": 512, "dtype": "bf16",
        "data": "synthetic: seeded random weights and uniform random token ids",
    }


def run_case(args) -> dict:
    """A small, fixed workload around one kernel, a few launches long: what the ncu captures
    under profiles/ are taken on.  Inputs are larger than L2 where the kernel streams."""
    import torch

    from shrike_b200.ops.cuda_ops import CudaOps

    torch.cuda.set_device(0)
    dev = "cuda"
    ops = CudaOps(torch.bfloat16, dev)
    raw = MODEL_7B
    h, inter = raw["hidden_size"], raw["intermediate_size"]
    heads, kv, d = raw["num_attention_heads"], raw["num_key_value_heads"], raw["head_dim"]
    tokens = args.batch
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    times = []
    filler = []

    def keep_busy():
        """The device is kept busy (about 0.2 ms) while the host prepares the timed launch (plan, tensor
        maps: about 25 us), so that the events bracket the kernel and not the host's work before it."""
        if hasattr(torch.cuda, "_sleep"):
            torch.cuda._sleep(400_000)
        else:
            if not filler:
                filler.append(torch.empty(1 << 30, dtype=torch.uint8, device=dev))
            filler[0].zero_()
    if args.case.startswith("gemm_"):
        shapes = {"gemm_gate_up": (2 * inter, h), "gemm_down": (h, inter), "gemm_qkv": ((heads + 2 * kv) * d, h)}
        n, k = shapes[args.case]
        weights = [torch.randn(n, k, device=dev, dtype=torch.bfloat16) for _ in range(3)]   # rotated: every call reads HBM
        x = torch.randn(tokens, k, device=dev, dtype=torch.bfloat16)
        out = torch.empty(tokens, n, device=dev, dtype=torch.bfloat16 if args.case == "gemm_gate_up" else torch.float32)
        for i in range(6):
            keep_busy()
            start.record()
            ops.linear(x, weights[i % 3], out, allow_partials=args.case != "gemm_gate_up")
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": n * k * 2}
    elif args.case == "branch_norm":
        # resid += LN(branch) and the sum in bfloat16, rows of 7B width: --batch rows (16,384 rows: inputs beyond L2)
        rows = tokens
        resid = torch.randn(rows, h, device=dev, dtype=torch.float32)
        branch = torch.randn(rows, h, device=dev, dtype=torch.float32)
        weight, bias = torch.ones(h, device=dev), torch.zeros(h, device=dev)
        out = torch.empty(rows, h, device=dev, dtype=torch.bfloat16)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.norm_add(resid, branch, weight, bias, 1e-6, out)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": rows * h * (4 + 4 + 4 + 2)}
    elif args.case == "tanh_norm":
        # resid += three pending branch outputs, then two tanh norms of the sum, rows of 7B width (--batch rows)
        rows = tokens
        resid = torch.randn(rows, h, device=dev, dtype=torch.float32)
        pending = [(torch.randn(rows, h, device=dev, dtype=torch.float32), scale) for scale in (0.8, 1.1, 1.0)]
        weight, bias = torch.ones(h, device=dev), torch.zeros(h, device=dev)
        outs = [torch.empty(rows, h, device=dev, dtype=torch.bfloat16) for _ in range(2)]
        for _ in range(6):
            keep_busy()
            start.record()
            ops.tanh_norm(resid, pending, norms=[(0.5, weight, bias, outs[0]), (0.7, weight, bias, outs[1])])
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": rows * h * (4 + 3 * 4 + 4 + 2 + 2)}
    elif args.case == "head_prep":
        # q|k|v|gate of 7B heads from the fused product's float32 result: per-head norms, rotation, pages (--batch tokens)
        total = -(-((heads + 2 * kv) * d + heads) // 16) * 16
        fused = torch.randn(tokens, total, device=dev, dtype=torch.float32)
        bias = torch.zeros(total, device=dev)
        positions = torch.arange(tokens, dtype=torch.int32, device=dev)
        inv_freq = torch.tensor([1e6 ** (-2.0 * i / d) for i in range(d // 2)], device=dev)
        weight = torch.ones(d, device=dev)
        q = torch.empty(tokens, heads * d, device=dev, dtype=torch.bfloat16)
        pages = -(-tokens // BLOCK_SIZE)
        keys = torch.empty(pages, BLOCK_SIZE, kv, d, device=dev, dtype=torch.bfloat16)
        values = torch.empty_like(keys)
        gate = torch.empty(tokens, heads, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.head_prep(fused, bias, positions, inv_freq, d, weight, weight, 1e-6, q, keys, values, positions, gate, heads, kv, d, d, d)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * (total * 4 + (heads + 2 * kv) * d * 2 + heads * 4)}
    elif args.case in ("decay_scan", "decay_scan_single"):
        # linear attention with a decay per head at the 7B-width shape (28 heads of 128 x 128): one prompt of
        # --prefill-tokens tokens (runs of 64 tokens), or --batch sequences one token each (the walk)
        lh, ld, lv = heads, d, d
        single = args.case.endswith("_single")
        seqs, q_len = (tokens, 1) if single else (1, args.prefill_tokens)
        n = seqs * q_len
        total = -(-(2 * lh * ld + 2 * lh * lv) // 16) * 16
        fused = torch.randn(n, total, device=dev, dtype=torch.float32) * 0.3
        decays = torch.tensor([math.exp(-1.0 / (8.0 * 2.0 ** (7.0 * i / (lh - 1)))) for i in range(lh)], device=dev)
        state = torch.zeros(seqs, lh, ld * lv, device=dev)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        slots = torch.arange(seqs, dtype=torch.int32, device=dev)
        out = torch.empty(n, lh * lv, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.decay_scan(fused, decays, state, q_start, slots, out, seqs, lh, ld, lv, longest=q_len)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        chunks = -(-q_len // 64)
        # per head and run of 64 tokens: scores 64 x 64 x dim, their outputs 64 x 64 x vdim, the state's addition and the
        # state's part of the outputs 2 x 64 x dim x vdim (2 flops a multiply-add)
        work = {"bytes": seqs * lh * ld * lv * 4 * 2 + n * (2 * lh * ld + lh * lv) * 4 + n * lh * lv * 4} if single else \
               {"flops": 2.0 * seqs * lh * chunks * (64 * 64 * ld + 64 * 64 * lv + 2 * 64 * ld * lv)}
    elif args.case == "latent_rope_store":
        # queries, latent and shared key part of the 7B-width latent attention (28 heads, rank 192 + 64 rotated) from the
        # fused product's float32 result: the latent's norm, the rotation, casts, page rows (--batch tokens)
        rank, rot = 192, 64
        padded = rank + rot
        total = -(-(heads * padded + padded) // 16) * 16
        fused = torch.randn(tokens, total, device=dev, dtype=torch.float32)
        positions = torch.arange(tokens, dtype=torch.int32, device=dev)
        inv_freq = torch.tensor([1e4 ** (-2.0 * i / rot) for i in range(rot // 2)], device=dev)
        weight = torch.ones(rank, device=dev)
        q = torch.empty(tokens, heads * padded, device=dev, dtype=torch.bfloat16)
        pages = -(-tokens // BLOCK_SIZE)
        latents = torch.empty(pages, BLOCK_SIZE, 1, padded, device=dev, dtype=torch.bfloat16)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.latent_rope_store(fused, weight, 1e-6, positions, inv_freq, 1.0, q, latents, positions, heads, rank, rot, padded)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * (total * 4 + (heads + 1) * padded * 2)}
    elif args.case in ("matrix_memory", "matrix_memory_single"):
        # the matrix memory of the 7B-width shape (8 heads of 128 x 256): one prompt of --prefill-tokens tokens (chunk
        # kernels), or --batch sequences one token each (the walk)
        mh, md, mv = 8, 128, 256
        single = args.case.endswith("_single")
        seqs, q_len = (tokens, 1) if single else (1, args.prefill_tokens)
        n = seqs * q_len
        total = -(-(2 * mh * md + 2 * mh * mv + 2 * mh) // 16) * 16
        fused = torch.randn(n, total, device=dev, dtype=torch.float32) * 0.3
        gate_bias = torch.zeros(2 * mh, device=dev)
        state = torch.zeros(seqs, mh, md * mv + md + 4, device=dev)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        slots = torch.arange(seqs, dtype=torch.int32, device=dev)
        num, den = torch.empty(n, mh * mv, device=dev), torch.empty(n, mh, device=dev)
        out = torch.empty(n, mh * mv, device=dev, dtype=torch.bfloat16)
        weight = torch.ones(mh * mv, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.matrix_memory(fused, gate_bias, state, q_start, slots, num, den, weight, 1e-6, out, seqs, mh, md, mv, 15.0, 1e-6,
                              longest=q_len)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        chunks = -(-q_len // 64)
        # per head and chunk: scores 64 x 64 x dim, their outputs 64 x 64 x vdim, the state's addition and the state's
        # part of the outputs 2 x 64 x dim x vdim (2 flops a multiply-add)
        work = {"bytes": seqs * mh * (md * mv + md) * 4 * 2 + n * total * 4} if single else \
               {"flops": 2.0 * seqs * mh * chunks * (64 * 64 * md + 64 * 64 * mv + 2 * 64 * md * mv)}
    elif args.case in ("gated_scan", "gated_scan_single"):
        # the gated linear recurrence at the 7B-width shape (8 heads of 128 x 128): one prompt of --prefill-tokens tokens
        # (runs of 64 tokens, each walked twice), or --batch sequences one token each (one walk)
        lh, ld, lv = 8, d, d
        single = args.case.endswith("_single")
        seqs, q_len = (tokens, 1) if single else (1, args.prefill_tokens)
        n = seqs * q_len
        total = -(-(2 * lh * ld + lh * lv) // 16) * 16
        fused = torch.randn(n, total, device=dev, dtype=torch.float32)
        bias, lower = torch.randn(lh * ld, device=dev), torch.rand(lh * ld, device=dev) * 0.9
        state = torch.zeros(seqs, lh, ld * lv, device=dev)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        slots = torch.arange(seqs, dtype=torch.int32, device=dev)
        out = torch.empty(n, lh * lv, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.gated_scan(fused, bias, lower, state, q_start, slots, out, seqs, lh, ld, lv, q_lens=[q_len] * seqs)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        # a token and head: dim x vdim multiply-adds for the state and as many for the output (2 flops each); a prompt's
        # runs are walked twice, which the count leaves out (it is the recurrence's own arithmetic)
        work = {"bytes": seqs * lh * ld * lv * 4 * 2 + n * total * 4 + n * lh * lv * 4} if single else \
               {"flops": 4.0 * n * lh * ld * lv}
    elif args.case == "stream_norm":
        # --batch rows of four streams of the 7B width with a two-term pending result and a layer scale
        count = 4
        streams = torch.randn(tokens, count, h, device=dev)
        terms = [(torch.randn(tokens, h, device=dev), 1.0), (torch.randn(tokens, h, device=dev), 0.9)]
        join = (torch.eye(count, device=dev) + 0.1, torch.ones(count, device=dev), torch.ones(h, device=dev))
        in_w, weight = torch.ones(count, device=dev), torch.ones(h, device=dev)
        out = torch.empty(tokens, h, device=dev, dtype=torch.bfloat16)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.stream_norm(streams, terms, join, in_w, weight, 1e-6, out)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * h * (2 * count * 4 + 2 * 4 + 2)}
    elif args.case in ("delta_scan", "delta_scan_single"):
        # the delta rule with a decay per key channel at the 7B-width shape (28 heads of 128 x 128): one prompt of
        # --prefill-tokens tokens, or --batch sequences one token each
        single = args.case.endswith("_single")
        seqs, q_len = (tokens, 1) if single else (1, args.prefill_tokens)
        n = seqs * q_len
        mixed = torch.randn(n, 3 * heads * d, device=dev)
        mixed[:, : 2 * heads * d] = torch.nn.functional.normalize(mixed[:, : 2 * heads * d].view(n, 2 * heads, d), dim=-1).view(n, -1)
        beta, gates = torch.rand(n, heads, device=dev), torch.randn(n, 2 * heads * d, device=dev) - 3.0
        rate, bias = torch.ones(heads, device=dev), torch.zeros(heads * d, device=dev)
        state = torch.zeros(seqs, heads, d * d, device=dev)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        slots = torch.arange(seqs, dtype=torch.int32, device=dev)
        out = torch.empty(n, heads * d, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.delta_scan(mixed, beta, gates, rate, bias, state, q_start, slots, out, seqs, heads, heads, d, d, q_lens=[q_len] * seqs)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        # a token and head: dim x vdim each of the decay (1 flop), S^T k, k u^T and S^T q (2 flops a multiply-add)
        work = {"bytes": seqs * heads * d * d * 4 * 2 + n * heads * (5 * d + 1) * 4} if single else {"flops": 7.0 * n * heads * d * d}
    elif args.case in ("head_delta_scan", "head_delta_scan_single", "gla_scan", "gla_scan_single"):
        # the delta rule with one decay a head (--heads value heads on half as many key heads, default 8) and linear attention
        # with decays per key channel (default 28 heads), heads of 128 x 128: one prompt of --prefill-tokens tokens, or
        # --batch sequences one token each
        single, delta = args.case.endswith("_single"), args.case.startswith("head_delta")
        count = args.heads or (8 if delta else 28)
        groups = count // 2 if delta and count % 2 == 0 else count
        seqs, q_len = (tokens, 1) if single else (1, args.prefill_tokens)
        n = seqs * q_len
        width = (2 * groups + count) * d
        mixed = torch.randn(n, width, device=dev)
        mixed[:, : 2 * groups * d] = torch.nn.functional.normalize(mixed[:, : 2 * groups * d].view(n, 2 * groups, d), dim=-1).view(n, -1)
        beta = torch.rand(n, count, device=dev) if delta else None
        gates = torch.randn(n, count if delta else count * d, device=dev) - (3.0 if delta else -3.0)
        rate, bias = torch.full((count,), 1.0 if delta else 1 / 16.0, device=dev), torch.zeros(gates.shape[1], device=dev)
        state = torch.zeros(seqs, count, d * d, device=dev)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        slots = torch.arange(seqs, dtype=torch.int32, device=dev)
        out = torch.empty(n, count * d, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.delta_scan(mixed, beta, gates, rate, bias, state, q_start, slots, out, seqs, count, groups, d, d, q_lens=[q_len] * seqs,
                           per_head=delta, sign=1.0 if delta else -1.0)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        # a token and head: dim x vdim of the decay (1 flop), k u^T and S^T q, with the delta rule also S^T k (2 flops each)
        work = {"bytes": seqs * count * d * d * 4 * 2 + n * (width + gates.shape[1] + count * d) * 4} if single else \
               {"flops": (7.0 if delta else 5.0) * n * count * d * d}
    elif args.case == "sum_norm":
        # --batch rows of the 7B width: two pending sums, and rows with a factor each of which a fifth is not zero
        resid, weight = torch.randn(tokens, h, device=dev), torch.ones(h, device=dev)
        terms = [(torch.randn(tokens, h, device=dev), 0.6), (torch.randn(tokens, h, device=dev), 0.4)]
        out = torch.randn(tokens, h, device=dev).to(torch.bfloat16)
        factors = torch.rand(tokens, device=dev)
        factors[torch.arange(tokens, device=dev) % 5 > 0] = 0.0
        for _ in range(6):
            keep_busy()
            start.record()
            ops.sum_norm(resid, terms, weight, 1e-6, out, row_term=(out, factors, 0.6))
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * h * (4 + 2 * 4 + 4 + 2 + 2 / 5)}
    elif args.case == "element_gate":
        # --batch rows of 28 heads of 128, gates from a fused q | k | v | gate product
        x = torch.randn(tokens, heads * d, device=dev).to(torch.bfloat16)
        fused = torch.randn(tokens, (2 * heads + 2 * kv) * d, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.element_gate(x, fused, (heads + 2 * kv) * d, heads, d)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * heads * d * (4 + 2 + 2)}
    elif args.case == "act_blocks":
        # --batch rows of 8 experts of 7,104 columns, two chosen a row: those are read, all are written
        x = torch.randn(tokens, 8 * 7104, device=dev).to(torch.bfloat16)
        share = torch.zeros(tokens, 9, device=dev)
        share[:, :2] = 0.4
        for _ in range(6):
            keep_busy()
            start.record()
            ops.act_blocks(x, share, 8, 7104, "gelu")
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * 7104 * 2 * (8 + 2)}
    elif args.case == "low_rank":
        # --batch rows: 3,584 decays from a rank of 16
        fused = torch.randn(tokens, 4 * heads * d + 16, device=dev)
        matrix = torch.randn(heads * d, 16, device=dev).to(torch.bfloat16)
        out = torch.empty(tokens, heads * d, device=dev)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.low_rank(fused, 4 * heads * d, 16, matrix, out)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * (heads * d * 4 + 64)}
    elif args.case == "delta_prep":
        # --batch tokens of one sequence, q, k and v of 28 heads of 128 behind four taps, beta and two low-rank rows of 128
        channels = 3 * heads * d
        total = channels + heads + 2 * 128 + 4
        fused = torch.randn(tokens, total, device=dev)
        taps = torch.randn(channels, 4, device=dev)
        state = torch.zeros(1, 3, channels, device=dev)
        q_start = torch.tensor([0, tokens], dtype=torch.int32, device=dev)
        zeros = torch.zeros(tokens, dtype=torch.int32, device=dev)
        mixed, beta = torch.empty(tokens, channels, device=dev), torch.empty(tokens, heads, device=dev)
        low = torch.empty(tokens, 256, device=dev, dtype=torch.bfloat16)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.delta_prep(fused, taps, state, q_start, zeros[:1], zeros, mixed, beta, low, 1, heads, heads, d, d, channels,
                           channels + heads, 1e-6, longest=tokens)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * (total * 4 + channels * 4 + heads * 4 + 256 * 2)}
    elif args.case == "norm_join":
        resid, branch = torch.randn(tokens, h, device=dev), torch.randn(tokens, h, device=dev)
        weight = torch.ones(h, device=dev)
        out = torch.empty(tokens, h, device=dev, dtype=torch.bfloat16)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.norm_join(resid, branch, weight, 1e-6, None, weight, 1e-6, out)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * h * (4 + 4 + 4 + 2)}
    elif args.case == "head_rms":
        # --batch rows of 28 heads of 128 with an output gate from a fused product
        x, gates = torch.randn(tokens, heads * d, device=dev), torch.randn(tokens, 2 * heads * d, device=dev)
        weight = torch.ones(d, device=dev)
        out = torch.empty(tokens, heads * d, device=dev, dtype=torch.bfloat16)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.head_rms(x, weight, 1e-6, out, heads, gate_source=gates, gate_at=heads * d)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * heads * d * (4 + 4 + 2)}
    elif args.case == "short_conv":
        # --batch tokens of one sequence, the fused q | k | v projection of the 7B-width shape, four taps
        channels = (heads + 2 * kv) * d
        fused = torch.randn(tokens, channels, device=dev)
        taps = torch.randn(channels, 4, device=dev)
        state = torch.zeros(1, 3, channels, device=dev)
        q_start = torch.tensor([0, tokens], dtype=torch.int32, device=dev)
        out = torch.empty_like(fused)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.short_conv(fused, None, taps, state, q_start, torch.zeros(1, dtype=torch.int32, device=dev),
                           torch.zeros(tokens, dtype=torch.int32, device=dev), out, 1, channels)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        work = {"bytes": tokens * channels * 4 * 2}
    elif args.case in ("attention_single_kept", "attention_portions_kept"):
        # a window of 4,096 keys that keeps the first four, soft-capped: --batch sequences of 8,192 keys one token each,
        # or a prompt of --prefill-tokens
        single = args.case.startswith("attention_single")
        seqs = tokens if single else 1
        ctx_len = 8192 if single else args.prefill_tokens
        q_len = 1 if single else args.prefill_tokens
        window = 4096
        blocks = -(-ctx_len // BLOCK_SIZE)
        keys = torch.randn(seqs * blocks + 8, BLOCK_SIZE, kv, d, device=dev, dtype=torch.bfloat16)
        values = torch.randn_like(keys)
        q = torch.randn(seqs * q_len, heads * d, device=dev, dtype=torch.bfloat16)
        width = max(8, 1 << (blocks - 1).bit_length())
        table = torch.full((seqs, width), -1, dtype=torch.int32, device=dev)
        table[:, :blocks] = torch.arange(seqs * blocks, dtype=torch.int32, device=dev).view(seqs, blocks)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        ctx = torch.full((seqs,), ctx_len, dtype=torch.int32, device=dev)
        seq_of = torch.arange(seqs, dtype=torch.int32, device=dev).repeat_interleave(q_len)
        out = torch.empty_like(q)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.paged_attention(q, keys, values, table, q_start, ctx, seq_of, heads, kv, d, d ** -0.5, window, out,
                                max_q_len=q_len, min_q_len=q_len, q_lens=[q_len] * seqs, softcap=30.0, keep_first=4)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        seen = sum(min(p + 1, window + 4) for p in range(ctx_len - q_len, ctx_len))
        work = {"bytes": seqs * (window + 4) * 2 * kv * d * 2} if single else {"flops": 4.0 * heads * d * seen}
    elif args.case in ("attention_single", "attention_portions", "attention_single_scores", "attention_portions_scores",
                       "attention_single_latent", "attention_portions_latent", "attention_single_sink", "attention_portions_sink"):
        single = args.case.startswith("attention_single")
        if args.case.endswith("_latent"):   # one key/value head of 256 whose keys are its values, as a cached latent is read
            kv, d = 1, 256
        changed = args.case.endswith("_scores")   # a soft cap and a distance bias on every score
        softcap = 50.0 if changed else None
        slopes = torch.tensor([2.0 ** (-8.0 * (i + 1) / heads) for i in range(heads)], device=dev) if changed else None
        sinks = torch.linspace(-1.0, 1.0, heads, device=dev) if args.case.endswith("_sink") else None   # one more term of every denominator
        seqs = tokens if single else 1
        ctx_len = CONTEXT if single else args.prefill_tokens
        q_len = 1 if single else args.prefill_tokens
        blocks = -(-ctx_len // BLOCK_SIZE)
        pages = seqs * blocks + 8
        keys = torch.randn(pages, BLOCK_SIZE, kv, d, device=dev, dtype=torch.bfloat16)
        values = keys if args.case.endswith("_latent") else torch.randn_like(keys)
        q = torch.randn(seqs * q_len, heads * d, device=dev, dtype=torch.bfloat16)
        width = max(8, 1 << (blocks - 1).bit_length())
        table = torch.full((seqs, width), -1, dtype=torch.int32, device=dev)
        table[:, :blocks] = torch.arange(seqs * blocks, dtype=torch.int32, device=dev).view(seqs, blocks)
        q_start = torch.arange(seqs + 1, dtype=torch.int32, device=dev) * q_len
        ctx = torch.full((seqs,), ctx_len, dtype=torch.int32, device=dev)
        seq_of = torch.arange(seqs, dtype=torch.int32, device=dev).repeat_interleave(q_len)
        out = torch.empty_like(q)
        for _ in range(6):
            keep_busy()
            start.record()
            ops.paged_attention(q, keys, values, table, q_start, ctx, seq_of, heads, kv, d, d ** -0.5, None, out,
                                max_q_len=q_len, min_q_len=q_len, q_lens=[q_len] * seqs, softcap=softcap, slopes=slopes, sinks=sinks)
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop) * 1e3)
        planes = 1 if args.case.endswith("_latent") else 2
        work = {"bytes": seqs * ctx_len * planes * kv * d * 2} if single else {"flops": 4.0 * heads * d * q_len * (q_len + 1) / 2}
    else:
        raise SystemExit(f"unknown case {args.case!r}")
    ops.check_status()
    best = min(times[2:])
    result = {"case": args.case, "tokens_or_sequences": tokens, "us": round(best, 2), "launch_times_us": [round(t, 1) for t in times]}
    if "bytes" in work:
        result["GBps"] = round(work["bytes"] / best / 1e3, 1)
    else:
        result["TFLOPs"] = round(work["flops"] / best / 1e6, 1)
    return result


def run_timeline(args) -> dict:
    """Where a captured decode step spends its time, kernel by kernel: start and end of every
    kernel of one step from CUPTI activity records (torch.profiler), on a model of the
    benchmark's widths with few layers.  Kernels overlap (each starts while the one before it
    runs), so the figure per kernel is `end - end of the kernel before it`: what the step
    would save if that kernel vanished from the chain.  Medians over the layers."""
    import numpy as np
    import torch
    from torch.profiler import ProfilerActivity, profile

    import shrike_b200.models  # noqa: F401
    from shrike_b200.config import parse_config
    from shrike_b200.engine.batch import StepEntry
    from shrike_b200.engine.llm_engine import LLMEngine
    from shrike_b200.weights.random_init import random_tensors

    torch.cuda.set_device(0)
    raw = dict(SHAPES[args.shape][1])
    context = args.context
    raw["num_hidden_layers"] = layers = args.layers or 6
    config = parse_config(raw)
    tensors = random_tensors(config, seed=0, device=torch.device("cuda:0"), dtype=torch.bfloat16)
    pages = args.batch * (-(-(context + 64) // BLOCK_SIZE)) + 64
    engine = LLMEngine(None, block_size=BLOCK_SIZE, num_blocks=pages, max_tokens_per_step=4096, max_running=64,
                       dtype="bfloat16", config=config, tensors=tensors)
    del tensors
    runner = engine.runner
    rng = np.random.default_rng(0)
    caches = []
    for _ in range(args.batch):
        cache = runner.cache.open()
        ids = rng.integers(0, raw["vocab_size"], context - 1).tolist()
        runner.cache.append(cache, 0, len(ids))
        runner.step([StepEntry(cache, ids, 0, [])])
        caches.append(cache)
    fed = [context - 1]

    def one_step():
        entries = []
        for cache in caches:
            runner.cache.append(cache, fed[0], 1)
            entries.append(StepEntry(cache, [5], fed[0], [0], (0.0, 1.0, 0)))
        _logits, drawn = runner.step(entries, sample=True)
        fed[0] += 1
        return drawn.tolist()

    for _ in range(6):
        one_step()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(3):
            one_step()
        torch.cuda.synchronize()
    kernels = sorted((e for e in prof.events() if e.device_type == torch.autograd.DeviceType.CUDA and "Memcpy" not in e.name),
                     key=lambda e: e.time_range.start)
    per_step = len(kernels) // 3
    step = kernels[-per_step:]
    rows, previous_end = [], step[0].time_range.start
    for event in step:
        rows.append((event.name.split("(")[0].split("<")[0].split("::")[-1], event.time_range.end - previous_end))
        previous_end = event.time_range.end
    norms = [i for i, (name, _) in enumerate(rows) if "add_rmsnorm" in name]
    first, per_layer = norms[0], norms[2] - norms[0]   # two norms a layer
    products = iter(["qkv product", "o product", "gate_up product", "down product"])
    seen_norms = 0
    labels = []
    for name, _ in rows[first + per_layer: first + 2 * per_layer]:
        if "add_rmsnorm" in name:
            labels.append("norm (feed-forward)" if seen_norms else "norm (mixer)")
            seen_norms += 1
        elif "gemm" in name or "nvjet" in name or "cutlass" in name:
            labels.append(next(products, "product"))
        elif "rope" in name:
            labels.append("rotary + cache store")
        elif "single_token" in name or "portions" in name or "attention" in name:
            labels.append("attention")
        elif "silu" in name:
            labels.append("SiLU product")
        else:
            labels.append(name)
    if "SiLU product" not in labels:
        labels = [label + " with SiLU" if label == "gate_up product" else label for label in labels]
    table = []
    for position in range(per_layer):
        samples = [rows[first + layer * per_layer + position] for layer in range(1, layers)]   # the first layer follows the embedding
        table.append({"kernel": labels[position], "name": samples[0][0], "in_situ_us": round(float(np.median([t for _, t in samples])), 2)})
    layer_us = round(sum(row["in_situ_us"] for row in table), 2)
    rest = rows[:first] + rows[first + layers * per_layer:]
    return {"case": "timeline", "shape": args.shape, "context": context, "batch": args.batch, "layers": layers, "layer_us": layer_us, "per_layer": table,
            "outside_layers": [{"name": name, "in_situ_us": round(t, 2)} for name, t in rest],
            "step_us": round(step[-1].time_range.end - step[0].time_range.start, 1)}


def run_design(args) -> dict:
    """A design (--arch sadodra, the default here, vupitar, kavedra, setotar, nulazen or radilix; the last three also beside the designs they are closest to) beside the Qwen2 decoder of the same widths, layer count and vocabulary (the
    closest model this engine serves), random weights: one 2,048-token prompt in one step, and decoding
    at --batch sequences of --context tokens, device-timed through the step function and the sampling
    kernel; for each, the kernels of one step by the time they take (CUPTI activity records).
    `--design 1.5b` or `7b` picks the pair of shape files; `--layers` cuts both models alike."""
    import numpy as np
    import torch
    from torch.profiler import ProfilerActivity, profile

    import shrike_b200.models  # noqa: F401
    from shrike_b200.config import parse_config
    from shrike_b200.engine.batch import StepEntry
    from shrike_b200.engine.llm_engine import LLMEngine
    from shrike_b200.shapes import shape_config
    from shrike_b200.weights.random_init import random_tensors

    torch.cuda.set_device(0)
    device = torch.device("cuda:0")
    context, batch = args.context, args.batch
    peaks = load_peaks()

    def kernels_of(run_step) -> list:
        with profile(activities=[ProfilerActivity.CUDA]) as prof:
            run_step()
            torch.cuda.synchronize()
        events = sorted((e for e in prof.events() if e.device_type == torch.autograd.DeviceType.CUDA
                         and "Memcpy" not in e.name and "Memset" not in e.name), key=lambda e: e.time_range.start)
        # kernels overlap (each may start while the one before it runs), so a kernel is charged the time
        # from the end of the kernel before it to its own end: what the step would save without it
        totals: dict = {}
        previous_end = events[0].time_range.start if events else 0
        for event in events:
            name = event.name.split("(")[0].split("<")[0].split("::")[-1].replace("void ", "")
            held = totals.setdefault(name, [0.0, 0])
            held[0] += max(0.0, event.time_range.end - max(previous_end, 0))
            held[1] += 1
            previous_end = max(previous_end, event.time_range.end)
        return [{"kernel": name, "us": round(us, 1), "launches": count}
                for name, (us, count) in sorted(totals.items(), key=lambda item: -item[1][0])][:14]

    def measure(name: str, raw: dict) -> dict:
        config = parse_config(raw)
        tensors = random_tensors(config, seed=0, device=device, dtype=torch.bfloat16)
        pages = batch * (-(-(context + args.steps + args.warmup + 16) // BLOCK_SIZE)) + -(-PREFILL_TOKENS // BLOCK_SIZE) + 64
        engine = LLMEngine(None, block_size=BLOCK_SIZE, num_blocks=pages, max_tokens_per_step=4096, max_running=64,
                           dtype="bfloat16", config=config, tensors=tensors)
        del tensors
        runner = engine.runner
        rng = np.random.default_rng(0)
        vocab = config.vocab_size

        def prefill_once():
            cache = runner.cache.open()
            ids = rng.integers(0, vocab, PREFILL_TOKENS).tolist()
            runner.cache.append(cache, 0, PREFILL_TOKENS)
            torch.cuda.synchronize()
            start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            runner.step([StepEntry(cache, ids, 0, [PREFILL_TOKENS - 1])])
            stop.record()
            torch.cuda.synchronize()
            runner.cache.free(cache)
            return start.elapsed_time(stop)

        runner.use_graphs = False
        prefill_ms = statistics.median([prefill_once() for _ in range(args.warmup + 5)][args.warmup:])
        prefill_kernels = kernels_of(prefill_once)
        runner.use_graphs = True

        caches = []
        for _ in range(batch):
            cache = runner.cache.open()
            ids = rng.integers(0, vocab, context - 1).tolist()
            runner.cache.append(cache, 0, len(ids))
            runner.step([StepEntry(cache, ids, 0, [])])
            caches.append(cache)
        fed = [context - 1]

        def decode_step():
            entries = []
            for index, cache in enumerate(caches):
                runner.cache.append(cache, fed[0], 1)
                entries.append(StepEntry(cache, [-1 - index] if fed[0] >= context else [5], fed[0], [0], (0.0, 1.0, 0)))
            fed[0] += 1
            return runner.step(entries, sample=True)[1]

        for _ in range(args.warmup):
            decode_step()
        torch.cuda.synchronize()
        launches = engine.ops.launches
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        for _ in range(args.steps):
            drawn = decode_step()
        stop.record()
        drawn.tolist()
        torch.cuda.synchronize()
        decode_ms = start.elapsed_time(stop) / args.steps
        launches = (engine.ops.launches - launches) // args.steps
        decode_kernels = kernels_of(decode_step)   # a replayed launch sequence: the records name its kernels all the same
        weight_bytes = engine.runner.model.weight_bytes()
        cache_bytes = runner.bytes_per_page / BLOCK_SIZE
        result = {
            "model": name, "layers": len(config.order), "weights_GB": round(weight_bytes / 1e9, 2),
            "cache_bytes_per_token": int(cache_bytes),
            "prefill": {"tokens": PREFILL_TOKENS, "ms": round(prefill_ms, 3), "tok_s": round(PREFILL_TOKENS * 1000.0 / prefill_ms, 1),
                        "kernels": prefill_kernels},
            "decode": {"batch": batch, "context": context, "ms_per_step": round(decode_ms, 4),
                       "tok_s": round(batch * 1000.0 / decode_ms, 1), "launches_per_step": launches,
                       "GBps_weights_and_cache": round((weight_bytes + batch * context * cache_bytes) / decode_ms / 1e6, 1),
                       "kernels": decode_kernels},
        }
        for cache in caches:
            runner.cache.free(cache)
        del engine, runner
        import gc

        gc.collect()
        torch.cuda.empty_cache()
        return result

    design = args.arch if args.arch != "qwen2" else "sadodra"
    ours = dict(shape_config(f"{design}-{args.design}"))
    theirs = dict(shape_config(f"qwen2.5-{args.design}"))
    if args.layers:
        # both models run `--layers` layers: a design that repeats some of its layers keeps its passes and
        # gives up distinct layers (never fewer than the repeated stretch)
        loop = ours.get("loop")
        extra = (loop["stop"] - loop["start"]) * (loop["times"] - 1) if loop else 0
        ours["layers"] = ours["layers"][: max(args.layers - extra, loop["stop"] if loop else 1)]
        theirs["num_hidden_layers"] = len(parse_config(ours).order)
    sampler = ClockSampler()
    sampler.start()
    t0 = time.perf_counter()
    results = [measure(f"{design.capitalize()} at Qwen2.5-{args.design.upper()} widths", ours)]
    # the designs it is closest to among those served: Setotar to Vupitar (attention beside a recurrent memory in one layer,
    # routed experts); Nulazen to Kavedra (latent attention, a linear recurrence) and for its experts to Vupitar; Radilix to
    # Setotar (attention beside a recurrence, experts in every layer) and for its recurrences to Nulazen
    for like in {"setotar": ("vupitar",), "nulazen": ("kavedra", "vupitar"), "radilix": ("setotar", "nulazen")}.get(design, ()):
        likeness = dict(shape_config(f"{like}-{args.design}"))
        if args.layers:
            loop = likeness.get("loop")
            extra = (loop["stop"] - loop["start"]) * (loop["times"] - 1) if loop else 0
            likeness["layers"] = likeness["layers"][: max(args.layers - extra, loop["stop"] if loop else 1)]
        results.append(measure(f"{like.capitalize()} at Qwen2.5-{args.design.upper()} widths", likeness))
    results.append(measure(f"Qwen2.5-{args.design.upper()} shape", theirs))
    sampler.stop()
    return {"case": "design", "design": design.capitalize(), "closest": "Qwen2ForCausalLM", "dtype": "bf16",
            "data": "synthetic: seeded random weights and uniform random token ids", "peaks": peaks,
            "models": results, "clocks": sampler.summary([(t0, time.perf_counter())])}


def run_reference(args) -> dict:
    reference = ROOT / "baseline" / "_ref"
    if not (reference / "shrike").is_dir():
        return {"impl": "reference", "unavailable": "the reference is not installed under baseline/_ref"}
    from baseline.reference_arm import run, run_mixed  # the unmodified reference through its own LLMEngine

    if args.workload == "mixed":
        return run_mixed(args, MODEL_1_5B)
    return run(args, SHAPES[args.shape][1], args.context)


def main():
    parser = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=50)
    parser.add_argument("--warmup", type=int, default=5)
    parser.add_argument("--impl", default="ours", choices=["ours", "reference"])
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--layers", type=int, default=0, help="fewer layers than the model has (0: all)")
    parser.add_argument("--shape", default="7b", choices=list(SHAPES), help="layer sizes of the decode workload")
    parser.add_argument("--context", type=int, default=1024, help="tokens each sequence holds when decoding is timed")
    parser.add_argument("--workload", default="decode", choices=["decode", "mixed"],
                        help="decode: the headline line; mixed: 64 requests through the scheduler at 1.5B shape")
    parser.add_argument("--arch", default="qwen2", choices=["qwen2", "sadodra", "vupitar", "kavedra", "setotar", "nulazen", "radilix"],
                        help="--workload mixed: the decoder the 64 requests run on (all at Qwen2.5-1.5B widths); "
                             "--case design: the design that is set beside the Qwen2 decoder (default there: sadodra)")
    parser.add_argument("--num-blocks", type=int, default=0, help="cache pages for --workload mixed (few pages force preemption)")
    parser.add_argument("--skip-mixed", action="store_true", help="leave the mixed workload out of the default line")
    parser.add_argument("--prefill-tokens", type=int, default=PREFILL_TOKENS,
                        help="prompt length of --case attention_portions")
    parser.add_argument("--heads", type=int, default=0, help="--case head_delta_scan / gla_scan: heads (0: those of the 7B-width shape)")
    parser.add_argument("--design", default="1.5b", choices=["1.5b", "7b"],
                        help="--case design: the widths at which the Sadodra decoder and the Qwen2 decoder are compared")
    parser.add_argument("--case", default=None,
                        help="run a small single-kernel workload instead (for profiling): gemm_gate_up, gemm_down, "
                             "gemm_qkv, attention_single, attention_portions (with _scores: soft-capped and distance-biased; with _latent: "
                             "one key/value head of 256 whose keys are its values; with _sink: a sink in every softmax), "
                             "branch_norm, tanh_norm, head_prep, matrix_memory (a prompt of --prefill-tokens), matrix_memory_single, "
                             "decay_scan (a prompt of --prefill-tokens), decay_scan_single, latent_rope_store, gated_scan, gated_scan_single, "
                             "head_delta_scan, gla_scan (a prompt of --prefill-tokens; --heads), the same with _single, sum_norm, element_gate, act_blocks, low_rank, "
                             "stream_norm, short_conv, delta_scan (a prompt of --prefill-tokens), delta_scan_single, delta_prep, norm_join, head_rms, "
                             "attention_single_kept, attention_portions_kept; "
                             "--batch gives tokens / sequences / rows.  timeline: per-kernel "
                             "times inside one captured decode step (--layers, default 6).  design: the Sadodra decoder "
                             "beside the Qwen2 decoder of equal widths (--design), prefill and decode")
    args = parser.parse_args()
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this engine runs on a single B200 (asked for {args.gpus})")
        sys.exit(2)
    args.warmup = max(3, args.warmup)
    if args.case == "timeline":
        print(json.dumps(run_timeline(args)))
        return
    if args.case == "design":
        print(json.dumps(run_design(args)))
        return
    if args.case:
        print(json.dumps(run_case(args)))
        return
    if args.workload == "mixed" and args.impl != "reference":
        print(json.dumps(run_mixed(args)))
        return
    result = run_reference(args) if args.impl == "reference" else run_ours(args)
    if args.impl != "reference" and args.shape == "7b" and not args.layers and not args.skip_mixed:
        # the scheduler end to end, beside the headline: 64 requests of mixed lengths at 1.5B widths
        import gc

        import torch

        gc.collect()
        torch.cuda.empty_cache()
        mixed_args = argparse.Namespace(**vars(args))
        mixed_args.layers, mixed_args.num_blocks = 0, 0
        mixed = run_mixed(mixed_args)
        result["mixed"] = {key: mixed[key] for key in ("value", "unit", "seconds", "steps", "requests", "model", "budget", "preemptions")}
    print(json.dumps(result))


if __name__ == "__main__":
    main()
