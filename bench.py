#!/usr/bin/env python3
"""Benchmark: decode throughput of GPT-2 small (random weights) on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A step is one decode step of a batch of 8 requests whose contexts end at the model's
context length (1024).  ``value`` is decoded tokens per second, timed on the device with CUDA
events around exactly K steps; ``e2e`` is the same metric through the Python entry point
(``LLM.generate``): token ids from the host in, sampled token ids to the host out, every
step.  The same line carries the prefill of 2,048 tokens (two prompts of 1024), the decode
step's memory roofline, and under ``points``: decode throughput at batch 1 and 64; the decode
workload as the target states it (512-token prompts, 256 greedy tokens, pages of 16, through
the scheduler) at batch 1, 8 and 64 with its fraction of the HBM roofline; a mixed serving
workload; the 32-bit path's decode and prompt steps.  ``reference_tokens`` says whether this
engine's 32-bit path and the reference's choose the same greedy tokens from the same weights.
``--model medium`` and ``--model xl`` run those sizes with their scheduler workloads (32 mixed
requests with prompts in portions of 512; 64 requests side by side at temperature 1.0).

The reference's counterparts are ``engine/bench/bench_batch.c:24-122`` (batched decode:
prefill untimed, one warm-up step, then timed steps) and ``engine/bench/bench.c`` (prefill).
"""

from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# The headline configuration: GPT-2 small.  Layers may be reduced with --layers where time or
# memory needs it; the line then names both numbers.
GPT2_SMALL = {"architectures": ["GPT2LMHeadModel"], "model_type": "gpt2", "n_layer": 12, "n_embd": 768, "n_head": 12,
              "n_inner": 3072, "vocab_size": 50257, "n_positions": 1024, "activation_function": "gelu_new",
              "layer_norm_epsilon": 1e-5, "tie_word_embeddings": True}
# The other GPT-2 sizes, for runs beside the headline one (--model).
SIZES = {"small": {}, "medium": {"n_layer": 24, "n_embd": 1024, "n_head": 16, "n_inner": 4096},
         "large": {"n_layer": 36, "n_embd": 1280, "n_head": 20, "n_inner": 5120},
         "xl": {"n_layer": 48, "n_embd": 1600, "n_head": 25, "n_inner": 6400}}
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def parse_args():
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=128)
    parser.add_argument("--warmup", type=int, default=8)
    parser.add_argument("--impl", default="ours", choices=("ours", "reference"))
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    parser.add_argument("--layers", type=int, default=None, help="fewer layers than the model has (named in the line)")
    parser.add_argument("--model", default="small", choices=sorted(SIZES), help="GPT-2 size; the headline run is small")
    parser.add_argument("--plain-kernels", action="store_true")
    parser.add_argument("--no-extras", action="store_true", help="skip prefill, batch 1/64 and the end-to-end run")
    parser.add_argument("--page-size", type=int, default=None, help="tokens per cache page (the engine's default if not given)")
    parser.add_argument("--only-prefill", action="store_true",
                        help="run the 2,048-token prompt step alone and print its own line (for profiling)")
    parser.add_argument("--kernels", action="store_true",
                        help="time single kernels (matrix products at forced tile widths, prompt attention) back to "
                             "back in a replayed graph and print one line each: the tables of profiles/ come from this")
    parser.add_argument("--compare", default=None, choices=("fuvolix", "sumozen", "lipulorn", "deluvik", "nufavik", "kerepel"),
                        help="fuvolix: prefill and decode of Fuvolix stacks at sizes of real layers (random weights), beside "
                             "GPT-2 of equal width, depth and inner size, and their mixers' kernels alone; sumozen: Sumozen "
                             "stacks beside Fuvolix stacks of equal width, depth and inner size, and its kernels alone; "
                             "lipulorn: Lipulorn stacks beside Fuvolix stacks of equal width, depth and feed-forward weights, and "
                             "its kernels alone beside the like kernels of Fuvolix and Sumozen; deluvik: Deluvik stacks beside "
                             "Sumozen stacks of equal width, depth and experts, and its kernels alone beside Sumozen's like kernels; "
                             "nufavik: Nufavik stacks beside Deluvik stacks of equal width, depth, heads and experts, and its kernels "
                             "alone beside Deluvik's like kernels; "
                             "kerepel: Kerepel stacks beside Deluvik stacks of equal width, depth, heads and feed-forward weights, and its "
                             "kernels alone beside the closest designs' like kernels; "
                             "one line each")
    parser.add_argument("--tokens-out", default=None,
                        help="(--impl reference) write the greedy tokens of the fixed check workload to this file "
                             "and print nothing else")
    return parser.parse_args()


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as handle:
                raw = json.load(handle)
            out = dict(FALLBACK_PEAKS)
            for key in out:
                if isinstance(raw.get(key), (int, float)):
                    out[key] = float(raw[key])
            out["source"] = "measured"
            return out
        except (OSError, ValueError):
            pass
    return {**FALLBACK_PEAKS, "source": "fallback"}


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
    NAMES = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")

    def __init__(self):
        self.process = None
        self.file = None

    def start(self):
        try:
            self.file = tempfile.NamedTemporaryFile("w+", suffix=".csv", delete=False)
            self.process = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                             "-i", "0", "-lms", "100"], stdout=self.file, stderr=subprocess.DEVNULL)
        except OSError:
            self.process = None

    def stop(self) -> dict:
        if self.process is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.process.terminate()
        self.process.wait()
        self.file.flush()
        self.file.seek(0)
        clocks, top, reasons = [], None, set()
        for line in self.file.read().splitlines():
            cells = [c.strip() for c in line.split(",")]
            if len(cells) < 6:
                continue
            try:
                clocks.append(float(cells[0]))
                top = float(cells[1])
            except ValueError:
                continue
            for name, cell in zip(self.NAMES, cells[2:6]):
                if cell.lower().startswith("active"):
                    reasons.add(name)
        self.file.close()
        os.unlink(self.file.name)
        return {"sm_mhz": statistics.median(clocks) if clocks else None, "sm_max_mhz": top,
                "reasons": sorted(reasons), "samples": len(clocks)}


def model_numbers(config: dict, dtype_bytes: int):
    e, i, v, layers = config["n_embd"], config["n_inner"], config["vocab_size"], config["n_layer"]
    matrix_params = layers * (e * 3 * e + e * e + 2 * e * i)
    vector_params = layers * (3 * e + e + i + e + 4 * e) + 2 * e
    weight_bytes = (matrix_params + v * e) * dtype_bytes + vector_params * 4      # every weight a decode step uses, once
    kv_bytes_per_token = layers * 2 * e * dtype_bytes
    return matrix_params, weight_bytes, kv_bytes_per_token


def prefill_flops(config: dict, n_prompts: int, length: int, wanted_rows: int) -> float:
    e, v, layers = config["n_embd"], config["vocab_size"], config["n_layer"]
    matrix_params, _, _ = model_numbers(config, 2)
    tokens = n_prompts * length
    gemm = 2.0 * tokens * matrix_params
    attention = layers * n_prompts * 2.0 * length * length * e          # causal half of QK^T and PV
    head = 2.0 * wanted_rows * v * e
    return gemm + attention + head


def make_model_folder(config: dict, folder: str) -> str:
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.weights import write_random_model
    return write_random_model(config_from_dict(config), 0, folder, recipe="gpt2", store_dtype="float32")


def decode_run(engine, batch: int, steps: int, warmup: int, context: int, vocab: int):
    """Device-timed decode: ``batch`` requests prefilled so that the timed steps end at
    ``context`` tokens.  Token ids are fixed in advance (nothing is read back inside the timed
    region); every step samples greedily on the device.  Returns (ms per step, launches per
    step, mean cached tokens per request during the timed steps)."""
    import numpy as np
    import torch
    from mini_llm_b200.engine import SamplingParams, StepEntry

    rng = np.random.default_rng(1234)
    prompt_len = context - steps - warmup
    if prompt_len < 1:
        raise SystemExit(f"--steps + --warmup must stay below the context length {context}")
    slots = [engine.open_request() for _ in range(batch)]
    for slot in slots:                                   # untimed prefill, one request per step
        engine.step([StepEntry(slot, rng.integers(0, vocab, prompt_len).tolist(), [])])
    feed = rng.integers(0, vocab, (steps + warmup, batch))
    greedy = [SamplingParams() for _ in range(batch)]

    def one(index):
        engine.step([StepEntry(slot, [int(feed[index, b])], [0]) for b, slot in enumerate(slots)], greedy)

    for index in range(warmup):
        one(index)
    torch.cuda.synchronize()
    launches_before = engine.kernels.launches
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for index in range(warmup, warmup + steps):
        one(index)
    stop.record()
    torch.cuda.synchronize()
    ms = start.elapsed_time(stop) / steps
    launches = (engine.kernels.launches - launches_before) / steps
    for slot in slots:
        engine.close_request(slot)
    mean_cached = prompt_len + warmup + (steps - 1) / 2.0
    return ms, launches, mean_cached


def prefill_run(engine, n_prompts: int, length: int, vocab: int, repeats: int = 5, from_idle: bool = False):
    """Milliseconds of one prompt step of ``n_prompts`` x ``length`` tokens.  The steps run one
    behind the other (a step's host work, the filling of its control block, then falls beside
    the step before it on the GPU, as in serving) between two events with a synchronise on
    both sides; the first five steps, which run eagerly and capture the graph, are not timed.
    ``from_idle``: each step alone instead, from an idle GPU, host work included (the median)."""
    import numpy as np
    import torch
    from mini_llm_b200.engine import StepEntry

    rng = np.random.default_rng(99)
    prompts = [rng.integers(0, vocab, length).tolist() for _ in range(n_prompts)]

    def one_step():
        slots = [engine.open_request() for _ in range(n_prompts)]
        engine.step([StepEntry(slot, prompt, [length - 1]) for slot, prompt in zip(slots, prompts)])
        for slot in slots:
            engine.close_request(slot)

    for _ in range(5):
        one_step()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if from_idle:
        times = []
        for _ in range(repeats):
            torch.cuda.synchronize()
            start.record()
            one_step()
            stop.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(stop))
        return statistics.median(times)
    torch.cuda.synchronize()
    start.record()
    for _ in range(repeats):
        one_step()
    stop.record()
    torch.cuda.synchronize()
    return start.elapsed_time(stop) / repeats


def e2e_run(folder, args, context: int, vocab: int):
    """The same decode metric through ``LLM.generate``: prompts go in as host token ids, every
    step uploads its control block from pinned host memory and reads the sampled ids back."""
    import numpy as np
    from mini_llm_b200.generate import LLM

    steps, warmup, batch = args.steps, args.warmup, args.batch
    rng = np.random.default_rng(4321)
    prompt_len = context - steps - warmup
    prompts = [rng.integers(0, vocab, prompt_len).tolist() for _ in range(batch)]
    # every prompt is admitted in the first step, so that all requests decode side by side to the end
    llm = LLM(folder, dtype=args.dtype, max_sessions=batch, cache_tokens=batch * context,
              max_tokens_per_step=batch * context, plain_kernels=args.plain_kernels)
    best = None
    for _ in range(2):                                     # the better of two runs (the host is a shared machine)
        stamps, uploads = [], []

        def on_token(index, token, reason):
            if index == batch - 1:
                stamps.append(time.perf_counter())
                uploads.append(llm.engine.control.last_upload_bytes)

        out = llm.generate(prompts, max_new_tokens=steps + warmup, temperature=0.0, on_token=on_token)
        assert all(len(tokens) == steps + warmup for tokens in out)
        seconds = stamps[-1] - stamps[warmup - 1]              # K steps after the warm-up steps
        if best is None or seconds < best[0]:
            best = (seconds, uploads[len(uploads) // 2])       # and the control block of a decode step, as copied
    seconds, control_bytes = best
    return {"value": batch * steps / seconds, "unit": "tokens/s", "h2d_bytes_per_step": control_bytes,
            "d2h_bytes_per_step": 4 * batch + 4, "ms_per_step": 1000.0 * seconds / steps, "runs": 2}


def serving_run(folder, args, vocab: int):
    """Tokens a second through the scheduler for a mixed workload: 64 requests, prompts of 16 to
    768 tokens, 32 to 256 new tokens each, temperature 0.8 and top-p 0.95, at most 32 live, a
    token budget of 512 per step (prompts in portions beside decoding requests)."""
    import numpy as np
    import torch
    from mini_llm_b200.engine.scheduler import Request
    from mini_llm_b200.generate import LLM

    rng = np.random.default_rng(3)
    prompts = [rng.integers(0, vocab, int(rng.integers(16, 769))).tolist() for _ in range(64)]
    lengths = [int(rng.integers(32, 257)) for _ in range(64)]
    llm = LLM(folder, dtype=args.dtype, max_sessions=32, cache_tokens=24 * 1024, max_tokens_per_step=512,
              max_prefill_chunk=512, plain_kernels=args.plain_kernels)
    # The same 64 requests pass after pass: a step shape with prompt portions is captured as a
    # CUDA graph the second time it is seen, so the first passes run some steps eagerly and pay
    # for captures; the passes go on until one ran every step from a graph or the one kernel
    # (eight at most).  Returns the first pass's and the best pass's tokens a second and the
    # number of passes.
    first, best, passes = 0.0, 0.0, 0
    for _ in range(8):
        requests = [Request(p, n, None, 0.8, 0.95, 100 + i) for i, (p, n) in enumerate(zip(prompts, lengths))]
        before = dict(llm.engine.step_kinds)
        torch.cuda.synchronize()
        start = time.perf_counter()
        for request in requests:
            llm.scheduler.submit(request)
        llm.scheduler.run()
        torch.cuda.synchronize()
        seconds = time.perf_counter() - start
        assert all(r.error is None and len(r.generated) == n for r, n in zip(requests, lengths))
        passes += 1
        rate = sum(lengths) / seconds
        first = first or rate
        best = max(best, rate)
        if all(llm.engine.step_kinds[kind] == before[kind] for kind in ("eager", "captured")):
            break
    return first, best, passes


def scheduled_decode_run(folder, args, batch: int, prompt_len: int, new_tokens: int, page_size: int, context: int,
                         vocab: int, weight_bytes: float, kv_per_token: float, hbm_gbs: float):
    """The decode workload as the target states it: ``batch`` requests, each a prompt of
    ``prompt_len`` uniform ids, ``new_tokens`` greedy tokens through the scheduler
    (``LLM.generate``), pages of ``page_size`` tokens.  The prompts are prefilled outside the
    timing: the clock runs from every request's first token to its last, host tokens out
    every step (the reference's bench_batch times its steps after untimed prefills too,
    engine/bench/bench_batch.c:74-114).  Returns tokens a second and the fraction of the HBM
    roofline at the mean context."""
    import numpy as np
    from mini_llm_b200.generate import LLM

    rng = np.random.default_rng(77 + batch)
    prompts = [rng.integers(0, vocab, prompt_len).tolist() for _ in range(batch)]
    llm = LLM(folder, dtype=args.dtype, page_size=page_size, max_sessions=batch, cache_tokens=batch * context,
              max_tokens_per_step=max(2048, batch * prompt_len), plain_kernels=args.plain_kernels)
    best = None
    for _ in range(2):                                  # the second pass finds its step shapes captured
        stamps = []

        def on_token(index, token, reason):
            if index == batch - 1:
                stamps.append(time.perf_counter())

        out = llm.generate(prompts, max_new_tokens=new_tokens, temperature=0.0, on_token=on_token)
        assert all(len(tokens) == new_tokens for tokens in out)
        seconds = stamps[-1] - stamps[0]                  # new_tokens - 1 decode steps
        best = seconds if best is None else min(best, seconds)
    steps = new_tokens - 1
    mean_context = prompt_len + new_tokens / 2.0
    step_bytes = weight_bytes + batch * mean_context * kv_per_token
    return batch * steps / best, step_bytes / (best / steps) / 1e9 / hbm_gbs


def workload_run(folder, args, vocab: int, context: int, n_requests: int, prompt_range, output_range, live: int,
                 budget: int, chunk: int, temperature: float, top_p: float, page_size: int):
    """A workload through the continuous-batching scheduler: ``n_requests`` requests with
    seeded prompt and output lengths, at most ``live`` at a time, a token budget per step and
    prompts in portions of at most ``chunk`` tokens beside decoding requests.  Returns
    generated tokens a second (wall clock, host tokens in and out) and the scheduler's
    counters."""
    import numpy as np
    import torch
    from mini_llm_b200.engine.scheduler import Request
    from mini_llm_b200.generate import LLM

    rng = np.random.default_rng(3)
    prompts = [rng.integers(0, vocab, int(rng.integers(prompt_range[0], prompt_range[1] + 1))).tolist()
               for _ in range(n_requests)]
    lengths = [int(rng.integers(output_range[0], output_range[1] + 1)) for _ in range(n_requests)]
    llm = LLM(folder, dtype=args.dtype, page_size=page_size, max_sessions=live, cache_tokens=live * context,
              max_tokens_per_step=budget, max_prefill_chunk=chunk, plain_kernels=args.plain_kernels)
    best, stats = 0.0, {}
    for _ in range(2):                                   # the second pass finds its step shapes captured
        requests = [Request(p, n, None, temperature, top_p, 100 + i) for i, (p, n) in enumerate(zip(prompts, lengths))]
        before = dict(llm.scheduler.counters)
        torch.cuda.synchronize()
        start = time.perf_counter()
        for request in requests:
            llm.scheduler.submit(request)
        llm.scheduler.run()
        torch.cuda.synchronize()
        seconds = time.perf_counter() - start
        assert all(r.error is None and len(r.generated) == n for r, n in zip(requests, lengths))
        if sum(lengths) / seconds > best:
            best = sum(lengths) / seconds
            after = llm.scheduler.counters
            steps = after["steps"] - before.get("steps", 0)
            tokens = (after["prefill_tokens"] + after["decode_tokens"] - before.get("prefill_tokens", 0)
                      - before.get("decode_tokens", 0))
            stats = {"steps": steps, "tokens_per_step": tokens / max(1, steps),
                     "preemptions": after["preemptions"] - before.get("preemptions", 0),
                     "pages": llm.engine.cache.groups[0].pool.n_pages}
    return best, stats


CHECK_PROMPT_SEED, CHECK_PROMPT_TOKENS, CHECK_NEW_TOKENS = 2024, 32, 16


def check_prompt(vocab: int):
    import numpy as np
    return np.random.default_rng(CHECK_PROMPT_SEED).integers(0, vocab, CHECK_PROMPT_TOKENS).tolist()


def compare_with_reference(folder, vocab: int) -> dict:
    """Whether the two arms choose the same greedy tokens: the 32-bit path of this engine and
    the reference's 32-bit GPU path, same seeded weights, a prompt of 32 ids and 16 new tokens.
    The reference runs in a process of its own (``--impl reference --tokens-out``)."""
    from mini_llm_b200.generate import generate
    if not os.path.isdir(os.path.join(REFERENCE, "mini_llm")):
        return {"unavailable": "the reference is not installed under baseline/_ref"}
    with tempfile.TemporaryDirectory() as scratch:
        path = os.path.join(scratch, "tokens.json")
        try:
            done = subprocess.run([sys.executable, os.path.abspath(__file__), "--impl", "reference", "--tokens-out", path],
                                  capture_output=True, text=True, timeout=600)
        except subprocess.TimeoutExpired:
            return {"unavailable": "the reference did not finish in ten minutes"}
        if done.returncode != 0 or not os.path.isfile(path):
            return {"unavailable": (done.stdout.strip() or done.stderr.strip())[-200:]}
        with open(path) as handle:
            theirs = json.load(handle)["tokens"]
    (mine,) = generate(folder, [check_prompt(vocab)], max_new_tokens=CHECK_NEW_TOKENS, temperature=0.0, dtype="float32",
                       page_size=16, max_sessions=2, cache_tokens=1024)
    same = 0
    while same < len(mine) and mine[same] == theirs[same]:
        same += 1
    return {"agree": same, "of": len(mine)}


def run_ours(args):
    import torch
    from mini_llm_b200.engine import Engine

    config = dict(GPT2_SMALL, **SIZES[args.model])
    layers_of_model = config["n_layer"]
    if args.layers is not None:
        config["n_layer"] = args.layers
    context, vocab = config["n_positions"], config["vocab_size"]
    dtype_bytes = 2 if args.dtype == "bfloat16" else 4
    peak = peaks()
    with tempfile.TemporaryDirectory() as folder:
        make_model_folder(config, folder)
        engine = Engine(folder, dtype=args.dtype, max_requests=64, cache_tokens=64 * context,
                        max_tokens_per_step=2048, plain_kernels=args.plain_kernels,
                        **({"page_size": args.page_size} if args.page_size else {}))
        _, weight_bytes, kv_per_token = model_numbers(config, dtype_bytes)

        if args.only_prefill:
            prefill_ms = prefill_run(engine, 2, 1024, vocab, repeats=max(1, args.steps))
            idle_ms = prefill_run(engine, 2, 1024, vocab, repeats=max(1, min(args.steps, 20)), from_idle=True)
            print(json.dumps({"metric": "prefill of 2,048 tokens", "ms": prefill_ms, "ms_from_idle": idle_ms,
                              "n_layer": config["n_layer"], "value": 2048 / (prefill_ms * 1e-3), "unit": "tokens/s"}))
            return 0
        sampler = ClockSampler()
        sampler.start()
        ms, launches, mean_cached = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
        clocks = sampler.stop()
        step_bytes = weight_bytes + args.batch * mean_cached * kv_per_token
        achieved = step_bytes / (ms * 1e-3) / 1e9
        line = {
            "metric": f"decode tokens/s, GPT-2 {args.model}, batch {args.batch}, context {context}", "value": args.batch / (ms * 1e-3),
            "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "ms_per_step": ms,
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16" if dtype_bytes == 2 else "fp32",
            "data": "synthetic: seeded random weights (N(0, 0.02)) and uniform random token ids", "impl": "ours",
            "config": {"model": f"gpt2-{args.model}", "n_layer": config["n_layer"], "n_layer_of_model": layers_of_model,
                       "n_embd": config["n_embd"], "n_head": config["n_head"], "n_inner": config["n_inner"],
                       "vocab_size": vocab, "n_positions": context, "global_batch": args.batch, "seq_len": context,
                       "prompt_tokens": context - args.steps - args.warmup, "page_size": engine.page_size,
                       "parallelism": "single GPU", "l2": "inputs larger than L2 (weights + cache per step)",
                       "peaks": peak["source"]},
            "gpu_launches": int(round(launches * args.steps)),
            "roofline": {"bound": "hbm", "achieved": achieved, "peak": peak["hbm_gbs"], "unit": "GB/s",
                         "frac": achieved / peak["hbm_gbs"], "bytes_per_step": step_bytes},
            "clocks": clocks,
        }
        if not args.no_extras:
            points = {}
            for batch in (1, 64):
                p_ms, _, _ = decode_run(engine, batch, min(args.steps, 64), max(3, min(args.warmup, 8)), context, vocab)
                points[f"decode_b{batch}"] = batch / (p_ms * 1e-3)
            line["points"] = points
            # K steps one behind the other between two events; and one step alone from an idle GPU,
            # which also holds the host's filling of the step's control block
            prefill_ms = prefill_run(engine, 2, 1024, vocab, repeats=32)
            idle_ms = prefill_run(engine, 2, 1024, vocab, repeats=7, from_idle=True)
            flops = prefill_flops(config, 2, 1024, 2)
            peak_flops = (peak["bf16_tflops"] if dtype_bytes == 2 else peak["bf16_tflops"]) * 1e12
            line["prefill"] = {"value": 2048 / (prefill_ms * 1e-3), "tokens": 2048, "ms": prefill_ms,
                               "frac": flops / (prefill_ms * 1e-3) / peak_flops, "flops": flops, "steps": 32,
                               "ms_from_idle": idle_ms}
            line["device"] = engine.device_info()
            del engine
            torch.cuda.empty_cache()
            line["e2e"] = e2e_run(folder, args, context, vocab)
            points = line["points"]
            if args.model == "small" and args.layers is None:
                # the decode workload as stated: 512-token prompts, 256 greedy tokens, pages of 16, through the scheduler
                for batch in (1, 8, 64):
                    value, frac = scheduled_decode_run(folder, args, batch, 512, 256, 16, context, vocab, weight_bytes,
                                                       kv_per_token, peak["hbm_gbs"])
                    points[f"sched_p16_b{batch}"] = value
                    points[f"sched_p16_b{batch}_hbm_frac"] = frac
                first, best, passes = serving_run(folder, args, vocab)
                points["serve_mixed_64"], points["serve_mixed_64_first_pass"], points["serve_mixed_64_passes"] = best, first, passes
                if args.dtype == "bfloat16":
                    # the true 32-bit path: the same decode step and prompt step through the plain kernels
                    plain = Engine(folder, dtype="float32", max_requests=8, cache_tokens=8 * context, max_tokens_per_step=2048)
                    f_ms, _, _ = decode_run(plain, 8, 16, 3, context, vocab)
                    points["decode_b8_float32"] = 8 / (f_ms * 1e-3)
                    points["prefill_2048_float32"] = 2048 / (prefill_run(plain, 2, 1024, vocab, repeats=2) * 1e-3)
                    del plain
                    torch.cuda.empty_cache()
                    line["reference_tokens"] = compare_with_reference(folder, vocab)
            elif args.model == "medium":
                # 32 requests, prompts of 16 to 768 tokens, 32 to 256 new tokens, prompts in portions of 512
                value, stats = workload_run(folder, args, vocab, context, 32, (16, 768), (32, 256), 32, 512, 512, 0.0, 1.0, 16)
                points["sched_medium_32"] = value
                points.update({f"sched_medium_32_{k}": v for k, v in stats.items()})
            elif args.model == "xl":
                # 64 requests side by side, 256-token prompts and 768 new tokens each, temperature 1.0, pages of 16
                value, stats = workload_run(folder, args, vocab, context, 64, (256, 256), (768, 768), 64, 2048, 2048, 1.0,
                                            1.0, 16)
                points["sched_xl_64"] = value
                points.update({f"sched_xl_64_{k}": v for k, v in stats.items()})
    print(json.dumps(line))
    return 0


REFERENCE = os.path.join(ROOT, "baseline", "_ref")


def unavailable(why: str) -> int:
    print(json.dumps({"impl": "reference", "unavailable": why}))
    return 0


def build_reference_library(target: str) -> str | None:
    """The reference's ``make gpu-lib`` (Makefile:165-180 of WillyBruhn/mini_llm) with its
    sources unchanged and only the target architecture replaced (it names sm_86 and sm_61)."""
    import glob
    import shutil
    engine = os.path.join(REFERENCE, "engine")
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.isdir(engine) or not os.path.isfile(nvcc):
        return "the reference's engine sources or nvcc are missing"
    pic = os.path.join(REFERENCE, "build", "pic")
    os.makedirs(pic, exist_ok=True)
    include = ["-I" + os.path.join(engine, "include"), "-I" + os.path.join(engine, "tests")]
    objects = []
    for source in sorted(glob.glob(os.path.join(engine, "src", "*.c"))):
        obj = os.path.join(pic, os.path.basename(source)[:-2] + ".o")
        done = subprocess.run(["gcc", "-O2", "-std=c11", *include, "-fPIC", "-c", "-o", obj, source], capture_output=True)
        if done.returncode != 0:
            return "gcc failed on the reference's sources"
        objects.append(obj)
    done = subprocess.run([nvcc, "-O2", "-lineinfo", "-gencode", "arch=compute_100a,code=sm_100a", *include, "-Xcompiler",
                           "-fPIC", "-shared", "-o", target, *sorted(glob.glob(os.path.join(engine, "src", "*.cu"))),
                           *objects, "-lm"], capture_output=True)
    return None if done.returncode == 0 else "nvcc failed on the reference's sources"


def export_reference_weights(config: dict, folder: str) -> None:
    """The same seeded random weights as our arm, in the reference's format: one raw
    little-endian fp32 file per tensor, named ``transformer.<name>.bin``
    (scripts/dump_weights.py:37-53, engine/src/gpt2.c:21-34,131-137)."""
    from mini_llm_b200.config import config_from_dict, describe_model
    from mini_llm_b200.weights import random_tensors
    for name, values in random_tensors(describe_model(config_from_dict(config)), 0, "gpt2").items():
        values.astype("<f4").tofile(os.path.join(folder, f"transformer.{name}.bin"))


def run_reference(args):
    """The unmodified reference through its own public API: ``NativeGPT2`` (ctypes binding),
    ``prefill_greedy`` per request, then ``decode_batch`` steps
    (pytorch/src/mini_llm/batch_api.py:44-70), fp16 decode weights as in its published runs."""
    if not os.path.isdir(os.path.join(REFERENCE, "mini_llm")):
        return unavailable("the reference is not installed under baseline/_ref")
    if args.batch > 16:
        return unavailable("the reference's batched decode takes at most 16 sequences")
    library = os.path.join(REFERENCE, "build", "libmini_llm_gpu.so")
    if not os.path.isfile(library):
        problem = build_reference_library(library)
        if problem:
            return unavailable(problem)
    import numpy as np
    import torch
    if not torch.cuda.is_available():
        return unavailable("no CUDA device")
    sys.path.insert(0, REFERENCE)
    try:
        from mini_llm.native import EngineOptions, NativeGPT2
    except Exception as error:
        return unavailable(f"the reference's binding does not import: {error}")
    config = dict(GPT2_SMALL)                # the reference's sizes are compile-time constants: GPT-2 small only
    context, vocab = config["n_positions"], config["vocab_size"]
    steps, warmup, batch = args.steps, args.warmup, args.batch
    prompt_len = context - steps - warmup
    rng = np.random.default_rng(1234)
    with tempfile.TemporaryDirectory() as folder:
        export_reference_weights(config, folder)
        engine = NativeGPT2(folder, library, backend="gpu",
                            options=EngineOptions(use_kv_cache=True, max_sessions=16, fp16_decode=not args.tokens_out))
    if args.tokens_out:
        # the fixed check workload, 32-bit weights: greedy tokens for the other arm to compare with
        cache = engine.try_take_cache()
        tokens = [engine.prefill_greedy(cache, check_prompt(vocab))]
        while len(tokens) < CHECK_NEW_TOKENS:
            tokens.append(engine.decode_batch([cache], [tokens[-1]])[0])
        engine.release_cache(cache)
        engine.close()
        with open(args.tokens_out, "w") as handle:
            json.dump({"tokens": [int(t) for t in tokens]}, handle)
        return 0
    sampler = ClockSampler()
    caches = [engine.try_take_cache() for _ in range(batch)]
    tokens = [engine.prefill_greedy(cache, rng.integers(0, vocab, prompt_len).tolist()) for cache in caches]
    for _ in range(warmup):
        tokens = engine.decode_batch(caches, tokens)
    torch.cuda.synchronize()
    sampler.start()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    wall = time.perf_counter()
    start.record()
    for _ in range(steps):
        tokens = engine.decode_batch(caches, tokens)       # host tokens in and out, every step
    stop.record()
    torch.cuda.synchronize()
    wall = time.perf_counter() - wall
    clocks = sampler.stop()
    ms = start.elapsed_time(stop) / steps
    for cache in caches:
        engine.release_cache(cache)
    line = {"metric": f"decode tokens/s, GPT-2 {args.model}, batch {args.batch}, context {context}", "value": batch / (ms * 1e-3),
            "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": ms,
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "fp16 weights, fp32 arithmetic",
            "data": "synthetic: seeded random weights (N(0, 0.02)) and uniform random token ids", "impl": "reference",
            "config": {"model": "gpt2-small", "n_layer": 12, "n_embd": 768, "n_head": 12, "n_inner": 3072,
                       "vocab_size": vocab, "n_positions": context, "global_batch": batch, "seq_len": context,
                       "prompt_tokens": prompt_len, "parallelism": "single GPU", "arch": "sources rebuilt for sm_100a"},
            "e2e": {"value": batch * steps / wall, "unit": "tokens/s", "h2d_bytes_per_step": 4 * batch,
                    "d2h_bytes_per_step": 4 * batch},
            "clocks": clocks}
    if not args.no_extras:
        cache = engine.try_take_cache()
        token = engine.prefill_greedy(cache, rng.integers(0, vocab, prompt_len).tolist())
        torch.cuda.synchronize()
        begin = time.perf_counter()
        for _ in range(min(steps, 64)):
            token = engine.decode_batch([cache], [token])[0]
        torch.cuda.synchronize()
        line["points"] = {"decode_b1": min(steps, 64) / (time.perf_counter() - begin)}
        engine.release_cache(cache)
        cache = engine.try_take_cache()
        prompts = [rng.integers(0, vocab, 1024).tolist() for _ in range(2)]
        torch.cuda.synchronize()
        begin = time.perf_counter()
        for prompt in prompts:                               # a prompt is never batched: one after the other
            engine.prefill_greedy(cache, prompt)
        torch.cuda.synchronize()
        seconds = time.perf_counter() - begin
        line["prefill"] = {"value": 2048 / seconds, "tokens": 2048, "ms": 1000.0 * seconds}
        engine.release_cache(cache)
    engine.close()
    print(json.dumps(line))
    return 0


def replayed_us(torch, launch, repeats=12):
    """Microseconds per call of ``launch(i)``, i = 0 .. repeats - 1 (each on operands of its own,
    so that nothing stays in L2 from call to call), captured once and replayed: the best of five."""
    import gc
    launch(0)
    torch.cuda.synchronize()
    gc.collect()             # a graph of an earlier call that is freed while this one is captured would end the capture
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(repeats):
            launch(i)
    for _ in range(3):
        graph.replay()
    torch.cuda.synchronize()
    first, last = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    best = float("inf")
    for _ in range(5):
        first.record()
        graph.replay()
        last.record()
        torch.cuda.synchronize()
        best = min(best, first.elapsed_time(last) * 1000.0 / repeats)
    graph.reset()
    return best


def run_kernels():
    """Single kernels at the sizes the profiles quote: the residual-sum product at every tile
    code the launcher knows (0: its own choice), and the prompt attention with one and with two
    tiles per CTA.  One JSON line per measurement."""
    import math
    import torch
    from mini_llm_b200.kernels import ops
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    codes = (0, 2064, 2096, 2128, 192, 256, 7002, 7004, 7102, 7104)
    shapes = ((640, 768, 3072), (1024, 768, 3072), (1536, 768, 3072), (2048, 768, 3072), (4096, 768, 3072),
              (2048, 768, 768), (1024, 1024, 4096), (2048, 1024, 4096), (1024, 1600, 6400), (2048, 1600, 6400))
    for m, n, k in shapes:
        xs = [torch.randn(m, k, device="cuda").bfloat16() for _ in range(12)]
        ws = [(torch.randn(n, k, device="cuda") / math.sqrt(k)).bfloat16() for _ in range(12)]
        bias, out = torch.randn(n, device="cuda"), torch.zeros(m, n, device="cuda")
        for code in codes:
            def launch(i, code=code):
                if code == 0:
                    ops.gemm_bf16(out, xs[i], ws[i], bias, "add", status)
                else:
                    ops.gemm_bf16_tile(out, xs[i], ws[i], bias, "add", status, code)
            print(json.dumps({"kernel": "gemm, residual sum", "m": m, "n": n, "k": k, "tile_code": code,
                              "us": round(replayed_us(torch, launch), 2)}), flush=True)
    heads, head, page = 12, 64, 64
    work = torch.zeros(2, dtype=torch.int32, device="cuda")
    for name, lengths, new in (("2 x 1024", [1024, 1024], [1024, 1024]), ("1 x 1024", [1024], [1024]),
                               ("4 x 512", [512] * 4, [512] * 4), ("8 x 256 after 768", [1024] * 8, [256] * 8),
                               ("700 + 300 + 1000 + 48 after 976", [700, 300, 1000, 1024], [700, 300, 1000, 48])):
        blocks = [-(-length // page) for length in lengths]
        k_pages = torch.randn(sum(blocks) + 1, page, heads, head, device="cuda").bfloat16()
        v_pages = torch.randn(sum(blocks) + 1, page, heads, head, device="cuda").bfloat16()
        table = torch.zeros(len(lengths), max(blocks), dtype=torch.int32)
        at = 0
        for i, count in enumerate(blocks):
            table[i, :count] = torch.arange(at, at + count, dtype=torch.int32)
            at += count
        table = table.cuda()
        q = torch.randn(sum(new), heads * head, device="cuda").bfloat16()
        out = torch.empty_like(q)
        offsets = [sum(new[:i]) for i in range(len(new))]
        starts = [length - count for length, count in zip(lengths, new)]
        tiles, _, _ = ops.attention_tiles(offsets, new, starts, split=False)
        tiles_d = torch.tensor(tiles, dtype=torch.int32, device="cuda")
        units, n_split, most = ops.attention_units(offsets, new, starts, heads, torch.cuda.get_device_properties(0).multi_processor_count)
        units_d = torch.tensor(units, dtype=torch.int32, device="cuda")
        scratch = None
        if n_split:
            scratch = (torch.empty(n_split * heads * most * ops.ATTENTION_UNIT * (head + 4), device="cuda"),
                       torch.zeros(2 * n_split * heads, dtype=torch.int32, device="cuda"))
        one = replayed_us(torch, lambda i: ops.attention_prefill(out, q, k_pages, v_pages, table, tiles_d, len(tiles), heads, heads,
                                                                head, page, 0.125, 0, status, work))
        two = replayed_us(torch, lambda i: ops.attention_prefill_two_tiles(out, q, k_pages, v_pages, table, units_d, len(units), heads,
                                                                          heads, head, page, 0.125, 0, status, work, scratch, n_split,
                                                                          most))
        print(json.dumps({"kernel": "prompt attention, 12 heads of 64", "prompts": name, "one_tile_per_cta_us": round(one, 2),
                          "two_tiles_per_cta_us": round(two, 2)}), flush=True)
    if int(status.item()) != 0:
        print(json.dumps({"error": "a bounded wait inside a kernel ran out", "status": int(status.item())}))
        return 1
    return 0


# Fuvolix stacks beside GPT-2 of equal width, depth and inner size: layers in threes (attention over a
# latent with a feed-forward, a gated matrix memory, a decaying matrix memory with a feed-forward).
FUVOLIX_SIZES = {
    "small": {"width": 768, "layers": 12, "ff": 3072, "gpt2": "small",
              "latent": {"heads": 12, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256},
              "mlstm": {"heads": 4, "dim": 96, "vdim": 192}, "lightning": {"heads": 12, "dim": 64, "vdim": 64}},
    "medium": {"width": 1024, "layers": 24, "ff": 4096, "gpt2": "medium",
               "latent": {"heads": 16, "dim": 64, "rot_dim": 64, "vdim": 64, "kv_rank": 512},
               "mlstm": {"heads": 4, "dim": 128, "vdim": 256}, "lightning": {"heads": 16, "dim": 64, "vdim": 64}},
}
FP32_FMA_TFLOPS_NOMINAL = 148 * 128 * 2 * 1.965e9 / 1e12      # 32-bit FMA of 148 SMs at the highest clock: no measured figure exists


def fuvolix_config(size: dict, vocab: int) -> dict:
    lat, mem, lit = size["latent"], size["mlstm"], size["lightning"]
    three = [
        {"type": "latent_attention", "mlp": {"kind": "dense", "ff": size["ff"]},
         "mixer": dict(lat, scale=(lat["dim"] + lat["rot_dim"]) ** -0.5, rot={"base": 10000.0, "dims": lat["rot_dim"]})},
        {"type": "mlstm", "mlp": None, "mixer": dict(mem, gate_cap=15.0)},
        {"type": "lightning", "mlp": {"kind": "dense", "ff": size["ff"]},
         "mixer": dict(lit, decay=[1.0 - 2.0 ** -(2 + 6 * h / max(lit["heads"] - 1, 1)) for h in range(lit["heads"])])},
    ]
    return {"architecture": "Fuvolix", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5, "groups": 4},
            "canon": {"taps": 4}, "layers": [three[i % 3] for i in range(size["layers"])]}


def mixer_kernels(torch, size: dict, peak: dict, memories=("mlstm", "lightning")):
    """The mixers' kernels alone, replayed back to back on operands of their own: prompt portions
    (2 x 1,024 tokens) and single tokens (8 requests at 1,023 cached tokens), each with the work it
    must do and the fraction of its bound: 32-bit FMA (nominal) where the sums are 32-bit by the
    design's rule, measured HBM copy bandwidth where the state or the cache is streamed."""
    from mini_llm_b200.kernels import ops
    lines = []
    page, fma_peak = 64, FP32_FMA_TFLOPS_NOMINAL
    dev = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def add(kernel, us, flops=None, bytes_moved=None, **more):
        line = {"kernel": kernel, "us": round(us, 2), **more}
        if flops is not None:
            line.update(tflops=round(flops / us / 1e6, 2), frac_fp32_fma_nominal=round(flops / us / 1e6 / fma_peak, 3))
        if bytes_moved is not None:
            line.update(gbs=round(bytes_moved / us / 1e3, 1), frac_hbm_measured=round(bytes_moved / us / 1e3 / peak["hbm_gbs"], 3))
        lines.append(line)

    # ---- attention over the latent, beside GPT-2's attention of as many heads of 64 ----
    lat = size["latent"]
    heads, rank, rot = lat["heads"], lat["kv_rank"], lat["rot_dim"]
    row = rank + rot
    for name, lengths, new in (("prompts, 2 x 1024", [1024, 1024], [1024, 1024]), ("single tokens, 8 x 1024", [1024] * 8, [1] * 8)):
        blocks = [-(-n // page) for n in lengths]
        table = torch.zeros(len(lengths), max(blocks), dtype=torch.int32)
        at = 0
        for i, count in enumerate(blocks):
            table[i, :count] = torch.arange(at, at + count, dtype=torch.int32)
            at += count
        table = table.cuda()
        n = sum(new)
        offsets = [sum(new[:i]) for i in range(len(new))]
        starts = [length - count for length, count in zip(lengths, new)]
        positions = torch.cat([torch.arange(s, s + m) for s, m in zip(starts, new)]).int().cuda()
        token_item = torch.cat([torch.full((m,), i) for i, m in enumerate(new)]).int().cuda()
        pairs = sum(sum(range(s + 1, s + m + 1)) for s, m in zip(starts, new)) * heads         # (query row, key) pairs
        pages = [torch.randn(sum(blocks) + 1, page, 1, row, device="cuda").bfloat16() for _ in range(4)]
        q_eff = torch.randn(n, heads * row, device="cuda")
        out = torch.empty(n, heads * rank, device="cuda")
        if len(new) == 2:
            tiles, _, _ = ops.attention_tiles(offsets, new, starts, split=False)
            tiles_d = dev(tiles)
            us = replayed_us(torch, lambda i: ops.latent_attention_tiled(out, q_eff, pages[i % 4], table, positions, token_item, heads,
                                                                         rank, rot, page, 0.1, tiles=tiles_d, n_tiles=len(tiles)))
            add(f"latent attention in tiles, {name}", us, flops=2.0 * pairs * (row + rank), heads=heads, row=row)
        else:
            parts = max(1, min(32, 296 // (n * (1 if heads <= 16 else -(-heads // 32)))))
            scratch = (torch.empty(n * heads * parts * rank, device="cuda"), torch.empty(n * heads * parts * 2, device="cuda"))
            us = replayed_us(torch, lambda i: ops.latent_attention_tiled(out, q_eff, pages[i % 4], table, positions, token_item, heads,
                                                                         rank, rot, page, 0.1, parts=parts, scratch=scratch))
            add(f"latent attention in parts, {name}", us, bytes_moved=sum(lengths) * row * 2.0, heads=heads, row=row, parts=parts)
        # GPT-2's kernels at as many heads of 64
        head = 64
        k_pages = [torch.randn(sum(blocks) + 1, page, heads, head, device="cuda").bfloat16() for _ in range(4)]
        v_pages = [torch.randn(sum(blocks) + 1, page, heads, head, device="cuda").bfloat16() for _ in range(4)]
        q = torch.randn(n, heads * head, device="cuda").bfloat16()
        o = torch.empty_like(q)
        status, work = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.zeros(2, dtype=torch.int32, device="cuda")
        if len(new) == 2:
            units, n_split, most = ops.attention_units(offsets, new, starts, heads, torch.cuda.get_device_properties(0).multi_processor_count)
            units_d = dev(units)
            scratch = None
            if n_split:
                scratch = (torch.empty(n_split * heads * most * ops.ATTENTION_UNIT * (head + 4), device="cuda"),
                           torch.zeros(2 * n_split * heads, dtype=torch.int32, device="cuda"))
            us = replayed_us(torch, lambda i: ops.attention_prefill_two_tiles(o, q, k_pages[i % 4], v_pages[i % 4], table, units_d, len(units),
                                                                              heads, heads, head, page, 0.125, 0, status, work, scratch,
                                                                              n_split, most))
            flops = 2.0 * pairs * 2 * head
            lines.append({"kernel": f"GPT-2 attention (tensor cores), {name}", "us": round(us, 2), "tflops": round(flops / us / 1e6, 2),
                          "frac_bf16_measured": round(flops / us / 1e6 / peak["bf16_tflops"], 3), "heads": heads})
        else:
            chunk, reach = 128, table.shape[1] * page
            acc = torch.empty(64 * heads * (reach // 64) * head, device="cuda")
            ml = torch.empty(64 * heads * (reach // 64) * 2, device="cuda")
            counters = torch.zeros(64 * heads, dtype=torch.int32, device="cuda")
            us = replayed_us(torch, lambda i: ops.split_attention(o, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item, heads,
                                                                  heads, head, page, 0.125, 0, chunk, -(-reach // chunk), acc, ml, counters))
            add(f"GPT-2 attention over split keys, {name}", us, bytes_moved=sum(lengths) * heads * head * 2 * 2.0, heads=heads)
    # ---- the matrix memories ----
    for kind in memories:
        mem = size[kind]
        h, dim, vdim = mem["heads"], mem["dim"], mem["vdim"]
        gated = kind == "mlstm"
        floats = ops.memory_state_floats(h, dim, vdim, gated)
        for name, counts, chunked in (("prompts, 2 x 1024", [1024, 1024], "passes"), ("prompts, 2 x 1024", [1024, 1024], True),
                                      ("single tokens, 8", [1] * 8, False)):
            n = sum(counts)
            projected = [torch.randn(n, 2 * h * dim + h * vdim, device="cuda").bfloat16() for _ in range(4)]
            states = [torch.zeros(len(counts), floats, device="cuda") for _ in range(4)]
            out = torch.empty(n, h * vdim, device="cuda")
            how = (dict(gates=torch.randn(n, 2 * h, device="cuda"), gate_bias=torch.zeros(2 * h, device="cuda"), gate_cap=15.0,
                        q_scale=dim ** -0.5) if gated else dict(decay=torch.full((h,), 0.98, device="cuda"), silu=True))
            slots, offs = dev(list(range(len(counts)))), dev([sum(counts[:i]) for i in range(len(counts))])
            cnts = dev(counts)
            passes = None
            if chunked == "passes":
                passes = [torch.empty(floats, device="cuda") for floats in ops.memory_passes_scratch(n, len(counts), h, dim, vdim)]

            def launch(i):
                x = projected[i % 4]
                ops.memory_scan(out, x[:, :h * dim], x[:, h * dim:2 * h * dim], x[:, 2 * h * dim:], states[i % 4], slots, offs, cnts,
                                h, dim, vdim, chunked=chunked is True, passes=passes, **how)
            us = replayed_us(torch, launch)
            if chunked == "passes":
                slices = -(-vdim // 32)
                per_chunk = slices * 32 * 32 * dim + 32 * vdim * (dim + 16) + dim * vdim * 32
                add(f"{kind} memory, chunks side by side, {name}", us, flops=2.0 * per_chunk * (n // 32) * h, heads=h, dim=dim, vdim=vdim)
            elif chunked:
                # per chunk of 32 tokens and head: 32 x 32 x dim scores (once per slice of 32 value columns),
                # 32 x vdim x (dim + 32 / 2) for the outputs, dim x vdim x 32 for the state
                slices = -(-vdim // 32)
                per_chunk = slices * 32 * 32 * dim + 32 * vdim * (dim + 16) + dim * vdim * 32
                add(f"{kind} memory, 32 tokens at a time, {name}", us, flops=2.0 * per_chunk * (n // 32) * h, heads=h, dim=dim, vdim=vdim)
            else:
                add(f"{kind} memory, token by token, {name}", us, bytes_moved=2.0 * len(counts) * floats * 4, heads=h, dim=dim, vdim=vdim)
    return lines


# Sumozen stacks beside Fuvolix of equal width, depth and inner size: layers in threes (two with an
# attention and a gated delta rule side by side, one state-space layer), every layer with a routed
# feed-forward whose chosen experts plus the shared one have the inner size of the dense one.
SUMOZEN_SIZES = {
    "small": {"width": 768, "layers": 12, "ff": 3072, "fuvolix": "small",
              "left": {"heads": 12, "kv_heads": 4, "dim": 64, "vdim": 64}, "right": {"heads": 6, "kv_heads": 3, "dim": 128, "vdim": 128},
              "mamba": {"heads": 24, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1},
              "moe": {"experts": 8, "top": 2, "ff": 768, "shared": 1536}},
    "medium": {"width": 1024, "layers": 24, "ff": 4096, "fuvolix": "medium",
               "left": {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 64}, "right": {"heads": 8, "kv_heads": 4, "dim": 128, "vdim": 128},
               "mamba": {"heads": 32, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1},
               "moe": {"experts": 8, "top": 2, "ff": 1024, "shared": 2048}},
}


def sumozen_config(size: dict, vocab: int) -> dict:
    left, right, moe = size["left"], size["right"], size["moe"]
    mlp = {"kind": "moe", "router": {"experts": moe["experts"], "top": moe["top"]}, "expert": {"ff": moe["ff"]},
           "shared": {"ff": moe["shared"]}}
    parallel = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": dict(left, conv=4, scale=left["dim"] ** -0.5, softcap=50.0,
                     rot={"base": 10000.0, "dims": left["dim"], "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}}),
        "right": dict(right, conv=4), "left_scale": 1.0, "right_scale": 1.0}}
    mamba = {"type": "mamba2", "mlp": mlp, "mixer": dict(size["mamba"], conv=4)}
    three = [parallel, parallel, mamba]
    return {"architecture": "Sumozen", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5},
            "layers": [three[i % 3] for i in range(size["layers"])]}


def sumozen_kernels(torch, size: dict, peak: dict, recurrences=("right", "mamba"), experts=True):
    """Sumozen's kernels alone, replayed back to back on operands of their own: prompt portions
    (2 x 1,024 tokens) and single tokens (8 requests at 1,023 cached tokens), each with the work it
    must do and the fraction of its bound: 32-bit FMA (nominal) where the sums are 32-bit by the
    design's rule, measured HBM copy bandwidth where the state, the cache or the weights are
    streamed, measured bf16 throughput for the products."""
    from mini_llm_b200.kernels import ops
    lines = []
    page, fma_peak = 64, FP32_FMA_TFLOPS_NOMINAL
    dev = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def add(kernel, us, flops=None, bytes_moved=None, tensor_flops=None, **more):
        line = {"kernel": kernel, "us": round(us, 2), **more}
        if flops is not None:
            line.update(tflops=round(flops / us / 1e6, 2), frac_fp32_fma_nominal=round(flops / us / 1e6 / fma_peak, 3))
        if tensor_flops is not None:
            line.update(tflops=round(tensor_flops / us / 1e6, 2), frac_bf16_measured=round(tensor_flops / us / 1e6 / peak["bf16_tflops"], 3))
        if bytes_moved is not None:
            line.update(gbs=round(bytes_moved / us / 1e3, 1), frac_hbm_measured=round(bytes_moved / us / 1e3 / peak["hbm_gbs"], 3))
        lines.append(line)

    # ---- the attention with capped scores ----
    left = size["left"]
    heads, kv_heads, dim, vdim = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
    for name, lengths, new in (("prompts, 2 x 1024", [1024, 1024], [1024, 1024]), ("single tokens, 8 x 1024", [1024] * 8, [1] * 8)):
        blocks = [-(-n // page) for n in lengths]
        table = torch.zeros(len(lengths), max(blocks), dtype=torch.int32)
        at = 0
        for i, count in enumerate(blocks):
            table[i, :count] = torch.arange(at, at + count, dtype=torch.int32)
            at += count
        table = table.cuda()
        n = sum(new)
        starts = [length - count for length, count in zip(lengths, new)]
        positions = torch.cat([torch.arange(s, s + m) for s, m in zip(starts, new)]).int().cuda()
        token_item = torch.cat([torch.full((m,), i) for i, m in enumerate(new)]).int().cuda()
        pairs = sum(sum(range(s + 1, s + m + 1)) for s, m in zip(starts, new)) * heads         # (query row, key) pairs
        k_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, dim, device="cuda").bfloat16() for _ in range(4)]
        v_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, vdim, device="cuda").bfloat16() for _ in range(4)]
        q = torch.randn(n, heads * dim, device="cuda").bfloat16()
        out = torch.empty(n, heads * vdim, device="cuda", dtype=torch.bfloat16)
        if len(new) == 2:
            us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                   heads, kv_heads, dim, vdim, page, 0.125, 50.0, 0, tiled=True))
            add(f"capped attention in tiles, {name}", us, flops=2.0 * pairs * (dim + vdim), heads=heads, kv_heads=kv_heads, dim=dim)
        else:
            chunk, reach = 128, table.shape[1] * page
            chunks = -(-reach // chunk)
            scratch = (torch.empty(n * heads * chunks * dim, device="cuda"), torch.empty(n * heads * chunks * 2, device="cuda"),
                       torch.zeros(n * heads, dtype=torch.int32, device="cuda"))
            us = replayed_us(torch, lambda i: ops.split_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                  heads, kv_heads, dim, page, 0.125, 0, chunk, chunks, *scratch, cap=50.0))
            add(f"capped attention over split keys, {name}", us, bytes_moved=sum(lengths) * kv_heads * (dim + vdim) * 2.0,
                heads=heads, kv_heads=kv_heads, dim=dim)
            us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                   heads, kv_heads, dim, vdim, page, 0.125, 50.0, 0))
            add(f"capped attention, one block per (token, head), {name}", us, bytes_moved=sum(lengths) * kv_heads * (dim + vdim) * 2.0,
                heads=heads, kv_heads=kv_heads, dim=dim)
    # ---- the recurrences ----
    for kind in recurrences:
        mem = size[kind]
        delta = kind == "right"
        h, vd = mem["heads"], mem["vdim"]
        qk_heads, kd = (mem["kv_heads"], mem["dim"]) if delta else (mem["groups"], mem["state"])
        for name, counts in (("prompts, 2 x 1024", [1024, 1024]), ("single tokens, 8", [1] * 8)):
            n = sum(counts)
            projected = [torch.randn(n, 2 * qk_heads * kd + h * vd, device="cuda").bfloat16() for _ in range(4)]
            states = [torch.zeros(len(counts), h * kd * vd, device="cuda") for _ in range(4)]
            out = torch.empty(n, h * vd, device="cuda")
            gate_a, gate_b = torch.randn(n, h, device="cuda"), torch.randn(n, h, device="cuda")
            rate, bias, skip = torch.zeros(h, device="cuda"), torch.zeros(h, device="cuda"), torch.ones(h, device="cuda")
            slots, offs, cnts = dev(list(range(len(counts)))), dev([sum(counts[:i]) for i in range(len(counts))]), dev(counts)

            def launch(i):
                x = projected[i % 4]
                ops.linear_recurrence(out, x[:, :qk_heads * kd], x[:, qk_heads * kd:2 * qk_heads * kd], x[:, 2 * qk_heads * kd:], gate_a,
                                      gate_b if delta else None, rate, bias, states[i % 4], slots, offs, cnts, h, qk_heads, kd, vd,
                                      delta, unit_norm=delta, q_scale=kd ** -0.5 if delta else 1.0, skip=None if delta else skip)
            us = replayed_us(torch, launch)
            label = "gated delta rule" if delta else "state-space recurrence"
            if len(counts) == 2:
                # per token and head: two sums over the old state and the state's update, four FMAs an entry
                add(f"{label}, token by token, {name}", us, flops=2.0 * 4 * kd * vd * h * n, heads=h, dim=kd, vdim=vd)
            else:
                add(f"{label}, {name}", us, bytes_moved=2.0 * len(counts) * h * kd * vd * 4, heads=h, dim=kd, vdim=vd)
    if not experts:
        return lines
    # ---- the routed feed-forward ----
    moe, width = size["moe"], size["width"]
    experts, top, inner, shared = moe["experts"], moe["top"], moe["ff"], moe["shared"]
    total, pairs = experts * inner + shared, top + 1
    up = [(torch.randn(2 * total, width, device="cuda") * 0.02).bfloat16() for _ in range(4)]
    down = [(torch.randn(width, total, device="cuda") * 0.02).bfloat16() for _ in range(4)]
    router, shared_gate = (torch.randn(experts, width, device="cuda") * 0.5).bfloat16(), (torch.randn(1, width, device="cuda") * 0.1).bfloat16()
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    starts = [e * inner for e in range(experts)] + [experts * inner]
    inner_of = dev([inner] * experts + [shared])
    for name, n in (("2,048 tokens", 2048), ("8 tokens", 8)):
        x = torch.randn(n, width, device="cuda").bfloat16()
        hidden = torch.zeros(n, width, device="cuda")
        choice = torch.zeros(n * pairs, dtype=torch.int32, device="cuda")
        in_weight, out_weight = torch.zeros(n * pairs, device="cuda"), torch.zeros(n * pairs, device="cuda")
        us = replayed_us(torch, lambda i: ops.route(x, router, shared_gate, top, choice, in_weight, out_weight))
        add(f"router, {name}", us, bytes_moved=n * width * 2.0 + experts * width * 2.0, experts=experts, top=top)
        needed = 2.0 * n * 3 * width * (top * inner + shared)                 # the flops the chosen experts need
        if n >= 32:
            gu = torch.empty(n, 2 * total, device="cuda", dtype=torch.bfloat16)
            act = torch.empty(n, total, device="cuda", dtype=torch.bfloat16)

            def launch(i):
                ops.gemm_bf16(gu, x, up[i % 4], None, "store", status)
                ops.expert_combine(act, gu, choice, in_weight, out_weight, experts, inner, top, pairs)
                ops.gemm_bf16(hidden, act, down[i % 4], None, "add", status)
            us = replayed_us(torch, launch)
            add(f"experts, two products over all experts, {name}", us, tensor_flops=needed, executed_tflops=round(2.0 * n * 3 * width * total / us / 1e6, 1),
                experts=experts, top=top, inner=inner, shared=shared)
            # the dense feed-forward of equal inner size (the closest model's), the same two products
            fc = [(torch.randn(size["ff"], width, device="cuda") * 0.02).bfloat16() for _ in range(4)]
            back = [(torch.randn(width, size["ff"], device="cuda") * 0.02).bfloat16() for _ in range(4)]
            mid = torch.empty(n, size["ff"], device="cuda", dtype=torch.bfloat16)

            def dense(i):
                ops.gemm_bf16(mid, x, fc[i % 4], None, "relu_squared", status)
                ops.gemm_bf16(hidden, mid, back[i % 4], None, "add", status)
            us = replayed_us(torch, dense)
            add(f"dense feed-forward of inner {size['ff']}, {name}", us, tensor_flops=2.0 * n * 2 * width * size["ff"])
        else:
            act = torch.empty(n * pairs, max(inner, shared), device="cuda", dtype=torch.bfloat16)

            tables = []
            for i in range(4):
                size_of = up[i].element_size()
                tables.append((torch.tensor([up[i].data_ptr() + s_ * width * size_of for s_ in starts], dtype=torch.int64, device="cuda"),
                               torch.tensor([up[i].data_ptr() + (total + s_) * width * size_of for s_ in starts], dtype=torch.int64, device="cuda"),
                               torch.tensor([down[i].data_ptr() + s_ * size_of for s_ in starts], dtype=torch.int64, device="cuda")))
            us = replayed_us(torch, lambda i: ops.experts(hidden, act, x, choice, in_weight, out_weight, *tables[i % 4], inner_of,
                                                          max(inner, shared), pairs, ld_down=total))
            # at most every expert once, and the shared one
            read = min(n * top, experts) * 3 * inner * width * 2.0 + 3 * shared * width * 2.0
            add(f"experts, pair by pair, {name}", us, bytes_moved=read, experts=experts, top=top, inner=inner, shared=shared)
    return lines


def run_compare_sumozen(args):
    """Sumozen beside Fuvolix of equal width, depth and inner size: the prompt step of 2,048 tokens
    (2 x 1,024) and the decode step of ``--batch`` requests at a context of 1,024, in bfloat16,
    through ``Engine.step``; then the kernels alone, Sumozen's and Fuvolix's.  One JSON line per measurement."""
    import torch
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.engine import Engine
    from mini_llm_b200.weights import write_random_model
    peak = peaks()
    context, vocab = 1024, GPT2_SMALL["vocab_size"]
    for name, size in SUMOZEN_SIZES.items():
        for design in ("sumozen", "fuvolix"):
            raw = sumozen_config(size, vocab) if design == "sumozen" else fuvolix_config(FUVOLIX_SIZES[size["fuvolix"]], vocab)
            with tempfile.TemporaryDirectory() as folder:
                write_random_model(config_from_dict(raw), 0, folder, recipe="gpt2", store_dtype="bfloat16")
                engine = Engine(folder, dtype="bfloat16", max_requests=16, cache_tokens=16 * context, max_tokens_per_step=2048,
                                **({"page_size": args.page_size} if args.page_size else {}))
                prefill_ms = prefill_run(engine, 2, 1024, vocab)
                decode_ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
                print(json.dumps({"design": design, "size": name, "width": size["width"], "layers": size["layers"], "inner": size["ff"],
                                  "prefill_2048_tokens_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(2048 / prefill_ms * 1e3),
                                  "decode_batch": args.batch, "decode_ms_per_step": round(decode_ms, 3),
                                  "decode_tokens_per_s": round(args.batch / decode_ms * 1e3), "launches_per_decode_step": launches,
                                  "weight_bytes": engine.model.weight_bytes, "step_kinds": engine.step_kinds}), flush=True)
                del engine
                torch.cuda.empty_cache()
        for line in sumozen_kernels(torch, size, peak):
            print(json.dumps(dict(line, design="sumozen", size=name)), flush=True)
        for line in mixer_kernels(torch, FUVOLIX_SIZES[size["fuvolix"]], peak):
            print(json.dumps(dict(line, design="fuvolix", size=name)), flush=True)
    return 0


# Lipulorn stacks beside Fuvolix of equal width and depth: layers in sixes (attention over a latent of its own within a
# window, attention in blocks, a channel delta memory, then the same three with the latent attention reading the first
# one's rows), four residual streams, every layer with a gated feed-forward of two thirds of the dense inner size (three
# matrices instead of two: as many weights).
LIPULORN_SIZES = {
    "small": {"width": 768, "layers": 12, "ff": 2048, "streams": 4, "fuvolix": "small", "sumozen": "small",
              "latent": {"heads": 12, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256, "q_rank": 384, "window": 512},
              "attention": {"heads": 12, "kv_heads": 4, "dim": 64, "vdim": 64, "chunk": 512},
              "delta": {"heads": 6, "kv_heads": 3, "dim": 128, "vdim": 128, "a_rank": 64, "g_rank": 64}},
    "medium": {"width": 1024, "layers": 24, "ff": 2816, "streams": 4, "fuvolix": "medium", "sumozen": "medium",
               "latent": {"heads": 16, "dim": 64, "rot_dim": 64, "vdim": 64, "kv_rank": 512, "q_rank": 512, "window": 512},
               "attention": {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 64, "chunk": 512},
               "delta": {"heads": 8, "kv_heads": 4, "dim": 128, "vdim": 128, "a_rank": 64, "g_rank": 64}},
    # a wider one; the like stack and the like kernels' sizes are given here, the other designs' tables stop at 1,024
    "large": {"width": 2048, "layers": 12, "ff": 5632, "streams": 4,
              "latent": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": 1536, "window": 512},
              "attention": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "chunk": 512},
              "delta": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "a_rank": 128, "g_rank": 128},
              "fuvolix": {"width": 2048, "layers": 12, "ff": 8192,
                          "latent": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512},
                          "mlstm": {"heads": 8, "dim": 128, "vdim": 256}, "lightning": {"heads": 16, "dim": 128, "vdim": 128}},
              "sumozen": {"left": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128},
                          "right": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128}}},
}


def lipulorn_config(size: dict, vocab: int) -> dict:
    lat, att, mem = size["latent"], size["attention"], size["delta"]
    mlp = {"kind": "dense", "ff": size["ff"]}

    def latent(source):
        mixer = {key: lat[key] for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")}
        mixer.update(scale=(lat["dim"] + lat["rot_dim"]) ** -0.5, mask={"size": lat["window"]},
                     rot={"base": 10000.0, "dims": lat["rot_dim"]})
        if source is not None:
            mixer["kv_from"] = source
        return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}
    attention = {"type": "attention", "mlp": mlp,
                 "mixer": {"heads": att["heads"], "kv_heads": att["kv_heads"], "dim": att["dim"], "vdim": att["vdim"],
                           "scale": att["dim"] ** -0.5, "mask": {"size": att["chunk"]}}}
    memory = {"type": "channel_delta", "mlp": mlp, "mixer": dict(mem, conv=4)}
    layers = []
    for index in range(size["layers"]):
        layers.append([latent(None), attention, memory, latent(index - 3), attention, memory][index % 6])
    return {"architecture": "Lipulorn", "vocab": vocab, "width": size["width"], "streams": size["streams"], "norm": {"eps": 1e-5},
            "layers": layers}


def lipulorn_kernels(torch, size: dict, peak: dict):
    """Lipulorn's kernels alone, replayed back to back on operands of their own: prompt portions
    (2 x 1,024 tokens) and single tokens (8 requests at 1,023 cached tokens), each with the work it
    must do and the fraction of its bound: 32-bit FMA (nominal) where the sums are 32-bit by the
    design's rule, measured HBM copy bandwidth where streams, state or cache are streamed."""
    from mini_llm_b200.kernels import ops
    lines = []
    page, fma_peak = 64, FP32_FMA_TFLOPS_NOMINAL
    dev = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def add(kernel, us, flops=None, bytes_moved=None, **more):
        line = {"kernel": kernel, "us": round(us, 2), **more}
        if flops is not None:
            line.update(tflops=round(flops / us / 1e6, 2), frac_fp32_fma_nominal=round(flops / us / 1e6 / fma_peak, 3))
        if bytes_moved is not None:
            line.update(gbs=round(bytes_moved / us / 1e3, 1), frac_hbm_measured=round(bytes_moved / us / 1e3 / peak["hbm_gbs"], 3))
        lines.append(line)

    def batch(lengths, new):
        blocks = [-(-n // page) for n in lengths]
        table = torch.zeros(len(lengths), max(blocks), dtype=torch.int32)
        at = 0
        for i, count in enumerate(blocks):
            table[i, :count] = torch.arange(at, at + count, dtype=torch.int32)
            at += count
        starts = [length - count for length, count in zip(lengths, new)]
        positions = torch.cat([torch.arange(s, s + m) for s, m in zip(starts, new)]).int().cuda()
        token_item = torch.cat([torch.full((m,), i) for i, m in enumerate(new)]).int().cuda()
        return table.cuda(), sum(blocks), starts, positions, token_item

    shapes = (("prompts, 2 x 1024", [1024, 1024], [1024, 1024]), ("single tokens, 8 x 1024", [1024] * 8, [1] * 8))
    # ---- attention over the latent within a window ----
    lat = size["latent"]
    heads, rank, rot, window = lat["heads"], lat["kv_rank"], lat["rot_dim"], lat["window"]
    row = rank + rot
    for name, lengths, new in shapes:
        table, n_blocks, starts, positions, token_item = batch(lengths, new)
        n = sum(new)
        offsets = [sum(new[:i]) for i in range(len(new))]
        seen = sum(sum(min(p + 1, window) for p in range(s, s + m)) for s, m in zip(starts, new))     # (query token, key) pairs
        pages = [torch.randn(n_blocks + 1, page, 1, row, device="cuda").bfloat16() for _ in range(4)]
        q_eff = torch.randn(n, heads * row, device="cuda")
        out = torch.empty(n, heads * rank, device="cuda")
        if len(new) == 2:
            tiles, _, _ = ops.attention_tiles(offsets, new, starts, split=False)
            tiles_d = dev(tiles)
            us = replayed_us(torch, lambda i: ops.latent_attention_tiled(out, q_eff, pages[i % 4], table, positions, token_item, heads,
                                                                         rank, rot, page, 0.1, tiles=tiles_d, n_tiles=len(tiles), window=window))
            add(f"latent attention in tiles, window {window}, {name}", us, flops=2.0 * seen * heads * (row + rank), heads=heads, row=row)
        else:
            parts = max(1, min(32, 296 // (n * (1 if heads <= 16 else -(-heads // 32)))))
            scratch = (torch.empty(n * heads * parts * rank, device="cuda"), torch.empty(n * heads * parts * 2, device="cuda"))
            us = replayed_us(torch, lambda i: ops.latent_attention_tiled(out, q_eff, pages[i % 4], table, positions, token_item, heads,
                                                                         rank, rot, page, 0.1, parts=parts, scratch=scratch, window=window))
            add(f"latent attention in parts, window {window}, {name}", us, bytes_moved=seen * row * 2.0, heads=heads, row=row, parts=parts)
    # ---- attention in blocks of positions, normed heads, a gate per head ----
    att = size["attention"]
    heads, kv_heads, dim, vdim, chunk = att["heads"], att["kv_heads"], att["dim"], att["vdim"], att["chunk"]
    for name, lengths, new in shapes:
        table, n_blocks, starts, positions, token_item = batch(lengths, new)
        n = sum(new)
        seen = sum(sum(p % chunk + 1 for p in range(s, s + m)) for s, m in zip(starts, new))
        k_pages = [torch.randn(n_blocks + 1, page, kv_heads, dim, device="cuda").bfloat16() for _ in range(4)]
        v_pages = [torch.randn(n_blocks + 1, page, kv_heads, vdim, device="cuda").bfloat16() for _ in range(4)]
        qkv = [torch.randn(n, (heads + kv_heads) * dim + kv_heads * vdim, device="cuda").bfloat16() for _ in range(4)]
        gate = torch.randn(n, 16, device="cuda")
        out = torch.empty(n, heads * vdim, device="cuda", dtype=torch.bfloat16)
        us = replayed_us(torch, lambda i: ops.head_norm_store(qkv[i % 4], heads * dim, (heads + kv_heads) * dim, heads, kv_heads, dim, vdim, 1e-5,
                                                              positions, token_item, table, page, k_pages[i % 4], v_pages[i % 4]))
        add(f"head norms + cache store, {name}", us, bytes_moved=n * ((2 * heads + 2 * kv_heads) * dim + 2 * kv_heads * vdim) * 2.0)
        q = qkv[0][:, :heads * dim]
        if len(new) == 2:
            us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                   heads, kv_heads, dim, vdim, page, 0.125, 0.0, 0, tiled=True, chunk=chunk, gate=gate))
            add(f"gated attention in tiles, blocks of {chunk}, {name}", us, flops=2.0 * seen * heads * (dim + vdim), heads=heads, kv_heads=kv_heads, dim=dim)
        else:
            span, reach = 128, table.shape[1] * page
            spans = -(-reach // span)
            scratch = (torch.empty(n * heads * spans * dim, device="cuda"), torch.empty(n * heads * spans * 2, device="cuda"),
                       torch.zeros(n * heads, dtype=torch.int32, device="cuda"))
            us = replayed_us(torch, lambda i: ops.split_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                  heads, kv_heads, dim, page, 0.125, 0, span, spans, *scratch,
                                                                  block=chunk, gate=gate))
            add(f"gated attention over split keys, blocks of {chunk}, {name}", us, bytes_moved=seen * kv_heads * (dim + vdim) * 2.0,
                heads=heads, kv_heads=kv_heads, dim=dim)
            us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                   heads, kv_heads, dim, vdim, page, 0.125, 0.0, 0, chunk=chunk, gate=gate))
            add(f"gated attention, one block per (token, head), blocks of {chunk}, {name}", us,
                bytes_moved=seen * kv_heads * (dim + vdim) * 2.0, heads=heads, kv_heads=kv_heads, dim=dim)
    # ---- the delta memory with a decay per key channel ----
    mem = size["delta"]
    h, qk_heads, kd, vd = mem["heads"], mem["kv_heads"], mem["dim"], mem["vdim"]
    for name, counts in (("prompts, 2 x 1024", [1024, 1024]), ("single tokens, 8", [1] * 8)):
        n = sum(counts)
        projected = [torch.randn(n, 2 * qk_heads * kd + h * vd, device="cuda").bfloat16() for _ in range(4)]
        states = [torch.zeros(len(counts), h * kd * vd, device="cuda") for _ in range(4)]
        out = torch.empty(n, h * vd, device="cuda")
        steps, writes = torch.randn(n, h * kd, device="cuda"), torch.randn(n, 16, device="cuda")
        rate, bias = torch.zeros(h, device="cuda"), torch.zeros(h * kd, device="cuda")
        slots, offs, cnts = dev(list(range(len(counts)))), dev([sum(counts[:i]) for i in range(len(counts))]), dev(counts)

        def launch(i):
            x = projected[i % 4]
            ops.linear_recurrence(out, x[:, :qk_heads * kd], x[:, qk_heads * kd:2 * qk_heads * kd], x[:, 2 * qk_heads * kd:], steps,
                                  writes[:, :h], rate, bias, states[i % 4], slots, offs, cnts, h, qk_heads, kd, vd, True,
                                  unit_norm=True, q_scale=kd ** -0.5, channel_decay=True)
        us = replayed_us(torch, launch)
        if len(counts) == 2:
            add(f"channel delta rule, token by token, {name}", us, flops=2.0 * 4 * kd * vd * h * n, heads=h, dim=kd, vdim=vd)
        else:
            add(f"channel delta rule, {name}", us, bytes_moved=2.0 * len(counts) * h * kd * vd * 4, heads=h, dim=kd, vdim=vd)
    # ---- the residual streams and the gated activation ----
    width, count, inner = size["width"], size["streams"], size["ff"]
    for name, n in (("2,048 tokens", 2048), ("8 tokens", 8)):
        streams = [torch.randn(n, count, width, device="cuda") for _ in range(4)]
        y = [torch.randn(n, width, device="cuda") for _ in range(4)]
        normed = torch.empty(n, width, device="cuda", dtype=torch.bfloat16)
        mix = torch.eye(count, device="cuda").contiguous()
        w_in, w_out, gain = torch.ones(count, device="cuda"), torch.ones(count, device="cuda"), torch.ones(width, device="cuda")
        us = replayed_us(torch, lambda i: ops.streams_step(streams[i % 4], y=y[i % 4], mix=mix, w_out=w_out, read=True, w_in=w_in,
                                                           normed=normed, gain=gain, eps=1e-5))
        add(f"streams: write, read-out and norm in one pass, {name}", us, bytes_moved=n * width * (8.0 * count + 4 + 2), streams=count)
        x = [torch.randn(n, width, device="cuda") for _ in range(4)]
        us = replayed_us(torch, lambda i: ops.grouped_rms_norm(normed, x[i % 4], gain, 1, 1e-5))
        add(f"one residual: norm alone, {name}", us, bytes_moved=n * width * (4.0 + 2))
        gu = [torch.randn(n, 2 * inner, device="cuda").bfloat16() for _ in range(4)]
        act = torch.empty(n, inner, device="cuda", dtype=torch.bfloat16)
        us = replayed_us(torch, lambda i: ops.gated_act(act, gu[i % 4], "silu"))
        add(f"gated activation, {name}", us, bytes_moved=n * inner * 6.0, inner=inner)
    return lines




def run_compare_lipulorn(args):
    """Lipulorn beside Fuvolix of equal width and depth (and as many feed-forward weights): the prompt step of
    2,048 tokens (2 x 1,024) and the decode step of ``--batch`` requests at a context of 1,024, in bfloat16,
    through ``Engine.step``; then the kernels alone: Lipulorn's, and the like kernels of Fuvolix (attention
    over a latent) and Sumozen (attention with grouped heads, the delta rule).  One JSON line per measurement."""
    import torch
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.engine import Engine
    from mini_llm_b200.weights import write_random_model
    peak = peaks()
    context, vocab = 1024, GPT2_SMALL["vocab_size"]
    for name, size in LIPULORN_SIZES.items():
        fuvolix = size["fuvolix"] if isinstance(size["fuvolix"], dict) else FUVOLIX_SIZES[size["fuvolix"]]
        sumozen = size["sumozen"] if isinstance(size["sumozen"], dict) else SUMOZEN_SIZES[size["sumozen"]]
        for design in ("lipulorn", "fuvolix"):
            raw = lipulorn_config(size, vocab) if design == "lipulorn" else fuvolix_config(fuvolix, vocab)
            with tempfile.TemporaryDirectory() as folder:
                write_random_model(config_from_dict(raw), 0, folder, recipe="gpt2", store_dtype="bfloat16")
                engine = Engine(folder, dtype="bfloat16", max_requests=16, cache_tokens=16 * context, max_tokens_per_step=2048,
                                **({"page_size": args.page_size} if args.page_size else {}))
                prefill_ms = prefill_run(engine, 2, 1024, vocab)
                decode_ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
                print(json.dumps({"design": design, "size": name, "width": size["width"], "layers": size["layers"],
                                  "inner": size["ff"] if design == "lipulorn" else fuvolix["ff"],
                                  "prefill_2048_tokens_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(2048 / prefill_ms * 1e3),
                                  "decode_batch": args.batch, "decode_ms_per_step": round(decode_ms, 3),
                                  "decode_tokens_per_s": round(args.batch / decode_ms * 1e3), "launches_per_decode_step": launches,
                                  "weight_bytes": engine.model.weight_bytes, "step_kinds": engine.step_kinds}), flush=True)
                del engine
                torch.cuda.empty_cache()
        for line in lipulorn_kernels(torch, size, peak):
            print(json.dumps(dict(line, design="lipulorn", size=name)), flush=True)
        for line in mixer_kernels(torch, fuvolix, peak, memories=()):
            if line["kernel"].startswith("latent attention"):
                print(json.dumps(dict(line, design="fuvolix", size=name)), flush=True)
        for line in sumozen_kernels(torch, sumozen, peak, recurrences=("right",), experts=False):
            print(json.dumps(dict(line, design="sumozen", size=name)), flush=True)
    return 0


# Deluvik stacks beside Sumozen of equal width, depth and experts: layers in fours (attention with convolved
# projections, attention whose values are its keys, a sliding-window attention beside the gated linear recurrence, and
# attention with convolved queries over the first layer's keys and values), every layer with the routed feed-forward
# that the Sumozen stack has (the first of every four a dense one of the same inner size).
DELUVIK_SIZES = {
    "small": {"width": 768, "layers": 12, "ff": 3072, "sumozen": "small",
              "attention": {"heads": 12, "kv_heads": 4, "dim": 64, "vdim": 64}, "window": 512,
              "unit": {"width": 768, "blocks": 12}, "moe": {"experts": 8, "top": 2, "ff": 768, "shared": 1536}},
    "medium": {"width": 1024, "layers": 24, "ff": 4096, "sumozen": "medium",
               "attention": {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 64}, "window": 512,
               "unit": {"width": 1024, "blocks": 16}, "moe": {"experts": 8, "top": 2, "ff": 1024, "shared": 2048}},
}


def deluvik_config(size: dict, vocab: int) -> dict:
    att, moe = size["attention"], size["moe"]
    routed = {"kind": "moe", "router": {"experts": moe["experts"], "top": moe["top"]}, "expert": {"ff": moe["ff"]},
              "shared": {"ff": moe["shared"]}}
    rot = {"base": 10000.0, "dims": att["dim"]}
    banded = dict(rot, scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1024})
    common = dict(att, scale=att["dim"] ** -0.5)

    def four(first):
        return [{"type": "attention_2", "mixer": dict(common, conv=4, rot=rot), "mlp": {"kind": "dense", "ff": size["ff"]}},
                {"type": "attention", "mixer": dict(common, kv_heads=1, rot=banded, softcap=50.0), "mlp": routed},
                {"type": "parallel", "mlp": routed, "mixer": {
                    "left": dict(common, kv_heads=1, rot=dict(rot, dims=att["dim"] // 2), mask={"size": size["window"]}),
                    "right": dict(size["unit"], conv=4), "left_scale": 1.0, "right_scale": 1.0}},
                {"type": "attention_2", "mixer": dict(common, conv=4, rot=rot, kv_from=first), "mlp": routed}]
    layers = []
    while len(layers) < size["layers"]:
        layers += four(len(layers))
    return {"architecture": "Deluvik", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": layers[:size["layers"]]}


def deluvik_kernels(torch, size: dict, peak: dict):
    """Deluvik's own kernels alone, replayed back to back on operands of their own: prompt portions (2 x 1,024 tokens)
    and single tokens (8 requests at 1,023 cached tokens), each with the work it must do and the fraction of its
    bound (32-bit FMA, nominal, where the sums are 32-bit by the design's rule; measured HBM copy bandwidth where
    rows, the cache or the state are streamed)."""
    from mini_llm_b200.kernels import ops
    lines = []
    page, fma_peak = 64, FP32_FMA_TFLOPS_NOMINAL
    dev = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def add(kernel, us, flops=None, bytes_moved=None, **more):
        line = {"kernel": kernel, "us": round(us, 2), **more}
        if flops is not None:
            line.update(tflops=round(flops / us / 1e6, 2), frac_fp32_fma_nominal=round(flops / us / 1e6 / fma_peak, 3))
        if bytes_moved is not None:
            line.update(gbs=round(bytes_moved / us / 1e3, 1), frac_hbm_measured=round(bytes_moved / us / 1e3 / peak["hbm_gbs"], 3))
        lines.append(line)

    att = size["attention"]
    heads, kv_heads, dim, vdim, width = att["heads"], att["kv_heads"], att["dim"], att["vdim"], size["width"]
    for name, lengths, new in (("prompts, 2 x 1024", [1024, 1024], [1024, 1024]), ("single tokens, 8 x 1024", [1024] * 8, [1] * 8)):
        blocks = [-(-n // page) for n in lengths]
        table = torch.zeros(len(lengths), max(blocks), dtype=torch.int32)
        at = 0
        for i, count in enumerate(blocks):
            table[i, :count] = torch.arange(at, at + count, dtype=torch.int32)
            at += count
        table = table.cuda()
        n = sum(new)
        starts = [length - count for length, count in zip(lengths, new)]
        positions = torch.cat([torch.arange(s, s + m) for s, m in zip(starts, new)]).int().cuda()
        token_item = torch.cat([torch.full((m,), i) for i, m in enumerate(new)]).int().cuda()
        k_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, dim, device="cuda").bfloat16() for _ in range(4)]
        v_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, vdim, device="cuda").bfloat16() for _ in range(4)]
        q = torch.randn(n, heads * dim, device="cuda").bfloat16()
        out = torch.empty(n, heads * vdim, device="cuda", dtype=torch.bfloat16)
        sink = torch.randn(heads, device="cuda")
        window = size["window"]
        if len(new) == 2:
            pairs = sum(sum(range(s + 1, s + m + 1)) for s, m in zip(starts, new)) * heads         # (query row, key) pairs
            us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                   heads, kv_heads, dim, vdim, page, 0.125, 50.0, 0, tiled=True, sink=sink))
            add(f"attention in tiles with a sink, {name}", us, flops=2.0 * pairs * (dim + vdim), heads=heads, kv_heads=kv_heads, dim=dim)
            seen = sum(sum(min(p + 1, window) for p in range(s, s + m)) for s, m in zip(starts, new)) * heads
            us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                   heads, kv_heads, dim, vdim, page, 0.125, 0.0, window, tiled=True))
            add(f"attention in tiles within a window of {window}, {name}", us, flops=2.0 * seen * (dim + vdim), heads=heads,
                kv_heads=kv_heads, dim=dim)
        else:
            chunk, reach = 128, table.shape[1] * page
            chunks = -(-reach // chunk)
            scratch = (torch.empty(n * heads * chunks * dim, device="cuda"), torch.empty(n * heads * chunks * 2, device="cuda"),
                       torch.zeros(n * heads, dtype=torch.int32, device="cuda"))
            us = replayed_us(torch, lambda i: ops.split_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                  heads, kv_heads, dim, page, 0.125, 0, chunk, chunks, *scratch, cap=50.0,
                                                                  sink=sink))
            add(f"attention over split keys with a sink, {name}", us, bytes_moved=sum(lengths) * kv_heads * (dim + vdim) * 2.0,
                heads=heads, kv_heads=kv_heads, dim=dim)
        # norm, rotation and the cache store: reads the 32-bit projections, writes the queries and the pages
        row = (heads + 2 * kv_heads) * dim
        projected = [torch.randn(n, row, device="cuda") for _ in range(4)]
        q_gain, k_gain = torch.ones(heads * dim, device="cuda"), torch.ones(kv_heads * dim, device="cuda")
        inv_freq = torch.tensor([10000.0 ** (-2.0 * i / dim) for i in range(dim // 2)], dtype=torch.float64, device="cuda")
        us = replayed_us(torch, lambda i: ops.norm_rotary_store(projected[i % 4], heads * dim, (heads + kv_heads) * dim, heads, kv_heads, dim,
                                                                vdim, q, q_gain, k_gain, "whole", 1e-5, dim, "half", inv_freq, positions,
                                                                token_item, table, page, k_pages[i % 4], v_pages[i % 4]))
        add(f"query and key norm, rotation and cache store, {name}", us, bytes_moved=n * row * 6.0, heads=heads, kv_heads=kv_heads, dim=dim)
        # the like kernel of the closest design: rotation and cache store (16-bit rows in place)
        rows16 = [torch.randn(n, row, device="cuda").bfloat16() for _ in range(4)]
        us = replayed_us(torch, lambda i: ops.rotary_store(rows16[i % 4], heads * dim, (heads + kv_heads) * dim, heads, kv_heads, dim, vdim, dim,
                                                           inv_freq, 1.0, positions, token_item, table, page, k_pages[i % 4], v_pages[i % 4]))
        add(f"(Sumozen) rotation and cache store, {name}", us, bytes_moved=n * ((heads + kv_heads) * dim * 4.0 + 2 * kv_heads * dim * 2.0 + kv_heads * dim * 2.0),
            heads=heads, kv_heads=kv_heads, dim=dim)
    # ---- the gated linear recurrence, the sum with the norm, the router ----
    inner, parts = size["unit"]["width"], size["unit"]["blocks"]
    for name, counts in (("prompts, 2 x 1024", [1024, 1024]), ("single tokens, 8", [1] * 8)):
        n = sum(counts)
        both = [torch.randn(n, 2 * inner, device="cuda").bfloat16() for _ in range(4)]
        u = [torch.randn(n, inner, device="cuda").bfloat16() for _ in range(4)]
        gates = [torch.randn(n, 2 * inner, device="cuda") for _ in range(4)]
        states = [torch.zeros(len(counts), inner, device="cuda") for _ in range(4)]
        out = torch.empty(n, inner, device="cuda", dtype=torch.bfloat16)
        bias_r, bias_i, lam = torch.zeros(inner, device="cuda"), torch.zeros(inner, device="cuda"), torch.randn(inner, device="cuda")
        slots, offs, cnts = dev(list(range(len(counts)))), dev([sum(counts[:i]) for i in range(len(counts))]), dev(counts)
        us = replayed_us(torch, lambda i: ops.gated_recurrence(out, u[i % 4], both[i % 4][:, :inner], gates[i % 4], bias_r, bias_i, lam, 8.0,
                                                               states[i % 4], slots, offs, cnts, inner // parts))
        add(f"gated linear recurrence, {name}", us, bytes_moved=n * inner * (2 + 2 + 8 + 2.0) + 2.0 * len(counts) * inner * 4, inner=inner)
        hidden = [torch.randn(n, width, device="cuda") for _ in range(4)]
        y = [torch.randn(n, width, device="cuda") for _ in range(4)]
        gain = torch.ones(width, device="cuda")
        rounded = torch.empty(n, width, device="cuda", dtype=torch.bfloat16)
        us = replayed_us(torch, lambda i: ops.add_normed_cast(hidden[i % 4], y[i % 4], gain, 1e-5, rounded))
        add(f"residual sum of a normed result with the rounded rows, {name}", us, bytes_moved=n * width * (4 + 4 + 4 + 2.0), width=width)
        normed = torch.empty(n, width, device="cuda", dtype=torch.bfloat16)
        us = replayed_us(torch, lambda i: ops.grouped_rms_norm(normed, hidden[i % 4], gain, 1, 1e-5))
        add(f"(Sumozen) norm of the stream, {name}", us, bytes_moved=n * width * (4 + 2.0), width=width)
        moe = size["moe"]
        x = torch.randn(n, width, device="cuda").bfloat16()
        router = (torch.randn(moe["experts"], width, device="cuda") * 0.5).bfloat16()
        router_bias = torch.randn(moe["experts"], device="cuda")
        shared_gate = (torch.randn(1, width, device="cuda") * 0.1).bfloat16()
        pairs = moe["top"] + 1
        choice = torch.zeros(n * pairs, dtype=torch.int32, device="cuda")
        in_weight, out_weight = torch.zeros(n * pairs, device="cuda"), torch.zeros(n * pairs, device="cuda")
        us = replayed_us(torch, lambda i: ops.route(x, router, None, moe["top"], choice, in_weight, out_weight, bias=router_bias,
                                                    rule="softmax_of_chosen", shared_plain=True))
        add(f"router with the softmax of the chosen logits, {name}", us, bytes_moved=n * width * 2.0 + moe["experts"] * width * 2.0)
        us = replayed_us(torch, lambda i: ops.route(x, router, shared_gate, moe["top"], choice, in_weight, out_weight))
        add(f"(Sumozen) router with sigmoid scores, {name}", us, bytes_moved=n * width * 2.0 + (moe["experts"] + 1) * width * 2.0)
    return lines


def run_compare_deluvik(args):
    """Deluvik beside Sumozen of equal width, depth and experts: the prompt step of 2,048 tokens (2 x 1,024) and the
    decode step of ``--batch`` requests at a context of 1,024, in bfloat16, through ``Engine.step``; then the kernels
    alone, Deluvik's own and Sumozen's like ones.  One JSON line per measurement."""
    import torch
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.engine import Engine
    from mini_llm_b200.weights import write_random_model
    peak = peaks()
    context, vocab = 1024, GPT2_SMALL["vocab_size"]
    for name, size in DELUVIK_SIZES.items():
        for design in ("deluvik", "sumozen"):
            raw = deluvik_config(size, vocab) if design == "deluvik" else sumozen_config(SUMOZEN_SIZES[size["sumozen"]], vocab)
            with tempfile.TemporaryDirectory() as folder:
                write_random_model(config_from_dict(raw), 0, folder, recipe="gpt2", store_dtype="bfloat16")
                engine = Engine(folder, dtype="bfloat16", max_requests=16, cache_tokens=16 * context, max_tokens_per_step=2048,
                                **({"page_size": args.page_size} if args.page_size else {}))
                prefill_ms = prefill_run(engine, 2, 1024, vocab)
                decode_ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
                print(json.dumps({"design": design, "size": name, "width": size["width"], "layers": size["layers"], "inner": size["ff"],
                                  "prefill_2048_tokens_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(2048 / prefill_ms * 1e3),
                                  "decode_batch": args.batch, "decode_ms_per_step": round(decode_ms, 3),
                                  "decode_tokens_per_s": round(args.batch / decode_ms * 1e3), "launches_per_decode_step": launches,
                                  "weight_bytes": engine.model.weight_bytes, "step_kinds": engine.step_kinds}), flush=True)
                del engine
                torch.cuda.empty_cache()
        for line in deluvik_kernels(torch, size, peak):
            print(json.dumps(dict(line, design="deluvik", size=name)), flush=True)
        for line in sumozen_kernels(torch, SUMOZEN_SIZES[size["sumozen"]], peak, recurrences=("mamba",), experts=False):
            print(json.dumps(dict(line, design="sumozen", size=name)), flush=True)
    return 0


# Nufavik stacks beside Deluvik stacks of equal width, depth, heads and experts: every Deluvik layer an "attention_2"
# (convolved projections, a sink) with routed experts, which have three matrices each there and two here.
NUFAVIK_SIZES = {
    "768 wide": {"width": 768, "layers": 12, "attention": {"heads": 12, "kv_heads": 4, "dim": 64, "vdim": 64}, "taps": 4, "window": 512,
                 "keep_first": 64, "moe": {"experts": 8, "identity": 2, "top": 2, "ff": 768}},
    "1,024 wide": {"width": 1024, "layers": 24, "attention": {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 96}, "taps": 4, "window": 512,
                   "keep_first": 64, "moe": {"experts": 8, "identity": 2, "top": 2, "ff": 1024}},
    "2,048 wide": {"width": 2048, "layers": 16, "attention": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128}, "taps": 4, "window": 512,
                   "keep_first": 64, "moe": {"experts": 16, "identity": 4, "top": 4, "ff": 1024}},
}


def nufavik_config(size: dict, vocab: int) -> dict:
    att, moe = size["attention"], size["moe"]
    layer = {"type": "attention",
             "mixer": dict(att, conv=size["taps"], scale=att["dim"] ** -0.5, rot={"base": 10000.0, "dims": att["dim"]},
                           mask={"size": size["window"], "keep_first": size["keep_first"]}),
             "mlp": {"kind": "moe", "router": {"experts": moe["experts"], "identity": moe["identity"], "top": moe["top"], "scale": 1.5},
                     "expert": {"ff": moe["ff"]}}}
    return {"architecture": "Nufavik", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "layers": [layer] * size["layers"]}


def nufavik_like_config(size: dict, vocab: int) -> dict:
    att, moe = size["attention"], size["moe"]
    layer = {"type": "attention_2", "mixer": dict(att, conv=size["taps"], scale=att["dim"] ** -0.5, rot={"base": 10000.0, "dims": att["dim"]}),
             "mlp": {"kind": "moe", "router": {"experts": moe["experts"], "top": moe["top"]}, "expert": {"ff": moe["ff"]}, "shared": None}}
    return {"architecture": "Deluvik", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": [layer] * size["layers"]}


def nufavik_kernels(torch, size: dict, peak: dict):
    """Nufavik's kernels alone, replayed back to back on operands of their own, each followed by Deluvik's like kernel
    at the same sizes: prompt portions (2 x 1,024 tokens) and single tokens (8 requests at 1,023 cached tokens), each
    with the work it must do and the fraction of its bound."""
    from mini_llm_b200.kernels import ops
    lines = []
    page, fma_peak = 64, FP32_FMA_TFLOPS_NOMINAL
    dev = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def add(kernel, us, flops=None, bytes_moved=None, tensor_flops=None, **more):
        line = {"kernel": kernel, "us": round(us, 2), **more}
        if flops is not None:
            line.update(tflops=round(flops / us / 1e6, 2), frac_fp32_fma_nominal=round(flops / us / 1e6 / fma_peak, 3))
        if tensor_flops is not None:
            line.update(tflops=round(tensor_flops / us / 1e6, 1), frac_bf16_measured=round(tensor_flops / us / 1e6 / peak["bf16_tflops"], 3))
        if bytes_moved is not None:
            line.update(gbs=round(bytes_moved / us / 1e3, 1), frac_hbm_measured=round(bytes_moved / us / 1e3 / peak["hbm_gbs"], 3))
        lines.append(line)

    att, moe, width, taps = size["attention"], size["moe"], size["width"], size["taps"]
    heads, kv_heads, dim, vdim = att["heads"], att["kv_heads"], att["dim"], att["vdim"]
    window, keep, scale = size["window"], size["keep_first"], dim ** -0.5
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    for name, lengths, new in (("prompts, 2 x 1024", [1024, 1024], [1024, 1024]), ("single tokens, 8 x 1024", [1024] * 8, [1] * 8)):
        blocks = [-(-n // page) for n in lengths]
        table = torch.stack([torch.arange(i * max(blocks), (i + 1) * max(blocks), dtype=torch.int32) for i in range(len(lengths))]).cuda()
        n, single = sum(new), len(new) > 2
        starts = [length - count for length, count in zip(lengths, new)]
        positions = torch.cat([torch.arange(s, s + m) for s, m in zip(starts, new)]).int().cuda()
        token_item = torch.cat([torch.full((m,), i) for i, m in enumerate(new)]).int().cuda()
        k_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, dim, device="cuda").bfloat16() for _ in range(4)]
        v_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, vdim, device="cuda").bfloat16() for _ in range(4)]
        q = torch.randn(n, heads * dim, device="cuda").bfloat16()
        out = torch.empty(n, heads * vdim, device="cuda", dtype=torch.bfloat16)
        sink = torch.zeros(heads, device="cuda")
        sees = lambda p, w, k: p + 1 if not w else min(p + 1, w) + min(k, max(p + 1 - w, 0))
        for label, w, kept in ((f"attention within {window} and the first {keep}", window, keep), ("(Deluvik) attention over all keys", 0, 0)):
            seen = sum(sum(sees(p, w, kept) for p in range(s, s + m)) for s, m in zip(starts, new))
            if single:
                chunk, reach = 128, min(table.shape[1] * page, w + kept) if w else table.shape[1] * page
                chunks, row = -(-reach // chunk), ops.split_attention_row(dim, vdim)
                scratch = (torch.empty(n * heads * chunks * row, device="cuda"), torch.empty(n * heads * chunks * 2, device="cuda"),
                           torch.zeros(n * heads, dtype=torch.int32, device="cuda"))
                us = replayed_us(torch, lambda i: ops.split_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                      heads, kv_heads, dim, page, scale, w, chunk, chunks, *scratch, sink=sink,
                                                                      value_size=vdim, keep=kept))
                add(f"{label}, split keys, {name}", us, bytes_moved=seen * kv_heads * (dim + vdim) * 2.0, heads=heads, kv_heads=kv_heads,
                    dim=dim, vdim=vdim)
            else:
                us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                       heads, kv_heads, dim, vdim, page, scale, 0.0, w, tiled=True, sink=sink,
                                                                       keep=kept))
                add(f"{label}, tiles, {name}", us, flops=2.0 * seen * heads * (dim + vdim), heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
        # taps, rotation and the cache store: reads the 32-bit projections, writes the queries and the pages
        columns = heads * dim + kv_heads * (dim + vdim)
        projected = [torch.randn(n, columns, device="cuda") for _ in range(4)]
        weights = torch.randn(columns, taps, device="cuda")
        states = [torch.zeros(len(new), taps - 1, columns, device="cuda") for _ in range(4)]
        q_gain, k_gain = torch.ones(heads * dim, device="cuda"), torch.ones(kv_heads * dim, device="cuda")
        inv_freq = torch.tensor([10000.0 ** (-2.0 * i / dim) for i in range(dim // 2)], dtype=torch.float64, device="cuda")
        items = (dev(list(range(len(new)))), dev(starts), dev([sum(new[:i]) for i in range(len(new))]), dev(new))
        moved = n * columns * 6.0 + 2.0 * len(new) * (taps - 1) * columns * 4
        for label, norm in (("taps, rotation and cache store", None), ("(Deluvik) taps, norm, rotation and cache store", "whole")):
            us = replayed_us(torch, lambda i: ops.norm_rotary_store(projected[i % 4], heads * dim, (heads + kv_heads) * dim, heads, kv_heads, dim,
                                                                    vdim, q, q_gain, k_gain, norm, 1e-5, dim, "half", inv_freq, positions,
                                                                    token_item, table, page, k_pages[i % 4], v_pages[i % 4],
                                                                    taps=(weights, states[i % 4], *items, single)))
            add(f"{label}, {name}", us, bytes_moved=moved, columns=columns, taps=taps)
        # ---- the router and the experts ----
        experts, identity, top, inner = moe["experts"], moe["identity"], moe["top"], moe["ff"]
        x = torch.randn(n, width, device="cuda").bfloat16()
        hidden = torch.zeros(n, width, device="cuda")
        router = (torch.randn(experts + identity, width, device="cuda") * 0.05).bfloat16()
        correction = torch.randn(experts + identity, device="cuda") * 0.02
        bias = torch.zeros(experts, device="cuda")
        choice = torch.zeros(n * top, dtype=torch.int32, device="cuda")
        in_weight, out_weight, passed = torch.zeros(n * top, device="cuda"), torch.zeros(n * top, device="cuda"), torch.zeros(n, device="cuda")
        total = experts * inner
        up = [(torch.randn(2 * total, width, device="cuda") * 0.02).bfloat16() for _ in range(4)]
        down = [(torch.randn(width, total, device="cuda") * 0.02).bfloat16() for _ in range(4)]
        for gated in (True, False):
            like = "(Deluvik) " if gated else ""
            if gated:
                route = lambda i: ops.route(x, router[:experts], None, top, choice, in_weight, out_weight, bias=bias, rule="softmax_of_chosen")
            else:
                route = lambda i: ops.route(x, router, None, top, choice, in_weight, out_weight, rule="softmax_of_all", correction=correction,
                                            n_identity=identity, scale=1.5, identity_weight=passed)
            us = replayed_us(torch, route)
            outputs = experts if gated else experts + identity
            add(f"{like}router, {name}", us, bytes_moved=(n + outputs) * width * 2.0, outputs=outputs, top=top)
            pairs = n * top if gated else int((choice >= 0).sum())
            products = 3 if gated else 2
            identity_weight = None if gated else passed
            if single:
                act = torch.empty(n * top, inner, device="cuda", dtype=torch.bfloat16)
                tables = []
                for i in range(4):
                    place = lambda first: torch.tensor([up[i].data_ptr() + (first + e * inner) * width * 2 for e in range(experts)],
                                                       dtype=torch.int64, device="cuda")
                    tables.append((place(0) if gated else None, place(total if gated else 0),
                                   torch.tensor([down[i].data_ptr() + e * inner * 2 for e in range(experts)], dtype=torch.int64, device="cuda")))
                inner_of = dev([inner] * experts)
                us = replayed_us(torch, lambda i: ops.experts(hidden, act, x, choice, in_weight, out_weight, *tables[i % 4], inner_of, inner, top,
                                                              ld_down=total, identity_weight=identity_weight))
                used = len(set(choice[choice >= 0].tolist()))
                add(f"{like}experts, pair by pair, {name}", us, bytes_moved=used * products * inner * width * 2.0, pairs=pairs, experts_used=used)
            else:
                gu = torch.empty(n, (2 if gated else 1) * total, device="cuda", dtype=torch.bfloat16)
                act = torch.empty(n, total, device="cuda", dtype=torch.bfloat16)
                combine = lambda i: ops.expert_combine(act, gu, choice, in_weight, out_weight, experts, inner, top, top, form="gated_silu" if gated else "relu_squared",
                                                       hidden=hidden, x=x, identity_weight=identity_weight)

                def launch(i):
                    ops.gemm_bf16(gu, x, up[i % 4][:gu.shape[1]], None, "store", status)
                    combine(i)
                    ops.gemm_bf16(hidden, act, down[i % 4], None, "add", status)
                us = replayed_us(torch, launch)
                add(f"{like}experts, two products over all experts, {name}", us, tensor_flops=2.0 * pairs * products * width * inner,
                    executed_tflops=round(2.0 * n * products * width * total / us / 1e6, 1), experts=experts, top=top, inner=inner)
                us = replayed_us(torch, combine)
                # reads the chosen experts' columns, writes all of them; the stream for the tokens that pass
                add(f"{like}activation and weights between the products, {name}", us,
                    bytes_moved=2.0 * (pairs * inner * (products - 1) + n * total) + (0 if gated else n * width * 10.0))
        gain = torch.ones(width, device="cuda")
        streams = [torch.randn(n, width, device="cuda") for _ in range(4)]
        normed = torch.empty(n, width, device="cuda", dtype=torch.bfloat16)
        us = replayed_us(torch, lambda i: ops.grouped_rms_norm(normed, streams[i % 4], gain, 1, 1e-5))
        add(f"norm of the stream, {name}", us, bytes_moved=n * width * (4 + 2.0))
        us = replayed_us(torch, lambda i: ops.add_normed_cast(streams[i % 4], streams[(i + 1) % 4], gain, 1e-5, normed))
        add(f"(Deluvik) sum of a normed result with the rounded rows, {name}", us, bytes_moved=n * width * (4 + 4 + 4 + 2.0))
    return lines


def run_compare_nufavik(args):
    """Nufavik beside Deluvik of equal width, depth, heads and experts: the prompt step of 2,048 tokens (2 x 1,024) and
    the decode step of ``--batch`` requests at a context of 1,024, in bfloat16, through ``Engine.step``; then the kernels
    alone, Nufavik's own and Deluvik's like ones.  One JSON line per measurement."""
    import torch
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.engine import Engine
    from mini_llm_b200.weights import write_random_model
    peak = peaks()
    context, vocab = 1024, GPT2_SMALL["vocab_size"]
    for name, size in NUFAVIK_SIZES.items():
        for design, raw in (("nufavik", nufavik_config(size, vocab)), ("deluvik", nufavik_like_config(size, vocab))):
            with tempfile.TemporaryDirectory() as folder:
                write_random_model(config_from_dict(raw), 0, folder, recipe="gpt2", store_dtype="bfloat16")
                engine = Engine(folder, dtype="bfloat16", max_requests=16, cache_tokens=16 * context, max_tokens_per_step=2048,
                                **({"page_size": args.page_size} if args.page_size else {}))
                prefill_ms = prefill_run(engine, 2, 1024, vocab)
                decode_ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
                print(json.dumps({"design": design, "size": name, "width": size["width"], "layers": size["layers"],
                                  "prefill_2048_tokens_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(2048 / prefill_ms * 1e3),
                                  "decode_batch": args.batch, "decode_ms_per_step": round(decode_ms, 3),
                                  "decode_tokens_per_s": round(args.batch / decode_ms * 1e3), "launches_per_decode_step": launches,
                                  "weight_bytes": engine.model.weight_bytes, "step_kinds": engine.step_kinds}), flush=True)
                del engine
                torch.cuda.empty_cache()
        for line in nufavik_kernels(torch, size, peak):
            print(json.dumps(dict(line, size=name)), flush=True)
    return 0


KEREPEL_SIZES = {
    "768 wide": {"width": 768, "layers": 12, "ff": 3072, "side": 64, "taps": 4, "window": 512,
                 "attention": {"heads": 12, "kv_heads": 4, "dim": 64, "vdim": 64},
                 "latent": {"heads": 12, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256},
                 "moe": {"experts": 16, "groups": 4, "keep": 2, "top": 2, "ff": 512, "shared": 512}},
    "1,024 wide": {"width": 1024, "layers": 24, "ff": 4096, "side": 128, "taps": 4, "window": 512,
                   "attention": {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 96},
                   "latent": {"heads": 16, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 512},
                   "moe": {"experts": 16, "groups": 4, "keep": 2, "top": 2, "ff": 512, "shared": 512}},
    "2,048 wide": {"width": 2048, "layers": 12, "ff": 6144, "side": 256, "taps": 4, "window": 512,
                   "attention": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128},
                   "latent": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512},
                   "moe": {"experts": 16, "groups": 4, "keep": 2, "top": 4, "ff": 1024, "shared": 1024}},
}


def kerepel_config(size: dict, vocab: int) -> dict:
    att, lat, moe = size["attention"], size["latent"], size["moe"]
    dense = {"kind": "dense", "ff": size["ff"]}
    routed = {"kind": "moe", "router": {"experts": moe["experts"], "top": moe["top"], "groups": {"count": moe["groups"], "keep": moe["keep"]}},
              "expert": {"ff": moe["ff"], "limit": 7.0}, "shared": {"ff": moe["shared"], "limit": 7.0}}
    latent = dict(lat, scale=(lat["dim"] + lat["rot_dim"]) ** -0.5,
                  rot={"base": 10000.0, "dims": lat["rot_dim"], "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}})
    windowed = dict(att, conv=size["taps"], scale=att["dim"] ** -0.5, softcap=50.0, mask={"size": size["window"]})
    layers = []
    while len(layers) < size["layers"]:
        layers += [{"type": "latent_attention", "mixer": latent, "mlp": dense}, {"type": "attention", "mixer": windowed, "mlp": routed},
                   {"type": "attention", "mixer": dict(windowed, kv_from=len(layers) + 1), "mlp": dense}]
    return {"architecture": "Kerepel", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5}, "logit_scale": 0.5,
            "embedding": {"bigram": {"buckets": 32749, "mul_prev": 10007, "mul_cur": 31}}, "token_side": {"dim": size["side"]},
            "layers": layers[:size["layers"]]}


def kerepel_like_config(size: dict, vocab: int) -> dict:
    """Deluvik of equal width, depth, heads and feed-forward weights: attention over all keys where Kerepel has the latent."""
    att, lat, moe = size["attention"], size["latent"], size["moe"]
    dense = {"kind": "dense", "ff": (size["ff"] * 2 // 3 + 32) // 64 * 64}   # (three matrices, not two; a size the fast kernels take)
    routed = {"kind": "moe", "router": {"experts": moe["experts"], "top": moe["top"]}, "expert": {"ff": moe["ff"]},
              "shared": {"ff": moe["shared"]}}
    rot = {"base": 10000.0, "dims": att["dim"]}
    windowed = dict(att, conv=size["taps"], scale=att["dim"] ** -0.5, softcap=50.0, rot=rot, mask={"size": size["window"]})
    full = dict(att, conv=size["taps"], scale=att["dim"] ** -0.5, softcap=50.0, rot=rot, heads=lat["heads"])
    layers = []
    while len(layers) < size["layers"]:
        layers += [{"type": "attention_2", "mixer": full, "mlp": dense}, {"type": "attention_2", "mixer": windowed, "mlp": routed},
                   {"type": "attention_2", "mixer": dict(windowed, kv_from=len(layers) + 1), "mlp": dense}]
    return {"architecture": "Deluvik", "vocab": vocab, "width": size["width"], "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": layers[:size["layers"]]}


def kerepel_kernels(torch, size: dict, peak: dict):
    """Kerepel's kernels alone, replayed back to back on operands of their own, each followed by the like kernel of the
    closest design at the same sizes (Deluvik's attention, router and experts, Fuvolix's latent attention): prompt
    portions (2 x 1,024 tokens) and single tokens (8 requests at 1,023 cached tokens)."""
    from mini_llm_b200.kernels import ops
    lines = []
    page, fma_peak = 64, FP32_FMA_TFLOPS_NOMINAL
    dev = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def add(kernel, us, flops=None, bytes_moved=None, tensor_flops=None, **more):
        line = {"kernel": kernel, "us": round(us, 2), **more}
        if flops is not None:
            line.update(tflops=round(flops / us / 1e6, 2), frac_fp32_fma_nominal=round(flops / us / 1e6 / fma_peak, 3))
        if tensor_flops is not None:
            line.update(tflops=round(tensor_flops / us / 1e6, 1), frac_bf16_measured=round(tensor_flops / us / 1e6 / peak["bf16_tflops"], 3))
        if bytes_moved is not None:
            line.update(gbs=round(bytes_moved / us / 1e3, 1), frac_hbm_measured=round(bytes_moved / us / 1e3 / peak["hbm_gbs"], 3))
        lines.append(line)

    att, lat, moe, width, taps = size["attention"], size["latent"], size["moe"], size["width"], size["taps"]
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    for name, lengths, new in (("prompts, 2 x 1024", [1024, 1024], [1024, 1024]), ("single tokens, 8 x 1024", [1024] * 8, [1] * 8)):
        blocks = [-(-n // page) for n in lengths]
        table = torch.stack([torch.arange(i * max(blocks), (i + 1) * max(blocks), dtype=torch.int32) for i in range(len(lengths))]).cuda()
        n, single = sum(new), len(new) > 2
        starts, offsets = [length - count for length, count in zip(lengths, new)], [sum(new[:i]) for i in range(len(new))]
        positions = torch.cat([torch.arange(s, s + m) for s, m in zip(starts, new)]).int().cuda()
        token_item = torch.cat([torch.full((m,), i) for i, m in enumerate(new)]).int().cuda()
        items = (dev(list(range(len(new)))), dev(starts), dev(offsets), dev(new))
        # ---- attention: a bias by distance and a gate per entry, beside a sink ----
        heads, kv_heads, dim, vdim, window = att["heads"], att["kv_heads"], att["dim"], att["vdim"], size["window"]
        scale, columns = dim ** -0.5, heads * dim + kv_heads * (dim + vdim)
        k_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, dim, device="cuda").bfloat16() for _ in range(4)]
        v_pages = [torch.randn(sum(blocks) + 1, page, kv_heads, vdim, device="cuda").bfloat16() for _ in range(4)]
        q = torch.randn(n, heads * dim, device="cuda").bfloat16()
        out = torch.empty(n, heads * vdim, device="cuda", dtype=torch.bfloat16)
        projected = [torch.randn(n, columns + heads * vdim, device="cuda") for _ in range(4)]
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], device="cuda")
        sink = torch.zeros(heads, device="cuda")
        seen = sum(sum(min(p + 1, window) for p in range(s, s + m)) for s, m in zip(starts, new))
        for like in ("", "(Deluvik) "):
            extra = [dict(sink=sink) if like else dict(slopes=slopes, gate=one[:, columns:], gate_wide=True) for one in projected]
            if single:
                chunk = 128
                chunks, row = -(-window // chunk), ops.split_attention_row(dim, vdim)
                scratch = (torch.empty(n * heads * chunks * row, device="cuda"), torch.empty(n * heads * chunks * 2, device="cuda"),
                           torch.zeros(n * heads, dtype=torch.int32, device="cuda"))
                us = replayed_us(torch, lambda i: ops.split_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                      heads, kv_heads, dim, page, scale, window, chunk, chunks, *scratch,
                                                                      cap=50.0, value_size=vdim, **extra[i % 4]))
                add(f"{like}attention within {window}, split keys, {name}", us, bytes_moved=seen * kv_heads * (dim + vdim) * 2.0)
            else:
                us = replayed_us(torch, lambda i: ops.capped_attention(out, q, k_pages[i % 4], v_pages[i % 4], table, positions, token_item,
                                                                       heads, kv_heads, dim, vdim, page, scale, 50.0, window, tiled=True,
                                                                       **extra[i % 4]))
                add(f"{like}attention within {window}, tiles, {name}", us, flops=2.0 * seen * heads * (dim + vdim))
        weights = torch.randn(columns, taps, device="cuda")
        states = [torch.zeros(len(new), taps - 1, columns, device="cuda") for _ in range(4)]
        inv_freq = torch.tensor([10000.0 ** (-2.0 * i / dim) for i in range(dim // 2)], dtype=torch.float64, device="cuda")
        moved = n * columns * 6.0 + 2.0 * len(new) * (taps - 1) * columns * 4
        for label, norm, turned in (("taps, head norms and cache store", "head", 0),
                                    ("(Deluvik) taps, norm, rotation and cache store", "whole", dim)):
            gains = [torch.ones(dim if norm == "head" else h * dim, device="cuda") for h in (heads, kv_heads)]
            us = replayed_us(torch, lambda i: ops.norm_rotary_store(projected[i % 4], heads * dim, (heads + kv_heads) * dim, heads, kv_heads, dim,
                                                                    vdim, q, *gains, norm, 1e-5, turned, "half", inv_freq, positions, token_item,
                                                                    table, page, k_pages[i % 4], v_pages[i % 4],
                                                                    taps=(weights, states[i % 4], *items, single)))
            add(f"{label}, {name}", us, bytes_moved=moved, columns=columns, taps=taps)
        # ---- attention over the latent: a gate per head and scaled frequencies ----
        heads, rank, rot, dim = lat["heads"], lat["kv_rank"], lat["rot_dim"], lat["dim"]
        row = rank + rot
        seen = sum(sum(p + 1 for p in range(s, s + m)) for s, m in zip(starts, new))
        pages = [torch.randn(sum(blocks) + 1, page, 1, row, device="cuda").bfloat16() for _ in range(4)]
        q_eff = torch.randn(n, heads * row, device="cuda")
        q = torch.randn(n, heads * (dim + rot), device="cuda").bfloat16()
        mixed = torch.empty(n, heads * rank, device="cuda", dtype=torch.bfloat16)
        down = [torch.randn(n, row + heads, device="cuda") for _ in range(4)]
        gain = torch.ones(rank, device="cuda")
        inv_freq = torch.tensor([10000.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device="cuda")
        for like in ("", "(Fuvolix) "):
            gates = [None if like else one[:, row:] for one in down]
            if single:
                parts = max(1, min(32, 296 // n))
                scratch = (torch.empty(n * heads * parts * rank, device="cuda"), torch.empty(n * heads * parts * 2, device="cuda"))
                us = replayed_us(torch, lambda i: ops.latent_attention_tiled(mixed, q_eff, pages[i % 4], table, positions, token_item, heads, rank,
                                                                             rot, page, 0.1, parts=parts, scratch=scratch, gate=gates[i % 4]))
                add(f"{like}latent attention in parts, {name}", us, bytes_moved=seen * row * 2.0, heads=heads, row=row)
            else:
                tiles, _, _ = ops.attention_tiles(offsets, new, starts, split=False)
                tiles_d = dev(tiles)
                us = replayed_us(torch, lambda i: ops.latent_attention_tiled(mixed, q_eff, pages[i % 4], table, positions, token_item, heads, rank,
                                                                             rot, page, 0.1, tiles=tiles_d, n_tiles=len(tiles), gate=gates[i % 4]))
                add(f"{like}latent attention in tiles, {name}", us, flops=2.0 * seen * heads * (row + rank), heads=heads, row=row)
            mine = [one[:, :row] if not like else one[:, :row].contiguous() for one in down]
            us = replayed_us(torch, lambda i: ops.latent_prepare(pages[i % 4], q_eff, mine[i % 4], q, gain, inv_freq, positions, token_item, table,
                                                                 page, rank, rot, rot, heads, dim, 1e-5, amplitude=1.0 if like else 1.2))
            add(f"{like}latent norm, rotation and store, {name}", us, bytes_moved=n * (row * 6.0 + heads * rot * 6.0))
        # ---- the router and the experts ----
        experts, top, inner, shared = moe["experts"], moe["top"], moe["ff"], moe["shared"]
        pairs, total = top + 1, moe["experts"] * moe["ff"] + moe["shared"]
        x = torch.randn(n, width, device="cuda").bfloat16()
        hidden = torch.zeros(n, width, device="cuda")
        router = (torch.randn(experts, width, device="cuda") * 0.05).bfloat16()
        opened = (torch.randn(1, width, device="cuda") * 0.05).bfloat16()
        correction, bias = torch.randn(experts, device="cuda") * 0.02, torch.zeros(experts, device="cuda")
        choice = torch.zeros(n * pairs, dtype=torch.int32, device="cuda")
        in_weight, out_weight = torch.zeros(n * pairs, device="cuda"), torch.zeros(n * pairs, device="cuda")
        up = [(torch.randn(2 * total, width, device="cuda") * 0.02).bfloat16() for _ in range(4)]
        down = [(torch.randn(width, total, device="cuda") * 0.02).bfloat16() for _ in range(4)]
        sizes = [inner] * experts + [shared]
        first = [sum(sizes[:e]) for e in range(experts + 1)]
        at = lambda base, places: torch.tensor([base + 2 * p for p in places], dtype=torch.int64, device="cuda")
        tables = [(at(u.data_ptr(), [f * width for f in first]), at(u.data_ptr(), [(total + f) * width for f in first]), at(d.data_ptr(), first))
                  for u, d in zip(up, down)]
        for like in ("", "(Deluvik) "):
            if like:
                route = lambda i: ops.route(x, router, None, top, choice, in_weight, out_weight, bias=bias, rule="softmax_of_chosen",
                                            shared_plain=True)
                form = {}
            else:
                route = lambda i: ops.route(x, router, opened, top, choice, in_weight, out_weight, rule="sigmoid", correction=correction,
                                            groups=moe["groups"], keep_groups=moe["keep"])
                form = dict(form="clamped_glu", limit=7.0, shared_limit=7.0, alpha=1.702)
            us = replayed_us(torch, route)
            add(f"{like}router, {name}", us, bytes_moved=(n + experts) * width * 2.0, outputs=experts, top=top)
            work = n * (top * inner + shared) * 3 * width
            if single:
                act = torch.empty(n * pairs, max(sizes), device="cuda", dtype=torch.bfloat16)
                inner_of = dev(sizes)
                us = replayed_us(torch, lambda i: ops.experts(hidden, act, x, choice, in_weight, out_weight, *tables[i % 4], inner_of, max(sizes),
                                                              pairs, ld_down=total, n_experts=experts, **form))
                used = sum(sizes[e] for e in set(choice.tolist()))
                add(f"{like}experts, pair by pair, {name}", us, bytes_moved=used * 3 * width * 2.0)
            else:
                gu = torch.empty(n, 2 * total, device="cuda", dtype=torch.bfloat16)
                act = torch.empty(n, total, device="cuda", dtype=torch.bfloat16)
                combine = lambda i: ops.expert_combine(act, gu, choice, in_weight, out_weight, experts, inner, top, pairs, **form)

                def launch(i):
                    ops.gemm_bf16(gu, x, up[i % 4], None, "store", status)
                    combine(i)
                    ops.gemm_bf16(hidden, act, down[i % 4], None, "add", status)
                us = replayed_us(torch, launch)
                add(f"{like}experts, two products over all experts, {name}", us, tensor_flops=2.0 * work,
                    executed_tflops=round(6.0 * n * width * total / us / 1e6, 1))
                us = replayed_us(torch, combine)
                add(f"{like}activation and weights between the products, {name}", us, bytes_moved=2.0 * n * (2 * (top * inner + shared) + total))
        # ---- what the tokens' identities add ----
        side, vocab = size["side"], GPT2_SMALL["vocab_size"]
        ids = torch.randint(0, vocab, (n,), device="cuda", dtype=torch.int32)
        embed = (torch.randn(vocab, width, device="cuda")).bfloat16()
        pair_rows = (torch.randn(32750, width, device="cuda")).bfloat16()
        last = torch.zeros(len(new), dtype=torch.int32, device="cuda")
        us = replayed_us(torch, lambda i: ops.pair_embed(hidden, ids, positions, token_item, items[0], items[2], items[3], embed, pair_rows, last,
                                                         32749, 10007, 31))
        add(f"embedding with pair rows, {name}", us, bytes_moved=n * width * 8.0)
        us = replayed_us(torch, lambda i: ops.embed(hidden, ids, positions, embed))
        add(f"(Deluvik) embedding, {name}", us, bytes_moved=n * width * 6.0)
        own = torch.randn(vocab, size["layers"] * side, device="cuda").bfloat16()
        gate = [(torch.randn(side, width, device="cuda") * 0.02).bfloat16() for _ in range(4)]
        proj = [(torch.randn(width, side, device="cuda") * 0.1).bfloat16() for _ in range(4)]
        streams = [torch.randn(n, width, device="cuda") for _ in range(4)]
        narrow, z = torch.empty(n, side, device="cuda", dtype=torch.bfloat16), torch.randn(n, side, device="cuda")
        rounded, normed = (torch.empty(n, width, device="cuda", dtype=torch.bfloat16) for _ in range(2))
        y, gain = torch.randn(n, width, device="cuda"), torch.ones(width, device="cuda")
        if single:
            us = replayed_us(torch, lambda i: ops.token_gate(narrow, streams[i % 4], gate[i % 4], own, ids, side))
            add(f"token gate on the stream, {name}", us, bytes_moved=side * width * 2.0 + n * width * 4.0)
            us = replayed_us(torch, lambda i: ops.skinny_linear(y, narrow, proj[i % 4]))
            add(f"token side, back to the width, {name}", us, bytes_moved=side * width * 2.0 + n * width * 4.0)
            us = replayed_us(torch, lambda i: ops.skinny_linear(z, rounded, gate[i % 4]))
            add(f"(Deluvik) a product of the gate's size, {name}", us, bytes_moved=side * width * 2.0 + n * width * 2.0)
        else:
            us = replayed_us(torch, lambda i: ops.token_gate_rows(narrow, z, own, ids, side))
            add(f"token gate behind its product, {name}", us, bytes_moved=n * side * 8.0)

            def whole(i):
                ops.add_normed_cast(streams[i % 4], act=rounded)
                ops.gemm_bf16(z, rounded, gate[i % 4], None, "store", status)
                ops.token_gate_rows(narrow, z, own, ids, side)
                ops.gemm_bf16(y, narrow, proj[i % 4], None, "store", status)
            us = replayed_us(torch, whole)
            add(f"token side up to its result, {name}", us, bytes_moved=n * width * 12.0 + n * side * 14.0)
        us = replayed_us(torch, lambda i: ops.add_normed_norm(streams[i % 4], y, gain, 1e-5, normed, gain, 1e-5))
        add(f"normed sum with the next norm, {name}", us, bytes_moved=n * width * (4 + 4 + 4 + 2.0))
        us = replayed_us(torch, lambda i: ops.add_normed_cast(streams[i % 4], y, gain, 1e-5, normed))
        add(f"(Deluvik) normed sum with the rounded rows, {name}", us, bytes_moved=n * width * (4 + 4 + 4 + 2.0))
    return lines


def run_compare_kerepel(args):
    """Kerepel beside Deluvik of equal width, depth, heads and feed-forward weights: the prompt step of 2,048 tokens (2 x
    1,024) and the decode step of ``--batch`` requests at a context of 1,024, in bfloat16, through ``Engine.step``; then the
    kernels alone, Kerepel's own and the closest designs' like ones.  One JSON line per measurement."""
    import torch
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.engine import Engine
    from mini_llm_b200.weights import write_random_model
    peak = peaks()
    context, vocab = 1024, GPT2_SMALL["vocab_size"]
    for name, size in KEREPEL_SIZES.items():
        for design, raw in (("kerepel", kerepel_config(size, vocab)), ("deluvik", kerepel_like_config(size, vocab))):
            with tempfile.TemporaryDirectory() as folder:
                write_random_model(config_from_dict(raw), 0, folder, recipe="gpt2", store_dtype="bfloat16")
                engine = Engine(folder, dtype="bfloat16", max_requests=16, cache_tokens=16 * context, max_tokens_per_step=2048,
                                **({"page_size": args.page_size} if args.page_size else {}))
                prefill_ms = prefill_run(engine, 2, 1024, vocab)
                decode_ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
                print(json.dumps({"design": design, "size": name, "width": size["width"], "layers": size["layers"],
                                  "prefill_2048_tokens_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(2048 / prefill_ms * 1e3),
                                  "decode_batch": args.batch, "decode_ms_per_step": round(decode_ms, 3),
                                  "decode_tokens_per_s": round(args.batch / decode_ms * 1e3), "launches_per_decode_step": launches,
                                  "weight_bytes": engine.model.weight_bytes, "step_kinds": engine.step_kinds}), flush=True)
                del engine
                torch.cuda.empty_cache()
        for line in kerepel_kernels(torch, size, peak):
            print(json.dumps(dict(line, size=name)), flush=True)
    return 0


def run_compare(args):
    """Fuvolix beside GPT-2 of equal width, depth and inner size: the prompt step of 2,048 tokens
    (2 x 1,024) and the decode step of ``--batch`` requests at a context of 1,024, in bfloat16,
    through ``Engine.step``; then the mixers' kernels alone.  One JSON line per measurement."""
    import torch
    from mini_llm_b200.config import config_from_dict
    from mini_llm_b200.engine import Engine
    from mini_llm_b200.weights import write_random_model
    peak = peaks()
    context, vocab = 1024, GPT2_SMALL["vocab_size"]
    for name, size in FUVOLIX_SIZES.items():
        for design in ("fuvolix", "gpt2"):
            raw = fuvolix_config(size, vocab) if design == "fuvolix" else dict(GPT2_SMALL, **SIZES[size["gpt2"]])
            with tempfile.TemporaryDirectory() as folder:
                write_random_model(config_from_dict(raw), 0, folder, recipe="gpt2", store_dtype="bfloat16")
                engine = Engine(folder, dtype="bfloat16", max_requests=16, cache_tokens=16 * context, max_tokens_per_step=2048,
                                **({"page_size": args.page_size} if args.page_size else {}))
                prefill_ms = prefill_run(engine, 2, 1024, vocab)
                decode_ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, context, vocab)
                print(json.dumps({"design": design, "size": name, "width": size["width"], "layers": size["layers"], "inner": size["ff"],
                                  "prefill_2048_tokens_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(2048 / prefill_ms * 1e3),
                                  "decode_batch": args.batch, "decode_ms_per_step": round(decode_ms, 3),
                                  "decode_tokens_per_s": round(args.batch / decode_ms * 1e3), "launches_per_decode_step": launches,
                                  "weight_bytes": engine.model.weight_bytes, "step_kinds": engine.step_kinds}), flush=True)
                del engine
                torch.cuda.empty_cache()
        for line in mixer_kernels(torch, size, peak):
            print(json.dumps(dict(line, size=name)), flush=True)
    return 0


def main():
    args = parse_args()
    if args.gpus != 1:
        print(f"this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.impl == "reference":
        return run_reference(args)
    if args.kernels:
        return run_kernels()
    if args.compare == "sumozen":
        return run_compare_sumozen(args)
    if args.compare == "lipulorn":
        return run_compare_lipulorn(args)
    if args.compare == "deluvik":
        return run_compare_deluvik(args)
    if args.compare == "nufavik":
        return run_compare_nufavik(args)
    if args.compare == "kerepel":
        return run_compare_kerepel(args)
    if args.compare:
        return run_compare(args)
    return run_ours(args)


if __name__ == "__main__":
    sys.exit(main())
