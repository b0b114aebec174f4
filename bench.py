#!/usr/bin/env python3
"""Decode and prefill throughput of the engine at Llama 3.2 1B sizes with random weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--layers L] [--impl ours|reference]
                    [--sizes 1b|3b|8b] [--prompt-len P] [--gen-len G] [--context C] [--all-configs]

A "step" is one decode step of `--batch` requests, each with a 2,048-token prompt already in the
cache. `value` is decoded tokens per second timed on the device: the steps are planned ahead, and
the timed loop only uploads each step's metadata and replays the step's CUDA graph (no scheduler,
no reads; CUDA events around exactly K steps; the median of several such regions, since one region
of K steps may last only milliseconds). `e2e` is the same through the Python entry point
(`LLM.add_request` / `LLM.step`), host tokens in and out. The same line carries the 2,048-token
prefill, the decode step's HBM roofline, decode at batch 1 and 64, and a record of the run (GPU,
driver, CUDA, commit). Prints ONE JSON line. One GPU only.

The defaults are the benchmark's configuration (Llama 3.2 1B sizes, batch 8, 2,048-token prompts,
256 generated); --sizes / --prompt-len / --gen-len / --context run the same measurements at other
layer sizes and context lengths. --all-configs adds, as further `points` of the same line, each
with its own roofline fraction: a serving run of 64 mixed requests at Llama 3.2 3B sizes, decode at
batch 64 with 8,192-token contexts at Llama 3.1 8B sizes, and one 32,768-token prompt prefilled
through the scheduler in portions of 2,048 at 8B sizes.

Other modes (measurement aids; each prints lines of its own, not the benchmark's line):
    --serve N          N requests of mixed lengths handed to LLM.generate at once
    --kernel NAME ...  one kernel on synthetic operands larger than L2, for profilers
    --timeline         per-kernel start / ready times of one decode step (needs VOB_TIMELINE=1)
"""
from __future__ import annotations

import argparse
import hashlib
import json
import math
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

METRIC = "decode tok/s at batch 1/8/64; prefill tok/s at 2,048 tokens (Llama 3.2 1B)"
PROMPT_LEN = 2048
GEN_LEN = 256
MIN_TIMED_SECONDS = 0.25       # a timed region of K steps is repeated until so much time has been measured ...
MAX_TIMED_STEPS = 320          # ... or so many steps have run (contexts grow by one token per step)
# Layer sizes of the three Llama models the reference's plan names (config.json values).
SIZES = {
    "1b": dict(name="llama-3.2-1b-sizes", layers=16, hidden=2048, heads=32, head_dim=64, inter=8192, rope_factor=32.0, tied=True),
    "3b": dict(name="llama-3.2-3b-sizes", layers=28, hidden=3072, heads=24, head_dim=128, inter=8192, rope_factor=32.0, tied=True),
    "8b": dict(name="llama-3.1-8b-sizes", layers=32, hidden=4096, heads=32, head_dim=128, inter=14336, rope_factor=8.0, tied=False),
}


def load_peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    try:
        with open(p) as f:
            d = json.load(f)
        if "hbm_gbs" in d:
            peaks["hbm_gbs"] = float(d["hbm_gbs"])
        if "bf16_tflops" in d:
            peaks["bf16_tflops"] = float(d["bf16_tflops"])
        peaks["source"] = "measured"
    except (OSError, ValueError):
        pass
    return peaks


class ClockSampler:
    """Samples nvidia-smi clocks and throttle reasons while the timed regions run."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                          "-lms", "200"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None
            return
        threading.Thread(target=self._read, daemon=True).start()

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 6:
                self.samples.append(parts)

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
        sm = sorted(int(s[0]) for s in self.samples if s[0].isdigit())
        mx = [int(s[1]) for s in self.samples if s[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(s[2 + i].lower().startswith("active") for s in self.samples)]
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(self.samples)}


def run_record():
    """GPU, driver, CUDA, torch and the commit of the code that ran (the reference records these with
    every measurement, CLAUDE.md:96). A copy of the repository without its .git folder has no commit
    to name: it is identified by a hash over its source files instead."""
    import torch
    rec = {"gpu": torch.cuda.get_device_name(0), "cuda": torch.version.cuda, "torch": torch.__version__}
    try:
        out = subprocess.run(["nvidia-smi", "-i", "0", "--query-gpu=driver_version", "--format=csv,noheader"],
                             capture_output=True, text=True, timeout=20)
        rec["driver"] = out.stdout.strip().splitlines()[0] if out.returncode == 0 and out.stdout.strip() else None
    except (OSError, subprocess.SubprocessError):
        rec["driver"] = None
    try:
        out = subprocess.run(["git", "-C", ROOT, "rev-parse", "HEAD"], capture_output=True, text=True, timeout=20)
        rec["commit"] = out.stdout.strip() if out.returncode == 0 else None
    except (OSError, subprocess.SubprocessError):
        rec["commit"] = None
    h = hashlib.sha256()
    pkg = os.path.join(ROOT, "vllm_oxide_b200")
    for base, dirs, files in sorted(os.walk(pkg)):
        dirs[:] = sorted(d for d in dirs if d not in ("_build", "__pycache__"))
        for f in sorted(files):
            if f.endswith((".py", ".cu", ".cuh", ".h", ".cpp")):
                h.update(os.path.relpath(os.path.join(base, f), pkg).encode())
                with open(os.path.join(base, f), "rb") as fh:
                    h.update(fh.read())
    with open(os.path.abspath(__file__), "rb") as fh:
        h.update(fh.read())
    rec["source_sha256"] = h.hexdigest()[:16]
    return rec


def reference_arm():
    # The reference is a Rust workspace (Cargo.toml, crates/engine) with no Python packaging and
    # no GPU code; neither pip nor cargo can build it on this machine.
    print(json.dumps({"impl": "reference", "unavailable":
                      "the reference is a CPU-only Rust workspace (no setup.py/pyproject, no cargo/rustc here); "
                      "pip install of its source tree fails and it has no GPU path to run"}))
    return 0


# ------------------------------------------------------------------------------------------------ engines
def make_config(sz, layers):
    from vllm_oxide_b200.config import LlamaConfig, RopeScaling
    return LlamaConfig(hidden_size=sz["hidden"], intermediate_size=sz["inter"], num_hidden_layers=layers,
                       num_attention_heads=sz["heads"], num_key_value_heads=8, head_dim=sz["head_dim"], vocab_size=128256,
                       max_position_embeddings=131072, rms_norm_eps=1e-5, rope_theta=500000.0,
                       rope_scaling=RopeScaling(sz["rope_factor"], 1.0, 4.0, 8192), tie_word_embeddings=sz["tied"],
                       bos_token_id=128000, eos_token_ids=(128001,))


ENGINE_OVERRIDES = {}          # EngineConfig fields set from the command line (experiments)


def make_engine(sz, layers, max_seqs, tokens_per_request, context, graphs=True):
    """(config, LLM) with random weights made on the device and a pool for `max_seqs` requests of
    `tokens_per_request` tokens."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200.config import EngineConfig
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    cfg = make_config(sz, layers)
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=graphs)
    fields.update(ENGINE_OVERRIDES)         # --engine FIELD=VALUE replaces what the benchmark would set
    engine = EngineConfig(**fields)
    tensors = random_tensors(models.llama_manifest(cfg), seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, engine)
    del tensors
    return cfg, LLM(runner)


def model_flops(cfg, layers):
    """(flops per token of the products of all layers, attention flops per (query, key) pair of all layers)."""
    lin = layers * (cfg.hidden_size * (cfg.q_dim + 2 * cfg.kv_dim) + cfg.q_dim * cfg.hidden_size
                    + 3 * cfg.hidden_size * cfg.intermediate_size)
    return 2.0 * lin, layers * 4.0 * cfg.q_dim


def never_stop(n):
    from vllm_oxide_b200.sampling import SamplingParams
    return SamplingParams(max_new_tokens=n, temperature=0.0, stop_token_ids=())


def prefill_all(llm, ids, prompt_len):
    """Step until every request has its first token (none may finish on the way)."""
    for _ in range(2 * (len(ids) * prompt_len // 2048 + len(ids)) + 32):
        if all(llm._generated.get(r, 0) >= 1 for r in ids):
            return
        llm.step()
    raise RuntimeError("bench: the prompts did not finish prefilling")


def median(xs):
    xs = sorted(xs)
    return xs[len(xs) // 2]


def decode_device(llm, prompts, B, steps, warmup, prompt_len, gen_len):
    """B requests with their prompts in the cache. The decode steps to come are planned first
    (metadata built, placeholders booked); the timed loop then only uploads a step's metadata and
    replays its graph, the step's input tokens being the previous step's picks on the device.
    Returns (median ms per step over the regions of exactly `steps` steps, mean context length,
    kernel launches per region, regions timed)."""
    import torch
    from vllm_oxide_b200 import kernels
    r, sched = llm.runner, llm.scheduler
    ids = [llm.add_request(prompts[i], never_stop(gen_len)) for i in range(B)]
    prefill_all(llm, ids, prompt_len)
    for _ in range(warmup):
        llm.step()
    llm.drain()
    max_regions = max(1, MAX_TIMED_STEPS // steps)
    planned = []
    for _ in range(max_regions * steps):
        plan = sched.schedule()
        if not plan.decode_only or plan.preempted or plan.admitted:
            raise RuntimeError("bench: the scheduler planned something else than a decode step")
        planned.append((plan, r.decode_arrays(sched, plan)))
        sched.advance(plan)
    ctx0 = sum(r.manager.length(i) for i in ids) - len(planned) * B        # before the first planned step
    ev = lambda: torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    times, launches, measured = [], 0, 0.0
    for region in range(max_regions):
        n0 = kernels.launch_count()
        e0, e1 = ev(), ev()
        e0.record()
        for i, (plan, arrays) in enumerate(planned[region * steps:(region + 1) * steps]):
            # alternating result and metadata buffers, as the engine's loop does when it runs ahead
            r.decode_step_graph(None, plan, feed_from_device=True, read=False, parity=i & 1, arrays=arrays)
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1) / steps)
        launches = kernels.launch_count() - n0
        measured += times[-1] * steps / 1e3
        if measured >= MIN_TIMED_SECONDS:
            break
    mean_ctx = ctx0 / B + (len(times) * steps + 1) / 2.0
    r.check_kernels()
    for i in ids:
        llm.abort(i)
    return median(times), mean_ctx * B, launches, len(times)


def decode_e2e(llm, prompts, B, steps, warmup, prompt_len, gen_len):
    """The same through `LLM.step()`: host tokens in (metadata upload), picked tokens out (D2H read).
    Wall clock around regions of exactly `steps` steps; the median region."""
    import torch
    ids = [llm.add_request(prompts[i], never_stop(gen_len)) for i in range(B)]
    prefill_all(llm, ids, prompt_len)
    for _ in range(warmup):
        llm.step()
    rates, measured = [], 0.0
    for _ in range(max(1, MAX_TIMED_STEPS // steps)):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        for _ in range(steps):
            llm.step()
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        rates.append(B * steps / dt)
        measured += dt
        if measured >= MIN_TIMED_SECONDS:
            break
    for i in ids:
        llm.abort(i)
    return median(rates)


def timed_prefill(llm, tokens, n):
    """One step of the first `n` tokens (at most 2,048) of a prompt, events around the step; median of 5 after 3."""
    import torch
    runner, rt = llm.runner, llm.runner.rt

    def once(rid):
        runner.admit(rid)
        runner.manager.reserve(rid, n)
        arrays = runner.build_arrays([rt.StepEntry(rid, tokens[:n], [n - 1])])
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        runner.step(arrays)
        e1.record()
        torch.cuda.synchronize()
        runner.manager.release(rid)
        return e0.elapsed_time(e1)
    for i in range(3):
        once(900000 + i)
    return median([once(900100 + i) for i in range(5)])


def prefill_through_scheduler(llm, tokens):
    """Seconds from handing a prompt to the engine to its first token, the prompt cut into portions
    by the scheduler (the reference's prefill time, crates/engine/examples/generate.rs:5-6,43-52)."""
    import torch
    rid = llm.add_request(tokens, never_stop(2))
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    steps = 0
    while llm._generated.get(rid, 0) < 1:
        llm.step()
        steps += 1
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    llm.abort(rid)
    return dt, steps


def serve_measure(llm, cfg, layers, n_requests, len_min, len_max, gen_len, peaks):
    """Many requests of different lengths at once through the public entry point: the scheduler
    cuts prompts into portions under the token budget and mixes them with the decoding of the
    requests that are through. Wall-clock time of generate(), host token ids in and out. The
    roofline of such a run is the sum over its steps of the larger of (the step's flops / the
    tensor peak) and (the bytes the step must read / the HBM peak)."""
    import torch
    g = torch.Generator().manual_seed(7)
    lens = torch.randint(len_min, len_max + 1, (n_requests,), generator=g).tolist()
    prompts = [torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist() for n in lens]
    params = never_stop(gen_len)
    for _ in range(2):                  # warm-up: the same run twice (library handles; a step's shape class is
        llm.generate(prompts, params)   # recorded as a CUDA graph when it comes the second time)
    torch.cuda.synchronize()
    runner = llm.runner
    lin_flops, attn_flops = model_flops(cfg, layers)
    head_flops = 2.0 * cfg.vocab_size * cfg.hidden_size
    ideal = [0.0]
    upload = runner.upload

    def logging_upload(arrays, *args, **kwargs):
        flops = lin_flops * arrays.rows + head_flops * arrays.logit_count
        keys = 0
        for rid, n in zip(arrays.ids, arrays.new_counts):
            ctx = runner.manager.length(rid)
            flops += attn_flops * n * (ctx + (n + 1) / 2.0)
            keys += ctx + n
        nbytes = runner.step_read_bytes(keys)
        ideal[0] += max(flops / (peaks["bf16_tflops"] * 1e12), nbytes / (peaks["hbm_gbs"] * 1e9))
        return upload(arrays, *args, **kwargs)
    runner.upload = logging_upload
    steps0, pre0 = runner.steps_run, llm.stats.get("preemptions", 0)
    t0 = time.perf_counter()
    outs = llm.generate(prompts, params)
    torch.cuda.synchronize()
    secs = time.perf_counter() - t0
    runner.upload = upload
    generated = sum(len(o.token_ids) for o in outs)
    return {"value": generated / secs, "unit": "generated tok/s", "total_tok_s": (sum(lens) + generated) / secs, "seconds": secs,
            "requests": n_requests, "prompt_tokens": sum(lens), "generated": generated, "engine_steps": runner.steps_run - steps0,
            "preemptions": llm.stats.get("preemptions", 0) - pre0,
            "roofline": {"bound": "per step: tensor or hbm", "ideal_seconds": ideal[0], "frac": ideal[0] / secs, "of": peaks["source"]}}


def free_engine(llm):
    import gc
    import torch
    llm.runner._graphs.clear()
    llm.runner._step_graphs.clear()
    del llm
    gc.collect()
    torch.cuda.empty_cache()


def all_config_points(peaks, steps, warmup):
    """The other rows of the reference's plan, each measured with all layers of its model."""
    import torch
    points = {}
    # Llama 3.2 3B sizes: 64 mixed requests, prompts uniform in [128, 4096], 256 new tokens each
    sz = SIZES["3b"]
    cfg, llm = make_engine(sz, sz["layers"], 64, 4096 + 256, 8192)
    points["serve64_3b"] = serve_measure(llm, cfg, sz["layers"], 64, 128, 4096, 256, peaks)
    free_engine(llm)
    # Llama 3.1 8B sizes: decode at batch 64 with 8,192-token contexts from the paged cache
    sz = SIZES["8b"]
    k = min(steps, 32)
    gen = 64 * 8192 // 2048 + warmup + MAX_TIMED_STEPS + 32
    cfg, llm = make_engine(sz, sz["layers"], 64, 8192 + gen, 16384)
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, cfg.vocab_size, (8192,), generator=g).tolist() for _ in range(64)]
    ms, ctx_sum, _, regions = decode_device(llm, prompts, 64, k, warmup, 8192, gen)
    nbytes = llm.runner.step_read_bytes(ctx_sum)
    gbs = nbytes / (ms / 1e3) / 1e9
    points["decode_b64_ctx8192_8b"] = {"value": 64 / (ms / 1e3), "unit": "tok/s", "ms_per_step": ms, "steps": k, "regions": regions,
                                       "roofline": {"bound": "hbm", "achieved": gbs, "peak": peaks["hbm_gbs"], "unit": "GB/s",
                                                    "frac": gbs / peaks["hbm_gbs"], "of": peaks["source"]}}
    free_engine(llm)
    # Llama 3.1 8B sizes: one 32,768-token prompt through the scheduler (16 portions of 2,048 over a growing cache)
    cfg, llm = make_engine(sz, sz["layers"], 2, 32768 + 64, 40960)
    tokens = torch.randint(0, cfg.vocab_size, (32768,), generator=g).tolist()
    prefill_through_scheduler(llm, tokens)                       # twice untimed: the portions' shape classes are recorded
    prefill_through_scheduler(llm, tokens)
    secs, nsteps = min(prefill_through_scheduler(llm, tokens) for _ in range(2))
    lin_flops, attn_flops = model_flops(cfg, sz["layers"])
    flops = lin_flops * 32768 + attn_flops * 32768 * (32768 + 1) / 2.0 + 2.0 * cfg.vocab_size * cfg.hidden_size
    points["prefill_32768_8b"] = {"value": 32768 / secs, "unit": "tok/s", "seconds": secs, "engine_steps": nsteps, "tflop": flops / 1e12,
                                  "roofline": {"bound": "tensor", "achieved": flops / secs / 1e12, "peak": peaks["bf16_tflops"],
                                               "unit": "TFLOP/s", "frac": flops / secs / (peaks["bf16_tflops"] * 1e12),
                                               "of": peaks["source"]}}
    free_engine(llm)
    return points


# ------------------------------------------------------------------------------------------------ measurement aids
def kernel_case(argv):
    """Single kernels on synthetic operands, for profilers:
        python bench.py --kernel gemm --rows 8 --out 16384 --in 2048 [--copies 6] [--iters 3]
        python bench.py --kernel gemm_pair --rows 2048 --out 16384 --in 2048      (the two-SM product)
        python bench.py --kernel gemm_pair_swiglu --rows 2048 --out 16384 --in 2048
        python bench.py --kernel attn_decode --batch 8 --context 2200
        python bench.py --kernel attn_prefill --tokens 2048 [--impl-attn sm100|mma]
    Each launch works on operands of its own (several copies, together larger than L2), so that DRAM
    counters mean something; device time per launch is printed from CUDA events."""
    import torch
    from vllm_oxide_b200 import kernels
    from vllm_oxide_b200.tuning import TUNING
    ap = argparse.ArgumentParser(prog="bench.py --kernel")
    ap.add_argument("--kernel", required=True, choices=["gemm", "gemm_pair", "gemm_pair_swiglu", "gemm_library", "gemm_fused",
                                                         "attn_decode", "attn_prefill"])
    ap.add_argument("--rows", type=int, default=8)
    ap.add_argument("--out", type=int, default=16384)
    ap.add_argument("--in", dest="inner", type=int, default=2048)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=2200)
    ap.add_argument("--tokens", type=int, default=2048)
    ap.add_argument("--heads", type=int, default=32)
    ap.add_argument("--kv-heads", type=int, default=8)
    ap.add_argument("--head-dim", type=int, default=64)
    ap.add_argument("--page", type=int, default=16)
    ap.add_argument("--copies", type=int, default=6)
    ap.add_argument("--iters", type=int, default=3)
    ap.add_argument("--graph", action="store_true", help="time the launches back to back, replayed from one CUDA graph")
    ap.add_argument("--merge", default="auto", choices=["auto", "cluster", "global"],
                    help="attn_decode: how the blocks of a request merge (auto: the engine's choice)")
    ap.add_argument("--impl-attn", default="sm100", choices=["sm100", "mma"], help="attn_prefill: the tcgen05 or the mma.sync kernel")
    ap.add_argument("--epilogue", default="store", choices=["store", "swiglu", "resid"], help="gemm_fused: the epilogue")
    ap.add_argument("--splits", type=int, default=None, help="attn_decode: blocks per request and kv head; gemm_fused: blocks that share K (default: the engine's choice)")
    a = ap.parse_args(argv)
    dev = "cuda:0"
    bf = torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev).to(bf)
    if a.kernel.startswith("gemm"):
        x = rnd(a.rows, a.inner)
        ws = [rnd(a.out, a.inner) for _ in range(a.copies)]
        if a.kernel == "gemm_pair_swiglu":          # --out counts the rows of [Wg; Wu]
            out = torch.empty(a.rows, a.out // 2, dtype=bf, device=dev)
            launches = [lambda w=w: kernels.gemm_pair_swiglu(x, w, out) for w in ws]
        elif a.kernel == "gemm_fused":
            fused = kernels.gemm_fused
            if a.epilogue == "swiglu":
                out = torch.empty(a.rows, a.out // 2, dtype=bf, device=dev)
                launches = [lambda w=w: fused(x, w, out, kernels.EPI_SWIGLU, a.out // 2, splits=a.splits) for w in ws]
            elif a.epilogue == "resid":
                out = torch.empty(a.rows, a.out, dtype=bf, device=dev)
                resid = torch.zeros(a.rows, a.out, dtype=torch.float32, device=dev)
                nw = torch.ones(a.out, dtype=torch.float32, device=dev)
                ssq = torch.zeros(-(-a.out // 128), 64, dtype=torch.float32, device=dev)
                ssq = torch.zeros(-(-a.out // 128), 64, dtype=torch.float32, device=dev)
                launches = [lambda w=w: fused(x, w, None, kernels.EPI_RESID, a.out, resid=(resid, nw, out, ssq), splits=a.splits) for w in ws]
            else:
                out = torch.empty(a.rows, a.out, dtype=bf, device=dev)
                launches = [lambda w=w: fused(x, w, out, kernels.EPI_STORE, a.out, splits=a.splits) for w in ws]
        else:
            out = torch.empty(a.rows, a.out, dtype=bf, device=dev)
            if a.kernel == "gemm_library":           # the library product the engine uses for many rows, for comparison
                launches = [lambda w=w: torch.mm(x, w.t(), out=out) for w in ws]
            else:
                fn = kernels.gemm_sm100 if a.kernel == "gemm" else kernels.gemm_sm100_pair
                launches = [lambda w=w: fn(x, w, out) for w in ws]
        nbytes = a.out * a.inner * 2 + a.rows * a.inner * 2 + out.numel() * 2
        flops = 2.0 * a.rows * a.out * a.inner
    else:
        H, KV, hd, page = a.heads, a.kv_heads, a.head_dim, a.page
        if a.kernel == "attn_decode":
            S, ctx, new = a.batch, a.context, 1
        else:
            S, ctx, new = 1, 0, a.tokens
        L = ctx + new
        pages_per = -(-L // page)
        caches = [(rnd(S * pages_per, KV, page, hd), rnd(S * pages_per, KV, page, hd)) for _ in range(a.copies)]
        bt = torch.arange(S * pages_per, dtype=torch.int32, device=dev).view(S, pages_per).contiguous()
        q = rnd(S * new, H * hd)
        out = torch.empty_like(q)
        scale = 1.0 / math.sqrt(hd)
        if a.kernel == "attn_decode":
            pos = torch.full((S,), L - 1, dtype=torch.int32, device=dev)
            # auto: the engine's choice (parts/attention.py decode_split_rule): a cluster of up to 8 blocks per
            # request and kv head, or, for few requests with long contexts, up to 64 that merge through global memory
            from vllm_oxide_b200.parts.attention import decode_split_rule
            sms = torch.cuda.get_device_properties(dev).multi_processor_count
            if a.merge == "auto":
                splits, wide = decode_split_rule(S, KV, sms, ctx > TUNING.long_context_keys)
            else:
                wide = a.merge == "global" and 3 * sms // (S * KV) >= 4
                splits = max(1, min(64, 3 * sms // (S * KV))) if wide else max(1, min(8, -(-2 * sms // (S * KV))))
            if a.splits:
                splits = a.splits
            partials = torch.empty(kernels.attn_decode_partial_floats(S, KV, hd, splits), device=dev) if wide else None
            arrived = torch.zeros(S * KV, dtype=torch.int32, device=dev) if wide else None
            launches = [lambda kc=kc, vc=vc: kernels.attn_decode_mma(q, out, kc, vc, bt, pos, H, KV, hd, scale, 0, splits,
                                                                     partials, arrived)
                        for kc, vc in caches]
            nbytes = 2 * S * L * KV * hd * 2
            flops = 4.0 * S * H * hd * L
        else:
            starts = torch.tensor([0, new], dtype=torch.int32, device=dev)
            ctxs = torch.zeros(1, dtype=torch.int32, device=dev)
            if a.impl_attn == "sm100":
                launches = [lambda kc=kc, vc=vc: kernels.attn_prefill_sm100(q, out, kc, vc, bt, starts, ctxs, 1, new, H, KV, hd, scale)
                            for kc, vc in caches]
            else:
                launches = [lambda kc=kc, vc=vc: kernels.attn_prefill_mma(q, out, kc, vc, bt, starts, ctxs, 1, new, H, KV, hd, scale, 0)
                            for kc, vc in caches]
            nbytes = 2 * L * KV * hd * 2 + 2 * new * H * hd * 2
            flops = 4.0 * H * hd * new * (new + 1) / 2
    for f in launches:
        f()
    torch.cuda.synchronize()
    kernels.gemm_sm100_check()
    if a.graph:
        kernels.set_pdl(True)
        gr = torch.cuda.CUDAGraph()
        with torch.cuda.graph(gr):
            for _ in range(2):
                for f in launches:
                    f()
        gr.replay()
        torch.cuda.synchronize()
        times = []
        for _ in range(max(a.iters, 3)):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            gr.replay()
            e1.record()
            torch.cuda.synchronize()
            times.append(e0.elapsed_time(e1) * 1e3 / (2 * len(launches)))
        us = median(times)
        print(f"{a.kernel}: {us:.1f} us per launch (events around a CUDA graph of {2 * len(launches)} launches back to back); "
              f"{nbytes / us / 1e3:.0f} GB/s of the bytes it must read; {flops / us / 1e6:.1f} TFLOP/s")
        return 0
    times = []
    for _ in range(a.iters):
        for f in launches:
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            f()
            e1.record()
            torch.cuda.synchronize()
            times.append(e0.elapsed_time(e1) * 1e3)
    us = median(times)
    print(f"{a.kernel}: {us:.1f} us per launch (events, single launches); {nbytes / us / 1e3:.0f} GB/s of the bytes it must read; "
          f"{flops / us / 1e6:.1f} TFLOP/s")
    return 0


KERNEL_TAGS = {1: "embed", 2: "add_rmsnorm", 4: "rope_kv_write", 5: "swiglu", 6: "paged_attention", 7: "attn_prefill_mma",
               8: "attn_decode_mma", 9: "pick_partial", 10: "pick_final", 11: "gemm_f32", 12: "gemm_sm100", 13: "gemm_sm100_persistent",
               14: "attn_prefill_sm100", 15: "gemm_sm100_pair"}


def timeline_of_a_decode_step(llm, prompts, B, prompt_len, gen_len):
    """With kernel libraries built with VOB_TIMELINE=1 in the environment (a different build: block 0
    of every kernel notes the global timer when it starts and when its wait for the kernel in front
    returns): the kernels of one decode step in order, with the time from each kernel's ready point
    to the next one's. Without that build nothing is recorded."""
    import collections
    import ctypes
    import torch
    from vllm_oxide_b200.csrc.build import _loaded
    ids = [llm.add_request(prompts[i], never_stop(gen_len)) for i in range(B)]
    prefill_all(llm, ids, prompt_len)
    for _ in range(6):
        llm.step()
    llm.drain()
    buf = torch.zeros(1 + 3 * 4096, dtype=torch.int64, device="cuda:0")

    def set_buffer(t):
        for name, lib in list(_loaded.items()):
            f = getattr(lib, f"vob_set_timeline_{name}", None)
            if f is not None:
                f.argtypes, f.restype = [ctypes.c_void_p], ctypes.c_int
                f(ctypes.c_void_p(t.data_ptr() if t is not None else 0))
    set_buffer(buf)
    torch.cuda.synchronize()
    llm.step()
    llm.drain()
    torch.cuda.synchronize()
    set_buffer(None)
    h = buf.cpu().tolist()
    n = min(h[0], 4096)
    rows = sorted(((KERNEL_TAGS.get(h[1 + 3 * e], str(h[1 + 3 * e])), h[2 + 3 * e], h[3 + 3 * e]) for e in range(n)), key=lambda x: x[2])
    if not rows:
        print("timeline: nothing recorded (build the kernel libraries with VOB_TIMELINE=1 in the environment)")
        return 1
    t0 = rows[0][1]
    print(f"{len(rows)} kernels; step span {(rows[-1][2] - t0) / 1000:.1f} us (batch {B})")
    agg = collections.OrderedDict()
    for i, (name, st, rd) in enumerate(rows):
        dur = (rows[i + 1][2] - rd) if i + 1 < len(rows) else 0
        c, d, lead = agg.get(name, (0, 0, 0))
        agg[name] = (c + 1, d + dur, lead + rd - st)
    for name, (c, d, lead) in agg.items():
        print(f"{name:22s} n={c:3d} time to next ready {d / 1000:8.1f} us (avg {d / c / 1000:6.2f})   avg waited at its wait {lead / c / 1000:6.2f} us")
    layers = llm.runner.config.num_hidden_layers
    per = max(1, (len(rows) - 4) // layers)
    mid = layers // 2
    print(f"layer {mid} in detail:")
    for i in range(1 + mid * per, min(len(rows) - 1, 1 + (mid + 1) * per + 1)):
        name, st, rd = rows[i]
        print(f"  {name:18s} start {(st - t0) / 1000:8.2f}  ready {(rd - t0) / 1000:8.2f}  (waited {(rd - st) / 1000:5.2f})"
              f"  -> next ready in {(rows[i + 1][2] - rd) / 1000:5.2f} us")
    for i in ids:
        llm.abort(i)
    return 0


# ------------------------------------------------------------------------------------------------ main
# ------------------------------------------------------------------------------------------------ Rotepel beside Llama
# Layer sizes at which the Rotepel design is measured beside the Llama decoder of the same width, feed-forward
# and layer count: per size the three mixers' heads and sizes (delta rule, retention, latent attention).
ROTEPEL_SIZES = {
    "1b": dict(llama="1b", width=2048, ff=8192, delta=dict(heads=32, dim=64, decay_rank=64),
               retention=dict(heads=16, dim=128, vdim=128), latent=dict(heads=32, dim=64, rot_dim=32, vdim=64, kv_rank=256)),
    "3b": dict(llama="3b", width=3072, ff=8192, delta=dict(heads=24, dim=128, decay_rank=96),
               retention=dict(heads=12, dim=128, vdim=256), latent=dict(heads=24, dim=128, rot_dim=64, vdim=128, kv_rank=512)),
}


def make_rotepel_engine(rs, blocks, max_seqs, tokens_per_request, context):
    """(config, LLM): `blocks` times the four layers [delta rule, retention, delta rule, latent attention], two streams,
    two norm groups, random weights drawn on the device."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200.config import EngineConfig, RotepelConfig, RotepelLayer
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    d, r, l = rs["delta"], rs["retention"], rs["latent"]
    delta = RotepelLayer(type="general_delta", ff=rs["ff"], **d)
    ret = RotepelLayer(type="retention", ff=rs["ff"], decay=tuple(1.0 - 2.0 ** -(5 + i % 6) for i in range(r["heads"])),
                       rot_dims=r["dim"], rot_base=1e6, **r)
    lat = RotepelLayer(type="latent_attention", ff=rs["ff"], scale=(l["dim"] + l["rot_dim"]) ** -0.5, rot_dims=l["rot_dim"],
                       rot_base=5e5, **l)
    cfg = RotepelConfig(vocab=128256, width=rs["width"], layers=(delta, ret, delta, lat) * blocks, norm_eps=1e-5, norm_groups=2, streams=2)
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=True)
    fields.update(ENGINE_OVERRIDES)
    tensors = random_tensors(models.rotepel_manifest(cfg), seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, EngineConfig(**fields))
    del tensors
    return cfg, LLM(runner)


def op_profile(llm, tokens, n, batch):
    """Device time op by op (CUDA events around every kernel wrapper, launches one by one) of one step of `n` prompt
    tokens and of one decode step of `batch` requests behind prompts of `n` tokens. Returns two lists of (op, calls, ms)."""
    import torch
    from vllm_oxide_b200 import kernels
    runner, rt = llm.runner, llm.runner.rt
    graphs, runner.graphs_enabled = runner.graphs_enabled, False
    ids = list(range(800000, 800000 + batch))
    try:
        for i, rid in enumerate(ids):
            runner.admit(rid)
            runner.manager.reserve(rid, n)
            arrays = runner.build_arrays([rt.StepEntry(rid, tokens[i][:n], [n - 1])])
            if i == batch - 1:
                with kernels.OpProfile() as prof:
                    runner.step(arrays)
                prefill = prof.totals()
            else:
                runner.step(arrays)
            runner.manager.commit(rid, n)
        decode = None
        for rep in range(3):
            for rid in ids:
                runner.manager.reserve(rid, 1)
            arrays = runner.build_arrays([rt.StepEntry(rid, [7], [0]) for rid in ids])
            if rep == 2:
                with kernels.OpProfile() as prof:
                    runner.step(arrays)
                decode = prof.totals()
            else:
                runner.step(arrays)
            for rid in ids:
                runner.manager.commit(rid, 1)
        torch.cuda.synchronize()
    finally:
        for rid in ids:
            runner.manager.release(rid)
        runner.graphs_enabled = graphs
    return prefill, decode


def rotepel_roofline(rs, blocks, n, batch, peaks, prefill, decode):
    """The new design's own kernels against their rooflines: algorithmic bytes (or FLOPs) of all their launches in one
    step over the measured time, as a fraction of the measured copy bandwidth (or the measured bfloat16 product rate)."""
    d, r, l = rs["delta"], rs["retention"], rs["latent"]
    W, S = rs["width"], 2
    norms = blocks * 4 * 2 + 1                       # two sublayers per layer, and the final norm (one row per request)
    out = {}

    def add(name, phase, totals, nbytes=None, flops=None):
        also = {name + "_tc"} | ({"latent_decode_tc"} if name == "latent_attend" else set())     # the tensor-core forms of a kernel count with it
        ms = sum(t for op, _, t in totals if op == name or op in also)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 3)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{name}"] = e
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        # read and write S streams of float32, read the sublayer's output, write the normed row
        add("stream_norm", phase, totals, nbytes=norms * rows * W * (2 * S * 4 + 2 + 2))
        seqs = 1 if phase == "prefill" else batch
        state = blocks * (2 * d["heads"] * d["dim"] * d["dim"] + r["heads"] * r["dim"] * r["vdim"]) * 4 * 2 * seqs
        per_token = blocks * (2 * d["heads"] * d["dim"] * (3 * 2 + 3 * 4 + 4) + r["heads"] * (2 * r["dim"] * 4 + r["vdim"] * (2 + 4)))
        # FLOPs of the recurrences as they are written (delta rule: 4 passes over K x V per token, retention 2)
        fl = blocks * rows * 2 * (2 * d["heads"] * d["dim"] * d["dim"] * 4 + r["heads"] * r["dim"] * r["vdim"] * 2)
        add("recurrence_scan", phase, totals, nbytes=state + rows * per_token, flops=fl)
        keys = rows * (n + 1) / 2 if phase == "prefill" else batch * (n + 3)
        add("latent_attend", phase, totals, nbytes=(blocks * batch * (n + 3) * (l["kv_rank"] + l["rot_dim"]) * 2) if phase == "decode" else None,
            flops=blocks * keys * l["heads"] * 2 * (2 * l["kv_rank"] + l["rot_dim"]))
    return out


def llama_roofline(cfg, layers, n, batch, peaks, prefill, decode):
    """The like kernels of the Llama decoder, the same way: the norm with the residual add, attention over the cache."""
    out = {}
    h, q, kv = cfg.hidden_size, cfg.q_dim, cfg.kv_dim

    def add(names, label, phase, totals, nbytes=None, flops=None):
        ms = sum(t for op, _, t in totals if op in names)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 3)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{label}"] = e
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        add(("add_rmsnorm",), "add_rmsnorm", phase, totals, nbytes=(2 * layers + 1) * rows * h * (2 * 4 + 2 + 2))
        keys = rows * (n + 1) / 2 if phase == "prefill" else batch * (n + 3)
        add(("attn_prefill_sm100", "attn_prefill_mma", "attn_decode_mma", "paged_attention"), "attention", phase, totals,
            nbytes=layers * batch * (n + 3) * 2 * kv * 2 if phase == "decode" else None, flops=layers * keys * 4 * q)
    return out


def rotepel_compare(a):
    """Prefill and decode of the Rotepel design beside the Llama decoder of the same width, feed-forward and number of
    layers; one JSON line. Device-timed like the benchmark's own points: one step of 2,048 prompt tokens (median of 5
    after 3), decode steps replayed from CUDA graphs (`--steps` steps a region, median region)."""
    import torch
    peaks = load_peaks()
    n, B, blocks = 2048, a.batch, 2
    gen = a.warmup + max(a.steps, MAX_TIMED_STEPS) + 64
    sampler = ClockSampler()
    sampler.start()
    points = []
    for key in a.rotepel.split(","):
        rs = ROTEPEL_SIZES[key]
        point = {"sizes": key, "layers": 4 * blocks, "prompt_len": n, "batch": B}
        for arch in ("rotepel", "llama"):
            if arch == "rotepel":
                cfg, llm = make_rotepel_engine(rs, blocks, B, n + gen, 8192)
                vocab = cfg.vocab
            else:
                cfg, llm = make_engine(SIZES[rs["llama"]], 4 * blocks, B, n + gen, 8192)
                vocab = cfg.vocab_size
            g = torch.Generator().manual_seed(1)
            prompts = [torch.randint(0, vocab, (n,), generator=g).tolist() for _ in range(B)]
            ms_prefill = timed_prefill(llm, prompts[0], n)
            ms_step, ctx_tokens, launches, regions = decode_device(llm, prompts, B, a.steps, a.warmup, n, gen)
            prefill, decode = op_profile(llm, prompts, n, B)
            e = {"prefill_tok_s": round(n / ms_prefill * 1e3, 1), "prefill_ms": round(ms_prefill, 3),
                 "decode_tok_s": round(B / ms_step * 1e3, 1), "decode_ms_per_step": round(ms_step, 4),
                 "decode_hbm_frac_of_measured": round(llm.runner.step_read_bytes(int(ctx_tokens)) / ms_step / 1e6 / peaks["hbm_gbs"], 3),
                 "launches_per_decode_step": launches // a.steps,
                 "ops_prefill_ms": {op: round(t, 4) for op, _, t in prefill}, "ops_decode_ms": {op: round(t, 4) for op, _, t in decode}}
            e["kernels"] = rotepel_roofline(rs, blocks, n, B, peaks, prefill, decode) if arch == "rotepel" else \
                llama_roofline(cfg, 4 * blocks, n, B, peaks, prefill, decode)
            point[arch] = e
            free_engine(llm)
            del llm
        points.append(point)
    clocks = sampler.stop()
    print(json.dumps({"metric": "Rotepel beside Llama at equal width, feed-forward and layer count: prefill and decode tok/s",
                      "dtype": "bf16", "data": "synthetic", "peaks": peaks, "points": points, "clocks": clocks, "run": run_record()}))
    return 0


# Layer sizes at which the Lomopel design is measured beside the Llama decoder of the same width, feed-forward,
# layer count and attention heads: per size the attention heads (shared by the full and the windowed attention),
# the window, and the gated delta rule's heads and sizes.
LOMOPEL_SIZES = {
    "1b": dict(llama="1b", width=2048, ff=8192, attn=dict(heads=32, kv_heads=8, dim=64, vdim=64), window=1024,
               delta=dict(heads=16, kv_heads=8, dim=128, vdim=128, conv=4, decay_rank=64, gate_rank=64)),
    "3b": dict(llama="3b", width=3072, ff=8192, attn=dict(heads=24, kv_heads=8, dim=128, vdim=128), window=1024,
               delta=dict(heads=24, kv_heads=12, dim=128, vdim=128, conv=4, decay_rank=96, gate_rank=96)),
}


def make_lomopel_engine(ls, blocks, max_seqs, tokens_per_request, context):
    """(config, LLM): `blocks` times the four layers [attention, parallel, parallel, attention], every attention layer
    mixing values, random weights drawn on the device."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200.config import EngineConfig, GatedDeltaConfig, LomopelConfig, LomopelLayer, SoftmaxMixerConfig
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    at = ls["attn"]
    full = SoftmaxMixerConfig(scale=at["dim"] ** -0.5, q_temp=(0.1, 1024), v_mix=True, **at)
    left = SoftmaxMixerConfig(scale=1.0 / 8, window=ls["window"], rot_dims=at["dim"] // 2, rot_base=1e4, **at)
    att = LomopelLayer("attention", attention=full, ff=ls["ff"])
    par = LomopelLayer("parallel", left=left, right=GatedDeltaConfig(**ls["delta"]), left_scale=1.0, right_scale=1.0, ff=ls["ff"])
    cfg = LomopelConfig(vocab=128256, width=ls["width"], layers=(att, par, par, att) * blocks, norm_eps=1e-5, embedding_scale=1.0)
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=True)
    fields.update(ENGINE_OVERRIDES)
    tensors = random_tensors(models.lomopel_manifest(cfg), seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, EngineConfig(**fields))
    del tensors
    return cfg, LLM(runner)


def lomopel_roofline(ls, blocks, n, batch, peaks, prefill, decode):
    """The new design's own kernels against their rooflines: algorithmic bytes (or FLOPs) of all their launches in one
    step over the measured time, as a fraction of the measured copy bandwidth (or the measured bfloat16 product rate)."""
    at, d, W, win = ls["attn"], ls["delta"], ls["width"], ls["window"]
    layers = 4 * blocks
    out = {}

    def add(names, label, phase, totals, nbytes=None, flops=None):
        ms = sum(t for op, _, t in totals if op in names)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 3)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{label}"] = e
    qd, kd, vd = at["heads"] * at["dim"], at["kv_heads"] * at["dim"], at["kv_heads"] * at["vdim"]
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        add(("add_rmsnorm",), "add_rmsnorm", phase, totals, nbytes=(2 * layers + 1) * rows * W * (2 * 4 + 2 + 2))
        # keys a row reads: all before it in the two full layers of a block, the window's in the two windowed ones
        if phase == "prefill":
            keys_full, keys_win = rows * (n + 1) / 2, sum(min(i + 1, win) for i in range(n))
        else:
            keys_full, keys_win = batch * (n + 3), batch * min(n + 3, win)
        fl = 2 * blocks * (keys_full + keys_win) * at["heads"] * 2 * (at["dim"] + at["vdim"])
        by = 2 * blocks * (keys_full + keys_win) * (kd + vd) * 2 if phase == "decode" else None
        add(("flex_attention", "attn_prefill_sm100", "attn_prefill_mma", "attn_decode_mma"), "attention", phase, totals, nbytes=by, flops=fl)
        # q, k, v read from the projection; q written, k and v written to the cache (and the values that layers share)
        add(("flex_prep",), "flex_prep", phase, totals, nbytes=layers * rows * (2 * qd + 2 * kd + 2 * vd) * 2)
        seqs = 1 if phase == "prefill" else batch
        H, K, V, G = d["heads"], d["dim"], d["vdim"], d["kv_heads"]
        state = 2 * blocks * H * K * V * 4 * 2 * seqs
        per_token = 2 * blocks * (2 * G * K * 4 + H * V * 2 + H * K * 4 + H * 4 + H * V * 4)
        add(("recurrence_scan",), "recurrence_scan", phase, totals, nbytes=state + rows * per_token,
            flops=2 * blocks * rows * 2 * H * K * V * 4)
        C = 2 * G * K + H * V
        add(("gated_delta_prep", "conv_state_update"), "gated_delta_prep", phase, totals,
            nbytes=2 * blocks * rows * (C * 2 + H * K * 2 + 2 * G * K * 4 + H * V * 2 + H * K * 4 + H * 4))
        add(("recurrence_post",), "recurrence_post", phase, totals, nbytes=2 * blocks * rows * H * V * (4 + 2 + 2))
    return out


def lomopel_compare(a):
    """Prefill and decode of the Lomopel design beside the Llama decoder of the same width, feed-forward, layer count
    and attention heads; one JSON line. Device-timed like the benchmark's own points: one step of 2,048 prompt tokens
    (median of 5 after 3), decode steps replayed from CUDA graphs (`--steps` steps a region, median region)."""
    import torch
    peaks = load_peaks()
    n, B, blocks = 2048, a.batch, 2
    gen = a.warmup + max(a.steps, MAX_TIMED_STEPS) + 64
    sampler = ClockSampler()
    sampler.start()
    points = []
    for key in a.lomopel.split(","):
        ls = LOMOPEL_SIZES[key]
        point = {"sizes": key, "layers": 4 * blocks, "prompt_len": n, "batch": B}
        for arch in ("lomopel", "llama"):
            if arch == "lomopel":
                cfg, llm = make_lomopel_engine(ls, blocks, B, n + gen, 8192)
                vocab = cfg.vocab
            else:
                cfg, llm = make_engine(SIZES[ls["llama"]], 4 * blocks, B, n + gen, 8192)
                vocab = cfg.vocab_size
            g = torch.Generator().manual_seed(1)
            prompts = [torch.randint(0, vocab, (n,), generator=g).tolist() for _ in range(B)]
            ms_prefill = timed_prefill(llm, prompts[0], n)
            ms_step, ctx_tokens, launches, regions = decode_device(llm, prompts, B, a.steps, a.warmup, n, gen)
            prefill, decode = op_profile(llm, prompts, n, B)
            e = {"prefill_tok_s": round(n / ms_prefill * 1e3, 1), "prefill_ms": round(ms_prefill, 3),
                 "decode_tok_s": round(B / ms_step * 1e3, 1), "decode_ms_per_step": round(ms_step, 4),
                 "decode_hbm_frac_of_measured": round(llm.runner.step_read_bytes(int(ctx_tokens)) / ms_step / 1e6 / peaks["hbm_gbs"], 3),
                 "launches_per_decode_step": launches // a.steps,
                 "ops_prefill_ms": {op: round(t, 4) for op, _, t in prefill}, "ops_decode_ms": {op: round(t, 4) for op, _, t in decode}}
            e["kernels"] = lomopel_roofline(ls, blocks, n, B, peaks, prefill, decode) if arch == "lomopel" else \
                llama_roofline(cfg, 4 * blocks, n, B, peaks, prefill, decode)
            point[arch] = e
            free_engine(llm)
            del llm
        points.append(point)
    clocks = sampler.stop()
    print(json.dumps({"metric": "Lomopel beside Llama at equal width, feed-forward, layer count and attention heads: prefill and decode tok/s",
                      "dtype": "bf16", "data": "synthetic", "peaks": peaks, "points": points, "clocks": clocks, "run": run_record()}))
    return 0


# Layer sizes at which the Bufulorn design is measured beside Lomopel, the closest design the engine has (attention with
# options, a gated delta rule), at the same width, feed-forward, layer count, attention heads and delta-rule sizes (those of
# LOMOPEL_SIZES): the length of a block of positions, and the routed experts (all experts together as large as the dense
# feed-forward, a token using two of them).
BUFULORN_SIZES = {
    "1b": dict(lomopel="1b", chunk=1536, softcap=30.0, moe=dict(ff=1024, experts=8, top=2, groups=4, keep=2)),
    "3b": dict(lomopel="3b", chunk=1536, softcap=30.0, moe=dict(ff=1024, experts=8, top=2, groups=4, keep=2)),
}


def make_bufulorn_engine(bs, blocks, max_seqs, tokens_per_request, context):
    """(config, LLM): `blocks` times the four layers [attention + dense, delta rule + experts, attention that reads the
    first layer's keys and values + dense, delta rule + dense], random weights drawn on the device."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200.config import (BufulornConfig, BufulornLayer, ChunkAttentionConfig, EngineConfig, FeedForwardConfig,
                                        HeadDecayDeltaConfig)
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    ls = LOMOPEL_SIZES[bs["lomopel"]]
    at, d = ls["attn"], ls["delta"]
    dense = FeedForwardConfig("dense", ls["ff"])
    moe = FeedForwardConfig("moe", **bs["moe"])
    delta = HeadDecayDeltaConfig(heads=d["heads"], kv_heads=d["kv_heads"], dim=d["dim"], vdim=d["vdim"], conv=d["conv"])
    layers = []
    for b in range(blocks):
        own = ChunkAttentionConfig(scale=at["dim"] ** -0.5, softcap=bs["softcap"], chunk=bs["chunk"], **at)
        reader = ChunkAttentionConfig(scale=at["dim"] ** -0.5, softcap=bs["softcap"], chunk=bs["chunk"], kv_from=4 * b, **at)
        layers += [BufulornLayer("attention", attention=own, mlp=dense), BufulornLayer("delta", delta=delta, mlp=moe),
                   BufulornLayer("attention", attention=reader, mlp=dense), BufulornLayer("delta", delta=delta, mlp=dense)]
    cfg = BufulornConfig(vocab=128256, width=ls["width"], norm_eps=1e-5, max_positions=context, layers=tuple(layers))
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=True)
    fields.update(ENGINE_OVERRIDES)
    tensors = random_tensors(models.bufulorn_manifest(cfg), seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, EngineConfig(**fields))
    del tensors
    return cfg, LLM(runner)


def bufulorn_roofline(bs, blocks, n, batch, peaks, prefill, decode):
    """The design's own kernels against their rooflines: algorithmic bytes (or FLOPs) of all their launches in one step
    over the measured time, as a fraction of the measured copy bandwidth (or the measured bfloat16 product rate)."""
    ls = LOMOPEL_SIZES[bs["lomopel"]]
    at, d, W, F, chunk, m = ls["attn"], ls["delta"], ls["width"], ls["ff"], bs["chunk"], bs["moe"]
    out = {}

    def add(names, label, phase, totals, nbytes=None, flops=None):
        ms = sum(t for op, _, t in totals if op in names)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 3)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{label}"] = e
    qd, kd, vd = at["heads"] * at["dim"], at["kv_heads"] * at["dim"], at["kv_heads"] * at["vdim"]
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        # every sub-layer: the result read, the float32 residual read and written, its rounding written
        add(("layernorm_add",), "layernorm_add", phase, totals, nbytes=8 * blocks * rows * W * (2 + 2 * 4 + 2))
        # keys a row reads: those of its own block of positions that are not behind it
        if phase == "prefill":
            keys = sum(i % chunk + 1 for i in range(n))
        else:
            keys = batch * ((n + 2) % chunk + 1)
        fl = 2 * blocks * keys * at["heads"] * 2 * (at["dim"] + at["vdim"])
        by = 2 * blocks * keys * (kd + vd) * 2 if phase == "decode" else None
        add(("flex_attention", "attn_prefill_mma_any", "attn_prefill_mma", "attn_decode_mma"), "attention", phase, totals, nbytes=by, flops=fl)
        # a layer with keys of its own: q, k, v read, q written, k and v written to the cache; a reader: q read and written
        add(("flex_prep",), "flex_prep", phase, totals, nbytes=blocks * rows * ((2 * qd + 2 * kd + 2 * vd) + 2 * qd) * 2)
        seqs = 1 if phase == "prefill" else batch
        H, K, V, G = d["heads"], d["dim"], d["vdim"], d["kv_heads"]
        state = 2 * blocks * H * K * V * 4 * 2 * seqs
        per_token = 2 * blocks * (2 * G * K * 4 + H * V * 2 + H * 4 * 2 + H * V * 4)
        add(("recurrence_scan",), "recurrence_scan", phase, totals, nbytes=state + rows * per_token,
            flops=2 * blocks * rows * 2 * H * K * V * 4)
        C = 2 * G * K + H * V
        add(("gated_delta_prep", "conv_state_update"), "gated_delta_prep", phase, totals,
            nbytes=2 * blocks * rows * (C * 2 + 2 * H * 2 + 2 * G * K * 4 + H * V * 2 + 2 * H * 4))
        add(("recurrence_post",), "recurrence_post", phase, totals, nbytes=2 * blocks * rows * H * V * (4 + 2 + 2))
        # the activation between the two products of a dense feed-forward: read and written in place
        add(("activation",), "xielu", phase, totals, nbytes=3 * blocks * rows * F * 2 * 2)
        # routed experts: the weights of every expert that is used are read once (decode), 3 products of ff x width a choice
        P, used = rows * m["top"], min(m["experts"], rows * m["top"])
        add(("moe_gate_up", "moe_down"), "expert products", phase, totals,
            nbytes=blocks * (used * 3 * m["ff"] * W * 2 + P * (W * 2 + 2 * m["ff"] * 2 + W * 4)), flops=blocks * P * 3 * 2 * m["ff"] * W)
        add(("moe_route", "moe_align", "moe_combine"), "election, order, sum", phase, totals,
            nbytes=blocks * (rows * W * 2 + m["experts"] * W * 4 + P * W * 4 + rows * W * 2))
    return out


def bufulorn_compare(a):
    """Prefill and decode of the Bufulorn design beside Lomopel of the same width, feed-forward, layer count, attention
    heads and delta-rule sizes; one JSON line. Device-timed like the benchmark's own points: one step of 2,048 prompt
    tokens (median of 5 after 3), decode steps replayed from CUDA graphs (`--steps` steps a region, median region)."""
    import torch
    peaks = load_peaks()
    n, B, blocks = 2048, a.batch, 2
    gen = a.warmup + max(a.steps, MAX_TIMED_STEPS) + 64
    sampler = ClockSampler()
    sampler.start()
    points = []
    for key in a.bufulorn.split(","):
        bs = BUFULORN_SIZES[key]
        ls = LOMOPEL_SIZES[bs["lomopel"]]
        point = {"sizes": key, "layers": 4 * blocks, "prompt_len": n, "batch": B}
        for arch in ("bufulorn", "lomopel"):
            if arch == "bufulorn":
                cfg, llm = make_bufulorn_engine(bs, blocks, B, n + gen, 8192)
            else:
                cfg, llm = make_lomopel_engine(ls, blocks, B, n + gen, 8192)
            g = torch.Generator().manual_seed(1)
            prompts = [torch.randint(0, cfg.vocab, (n,), generator=g).tolist() for _ in range(B)]
            ms_prefill = timed_prefill(llm, prompts[0], n)
            ms_step, ctx_tokens, launches, regions = decode_device(llm, prompts, B, a.steps, a.warmup, n, gen)
            prefill, decode = op_profile(llm, prompts, n, B)
            e = {"prefill_tok_s": round(n / ms_prefill * 1e3, 1), "prefill_ms": round(ms_prefill, 3),
                 "decode_tok_s": round(B / ms_step * 1e3, 1), "decode_ms_per_step": round(ms_step, 4),
                 "decode_hbm_frac_of_measured": round(llm.runner.step_read_bytes(int(ctx_tokens)) / ms_step / 1e6 / peaks["hbm_gbs"], 3),
                 "launches_per_decode_step": launches // a.steps,
                 "ops_prefill_ms": {op: round(t, 4) for op, _, t in prefill}, "ops_decode_ms": {op: round(t, 4) for op, _, t in decode}}
            e["kernels"] = bufulorn_roofline(bs, blocks, n, B, peaks, prefill, decode) if arch == "bufulorn" else \
                lomopel_roofline(ls, blocks, n, B, peaks, prefill, decode)
            point[arch] = e
            free_engine(llm)
            del llm
        points.append(point)
    clocks = sampler.stop()
    print(json.dumps({"metric": "Bufulorn beside Lomopel at equal width, feed-forward, layer count, attention heads and delta-rule sizes: "
                                "prefill and decode tok/s",
                      "dtype": "bf16", "data": "synthetic", "peaks": peaks, "points": points, "clocks": clocks, "run": run_record()}))
    return 0


# Layer sizes at which the Pironex design is measured beside Bufulorn, the closest design the engine has (attention with a cap
# that may read another layer's keys and values, a recurrent mixer with short convolutions, routed experts, layer norms on the
# sub-layers' results), at the same width, attention heads and recurrent sizes (those of LOMOPEL_SIZES): the window and the
# pooled blocks, the latent attention (the sizes of ROTEPEL_SIZES), the state-space mixer and the experts.
PIRONEX_SIZES = {
    "1b": dict(bufulorn="1b", window=1024, pool=64, softcap=30.0, taps=4, moe=dict(ff=1024, limit=7.0, experts=8, top=2, shared_ff=2048, shared_limit=7.0)),
    "3b": dict(bufulorn="3b", window=1024, pool=64, softcap=30.0, taps=4, moe=dict(ff=1024, limit=7.0, experts=8, top=2, shared_ff=2048, shared_limit=7.0)),
}


def pironex_parts(ps):
    ls = LOMOPEL_SIZES[BUFULORN_SIZES[ps["bufulorn"]]["lomopel"]]
    d, lat = ls["delta"], ROTEPEL_SIZES[ls["llama"]]["latent"]
    ssm = dict(heads=d["heads"], vdim=d["vdim"], state=d["dim"], groups=d["kv_heads"], norm_groups=d["kv_heads"], conv=d["conv"])
    return ls, ssm, lat


def make_pironex_engine(ps, blocks, max_seqs, tokens_per_request, context):
    """(config, LLM): `blocks` times the four layers [state space, latent attention in a window, attention with a window and
    pooled blocks, attention that reads that layer's keys and values], each with routed experts and a shared expert, random
    weights drawn on the device."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200.config import (ClampedExpertsConfig, EngineConfig, PironexConfig, PironexLayer, PooledAttentionConfig,
                                        StateSpaceConfig, WindowLatentConfig)
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    ls, ssm, lat = pironex_parts(ps)
    at = ls["attn"]
    moe = ClampedExpertsConfig(**ps["moe"])
    layers = []
    for b in range(blocks):
        common = dict(scale=at["dim"] ** -0.5, softcap=ps["softcap"], rot_dims=at["dim"] // 2, rot_base=5e5, window=ps["window"], pool=ps["pool"], **at)
        layers += [PironexLayer("mamba2", ssm=StateSpaceConfig(**ssm), mlp=moe),
                   PironexLayer("latent_attention", latent=WindowLatentConfig(scale=(lat["dim"] + lat["rot_dim"]) ** -0.5, rot_base=1e4,
                                                                              window=ps["window"], **lat), mlp=moe),
                   PironexLayer("attention", attention=PooledAttentionConfig(**common), mlp=moe),
                   PironexLayer("attention", attention=PooledAttentionConfig(kv_from=4 * b + 2, **common), mlp=moe)]
    cfg = PironexConfig(vocab=128256, width=ls["width"], norm_eps=1e-5, embedding_scale=1.0, canon_taps=ps["taps"], layers=tuple(layers))
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=True)
    fields.update(ENGINE_OVERRIDES)
    tensors = random_tensors(models.pironex_manifest(cfg), seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, EngineConfig(**fields))
    del tensors
    return cfg, LLM(runner)


def pironex_roofline(ps, blocks, n, batch, peaks, prefill, decode):
    """The design's own kernels against their rooflines: algorithmic bytes (or FLOPs) of all their launches in one step
    over the measured time, as a fraction of the measured copy bandwidth (or the measured bfloat16 product rate)."""
    ls, ssm, lat = pironex_parts(ps)
    at, W, win, pool, m, taps = ls["attn"], ls["width"], ps["window"], ps["pool"], ps["moe"], ps["taps"]
    layers = 4 * blocks
    out = {}

    def add(names, label, phase, totals, nbytes=None, flops=None):
        ms = sum(t for op, _, t in totals if op in names)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 3)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{label}"] = e
    qd, kd, vd = at["heads"] * at["dim"], at["kv_heads"] * at["dim"], at["kv_heads"] * at["vdim"]
    H, P, N, G = ssm["heads"], ssm["vdim"], ssm["state"], ssm["groups"]
    inner, chans = H * P, H * P + 2 * G * N
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        # in front of a sub-layer: the float32 residual read, its normed rounding written; behind it: the result read, the
        # residual read and written
        add(("layernorm_rows", "layernorm_add"), "layer norms", phase, totals, nbytes=2 * layers * rows * W * ((4 + 2) + (2 + 2 * 4)))
        # the convolutions in front of the sub-layers (read, written, the state moved on) and the state-space mixer's own
        add(("causal_conv", "conv_state_update"), "causal convolutions", phase, totals,
            nbytes=2 * layers * rows * W * (2 + 2) + blocks * rows * chans * (2 + 4))
        add(("depth_average",), "depth average", phase, totals, nbytes=sum(rows * W * 4 * (i + 4) for i in range(layers)))
        # keys a row scores: its window's tokens and every token of the pooled blocks behind it (each block is read whole)
        if phase == "prefill":
            keys = sum(min(i + 1, win) + max(0, (i - win + 1) // pool) * pool for i in range(n))
        else:
            keys = batch * (min(n + 3, win) + max(0, (n + 3 - win) // pool) * pool)
        add(("flex_attention", "attn_prefill_mma_any", "attn_prefill_mma", "attn_decode_mma"), "attention", phase, totals,
            nbytes=2 * blocks * keys * (kd + vd) * 2 if phase == "decode" else None, flops=2 * blocks * keys * at["heads"] * 2 * (at["dim"] + at["vdim"]))
        add(("flex_prep",), "flex_prep", phase, totals, nbytes=blocks * rows * ((2 * qd + 2 * kd + 2 * vd) + 2 * qd) * 2)
        lkeys = sum(min(i + 1, win) for i in range(n)) if phase == "prefill" else batch * min(n + 3, win)
        add(("latent_attend", "latent_attend_tc", "latent_decode_tc"), "latent attention", phase, totals,
            nbytes=blocks * lkeys * (lat["kv_rank"] + lat["rot_dim"]) * 2 if phase == "decode" else None,
            flops=blocks * lkeys * lat["heads"] * 2 * (2 * lat["kv_rank"] + lat["rot_dim"]))
        seqs = 1 if phase == "prefill" else batch
        add(("recurrence_scan",), "recurrence_scan", phase, totals,
            nbytes=blocks * (H * N * P * 4 * 2 * seqs + rows * (2 * G * N * 4 + H * P * 4 + 2 * H * 4 + H * P * 4)), flops=blocks * rows * 2 * H * N * P * 2)
        add(("ssm_steps", "ssm_post"), "state-space steps, gate and norm", phase, totals,
            nbytes=blocks * rows * (H * (2 + 8) + inner * (4 + 4 + 2 + 2)))
        Pn, used = rows * m["top"], min(m["experts"], rows * m["top"])
        add(("moe_gate_up", "moe_down"), "expert products", phase, totals,
            nbytes=layers * (used * 3 * m["ff"] * W * 2 + Pn * (W * 2 + 2 * m["ff"] * 2 + W * 4)), flops=layers * Pn * 3 * 2 * m["ff"] * W)
        add(("moe_route", "moe_align", "moe_combine", "glu_clamped"), "election, order, sum, shared gate", phase, totals,
            nbytes=layers * (rows * W * 2 + m["experts"] * W * 4 + Pn * W * 4 + 2 * rows * W * 2 + rows * 3 * m["shared_ff"] * 2))
    return out


def pironex_compare(a):
    """Prefill and decode of the Pironex design beside Bufulorn of the same width, attention heads and recurrent sizes; one
    JSON line. Device-timed like the benchmark's own points: one step of 2,048 prompt tokens (median of 5 after 3), decode
    steps replayed from CUDA graphs (`--steps` steps a region, median region)."""
    import torch
    peaks = load_peaks()
    n, B, blocks = 2048, a.batch, 2
    gen = a.warmup + max(a.steps, MAX_TIMED_STEPS) + 64
    sampler = ClockSampler()
    sampler.start()
    points = []
    for key in a.pironex.split(","):
        ps = PIRONEX_SIZES[key]
        bs = BUFULORN_SIZES[ps["bufulorn"]]
        point = {"sizes": key, "layers": 4 * blocks, "prompt_len": n, "batch": B}
        for arch in ("pironex", "bufulorn"):
            if arch == "pironex":
                cfg, llm = make_pironex_engine(ps, blocks, B, n + gen, 8192)
            else:
                cfg, llm = make_bufulorn_engine(bs, blocks, B, n + gen, 8192)
            g = torch.Generator().manual_seed(1)
            prompts = [torch.randint(0, cfg.vocab, (n,), generator=g).tolist() for _ in range(B)]
            ms_prefill = timed_prefill(llm, prompts[0], n)
            ms_step, ctx_tokens, launches, regions = decode_device(llm, prompts, B, a.steps, a.warmup, n, gen)
            prefill, decode = op_profile(llm, prompts, n, B)
            e = {"prefill_tok_s": round(n / ms_prefill * 1e3, 1), "prefill_ms": round(ms_prefill, 3),
                 "decode_tok_s": round(B / ms_step * 1e3, 1), "decode_ms_per_step": round(ms_step, 4),
                 "decode_hbm_frac_of_measured": round(llm.runner.step_read_bytes(int(ctx_tokens)) / ms_step / 1e6 / peaks["hbm_gbs"], 3),
                 "launches_per_decode_step": launches // a.steps,
                 "ops_prefill_ms": {op: round(t, 4) for op, _, t in prefill}, "ops_decode_ms": {op: round(t, 4) for op, _, t in decode}}
            e["kernels"] = pironex_roofline(ps, blocks, n, B, peaks, prefill, decode) if arch == "pironex" else \
                bufulorn_roofline(bs, blocks, n, B, peaks, prefill, decode)
            point[arch] = e
            free_engine(llm)
            del llm
        points.append(point)
    clocks = sampler.stop()
    print(json.dumps({"metric": "Pironex beside Bufulorn at equal width, layer count, attention heads and recurrent sizes: "
                                "prefill and decode tok/s",
                      "dtype": "bf16", "data": "synthetic", "peaks": peaks, "points": points, "clocks": clocks, "run": run_record()}))
    return 0


# Layer sizes at which the Fanopel design is measured beside Bufulorn, the closest design the engine has (capped scores with a
# distance bias, a gate on the heads' results, routed experts chosen among the best groups, layer norms), both built of the same
# number of layers of attention and experts with the same width, heads and experts (those of BUFULORN_SIZES).
FANOPEL_SIZES = {
    "1b": dict(bufulorn="1b", window=1024, keep_first=16, softcap=30.0, scale=2.5),
    "3b": dict(bufulorn="3b", window=1024, keep_first=16, softcap=30.0, scale=2.5),
}


def make_experts_engine(arch, fs, layers, max_seqs, tokens_per_request, context):
    """(config, LLM): `layers` layers of attention and routed experts, of the Fanopel or the Bufulorn design, random weights
    drawn on the device."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200 import config as cf
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    bs = BUFULORN_SIZES[fs["bufulorn"]]
    ls = LOMOPEL_SIZES[bs["lomopel"]]
    at = ls["attn"]
    common = dict(vocab=128256, width=ls["width"], norm_eps=1e-5, max_positions=context)
    if arch == "fanopel":
        a = cf.KeyValueAttentionConfig(heads=at["heads"], kv_heads=at["kv_heads"], dim=at["dim"], scale=at["dim"] ** -0.5, softcap=fs["softcap"],
                                       window=fs["window"], keep_first=fs["keep_first"])
        cfg = cf.FanopelConfig(layers=(cf.FanopelLayer(a, cf.PlainExpertsConfig(scale=fs["scale"], **bs["moe"])),) * layers, residual_mult=0.5, **common)
        manifest = models.fanopel_manifest(cfg)
    else:
        a = cf.ChunkAttentionConfig(scale=at["dim"] ** -0.5, softcap=bs["softcap"], chunk=bs["chunk"], **at)
        cfg = cf.BufulornConfig(layers=(cf.BufulornLayer("attention", attention=a, mlp=cf.FeedForwardConfig("moe", **bs["moe"])),) * layers, **common)
        manifest = models.bufulorn_manifest(cfg)
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=True)
    fields.update(ENGINE_OVERRIDES)
    tensors = random_tensors(manifest, seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, cf.EngineConfig(**fields))
    del tensors
    return cfg, LLM(runner)


def experts_roofline(arch, fs, layers, n, batch, peaks, prefill, decode):
    """The kernels of attention-and-experts layers against their rooflines: algorithmic bytes (or FLOPs) of all their launches in
    one step over the measured time, as a fraction of the measured copy bandwidth (or the measured bfloat16 product rate)."""
    bs = BUFULORN_SIZES[fs["bufulorn"]]
    ls = LOMOPEL_SIZES[bs["lomopel"]]
    at, W, m, new = ls["attn"], ls["width"], bs["moe"], arch == "fanopel"
    out = {}

    def add(names, label, phase, totals, nbytes=None, flops=None):
        ms = sum(t for op, _, t in totals if op in names)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 4)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{label}"] = e
    qd, kd, vd = at["heads"] * at["dim"], at["kv_heads"] * at["dim"], at["kv_heads"] * at["vdim"]

    def seen(p):       # keys a query at position p reads
        return min(p + 1, fs["window"]) + max(0, min(fs["keep_first"], p + 1 - fs["window"])) if new else p % bs["chunk"] + 1
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        # every norm: the float32 residual read and written, the sub-layer's result read, the type the next product reads written
        add(("add_layernorm", "layernorm_add", "layernorm_rows", "cast_rows"), "layer norms", phase, totals, nbytes=2 * layers * rows * W * (2 + 2 * 4 + 2))
        keys = sum(seen(i) for i in range(n)) if phase == "prefill" else batch * seen(n + 2)
        per_key = kd * 2 + 4 if new else (kd + vd) * 2
        add(("flex_attention", "attn_prefill_mma_any", "attn_prefill_mma", "attn_decode_mma"), "attention", phase, totals,
            nbytes=layers * keys * per_key if phase == "decode" else None, flops=layers * keys * at["heads"] * 2 * (at["dim"] + at["vdim"]))
        add(("flex_prep", "whole_norm_prep"), "preparation of q, k (and v)", phase, totals,
            nbytes=layers * rows * 2 * (qd + kd + (0 if new else vd)) * 2)
        P, used, mats = rows * m["top"], min(m["experts"], rows * m["top"]), 2 if new else 3
        add(("moe_gate_up", "moe_up", "moe_down"), "expert products", phase, totals,
            nbytes=layers * (used * mats * m["ff"] * W * 2 + P * (W * 2 + 2 * m["ff"] * 2 + W * 4)), flops=layers * P * mats * 2 * m["ff"] * W)
        add(("moe_route", "moe_align", "moe_combine"), "election, order, sum", phase, totals,
            nbytes=layers * (rows * W * 2 + m["experts"] * W * 4 + P * W * 4 + rows * W * 2))
    return out


def fanopel_compare(a):
    """Prefill and decode of the Fanopel design beside Bufulorn layers of attention and experts of the same width, layer count,
    heads and experts; one JSON line. Device-timed like the benchmark's own points: one step of 2,048 prompt tokens (median of 5
    after 3), decode steps replayed from CUDA graphs (`--steps` steps a region, median region)."""
    import torch
    peaks = load_peaks()
    n, B, layers = 2048, a.batch, 8
    gen = a.warmup + max(a.steps, MAX_TIMED_STEPS) + 64
    sampler = ClockSampler()
    sampler.start()
    points = []
    for key in a.fanopel.split(","):
        fs = FANOPEL_SIZES[key]
        point = {"sizes": key, "layers": layers, "prompt_len": n, "batch": B}
        for arch in ("fanopel", "bufulorn"):
            cfg, llm = make_experts_engine(arch, fs, layers, B, n + gen, 8192)
            g = torch.Generator().manual_seed(1)
            prompts = [torch.randint(0, cfg.vocab, (n,), generator=g).tolist() for _ in range(B)]
            ms_prefill = timed_prefill(llm, prompts[0], n)
            ms_step, ctx_tokens, launches, regions = decode_device(llm, prompts, B, a.steps, a.warmup, n, gen)
            prefill, decode = op_profile(llm, prompts, n, B)
            point[arch] = {"prefill_tok_s": round(n / ms_prefill * 1e3, 1), "prefill_ms": round(ms_prefill, 3),
                           "decode_tok_s": round(B / ms_step * 1e3, 1), "decode_ms_per_step": round(ms_step, 4),
                           "cache_bytes_per_token": llm.runner.pools.bytes_per_token(), "launches_per_decode_step": launches // a.steps,
                           "ops_prefill_ms": {op: round(t, 4) for op, _, t in prefill}, "ops_decode_ms": {op: round(t, 4) for op, _, t in decode},
                           "kernels": experts_roofline(arch, fs, layers, n, B, peaks, prefill, decode)}
            free_engine(llm)
            del llm
        points.append(point)
    clocks = sampler.stop()
    print(json.dumps({"metric": "Fanopel beside Bufulorn (attention and experts in every layer) at equal width, layer count, heads and experts: "
                                "prefill and decode tok/s",
                      "dtype": "bf16", "data": "synthetic", "peaks": peaks, "points": points, "clocks": clocks, "run": run_record()}))
    return 0


# Layer sizes at which the Robuvik design is measured beside Pironex, the closest design the engine has (latent attention with
# interleaved rotary positions, attention in a window, routed experts beside a shared one), both built of the same run of layers
# with the same width, heads, latent, window and experts; Pironex without its convolutions, pooled blocks and caps.
ROBUVIK_SIZES = {
    "1b": dict(lomopel="1b", window=1024, q_rank=768, moe=dict(ff=1024, experts=8, top=2, shared_ff=2048)),
    "3b": dict(lomopel="3b", window=1024, q_rank=1024, moe=dict(ff=1024, experts=8, top=2, shared_ff=2048)),
}
ROBUVIK_LAYERS, ROBUVIK_LOOP = "LAALA", (1, 4, 2)          # latent attention / attention; three layers run twice: LAALAALA


def robuvik_runs():
    """The kinds of the layers in the order they run."""
    a, b, times = ROBUVIK_LOOP
    return ROBUVIK_LAYERS[:a] + ROBUVIK_LAYERS[a:b] * times + ROBUVIK_LAYERS[b:]


def make_side_by_side_engine(arch, rs, max_seqs, tokens_per_request, context):
    """(config, LLM): eight runs of layers of the Robuvik design, or as many Pironex layers of the same kinds, random weights drawn
    on the device."""
    import torch
    from vllm_oxide_b200 import models
    from vllm_oxide_b200 import config as cf
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.weights import random_tensors
    ls = LOMOPEL_SIZES[rs["lomopel"]]
    at, lat, m = ls["attn"], ROTEPEL_SIZES[ls["llama"]]["latent"], rs["moe"]
    scale, lscale = at["dim"] ** -0.5, (lat["dim"] + lat["rot_dim"]) ** -0.5
    common = dict(vocab=128256, width=ls["width"], norm_eps=1e-5)
    if arch == "robuvik":
        def rot(n):
            return cf.StretchedRotaryConfig(dims=n, base=5e5, factor=8.0, original=8192.0, fast=32.0, slow=1.0)
        moe = cf.DenseOrExpertsConfig("moe", **m)
        kinds = {"A": cf.RobuvikLayer("attention", attention=cf.WindowAttentionConfig(scale=scale, rot=rot(at["dim"]), window=rs["window"], **at), mlp=moe),
                 "L": cf.RobuvikLayer("latent_attention", latent=cf.GatedLatentConfig(q_rank=rs["q_rank"], scale=lscale, rot=rot(lat["rot_dim"]), **lat), mlp=moe)}
        cfg = cf.RobuvikConfig(layers=tuple(kinds[k] for k in ROBUVIK_LAYERS), loop=ROBUVIK_LOOP,
                               bigram=cf.BigramConfig(buckets=65521, mul_prev=8191, mul_cur=131), **common)
        manifest = models.robuvik_manifest(cfg)
    else:
        moe = cf.ClampedExpertsConfig(limit=7.0, shared_limit=7.0, **m)
        kinds = {"A": cf.PironexLayer("attention", attention=cf.PooledAttentionConfig(scale=scale, rot_dims=at["dim"], rot_base=5e5, window=rs["window"], **at), mlp=moe),
                 "L": cf.PironexLayer("latent_attention", latent=cf.WindowLatentConfig(scale=lscale, rot_base=5e5, **lat), mlp=moe)}
        cfg = cf.PironexConfig(layers=tuple(kinds[k] for k in robuvik_runs()), **common)
        manifest = models.pironex_manifest(cfg)
    pages_per_req = -(-(tokens_per_request + 16) // 16)
    fields = dict(max_batch_tokens=2048, max_seqs=max_seqs, max_model_len=context, block_size=16,
                  num_pages=max_seqs * pages_per_req + 8, dtype="bfloat16", cuda_graphs=True)
    fields.update(ENGINE_OVERRIDES)
    tensors = random_tensors(manifest, seed=0, std=0.02, dtype=torch.bfloat16, device="cuda:0")
    runner = ModelRunner(cfg, tensors, cf.EngineConfig(**fields))
    del tensors
    return cfg, LLM(runner)


def side_by_side_roofline(arch, rs, n, batch, peaks, prefill, decode):
    """The kernels of both designs against their rooflines: algorithmic bytes (or FLOPs) of all their launches in one step over
    the measured time, as a fraction of the measured copy bandwidth (or the measured bfloat16 product rate)."""
    ls = LOMOPEL_SIZES[rs["lomopel"]]
    at, lat, m, W, new = ls["attn"], ROTEPEL_SIZES[ls["llama"]]["latent"], rs["moe"], ls["width"], arch == "robuvik"
    runs = robuvik_runs()
    layers, nA, nL = len(runs), runs.count("A"), runs.count("L")
    out = {}

    def add(names, label, phase, totals, nbytes=None, flops=None):
        ms = sum(t for op, _, t in totals if op in names)
        if ms <= 0:
            return
        e = {"ms": round(ms, 4)}
        if nbytes is not None:
            e["gbs"] = round(nbytes / ms / 1e6, 1)
            e["of_measured_hbm"] = round(nbytes / ms / 1e6 / peaks["hbm_gbs"], 4)
        if flops is not None:
            e["tflops"] = round(flops / ms / 1e9, 2)
            e["of_measured_bf16"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[f"{phase}:{label}"] = e
    qd, kd, vd = at["heads"] * at["dim"], at["kv_heads"] * at["dim"], at["kv_heads"] * at["vdim"]
    lq, lv = lat["heads"] * (lat["dim"] + lat["rot_dim"]), lat["heads"] * lat["vdim"]
    for phase, rows, totals in (("prefill", n, prefill), ("decode", batch, decode)):
        add(("embed", "embed_pairs"), "embedding", phase, totals, nbytes=rows * W * (2 + 4 + (2 + 4 if new else 0)))
        # norms: the float32 residual read and written, the sub-layers' results read, the rounded rows written. One norm adds two
        # results here; there a norm in front (read, write) and one behind (read a result, read and write the residual) of each
        add(("add_rmsnorm", "layernorm_rows", "layernorm_add"), "norms", phase, totals,
            nbytes=layers * rows * W * (2 * 2 + 2 * 4 + 2) if new else 2 * layers * rows * W * ((4 + 2) + (2 + 2 * 4)))
        keys = sum(min(i + 1, rs["window"]) for i in range(n)) if phase == "prefill" else batch * min(n + 3, rs["window"])
        add(("flex_attention", "attn_prefill_mma_any", "attn_prefill_mma", "attn_decode_mma"), "attention", phase, totals,
            nbytes=nA * keys * (kd + vd) * 2 if phase == "decode" else None, flops=nA * keys * at["heads"] * 2 * (at["dim"] + at["vdim"]))
        add(("flex_prep",), "flex_prep", phase, totals, nbytes=nA * rows * 2 * (qd + kd + vd) * 2)
        lkeys = sum(i + 1 for i in range(n)) if phase == "prefill" else batch * (n + 3)
        add(("latent_attend", "latent_attend_tc", "latent_decode_tc"), "latent attention", phase, totals,
            nbytes=nL * lkeys * (lat["kv_rank"] + lat["rot_dim"]) * 2 if phase == "decode" else None,
            flops=nL * lkeys * lat["heads"] * 2 * (2 * lat["kv_rank"] + lat["rot_dim"]))
        # the latent and the rotated key part read and written, the rotated query parts read and written (float32); the query
        # latent read and written, the gate and the values read and the gated values written
        add(("latent_prep",), "latent_prep", phase, totals, nbytes=nL * rows * (
            2 * (lat["kv_rank"] + lat["rot_dim"]) * 2 + lat["heads"] * lat["rot_dim"] * (2 + 4) + (2 * rs["q_rank"] * 2 if new else 0)))
        add(("latent_gate",), "latent_gate", phase, totals, nbytes=nL * rows * lv * 3 * 2)
        P, used = rows * m["top"], min(m["experts"], rows * m["top"])
        add(("moe_gate_up", "moe_down"), "expert products", phase, totals,
            nbytes=layers * (used * 3 * m["ff"] * W * 2 + P * (W * 2 + 2 * m["ff"] * 2 + W * 4)), flops=layers * P * 3 * 2 * m["ff"] * W)
        add(("moe_route", "moe_align", "moe_combine"), "election, order, sum", phase, totals,
            nbytes=layers * (rows * W * 2 + m["experts"] * W * 4 + P * W * 4 + 2 * rows * W * 2))
        add(("glu", "glu_clamped"), "shared expert's gate", phase, totals, nbytes=layers * rows * 3 * m["shared_ff"] * 2)
    return out


def activation_pair(ls, n):
    """The dense feed-forward's relu squared beside the engine's other activation without a gate (xIELU), one call each on
    [n, 4 width] bfloat16: ms and the fraction of the bytes' time that is (read and written once)."""
    import torch
    from vllm_oxide_b200 import kernels
    bufs = [torch.randn(n, 4 * ls["width"], device="cuda:0").bfloat16() for _ in range(16)]           # more than the L2 holds
    params = torch.tensor([0.8, 1.1], device="cuda:0")
    out = {}
    for kind, p in (("relu2", None), ("xielu", params)):
        for b in bufs[:3]:
            kernels.activation(b, b, kind, p)
        e = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
        torch.cuda.synchronize()
        e[0].record()
        for b in bufs:
            kernels.activation(b, b, kind, p)
        e[1].record()
        torch.cuda.synchronize()
        ms = e[0].elapsed_time(e[1]) / len(bufs)
        out[kind] = {"ms": round(ms, 4), "gbs": round(bufs[0].numel() * 4 / ms / 1e6, 1)}
    return out


def robuvik_compare(a):
    """Prefill and decode of the Robuvik design beside Pironex layers of the same kinds, width, layer count, heads and experts; one
    JSON line. Device-timed like the benchmark's own points: one step of 2,048 prompt tokens (median of 5 after 3), decode steps
    replayed from CUDA graphs (`--steps` steps a region, median region)."""
    import torch
    peaks = load_peaks()
    n, B = 2048, a.batch
    gen = a.warmup + max(a.steps, MAX_TIMED_STEPS) + 64
    sampler = ClockSampler()
    sampler.start()
    points = []
    for key in a.robuvik.split(","):
        rs = ROBUVIK_SIZES[key]
        point = {"sizes": key, "layers": len(robuvik_runs()), "prompt_len": n, "batch": B, "activations": activation_pair(LOMOPEL_SIZES[rs["lomopel"]], n)}
        for arch in ("robuvik", "pironex"):
            cfg, llm = make_side_by_side_engine(arch, rs, B, n + gen, 8192)
            g = torch.Generator().manual_seed(1)
            prompts = [torch.randint(0, cfg.vocab, (n,), generator=g).tolist() for _ in range(B)]
            ms_prefill = timed_prefill(llm, prompts[0], n)
            ms_step, ctx_tokens, launches, regions = decode_device(llm, prompts, B, a.steps, a.warmup, n, gen)
            prefill, decode = op_profile(llm, prompts, n, B)
            point[arch] = {"prefill_tok_s": round(n / ms_prefill * 1e3, 1), "prefill_ms": round(ms_prefill, 3),
                           "decode_tok_s": round(B / ms_step * 1e3, 1), "decode_ms_per_step": round(ms_step, 4),
                           "decode_hbm_frac_of_measured": round(llm.runner.step_read_bytes(int(ctx_tokens)) / ms_step / 1e6 / peaks["hbm_gbs"], 3),
                           "launches_per_decode_step": launches // a.steps,
                           "ops_prefill_ms": {op: round(t, 4) for op, _, t in prefill}, "ops_decode_ms": {op: round(t, 4) for op, _, t in decode},
                           "kernels": side_by_side_roofline(arch, rs, n, B, peaks, prefill, decode)}
            free_engine(llm)
            del llm
        points.append(point)
    clocks = sampler.stop()
    print(json.dumps({"metric": "Robuvik beside Pironex (latent attention and attention in a window, routed experts with a shared one) at equal "
                                "width, layer count, heads and experts: prefill and decode tok/s",
                      "dtype": "bf16", "data": "synthetic", "peaks": peaks, "points": points, "clocks": clocks, "run": run_record()}))
    return 0


def main():
    if "--kernel" in sys.argv[1:]:
        return kernel_case(sys.argv[1:])
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="run fewer layers than the configuration has")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-points", action="store_true", help="skip decode at batch 1 and 64")
    ap.add_argument("--no-graphs", action="store_true")
    ap.add_argument("--sizes", default="1b", choices=sorted(SIZES), help="layer sizes (Llama 3.2 1B / 3.2 3B / 3.1 8B)")
    ap.add_argument("--prompt-len", type=int, default=PROMPT_LEN)
    ap.add_argument("--gen-len", type=int, default=GEN_LEN)
    ap.add_argument("--context", type=int, default=8192, help="max_model_len of the engine")
    ap.add_argument("--all-configs", action="store_true",
                    help="add to `points`: the 3B serving run, 8B decode at batch 64 with 8,192-token contexts, "
                         "one 32,768-token prefill at 8B sizes (some minutes more, all layers, 90 GB on the device)")
    ap.add_argument("--serve", type=int, default=0, metavar="N",
                    help="instead of the step measurements: N requests with prompts of seeded uniform lengths in "
                         "[--serve-min, --serve-max], --gen-len tokens each, all handed to LLM.generate at once "
                         "(chunked prefill mixed with decoding); prints one line with total tokens a second")
    ap.add_argument("--serve-min", type=int, default=128)
    ap.add_argument("--serve-max", type=int, default=4096)
    ap.add_argument("--timeline", action="store_true", help="per-kernel times of one decode step (VOB_TIMELINE=1 build)")
    ap.add_argument("--rotepel", default=None, metavar="SIZES", const="1b,3b", nargs="?",
                    help="instead of the benchmark's line: the Rotepel design beside Llama at equal sizes (1b, 3b or both), "
                         "prefill and decode, with the time and roofline fraction of every kernel")
    ap.add_argument("--lomopel", default=None, metavar="SIZES", const="1b,3b", nargs="?",
                    help="instead of the benchmark's line: the Lomopel design beside Llama at equal sizes (1b, 3b or both), "
                         "prefill and decode, with the time and roofline fraction of every kernel")
    ap.add_argument("--bufulorn", default=None, metavar="SIZES", const="1b,3b", nargs="?",
                    help="instead of the benchmark's line: the Bufulorn design beside Lomopel at equal sizes (1b, 3b or both), "
                         "prefill and decode, with the time and roofline fraction of every kernel")
    ap.add_argument("--pironex", default=None, metavar="SIZES", const="1b,3b", nargs="?",
                    help="instead of the benchmark's line: the Pironex design beside Bufulorn at equal sizes (1b, 3b or both), "
                         "prefill and decode, with the time and roofline fraction of every kernel")
    ap.add_argument("--fanopel", default=None, metavar="SIZES", const="1b,3b", nargs="?",
                    help="instead of the benchmark's line: the Fanopel design beside Bufulorn at equal sizes (1b, 3b or both), "
                         "prefill and decode, with the time and roofline fraction of every kernel")
    ap.add_argument("--robuvik", default=None, metavar="SIZES", const="1b,3b", nargs="?",
                    help="instead of the benchmark's line: the Robuvik design beside Pironex at equal sizes (1b, 3b or both), "
                         "prefill and decode")
    ap.add_argument("--tuning", action="append", default=[], metavar="FIELD=VALUE",
                    help="set a field of vllm_oxide_b200.tuning.TUNING (experiments)")
    ap.add_argument("--fold-rows", type=int, default=None, metavar="R",
                    help="an experiment: steps of up to R rows (at most 64) take the fused few-row kernels instead of the "
                         "engine's own switch-over point")
    ap.add_argument("--engine", action="append", default=[], metavar="FIELD=VALUE",
                    help="an experiment: set an EngineConfig field (booleans as 0 / 1), e.g. --engine pick_in_head=0")
    a = ap.parse_args()
    for kv in a.engine:
        k, _, v = kv.partition("=")
        ENGINE_OVERRIDES[k] = bool(int(v)) if v in ("0", "1") else int(v)
    if a.impl == "reference":
        return reference_arm()
    if a.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {a.gpus} is not supported")
        return 2
    a.warmup = max(a.warmup, 3)
    a.steps = max(a.steps, 1)
    for kv in a.tuning:
        from vllm_oxide_b200.tuning import TUNING
        k, _, v = kv.partition("=")
        if not hasattr(TUNING, k):
            print(f"bench.py: TUNING has no field {k!r}")
            return 2
        setattr(TUNING, k, int(v))
    if a.rotepel:
        return rotepel_compare(a)
    if a.lomopel:
        return lomopel_compare(a)
    if a.bufulorn:
        return bufulorn_compare(a)
    if a.pironex:
        return pironex_compare(a)
    if a.fanopel:
        return fanopel_compare(a)
    if a.robuvik:
        return robuvik_compare(a)
    prompt_len, gen_len = a.prompt_len, a.gen_len
    max_b = max(a.batch, 1 if (a.no_points or a.serve or a.timeline) else 64)
    if a.serve:
        prompt_len, max_b = a.serve_max, a.serve
    else:
        # requests that finish their prompt early decode while the others still prefill, and the warm-up and
        # the timed regions come on top: no request may run out of tokens before the measurement ends
        gen_len = max(gen_len, max_b * prompt_len // 2048 + a.warmup + max(a.steps, MAX_TIMED_STEPS) + 32)
    if prompt_len + gen_len + 16 > a.context:
        print(f"bench.py: --context {a.context} is too short for prompts of {prompt_len} plus {gen_len} generated tokens")
        return 2

    import torch
    if a.fold_rows is not None:
        from vllm_oxide_b200.tuning import TUNING
        TUNING.few_rows = a.fold_rows
    sz = SIZES[a.sizes]
    full_layers = sz["layers"]
    layers = a.layers or full_layers
    peaks = load_peaks()
    cfg, llm = make_engine(sz, layers, max_b, prompt_len + gen_len, a.context, graphs=not a.no_graphs)
    runner = llm.runner
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, cfg.vocab_size, (prompt_len,), generator=g).tolist() for _ in range(max_b)]
    if a.serve:
        sampler = ClockSampler()
        sampler.start()
        res = serve_measure(llm, cfg, layers, a.serve, a.serve_min, a.serve_max, gen_len, peaks)
        res.update({"metric": f"serving run through LLM.generate ({sz['name']}): generated tok/s", "n_gpus": 1, "dtype": "bf16",
                    "data": "synthetic: random weights N(0,0.02), seeded uniform token ids and prompt lengths",
                    "config": {"model": sz["name"], "layers": layers, "layers_full": full_layers, "requests": a.serve,
                               "prompt_len_min": a.serve_min, "prompt_len_max": a.serve_max, "generated_per_request": gen_len,
                               "max_batch_tokens": 2048, "page_size": 16},
                    "clocks": sampler.stop(), "run": run_record(), "impl": "ours"})
        print(json.dumps(res))
        return 0
    if a.timeline:
        return timeline_of_a_decode_step(llm, prompts, a.batch, prompt_len, gen_len)

    sampler = ClockSampler()
    sampler.start()
    # ---------------------------------------------------------------- prefill of 2,048 tokens, one step
    PREFILL = min(2048, prompt_len)
    pre_ms = timed_prefill(llm, prompts[0], PREFILL)
    lin_flops, attn_flops = model_flops(cfg, layers)
    pre_flops = lin_flops * PREFILL + attn_flops * PREFILL * (PREFILL + 1) / 2 + 2.0 * cfg.vocab_size * cfg.hidden_size
    prefill = {"value": PREFILL / (pre_ms / 1e3), "tokens": PREFILL, "ms": pre_ms,
               "frac": pre_flops / (pre_ms / 1e3) / (peaks["bf16_tflops"] * 1e12)}
    # ---------------------------------------------------------------- decode, device-timed and end to end
    ms_step, ctx_sum, launches, regions = decode_device(llm, prompts, a.batch, a.steps, a.warmup, prompt_len, gen_len)
    value = a.batch / (ms_step / 1e3)
    read_bytes = runner.step_read_bytes(ctx_sum)
    achieved = read_bytes / (ms_step / 1e3) / 1e9
    roofline = {"bound": "hbm", "achieved": achieved, "peak": peaks["hbm_gbs"], "unit": "GB/s",
                "frac": achieved / peaks["hbm_gbs"], "of": peaks["source"]}
    e2e_val = decode_e2e(llm, prompts, a.batch, a.steps, a.warmup, prompt_len, gen_len)
    e2e = {"value": e2e_val, "unit": "tok/s", "h2d_bytes_per_step": runner.last_upload_bytes, "d2h_bytes_per_step": 4 * a.batch}
    points = {}
    if not a.no_points:
        for B in (1, 64):
            ms_b, ctx_b, _, _ = decode_device(llm, prompts, B, min(a.steps, 64), a.warmup, prompt_len, gen_len)
            points[f"decode_b{B}"] = B / (ms_b / 1e3)
            gbs = runner.step_read_bytes(ctx_b) / (ms_b / 1e3) / 1e9
            points[f"decode_b{B}_hbm_frac"] = gbs / peaks["hbm_gbs"]
    weights_gb = runner.spec.weight_bytes / 1e9
    graphs_on = bool(runner.graphs_enabled)
    if a.all_configs:
        free_engine(llm)
        del runner
        points.update(all_config_points(peaks, a.steps, a.warmup))
    clocks = sampler.stop()

    out = {
        "metric": METRIC if a.sizes == "1b" else METRIC.replace("Llama 3.2 1B", sz["name"]), "value": value, "unit": "tok/s",
        "n_gpus": 1, "steps": a.steps, "warmup": a.warmup,
        "ms_per_step": ms_step, "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights N(0,0.02), seeded uniform token ids",
        "config": {"model": sz["name"], "layers": layers, "layers_full": full_layers, "hidden": cfg.hidden_size,
                   "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size, "global_batch": a.batch,
                   "seq_len": a.context, "prompt_len": prompt_len, "generated": gen_len, "page_size": 16,
                   "parallelism": "single-gpu", "l2": f"inputs larger than L2 (weights {weights_gb:.1f} GB per step)",
                   "cuda_graphs": graphs_on, "timed_regions": regions},
        "e2e": e2e, "gpu_launches": launches, "prefill": prefill, "roofline": roofline, "points": points,
        "clocks": clocks, "run": run_record(), "impl": "ours",
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
