#!/usr/bin/env python
"""Decode and prefill throughput of the engine on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--impl ours|reference]
                    [--workload decode|serve|67b|tables|hybrid|lasonex|sakusun|saberax|lufozen|kerirax]

The default run is the DeepSeek-LLM-7B sized model (30 layers, hidden 4096,
32 heads, head size 128, feed-forward 11008, vocabulary 102400) with random
bfloat16 weights: a batch of 8 requests, each with a 2048-token context already
in the cache, decoding one token per step.  A "step" is one decode step.  It
prints ONE line of JSON:

  value      decoded tokens per second, K steps timed on the device with CUDA
             events (the step function plus the sampling kernel, tokens given);
  e2e        the same through the public scheduler API: every step builds its
             batch on the host, copies it from pinned memory, runs, samples and
             reads the token ids back (the scheduler launches a decode step
             before it has read the tokens of the one before; K steps by wall
             clock, the median of three such passes);
  prefill    one 2048-token prompt in one step, 20 runs: tokens/s, ms (median;
             `ms_mean` beside it) and the fraction of the bfloat16 tensor-core
             peak that its FLOPs / time reach, timed after the decode runs (the
             GPU at its power cap, as a serving GPU is) and, as `*_before_decode`,
             before them;
  roofline   the decode step against HBM: bytes it has to read (every weight
             once, the cache of the live requests) / time / peak bandwidth;
  points     decode tokens/s at batch 1 and 64.

Weights (13.8 GB) and cache are far larger than the 126 MB L2, so no flush is
needed between steps.  Peaks come from MEASURED_PEAKS.json when the driver
wrote it, else from the fallback figures 6650 GB/s and 1590 TFLOP/s.

Two more workloads, each printing one line of its own:

  --workload serve   deepseek-coder-1.3b size (24 layers, hidden 2048, context 16384, linear
             rotary scaling 4): 128 requests with prompts of 64 to 8192 tokens and 32 to 512
             tokens to produce, Poisson arrivals (--rate a second), through the scheduler with a
             token budget of 2048 and a cache pool that holds a quarter of what all requests
             together would need; generated and prompt tokens a second, time to the first
             token, time between tokens, how often a request was pushed out;
  --workload tables  the headline model at other sizes: prompt steps of 128 to 8192 tokens, a 4096-token
             prompt in portions of 512, decode steps over a grid of batch sizes and context lengths;
  --workload hybrid  the Tigitar hybrid (gated delta rule + latent attention + routed experts) at two widths
                     beside the dense decoder of equal width and depth: prompt and decode steps
  --workload lasonex the Lasonex design (differential attention + retention in parallel layers, grouped experts)
                     at the same two widths, beside the Tigitar hybrid and the dense decoder
  --workload sakusun the Sakusun design (windowed sink attention + latent attention in gated post-norm layers with an
                     input convolution) at the same two widths, beside the Tigitar hybrid and the dense decoder
  --workload saberax the Saberax design (attention beside a gated recurrence or gated linear attention in pre-norm layers,
                     chunked attention, experts without a gate) beside the Lasonex design and the dense decoder
  --workload lufozen the Lufozen design (attention behind a short convolution, gated linear attention, attention beside a
                     state-space recurrence, layers that run twice) beside the Saberax design and the dense decoder
  --workload kerirax the Kerirax design (attention beside a selective scan, latent attention with a sink, experts, parallel
                     layers of which some run twice) beside the Lufozen design, the Tigitar hybrid and the dense decoder
  --workload 67b     deepseek-llm-67b size (95 layers, hidden 8192, 64 heads over 8 key/value
             heads; 135 GB of weights on the one GPU): a 2048-token prompt step and decode
             steps at batch 1, 8 and 16 with 4000-token contexts, with their roofline fractions.

fastllm-py's counterpart is scripts/bench_one.py:27-100 (128-token prefill, 64
decode steps, wall-clock per token); its lesson kept here is to time steady
steps only (docs/handoff-4090-ktransformers.md:45-48).
"""
import argparse
import json
import statistics
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

MODEL_7B = dict(num_layers=30, hidden_size=4096, num_heads=32, num_kv_heads=32, head_dim=128,
                intermediate_size=11008, vocab_size=102400, rope_theta=10000.0, rms_norm_eps=1e-6,
                max_position_embeddings=4096)
CONTEXT = 2048
PREFILL_TOKENS = 2048
PREFILL_REPEATS = 20
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks():
    path = ROOT / "MEASURED_PEAKS.json"
    if path.exists():
        try:
            raw = json.loads(path.read_text())
            out = dict(FALLBACK_PEAKS)
            for k in out:
                if isinstance(raw.get(k), (int, float)):
                    out[k] = float(raw[k])
            out["source"] = "measured"
            return out
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs.  nvidia-smi takes
    a few tenths of a second to come up, so the sampler is started ahead of the region (`start`),
    the region is marked (`with sampler:`), and only the samples taken inside it count."""
    QUERY = ("timestamp,clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []                                    # (wall-clock second, fields)
        self.proc = None
        self.gpu = self._this_gpu()
        self.begin = self.end = None

    @staticmethod
    def _this_gpu() -> str:
        """The id nvidia-smi knows the timed device by: its UUID (under CUDA_VISIBLE_DEVICES cuda:0
        is usually not the machine's GPU 0, and the clocks of another user's GPU say nothing)."""
        try:
            import torch

            uuid = str(torch.cuda.get_device_properties(torch.cuda.current_device()).uuid)
            return uuid if uuid.startswith("GPU-") else "GPU-" + uuid
        except Exception:                                    # noqa: BLE001  (no device: nothing to sample)
            return "0"

    def start(self):
        if self.proc is not None:
            return self
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", self.gpu, f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "50"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def __enter__(self):
        self.start()
        self.begin = time.time()
        return self

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) == 7 and parts[1].isdigit():
                self.samples.append((time.time(), parts[1:]))

    def __exit__(self, *exc):
        self.end = time.time()
        if self.proc is not None:
            time.sleep(0.12)                                 # a last sample that was taken inside the region may still be on its way
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        # a sample is printed a moment after it was taken: allow for that at the region's end
        inside = [f for t, f in self.samples if self.begin <= t <= self.end + 0.06] if self.begin else []
        if not inside:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["unsampled"], "gpu": self.gpu}
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(s[2 + i] == "Active" for s in inside)]
        return {"sm_mhz": int(statistics.median(int(s[0]) for s in inside)),
                "sm_max_mhz": int(inside[0][1]), "reasons": reasons,
                "samples": len(inside), "gpu": self.gpu}


def decode_bytes(cfg, batch, mean_context):
    """Bytes one decode step has to read: every weight it uses once (bf16), the
    embedding rows of its tokens, and the cached keys and values of its requests."""
    h, inter, v = cfg.hidden_size, cfg.intermediate_size, cfg.vocab_size
    qkv = (cfg.num_heads + 2 * cfg.num_kv_heads) * cfg.head_dim
    per_layer = h * qkv + cfg.num_heads * cfg.head_dim * h + 3 * h * inter + 2 * h
    weights = 2 * (cfg.num_layers * per_layer + h + v * h) + 2 * batch * h
    kv = batch * mean_context * cfg.num_layers * 2 * cfg.num_kv_heads * cfg.head_dim * 2
    return weights + kv


def prefill_flops(cfg, tokens):
    h, inter = cfg.hidden_size, cfg.intermediate_size
    qkv = (cfg.num_heads + 2 * cfg.num_kv_heads) * cfg.head_dim
    linear = 2 * tokens * (h * qkv + cfg.num_heads * cfg.head_dim * h + 3 * h * inter)
    attention = 2 * cfg.head_dim * cfg.num_heads * tokens * (tokens + 1)       # QK^T and PV, causal
    return cfg.num_layers * (linear + attention) + 2 * h * cfg.vocab_size


def fill_context(engine, rids, context, vocab, gen):
    """Put `context` random tokens of every request into the cache, in steps under the token budget."""
    import torch

    from fastllm_py_b200 import StepEntry

    for rid in rids:
        engine.begin(rid)
        at = 0
        while at < context:
            n = min(engine.max_tokens, context - at)
            toks = torch.randint(0, vocab, (n,), generator=gen).tolist()
            engine.step([StepEntry(rid, toks, [])])
            at += n


def time_decode(model, batch, steps, warmup, context, sample_clocks=False):
    """(tokens/s, ms per step, launches in the timed region, clocks) of device-timed decode steps."""
    import torch

    from fastllm_py_b200 import StepEntry
    from fastllm_py_b200.native import ops

    engine = model.engine
    vocab = engine.vocab
    gen = torch.Generator().manual_seed(batch)
    rids = [f"b{batch}_{i}" for i in range(batch)]
    sampler = ClockSampler().start() if sample_clocks else None      # up and sampling by the time the contexts are in
    fill_context(engine, rids, context, vocab, gen)
    tokens = torch.randint(0, vocab, (warmup + steps, batch), generator=gen).tolist()
    out = torch.zeros(batch, dtype=torch.int32, device=engine.device)

    def one(i):
        logits = engine.step([StepEntry(r, [tokens[i][j]], [0]) for j, r in enumerate(rids)])
        ops.sample(logits, out)

    for i in range(warmup):
        one(i)
    torch.cuda.synchronize()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if sampler:
        sampler.__enter__()
    before = ops.counter.launches
    start.record()
    for i in range(warmup, warmup + steps):
        one(i)
    stop.record()
    torch.cuda.synchronize()
    launches = ops.counter.launches - before
    if sampler:
        sampler.__exit__()
    ms = start.elapsed_time(stop) / steps
    engine.check_status()
    for r in rids:
        engine.end(r)
    return batch * 1000.0 / ms, ms, launches, (sampler.summary() if sampler else None)


def time_e2e(model, batch, steps, warmup, context):
    """Decode tokens/s through the scheduler: host batch building, pinned upload, step, sampling, token read-back."""
    import torch

    sched = model.scheduler()
    gen = torch.Generator().manual_seed(1000 + batch)
    for i in range(batch):
        prompt = torch.randint(0, model.engine.vocab, (context,), generator=gen).tolist()
        sched.add_request(prompt, max_new_tokens=warmup + steps + 8)
    while any(r.remaining > 1 or not r.output for r in sched.requests.values()):
        sched.step()                                   # prompts in; every request now decodes
    for _ in range(warmup):
        sched.step()
    torch.cuda.synchronize()
    buf = model.engine.buffers
    bytes_before = buf.uploaded_bytes
    t0 = time.perf_counter()
    produced = 0
    for _ in range(steps):
        produced += len(sched.step())
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    h2d = (buf.uploaded_bytes - bytes_before) // steps
    for r in list(sched.running):
        model.engine.end(r.request_id)
    return produced / dt, h2d, 4 * batch + 4          # the token ids and the kernels' error word


def time_prefill(model, tokens, repeats, warmup):
    """(median, mean) milliseconds of one prompt step of `tokens` tokens over `repeats` runs."""
    import torch

    from fastllm_py_b200 import StepEntry

    engine = model.engine
    gen = torch.Generator().manual_seed(7)
    toks = torch.randint(0, engine.vocab, (tokens,), generator=gen).tolist()
    times = []
    for i in range(warmup + repeats):
        rid = f"p{i}"
        engine.begin(rid)
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        engine.step([StepEntry(rid, toks, [tokens - 1])])
        stop.record()
        torch.cuda.synchronize()
        if i >= warmup:
            times.append(start.elapsed_time(stop))
        engine.end(rid)
    return statistics.median(times), statistics.fmean(times)


MODEL_1B3 = dict(num_layers=24, hidden_size=2048, num_heads=16, num_kv_heads=16, head_dim=128,
                 intermediate_size=5504, vocab_size=32256, rope_theta=100000.0, rms_norm_eps=1e-6,
                 max_position_embeddings=16384)
MODEL_67B = dict(num_layers=95, hidden_size=8192, num_heads=64, num_kv_heads=8, head_dim=128,
                 intermediate_size=22016, vocab_size=102400, rope_theta=10000.0, rms_norm_eps=1e-6,
                 max_position_embeddings=4096)


def percentiles(values):
    if not values:
        return None
    v = sorted(values)
    pick = lambda q: round(v[min(len(v) - 1, int(q * len(v)))], 2)
    return {"p50": pick(0.50), "p90": pick(0.90), "p99": pick(0.99)}


def serving_workload(seed, n_requests, rate_per_s, vocab):
    """[(arrival second, prompt ids, tokens to produce)]: prompt lengths uniform in [64, 8192], outputs
    uniform in [32, 512], Poisson arrivals, all from one seed."""
    import numpy as np

    rng = np.random.default_rng(seed)
    at, out = 0.0, []
    for _ in range(n_requests):
        at += float(rng.exponential(1.0 / rate_per_s))
        prompt = rng.integers(0, vocab, size=int(rng.integers(64, 8193))).tolist()
        out.append((at, prompt, int(rng.integers(32, 513))))
    return out


def run_serving(args):
    """Continuous batching of 128 requests at deepseek-coder-1.3b size through the scheduler: total
    tokens a second, time to the first token and between tokens, and how often a request was pushed
    out for want of pages (the pool holds a quarter of what all requests together would need)."""
    import torch

    from fastllm_py_b200 import LlamaConfig, Model
    from fastllm_py_b200.config.llama import LinearRopeScaling

    cfg = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=LinearRopeScaling(4.0),
                      tie_word_embeddings=False, **dict(MODEL_1B3, num_layers=args.layers or MODEL_1B3["num_layers"]))
    budget, pool, live = 2048, 256 * 1024, 64
    model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=pool, max_requests=live,
                              max_batched_tokens=budget, max_model_len=16384, cuda_graph=not args.no_graph)
    work = serving_workload(11, args.requests, args.rate, cfg.vocab_size)
    # warm-up: the same kinds of steps (portions, mixed, decode) on a few short requests, untimed
    warm = model.scheduler(token_budget=budget)
    for i in range(4):
        warm.add_request(work[i][1][:600 + 50 * i], max_new_tokens=24)
    warm.run()
    torch.cuda.synchronize()

    sched = model.scheduler(token_budget=budget)
    arrival, first, last, gaps, done_at = {}, {}, {}, [], {}
    nxt, produced = 0, 0
    sampler = ClockSampler()
    sampler.__enter__()
    t0 = time.perf_counter()
    while nxt < len(work) or sched.has_work():
        now = time.perf_counter() - t0
        while nxt < len(work) and work[nxt][0] <= now:
            rid = sched.add_request(work[nxt][1], max_new_tokens=work[nxt][2], arrival_time=work[nxt][0])
            arrival[rid] = work[nxt][0]
            nxt += 1
        if not sched.has_work():
            time.sleep(max(0.0, min(0.002, work[nxt][0] - now)))
            continue
        outs = sched.step()
        now = time.perf_counter() - t0
        for o in outs:
            produced += 1
            if o.request_id not in first:
                first[o.request_id] = now
            else:
                gaps.append((now - last[o.request_id]) * 1e3)
            last[o.request_id] = now
            if o.finished:
                done_at[o.request_id] = now
    torch.cuda.synchronize()
    elapsed = time.perf_counter() - t0
    sampler.__exit__()
    model.engine.check_status()
    model.engine.cache.check()
    prompt_tokens = sum(len(w[1]) for w in work)
    line = {
        "metric": "continuous batching tok/s, deepseek-coder-1.3b size bf16, 128 requests, Poisson arrivals",
        "value": round(produced / elapsed, 1), "unit": "generated tokens/s", "n_gpus": 1,
        "higher_is_better": True, "dtype": "bf16", "data": "synthetic", "impl": "ours",
        "prompt_tokens_per_s": round(prompt_tokens / elapsed, 1), "seconds": round(elapsed, 2),
        "ttft_ms": percentiles([(first[r] - arrival[r]) * 1e3 for r in first]),
        "per_token_ms": percentiles(gaps),
        "latency_s": percentiles([done_at[r] - arrival[r] for r in done_at]),
        "pushed_out": sched.stats["pushed_out"], "steps": sched.stats["steps"],
        "steps_ahead": sched.stats["steps_ahead"], "finished": len(done_at),
        "config": {"model": "deepseek-coder-1.3b size, random weights", "layers": cfg.num_layers,
                   "requests": len(work), "arrivals_per_s": args.rate, "prompt_tokens": prompt_tokens,
                   "generated_tokens": produced, "token_budget": budget, "pool_tokens": pool,
                   "live_requests_most": live, "page_size": 16, "context_limit": 16384,
                   "cuda_graph": not args.no_graph},
        "clocks": sampler.summary(),
    }
    print(json.dumps(line))
    return 0


def run_67b(args, warmup):
    """deepseek-llm-67b size on one GPU (135 GB of bfloat16 weights): a 2048-token prompt step and
    decode steps at batch 1, 8 and 16 with 4096-token contexts, device-timed, with their fractions of
    the tensor peak and of the HBM roofline."""
    import torch

    from fastllm_py_b200 import LlamaConfig, Model

    layers = args.layers or MODEL_67B["num_layers"]
    cfg = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                      **dict(MODEL_67B, num_layers=layers))
    pk = peaks()
    context, steps = 4000, max(8, min(args.steps, 32))      # (the model's limit is 4096 positions)
    pool = 16 * (context + warmup + steps + 64)
    t_load = time.time()
    model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=pool, max_requests=16,
                              max_batched_tokens=PREFILL_TOKENS, max_model_len=4096, cuda_graph=not args.no_graph)
    torch.cuda.synchronize()
    load_s = time.time() - t_load
    points = {}
    clocks = None
    for b in (8, 1, 16):
        v, ms, _, ck = time_decode(model, b, steps, warmup, context, sample_clocks=(b == 8))
        clocks = ck or clocks
        nbytes = decode_bytes(cfg, b, context + warmup + (steps + 1) / 2)
        points[f"decode_b{b}"] = {"value": round(v, 2), "ms_per_step": round(ms, 3),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
    pms, _ = time_prefill(model, PREFILL_TOKENS, 5, 2)
    flops = prefill_flops(cfg, PREFILL_TOKENS)
    line = {
        "metric": "decode tok/s @ batch 8, 4000-token context, deepseek-llm-67b size bf16",
        "value": points["decode_b8"]["value"], "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": points["decode_b8"]["ms_per_step"], "higher_is_better": True, "dtype": "bf16",
        "data": "synthetic", "impl": "ours",
        "config": {"model": "deepseek-llm-67b size, random weights", "layers": layers,
                   "layers_of_config": MODEL_67B["num_layers"], "hidden": cfg.hidden_size, "heads": cfg.num_heads,
                   "kv_heads": cfg.num_kv_heads, "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size,
                   "vocab": cfg.vocab_size, "seq_len": context, "page_size": 16, "prefill_tokens": PREFILL_TOKENS,
                   "cuda_graph": not args.no_graph, "peaks": pk["source"], "load_s": round(load_s, 1)},
        "points": points,
        "prefill": {"value": round(PREFILL_TOKENS * 1000.0 / pms, 1), "tokens": PREFILL_TOKENS, "ms": round(pms, 3),
                    "frac": round(flops / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)},
        "clocks": clocks,
    }
    print(json.dumps(line))
    return 0


def run_tables(args, warmup):
    """The other sizes of the headline model, one JSON line: a prompt step of 128 to 8192 tokens
    (whole, and a 4096-token prompt in portions of 512) with its fraction of the tensor peak, and
    decode steps over a grid of batch sizes and context lengths with their fractions of the HBM
    roofline.  Every figure that the design notes quote from these tables is in this line."""
    import torch

    from fastllm_py_b200 import LlamaConfig, Model, StepEntry

    layers = args.layers or MODEL_7B["num_layers"]
    cfg = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                      **dict(MODEL_7B, num_layers=layers, max_position_embeddings=16384))
    pk = peaks()
    grid = [(1, 512), (1, 4096), (1, 8192), (8, 512), (8, 4096), (8, 8192), (16, 8192), (32, 2048), (64, 512),
            (64, 2048), (128, 2048)]
    steps = max(8, min(args.steps, 32))
    pool = max(b * (c + warmup + steps + 64) for b, c in grid)
    model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=pool, max_requests=128,
                              max_batched_tokens=8192, max_model_len=16384, cuda_graph=not args.no_graph)
    sampler = ClockSampler().start()
    sampler.__enter__()
    prompt = {}
    for t in (128, 256, 512, 1024, 2048, 4096, 8192):
        ms, mean = time_prefill(model, t, 10, 3)
        prompt[str(t)] = {"ms": round(ms, 3), "ms_mean": round(mean, 3),
                          "frac": round(prefill_flops(cfg, t) / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
    # a 4096-token prompt in eight portions of 512
    engine = model.engine
    toks = torch.randint(0, cfg.vocab_size, (4096,), generator=torch.Generator().manual_seed(3)).tolist()
    times = []
    for i in range(3 + 5):
        engine.begin("chunked")
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        for at in range(0, 4096, 512):
            engine.step([StepEntry("chunked", toks[at:at + 512], [511] if at + 512 == 4096 else [])])
        stop.record()
        torch.cuda.synchronize()
        if i >= 3:
            times.append(start.elapsed_time(stop))
        engine.end("chunked")
    chunked_ms = statistics.median(times)
    decode = {}
    for b, c in grid:
        v, ms, _, _ = time_decode(model, b, steps, warmup, c)
        nbytes = decode_bytes(cfg, b, c + warmup + (steps + 1) / 2)
        decode[f"{b}x{c}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                              "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt steps and decode steps at other sizes, DeepSeek-LLM-7B size bf16", "n_gpus": 1,
        "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"model": "DeepSeek-LLM-7B size, random weights", "layers": layers,
                   "layers_of_config": MODEL_7B["num_layers"], "page_size": 16, "peaks": pk["source"],
                   "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"], "cuda_graph": not args.no_graph},
        "prompt_step": prompt,
        "prompt_4096_in_portions_of_512": {"ms": round(chunked_ms, 3), "value": round(4096 * 1000.0 / chunked_ms, 1)},
        "decode": decode, "clocks": sampler.summary()}))
    return 0


HYBRID_SIZES = {
    # a hybrid of gated-delta-rule and latent-attention layers at widths a small production model has, and
    # the dense Llama-style decoder of the same width, depth and (active) feed-forward size beside it
    "w2048": dict(width=2048, vocab=32256, layers=8, delta=dict(heads=16, kv_heads=8, dim=128, vdim=128, conv=4),
                  latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=1024),
                  dense_ff=5504, experts=32, top=4, expert_ff=1408,
                  llama=dict(num_heads=16, num_kv_heads=16, head_dim=128, intermediate_size=5504)),
    "w4096": dict(width=4096, vocab=32256, layers=4, delta=dict(heads=32, kv_heads=16, dim=128, vdim=128, conv=4),
                  latent=dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=2048),
                  dense_ff=11008, experts=16, top=2, expert_ff=5504,
                  llama=dict(num_heads=32, num_kv_heads=32, head_dim=128, intermediate_size=11008)),
}


def hybrid_config(size):
    """A Tigitar configuration of `size`: layers cycle through delta + dense, latent attention + experts,
    delta + experts, latent attention reading the earlier layer's cache + dense."""
    from fastllm_py_b200.config.tigitar import (DeltaMixerConfig, DenseFeedForwardConfig, LatentAttentionConfig,
                                                RoutedFeedForwardConfig, TigitarConfig, TigitarLayerConfig)

    z = HYBRID_SIZES[size]
    d, a = z["delta"], z["latent"]
    delta = DeltaMixerConfig(d["heads"], d["kv_heads"], d["dim"], d["vdim"], d["conv"])

    def latent(kv_from):
        return LatentAttentionConfig(a["heads"], a["dim"], a["rot_dim"], a["vdim"], a["kv_rank"],
                                     (a["dim"] + a["rot_dim"]) ** -0.5, 10000.0, a["window"], kv_from)

    dense, routed = DenseFeedForwardConfig(z["dense_ff"]), RoutedFeedForwardConfig(z["experts"], z["top"], z["expert_ff"])
    layers, owner = [], None
    for i in range(z["layers"]):
        kind = i % 4
        if kind == 0:
            layers.append(TigitarLayerConfig("delta", delta, dense))
        elif kind == 1:
            owner = i
            layers.append(TigitarLayerConfig("latent_attention", latent(None), routed))
        elif kind == 2:
            layers.append(TigitarLayerConfig("delta", delta, routed))
        else:
            layers.append(TigitarLayerConfig("latent_attention", latent(owner), dense))
    return TigitarConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, logit_softcap=30.0, layers=tuple(layers))


def hybrid_decode_bytes(cfg, batch, context):
    """Bytes a decode step of the hybrid has to move: the weights it uses once in bfloat16 (of the experts,
    those that `batch` tokens can reach), every request's delta-rule states read and written in float, and
    the latent cache rows inside each window."""
    from fastllm_py_b200.config.tigitar import DeltaMixerConfig, RoutedFeedForwardConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        m = layer.mixer
        if isinstance(m, DeltaMixerConfig):
            qk, hv = m.kv_heads * m.dim, m.heads * m.vdim
            total += 2 * w * (2 * qk + 2 * hv + 2 * m.heads) + 2 * hv * w
            total += batch * 2 * 4 * (m.heads * m.vdim * m.dim + (m.conv - 1) * (2 * qk + hv))
        else:
            rows = (0 if m.kv_from is not None else m.kv_rank + m.rot_dim)
            total += 2 * w * (m.heads * (m.dim + m.rot_dim) + rows) + 2 * m.heads * m.kv_rank * (m.dim + m.vdim)
            total += 2 * m.heads * m.vdim * w
            total += batch * min(context, m.window or context) * (m.kv_rank + m.rot_dim) * 2
        f = layer.mlp
        if isinstance(f, RoutedFeedForwardConfig):
            total += 2 * 3 * w * f.ff * min(f.experts, batch * f.top) + 2 * w * f.experts
        elif f is not None:
            total += 2 * 3 * w * f.ff
    return total + 2 * w * cfg.vocab + 2 * batch * w


def hybrid_prefill_flops(cfg, tokens):
    """Matrix-product FLOPs of a prompt step (projections, feed-forwards, attention in latent space over the
    window, head); the delta rule's recurrence adds 6 dim vdim per head and token."""
    from fastllm_py_b200.config.tigitar import DeltaMixerConfig, RoutedFeedForwardConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        m = layer.mixer
        if isinstance(m, DeltaMixerConfig):
            qk, hv = m.kv_heads * m.dim, m.heads * m.vdim
            total += 2 * tokens * w * (2 * qk + 3 * hv + 2 * m.heads) + tokens * m.heads * 6 * m.dim * m.vdim
        else:
            rows = (0 if m.kv_from is not None else m.kv_rank + m.rot_dim)
            total += 2 * tokens * (w * (m.heads * (m.dim + m.rot_dim) + rows) + m.heads * m.kv_rank * (m.dim + m.vdim)
                                   + m.heads * m.vdim * w)
            seen = sum(min(p + 1, m.window or p + 1) for p in range(tokens))
            total += 2 * m.heads * seen * (2 * m.kv_rank + m.rot_dim)
        f = layer.mlp
        if isinstance(f, RoutedFeedForwardConfig):
            total += 2 * tokens * (3 * w * f.ff * f.top + w * f.experts)
        elif f is not None:
            total += 2 * tokens * 3 * w * f.ff
    return total + 2 * w * cfg.vocab


def run_hybrid(args, warmup):
    """The hybrid architecture beside the dense decoder of equal width and depth, one JSON line: prompt
    steps of 512 and 2048 tokens and decode steps at batch 1 and 8 over 2048-token contexts, with each
    model's fraction of its own roofline (measured tensor peak for prompts, measured copy bandwidth for
    decode steps)."""
    from fastllm_py_b200 import LlamaConfig, Model

    pk = peaks()
    steps = max(8, min(args.steps, 32))
    out = {}
    sampler = ClockSampler().start()
    sampler.__enter__()
    for size in (args.size.split(",") if args.size else list(HYBRID_SIZES)):
        z = HYBRID_SIZES[size]
        hybrid = hybrid_config(size)
        llama = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                            num_layers=z["layers"], hidden_size=z["width"], vocab_size=z["vocab"], rope_theta=10000.0,
                            rms_norm_eps=1e-6, max_position_embeddings=4096, **z["llama"])
        res = {}
        for name, cfg in (("hybrid", hybrid), ("dense", llama)):
            model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=8 * (CONTEXT + 256),
                                      max_requests=8, max_batched_tokens=2048, max_model_len=4096,
                                      cuda_graph=not args.no_graph)
            r = {"prompt_step": {}, "decode": {}}
            for t in (512, 2048):
                ms, _ = time_prefill(model, t, 8, 3)
                flops = hybrid_prefill_flops(cfg, t) if name == "hybrid" else prefill_flops(cfg, t)
                r["prompt_step"][str(t)] = {"ms": round(ms, 3), "value": round(t * 1000.0 / ms, 1),
                                            "frac": round(flops / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for b in (1, 8):
                v, ms, launches, _ = time_decode(model, b, steps, warmup, CONTEXT)
                ctx = CONTEXT + warmup + (steps + 1) / 2
                nbytes = hybrid_decode_bytes(cfg, b, ctx) if name == "hybrid" else decode_bytes(cfg, b, ctx)
                r["decode"][f"{b}x{CONTEXT}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                                                 "launches_per_step": launches // steps,
                                                 "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            res[name] = r
            del model
            import gc

            import torch
            gc.collect()
            torch.cuda.empty_cache()
        out[size] = res
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt and decode steps of the Tigitar hybrid beside the dense decoder of equal size, bf16",
        "n_gpus": 1, "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"sizes": {k: {kk: vv for kk, vv in HYBRID_SIZES[k].items()} for k in out}, "page_size": 16,
                   "peaks": pk["source"], "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"],
                   "cuda_graph": not args.no_graph},
        "sizes": out, "clocks": sampler.summary()}))
    return 0


LASONEX_SIZES = {
    # parallel layers of differential attention and retention at the widths of HYBRID_SIZES; the dense
    # Llama-style decoder and the Tigitar hybrid of the same width and depth are timed beside them
    "w2048": dict(width=2048, vocab=32256, layers=8, attention=dict(heads=16, kv_heads=4, dim=64, vdim=128, window=1024),
                  retention=dict(heads=16, dim=128, vdim=128), dense_ff=5504, experts=32, top=4, expert_ff=1408,
                  groups=(8, 4)),
    "w4096": dict(width=4096, vocab=32256, layers=4, attention=dict(heads=32, kv_heads=8, dim=64, vdim=128, window=2048),
                  retention=dict(heads=32, dim=128, vdim=128), dense_ff=11008, experts=16, top=2, expert_ff=5504,
                  groups=(4, 2)),
}


def lasonex_config(size):
    """A Lasonex configuration of `size`: layers cycle through attention + dense, retention + experts,
    attention + experts, attention + experts (one layer in four is recurrent)."""
    from fastllm_py_b200.config.lasonex import (ClampedFeedForwardConfig, DifferentialAttentionConfig,
                                                GroupedExpertsConfig, LasonexConfig, LasonexLayerConfig,
                                                RetentionConfig, RotationConfig)

    z = LASONEX_SIZES[size]
    a, r = z["attention"], z["retention"]
    attention = DifferentialAttentionConfig(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["dim"] ** -0.5, 0.8,
                                            a["window"], RotationConfig(10000.0, a["dim"], ("yarn", 4.0, 4096.0, 32.0, 1.0)))
    decay = tuple(1.0 - 2.0 ** (-5.0 - 6.0 * h / max(1, r["heads"] - 1)) for h in range(r["heads"]))
    retention = RetentionConfig(r["heads"], r["dim"], r["vdim"], decay, RotationConfig(10000.0, r["dim"], None))
    dense = ClampedFeedForwardConfig(z["dense_ff"], 7.0)
    routed = GroupedExpertsConfig(z["experts"], z["top"], z["groups"][0], z["groups"][1], z["expert_ff"], 7.0)
    layers = []
    for i in range(z["layers"]):
        kind = i % 4
        if kind == 0:
            layers.append(LasonexLayerConfig("attention", attention, dense))
        elif kind == 1:
            layers.append(LasonexLayerConfig("retention", retention, routed))
        else:
            layers.append(LasonexLayerConfig("attention", attention, routed))
    return LasonexConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, embedding_scale=float(z["width"]) ** 0.5,
                         layers=tuple(layers))


def lasonex_decode_bytes(cfg, batch, context):
    """Bytes a decode step has to move: the weights it uses once in bfloat16 (of the experts, those that
    `batch` tokens can reach), every request's retention states read and written in float, and the cache
    rows (two key maps and a value per key/value head) inside each window."""
    from fastllm_py_b200.config.lasonex import GroupedExpertsConfig, RetentionConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        m = layer.mixer
        if isinstance(m, RetentionConfig):
            total += 2 * w * (2 * m.heads * m.dim + 3 * m.heads * m.vdim)
            total += batch * 2 * 4 * m.heads * m.vdim * m.dim
        else:
            total += 2 * w * (m.heads * 2 * m.dim + m.kv_heads * (2 * m.dim + m.vdim) + m.heads * m.vdim)
            total += batch * min(context, m.window or context) * m.kv_heads * (2 * m.dim + m.vdim) * 2
        f = layer.mlp
        if isinstance(f, GroupedExpertsConfig):
            total += 2 * 3 * w * f.ff * min(f.experts, batch * f.top) + 2 * w * f.experts
        elif f is not None:
            total += 2 * 3 * w * f.ff
    return total + 2 * w * cfg.vocab + 2 * batch * w


def lasonex_prefill_flops(cfg, tokens):
    """Matrix-product FLOPs of a prompt step (projections, feed-forwards, both attention maps over the window,
    head); the retention recurrence adds 4 dim vdim per head and token."""
    from fastllm_py_b200.config.lasonex import GroupedExpertsConfig, RetentionConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        m = layer.mixer
        if isinstance(m, RetentionConfig):
            total += 2 * tokens * w * (2 * m.heads * m.dim + 3 * m.heads * m.vdim) + tokens * m.heads * 4 * m.dim * m.vdim
        else:
            total += 2 * tokens * w * (m.heads * 2 * m.dim + m.kv_heads * (2 * m.dim + m.vdim) + m.heads * m.vdim)
            seen = sum(min(p + 1, m.window or p + 1) for p in range(tokens))
            total += 2 * m.heads * seen * 2 * (m.dim + m.vdim)
        f = layer.mlp
        if isinstance(f, GroupedExpertsConfig):
            total += 2 * tokens * (3 * w * f.ff * f.top + w * f.experts)
        elif f is not None:
            total += 2 * tokens * 3 * w * f.ff
    return total + 2 * w * cfg.vocab


def run_lasonex(args, warmup):
    """The Lasonex design beside the Tigitar hybrid and the dense decoder of equal width and depth, one JSON
    line: prompt steps of 512 and 2048 tokens and decode steps at batch 1 and 8 over 2048-token contexts, with
    each model's fraction of its own roofline (measured tensor peak for prompts, measured copy bandwidth for
    decode steps)."""
    from fastllm_py_b200 import LlamaConfig, Model

    pk = peaks()
    steps = max(8, min(args.steps, 32))
    out = {}
    sampler = ClockSampler().start()
    sampler.__enter__()
    for size in (args.size.split(",") if args.size else list(LASONEX_SIZES)):
        z, hz = LASONEX_SIZES[size], HYBRID_SIZES[size]
        llama = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                            num_layers=z["layers"], hidden_size=z["width"], vocab_size=z["vocab"], rope_theta=10000.0,
                            rms_norm_eps=1e-6, max_position_embeddings=4096, **hz["llama"])
        models = [("lasonex", lasonex_config(size), lasonex_prefill_flops, lasonex_decode_bytes),
                  ("hybrid", hybrid_config(size), hybrid_prefill_flops, hybrid_decode_bytes),
                  ("dense", llama, prefill_flops, decode_bytes)]
        res = {}
        for name, cfg, flops_of, bytes_of in models:
            if args.only and name not in args.only.split(","):
                continue
            model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=8 * (CONTEXT + 256),
                                      max_requests=8, max_batched_tokens=2048, max_model_len=4096,
                                      cuda_graph=not args.no_graph)
            r = {"prompt_step": {}, "decode": {}}
            for t in (512, 2048):
                ms, _ = time_prefill(model, t, 8, 3)
                r["prompt_step"][str(t)] = {"ms": round(ms, 3), "value": round(t * 1000.0 / ms, 1),
                                            "frac": round(flops_of(cfg, t) / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for b in (1, 8):
                v, ms, launches, _ = time_decode(model, b, steps, warmup, CONTEXT)
                ctx = CONTEXT + warmup + (steps + 1) / 2
                r["decode"][f"{b}x{CONTEXT}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                                                 "launches_per_step": launches // steps,
                                                 "frac": round(bytes_of(cfg, b, ctx) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            res[name] = r
            del model
            import gc

            import torch
            gc.collect()
            torch.cuda.empty_cache()
        out[size] = res
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt and decode steps of the Lasonex design beside the Tigitar hybrid and the dense decoder "
                  "of equal size, bf16",
        "n_gpus": 1, "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"sizes": {k: dict(LASONEX_SIZES[k]) for k in out}, "page_size": 16,
                   "peaks": pk["source"], "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"],
                   "cuda_graph": not args.no_graph},
        "sizes": out, "clocks": sampler.summary()}))
    return 0


SAKUSUN_SIZES = {
    # gated post-norm layers at the widths of HYBRID_SIZES: three latent-attention layers (queries through a latent of
    # their own, an output gate) to one windowed sink-attention layer, a dense gelu unit in every layer; the dense
    # Llama-style decoder of the same width, depth and feed-forward size is timed beside it
    "w2048": dict(width=2048, vocab=32256, layers=8, ff=5504, taps=3, buckets=100003,
                  attention=dict(heads=16, kv_heads=4, dim=128, vdim=128, window=1024, keep_first=64, bias_max=2048.0),
                  latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=768)),
    "w4096": dict(width=4096, vocab=32256, layers=4, ff=11008, taps=3, buckets=100003,
                  attention=dict(heads=32, kv_heads=8, dim=128, vdim=128, window=2048, keep_first=64, bias_max=4096.0),
                  latent=dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536)),
}


def sakusun_config(size):
    """A Sakusun configuration of `size`: layers cycle through latent attention, sink attention (blending its values
    with the first such layer's), latent attention, latent attention; a dense gelu unit in every layer."""
    from fastllm_py_b200.config.sakusun import (DenseConfig, QueryLatentAttentionConfig, SakusunConfig,
                                                SakusunLayerConfig, SinkAttentionConfig)

    z = SAKUSUN_SIZES[size]
    a, m = z["attention"], z["latent"]
    attention = SinkAttentionConfig(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["dim"] ** -0.5, 50.0, a["bias_max"],
                                    a["window"], a["keep_first"], True)
    latent = QueryLatentAttentionConfig(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"],
                                        (m["dim"] + m["rot_dim"]) ** -0.5, 10000.0)
    layers = [SakusunLayerConfig("attention", attention, DenseConfig(z["ff"])) if i % 4 == 1 else
              SakusunLayerConfig("latent_attention", latent, DenseConfig(z["ff"])) for i in range(z["layers"])]
    return SakusunConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, embedding_scale=1.0,
                         bigram_buckets=z["buckets"], bigram_mul_prev=31, bigram_mul_cur=7, taps=z["taps"],
                         layers=tuple(layers))


def sakusun_decode_bytes(cfg, batch, context):
    """Bytes a decode step has to move: the weights it uses once in bfloat16 (the gate matrices of the residual
    branches among them), the cache rows inside each window plus the kept first tokens, the latent rows of the whole
    context, and every request's kept convolution rows read and written in float."""
    from fastllm_py_b200.config.sakusun import SinkAttentionConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        m = layer.mixer
        subs = 1 if layer.mlp is None else 2
        total += subs * (2 * w * w + batch * 2 * 4 * max(cfg.taps - 1, 0) * w)
        if isinstance(m, SinkAttentionConfig):
            total += 2 * w * (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim) + m.heads * m.vdim)
            seen = min(context, (m.window + m.keep_first) if m.window else context)
            total += batch * seen * m.kv_heads * (m.dim + m.vdim) * 2
        else:
            total += 2 * (w * (m.q_rank + m.kv_rank + m.rot_dim + m.heads * m.vdim) + m.q_rank * m.heads * (m.dim + m.rot_dim)
                          + m.heads * m.kv_rank * (m.dim + m.vdim) + m.heads * m.vdim * w)
            total += batch * context * (m.kv_rank + m.rot_dim) * 2
        if layer.mlp is not None:
            total += 2 * 3 * w * layer.mlp.ff
    return total + 2 * w * cfg.vocab + 2 * batch * w


def sakusun_prefill_flops(cfg, tokens):
    """Matrix-product FLOPs of a prompt step: projections, residual gates, feed-forwards, sink attention over the
    window and the kept tokens, latent attention in latent space over every earlier token, head."""
    from fastllm_py_b200.config.sakusun import SinkAttentionConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        m = layer.mixer
        subs = 1 if layer.mlp is None else 2
        total += subs * 2 * tokens * w * w
        if isinstance(m, SinkAttentionConfig):
            total += 2 * tokens * w * (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim) + m.heads * m.vdim)
            seen = sum(min(p + 1, (m.window + m.keep_first) if m.window else p + 1) for p in range(tokens))
            total += 2 * m.heads * seen * (m.dim + m.vdim)
        else:
            total += 2 * tokens * (w * (m.q_rank + m.kv_rank + m.rot_dim + m.heads * m.vdim)
                                   + m.q_rank * m.heads * (m.dim + m.rot_dim) + m.heads * m.kv_rank * (m.dim + m.vdim)
                                   + m.heads * m.vdim * w)
            seen = sum(p + 1 for p in range(tokens))
            total += 2 * m.heads * seen * (2 * m.kv_rank + m.rot_dim)
        if layer.mlp is not None:
            total += 2 * tokens * 3 * w * layer.mlp.ff
    return total + 2 * w * cfg.vocab


def run_sakusun(args, warmup):
    """The Sakusun design beside the Tigitar hybrid (the model that shares its latent attention) and the dense decoder
    of equal width, depth and feed-forward size, one JSON line: prompt steps of 512 and 2048 tokens and decode steps at
    batch 1 and 8 over 2048-token contexts, with each model's fraction of its own roofline (measured tensor peak for
    prompts, measured copy bandwidth for decode steps)."""
    from fastllm_py_b200 import LlamaConfig, Model

    pk = peaks()
    steps = max(8, min(args.steps, 32))
    out = {}
    sampler = ClockSampler().start()
    sampler.__enter__()
    for size in (args.size.split(",") if args.size else list(SAKUSUN_SIZES)):
        z, hz = SAKUSUN_SIZES[size], HYBRID_SIZES[size]
        llama = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                            num_layers=z["layers"], hidden_size=z["width"], vocab_size=z["vocab"], rope_theta=10000.0,
                            rms_norm_eps=1e-6, max_position_embeddings=4096, **hz["llama"])
        models = [("sakusun", sakusun_config(size), sakusun_prefill_flops, sakusun_decode_bytes),
                  ("hybrid", hybrid_config(size), hybrid_prefill_flops, hybrid_decode_bytes),
                  ("dense", llama, prefill_flops, decode_bytes)]
        res = {}
        for name, cfg, flops_of, bytes_of in models:
            if args.only and name not in args.only.split(","):
                continue
            model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=8 * (CONTEXT + 256),
                                      max_requests=8, max_batched_tokens=2048, max_model_len=4096,
                                      cuda_graph=not args.no_graph)
            r = {"prompt_step": {}, "decode": {}}
            for t in (512, 2048):
                ms, _ = time_prefill(model, t, 8, 3)
                r["prompt_step"][str(t)] = {"ms": round(ms, 3), "value": round(t * 1000.0 / ms, 1),
                                            "frac": round(flops_of(cfg, t) / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for b in (1, 8):
                v, ms, launches, _ = time_decode(model, b, steps, warmup, CONTEXT)
                ctx = CONTEXT + warmup + (steps + 1) / 2
                r["decode"][f"{b}x{CONTEXT}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                                                 "launches_per_step": launches // steps,
                                                 "frac": round(bytes_of(cfg, b, ctx) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            res[name] = r
            del model
            import gc

            import torch
            gc.collect()
            torch.cuda.empty_cache()
        out[size] = res
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt and decode steps of the Sakusun design beside the Tigitar hybrid and the dense decoder "
                  "of equal size, bf16",
        "n_gpus": 1, "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"sizes": {k: dict(SAKUSUN_SIZES[k]) for k in out}, "page_size": 16,
                   "peaks": pk["source"], "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"],
                   "cuda_graph": not args.no_graph},
        "sizes": out, "clocks": sampler.summary()}))
    return 0


SABERAX_SIZES = {
    # pre-norm layers of attention beside a recurrent mixer at the widths of HYBRID_SIZES; layers cycle through
    # attention + recurrent unit with a dense unit, windowed attention + gated linear attention with routed experts,
    # the same with a dense unit, chunked attention with routed experts.  The Lasonex design (windowed attention and a
    # linear-attention state in parallel layers, grouped experts) and the dense Llama-style decoder of the same width
    # and depth are timed beside it
    "w2048": dict(width=2048, vocab=32256, layers=8, attention=dict(heads=16, kv_heads=4, dim=128, vdim=128, window=1024),
                  recurrent=dict(width=2048, blocks=8, conv=4), linear=dict(heads=16, dim=64, vdim=128, tau=16.0),
                  dense_ff=5504, experts=32, top=4, expert_ff=1408, shared_ff=1408, groups=(8, 4)),
    "w4096": dict(width=4096, vocab=32256, layers=4, attention=dict(heads=32, kv_heads=8, dim=128, vdim=128, window=2048),
                  recurrent=dict(width=4096, blocks=16, conv=4), linear=dict(heads=32, dim=64, vdim=128, tau=16.0),
                  dense_ff=11008, experts=16, top=2, expert_ff=5504, shared_ff=5504, groups=(4, 2)),
}


def saberax_config(size):
    from fastllm_py_b200.config.saberax import (AttentionConfig, DenseConfig, ExpertsConfig, GatedLinearAttentionConfig,
                                                PairConfig, RecurrentUnitConfig, RotationConfig, SaberaxConfig,
                                                SaberaxLayerConfig)

    z = SABERAX_SIZES[size]
    a, r, g = z["attention"], z["recurrent"], z["linear"]
    sizes = (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["dim"] ** -0.5)
    normed = AttentionConfig("normed", *sizes, None, None, (0.3, 128))
    windowed = AttentionConfig("windowed", *sizes, a["window"], RotationConfig(10000.0, 64, ("yarn", 4.0, 4096.0, 32.0, 1.0)), None)
    chunked = AttentionConfig("chunked", *sizes, a["window"], RotationConfig(250000.0, a["dim"], ("bands", 4.0, 2048.0, 1.0, 4.0)), None)
    first = PairConfig(normed, RecurrentUnitConfig(r["width"], r["blocks"], r["conv"]))
    second = PairConfig(windowed, GatedLinearAttentionConfig(g["heads"], g["dim"], g["vdim"], g["tau"]))
    dense = DenseConfig(z["dense_ff"])
    routed = ExpertsConfig(z["experts"], z["top"], 2.0, z["groups"][0], z["groups"][1], z["expert_ff"], z["shared_ff"])
    cycle = [("parallel", first, dense), ("parallel_2", second, routed), ("parallel_2", second, dense), ("attention", chunked, routed)]
    layers = tuple(SaberaxLayerConfig(*cycle[i % 4], None) for i in range(z["layers"]))
    return SaberaxConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-5, residual_mult=0.7, layers=layers)


def _saberax_layer_sizes(layer, w):
    """(weight elements a token's mixer products touch, state floats per request, [(attention config, reach)])."""
    from fastllm_py_b200.config.saberax import AttentionConfig, GatedLinearAttentionConfig, RecurrentUnitConfig

    def attention(m):
        v = 0 if m.role == "chunked" else m.kv_heads * m.vdim
        return w * (m.heads * m.dim + m.kv_heads * m.dim + v + m.heads * m.vdim + (m.heads if m.role == "chunked" else 0))

    m = layer.mixer
    if isinstance(m, AttentionConfig):
        return attention(m), 0, [m]
    weights, state = attention(m.left), 0
    r = m.right
    if isinstance(r, RecurrentUnitConfig):
        weights += 3 * w * r.width + 2 * r.width * (r.width // r.blocks)
        state = r.width * r.conv
    elif isinstance(r, GatedLinearAttentionConfig):
        weights += w * (2 * r.heads * r.dim + 3 * r.heads * r.vdim + r.rank) + r.heads * r.dim * r.rank
        state = r.heads * r.dim * r.vdim
    return weights, state, [m.left]


def saberax_decode_bytes(cfg, batch, context):
    """Bytes a decode step has to move: the weights it uses once in bfloat16 (of the experts, those that `batch`
    tokens can reach), every request's recurrent states read and written in float, and the cache rows that each
    attention sees (all of them, the window's, or on average half a chunk's)."""
    from fastllm_py_b200.config.saberax import ExpertsConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        weights, state, attentions = _saberax_layer_sizes(layer, w)
        total += 2 * weights + batch * 2 * 4 * state
        for m in attentions:
            seen = context if m.mask is None else min(context, m.mask) / (2 if m.role == "chunked" else 1)
            total += batch * seen * m.kv_heads * (m.dim + m.vdim) * 2
        f = layer.mlp
        if isinstance(f, ExpertsConfig):
            total += 2 * 2 * w * f.ff * min(f.experts, batch * f.top) + 2 * w * f.experts + 2 * 2 * w * (f.shared_ff or 0)
        elif f is not None:
            total += 2 * 3 * w * f.ff
    return total + 2 * w * cfg.vocab + 2 * batch * w


def saberax_prefill_flops(cfg, tokens):
    """Matrix-product FLOPs of a prompt step (projections, gates of the recurrent unit, feed-forwards, attention over what
    each query sees, head); the linear attention's recurrence adds 4 dim vdim per head and token."""
    from fastllm_py_b200.config.saberax import ExpertsConfig, GatedLinearAttentionConfig, PairConfig

    w, total = cfg.width, 0
    for layer in cfg.layers:
        weights, _, attentions = _saberax_layer_sizes(layer, w)
        total += 2 * tokens * weights
        if isinstance(layer.mixer, PairConfig) and isinstance(layer.mixer.right, GatedLinearAttentionConfig):
            r = layer.mixer.right
            total += tokens * r.heads * 4 * r.dim * r.vdim
        for m in attentions:
            if m.role == "chunked" and m.mask:
                seen = sum(p % m.mask + 1 for p in range(tokens))
            else:
                seen = sum(min(p + 1, m.mask or p + 1) for p in range(tokens))
            total += 2 * m.heads * seen * (m.dim + m.vdim)
        f = layer.mlp
        if isinstance(f, ExpertsConfig):
            total += 2 * tokens * (2 * w * f.ff * f.top + w * f.experts + 2 * w * (f.shared_ff or 0))
        elif f is not None:
            total += 2 * tokens * 3 * w * f.ff
    return total + 2 * w * cfg.vocab


def run_saberax(args, warmup):
    """The Saberax design beside the Lasonex design (the closest model: windowed attention and a recurrent state side
    by side in every layer, grouped experts) and the dense decoder of equal width and depth, one JSON line: prompt steps
    of 512 and 2048 tokens and decode steps at batch 1 and 8 over 2048-token contexts, with each model's fraction of its
    own roofline (measured tensor peak for prompts, measured copy bandwidth for decode steps)."""
    from fastllm_py_b200 import LlamaConfig, Model

    pk = peaks()
    steps = max(8, min(args.steps, 32))
    out = {}
    sampler = ClockSampler().start()
    sampler.__enter__()
    for size in (args.size.split(",") if args.size else list(SABERAX_SIZES)):
        z, hz = SABERAX_SIZES[size], HYBRID_SIZES[size]
        llama = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                            num_layers=z["layers"], hidden_size=z["width"], vocab_size=z["vocab"], rope_theta=10000.0,
                            rms_norm_eps=1e-6, max_position_embeddings=4096, **hz["llama"])
        models = [("saberax", saberax_config(size), saberax_prefill_flops, saberax_decode_bytes),
                  ("lasonex", lasonex_config(size), lasonex_prefill_flops, lasonex_decode_bytes),
                  ("dense", llama, prefill_flops, decode_bytes)]
        res = {}
        for name, cfg, flops_of, bytes_of in models:
            if args.only and name not in args.only.split(","):
                continue
            model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=8 * (CONTEXT + 256),
                                      max_requests=8, max_batched_tokens=2048, max_model_len=4096,
                                      cuda_graph=not args.no_graph)
            r = {"prompt_step": {}, "decode": {}}
            for t in (512, 2048):
                ms, _ = time_prefill(model, t, 8, 3)
                r["prompt_step"][str(t)] = {"ms": round(ms, 3), "value": round(t * 1000.0 / ms, 1),
                                            "frac": round(flops_of(cfg, t) / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for b in (1, 8):
                v, ms, launches, _ = time_decode(model, b, steps, warmup, CONTEXT)
                ctx = CONTEXT + warmup + (steps + 1) / 2
                r["decode"][f"{b}x{CONTEXT}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                                                 "launches_per_step": launches // steps,
                                                 "frac": round(bytes_of(cfg, b, ctx) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            res[name] = r
            del model
            import gc

            import torch
            gc.collect()
            torch.cuda.empty_cache()
        out[size] = res
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt and decode steps of the Saberax design beside the Lasonex design and the dense decoder "
                  "of equal size, bf16",
        "n_gpus": 1, "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"sizes": {k: dict(SABERAX_SIZES[k]) for k in out}, "page_size": 16,
                   "peaks": pk["source"], "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"],
                   "cuda_graph": not args.no_graph},
        "sizes": out, "clocks": sampler.summary()}))
    return 0


LUFOZEN_SIZES = {
    # pre-norm layers at the widths of HYBRID_SIZES: six layers of which two run twice, so eight runs, as many as the other
    # designs have layers.  The unit without a gate is as large as their gated ones.  The Saberax design (attention beside a
    # recurrent mixer in pre-norm layers) and the dense Llama-style decoder of the same width and depth are timed beside it
    "w2048": dict(width=2048, vocab=32256, attention=dict(heads=16, kv_heads=4, dim=128, vdim=128, conv=4),
                  linear=dict(heads=16, dim=64, vdim=128, tau=16.0),
                  state_space=dict(heads=64, vdim=64, state=128, groups=2, conv=4), ff=8192, runs=8),
    "w4096": dict(width=4096, vocab=32256, attention=dict(heads=32, kv_heads=8, dim=128, vdim=128, conv=4),
                  linear=dict(heads=32, dim=64, vdim=128, tau=16.0),
                  state_space=dict(heads=128, vdim=64, state=128, groups=4, conv=4), ff=16384, runs=4),
}


def lufozen_config(size):
    from fastllm_py_b200.config.lufozen import (AttentionConfig, DenseConfig, GatedLinearAttentionConfig, LoopConfig,
                                                LufozenConfig, LufozenLayerConfig, PairConfig, RotationConfig, StateSpaceConfig)

    z = LUFOZEN_SIZES[size]
    a, g, r = z["attention"], z["linear"], z["state_space"]
    sizes = (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["dim"] ** -0.5)
    rot = RotationConfig(500000.0, a["dim"], (8.0, 8192.0, 1.0, 4.0))
    lone = ("attention", AttentionConfig(*sizes, rot, a["conv"]))
    pair = ("parallel", PairConfig(AttentionConfig(*sizes, rot),
                                   StateSpaceConfig(r["heads"], r["vdim"], r["state"], r["groups"], r["conv"], r["groups"]), 0.7, 0.4))
    linear = ("gla", GatedLinearAttentionConfig(g["heads"], g["dim"], g["vdim"], g["tau"]))
    if z["runs"] == 8:
        kinds, loop = [lone, pair, linear, pair, lone, linear], LoopConfig(1, 3, 2)
    else:
        kinds, loop = [lone, pair, linear], LoopConfig(1, 2, 2)
    layers = tuple(LufozenLayerConfig(*k, DenseConfig(z["ff"])) for k in kinds)
    return LufozenConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-5, embedding_scale=8.0, bigram_buckets=65521,
                         bigram_mul_prev=17, bigram_mul_cur=5, logit_scale=0.5, loop=loop, layers=layers)


def _lufozen_layer_sizes(layer, w):
    """(weight elements a token's mixer products touch, state floats per request, [attention config], [(dim, vdim of a
    recurrence's state per head, heads)])."""
    from fastllm_py_b200.config.lufozen import AttentionConfig, GatedLinearAttentionConfig

    def attention(m):
        lone = m.conv is not None
        return w * (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim) + m.heads * m.vdim * (2 if lone else 1))

    m = layer.mixer
    if isinstance(m, AttentionConfig):
        return attention(m), (m.conv - 1) * (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)), [m], []
    if isinstance(m, GatedLinearAttentionConfig):
        weights = w * (2 * m.heads * m.dim + 3 * m.heads * m.vdim + m.rank) + m.heads * m.dim * m.rank
        return weights, m.heads * m.dim * m.vdim, [], [(m.dim, m.vdim, m.heads)]
    r = m.right
    inner, channels = r.heads * r.vdim, r.heads * r.vdim + 2 * r.groups * r.state
    weights = attention(m.left) + w * (2 * inner + channels + r.heads)
    return weights, inner * r.state + (r.conv - 1) * channels, [m.left], [(r.state, r.vdim, r.heads)]


def lufozen_decode_bytes(cfg, batch, context):
    """Bytes a decode step has to move: every run's weights in bfloat16 (a layer that runs twice is read twice), every
    request's states read and written in float, and the cache rows that the attentions see."""
    w, total = cfg.width, 0
    for i, _ in cfg.running_order():
        layer = cfg.layers[i]
        weights, state, attentions, _ = _lufozen_layer_sizes(layer, w)
        total += 2 * weights + batch * 2 * 4 * state
        for m in attentions:
            total += batch * context * m.kv_heads * (m.dim + m.vdim) * 2
        if layer.mlp is not None:
            total += 2 * 2 * w * layer.mlp.ff
    return total + 2 * w * cfg.vocab + 2 * batch * w * 2


def lufozen_prefill_flops(cfg, tokens):
    """Matrix-product FLOPs of a prompt step (projections, feed-forwards, attention, head) and 4 per state element and token
    of the two recurrences."""
    w, total = cfg.width, 0
    for i, _ in cfg.running_order():
        layer = cfg.layers[i]
        weights, _, attentions, states = _lufozen_layer_sizes(layer, w)
        total += 2 * tokens * weights
        for dim, vdim, heads in states:
            total += tokens * heads * 4 * dim * vdim
        for m in attentions:
            total += 2 * m.heads * (tokens * (tokens + 1) // 2) * (m.dim + m.vdim)
        if layer.mlp is not None:
            total += 2 * tokens * 2 * w * layer.mlp.ff
    return total + 2 * w * cfg.vocab


def run_lufozen(args, warmup):
    """The Lufozen design beside the Saberax design (the closest model: attention beside a recurrent mixer in pre-norm layers)
    and the dense decoder of equal width and number of layer runs, one JSON line: prompt steps of 512 and 2048 tokens and
    decode steps at batch 1 and 8 over 2048-token contexts, with each model's fraction of its own roofline (measured tensor
    peak for prompts, measured copy bandwidth for decode steps)."""
    from fastllm_py_b200 import LlamaConfig, Model

    pk = peaks()
    steps = max(8, min(args.steps, 32))
    out = {}
    sampler = ClockSampler().start()
    sampler.__enter__()
    for size in (args.size.split(",") if args.size else list(LUFOZEN_SIZES)):
        z, hz = LUFOZEN_SIZES[size], HYBRID_SIZES[size]
        llama = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                            num_layers=z["runs"], hidden_size=z["width"], vocab_size=z["vocab"], rope_theta=10000.0,
                            rms_norm_eps=1e-6, max_position_embeddings=4096, **hz["llama"])
        models = [("lufozen", lufozen_config(size), lufozen_prefill_flops, lufozen_decode_bytes),
                  ("saberax", saberax_config(size), saberax_prefill_flops, saberax_decode_bytes),
                  ("dense", llama, prefill_flops, decode_bytes)]
        res = {}
        for name, cfg, flops_of, bytes_of in models:
            if args.only and name not in args.only.split(","):
                continue
            model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=8 * (CONTEXT + 256),
                                      max_requests=8, max_batched_tokens=2048, max_model_len=4096,
                                      cuda_graph=not args.no_graph)
            r = {"prompt_step": {}, "decode": {}}
            for t in (512, 2048):
                ms, _ = time_prefill(model, t, 8, 3)
                r["prompt_step"][str(t)] = {"ms": round(ms, 3), "value": round(t * 1000.0 / ms, 1),
                                            "frac": round(flops_of(cfg, t) / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for b in (1, 8):
                v, ms, launches, _ = time_decode(model, b, steps, warmup, CONTEXT)
                ctx = CONTEXT + warmup + (steps + 1) / 2
                r["decode"][f"{b}x{CONTEXT}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                                                 "launches_per_step": launches // steps,
                                                 "frac": round(bytes_of(cfg, b, ctx) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            res[name] = r
            del model
            import gc

            import torch
            gc.collect()
            torch.cuda.empty_cache()
        out[size] = res
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt and decode steps of the Lufozen design beside the Saberax design and the dense decoder "
                  "of equal size, bf16",
        "n_gpus": 1, "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"sizes": {k: dict(LUFOZEN_SIZES[k]) for k in out}, "page_size": 16,
                   "peaks": pk["source"], "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"],
                   "cuda_graph": not args.no_graph},
        "sizes": out, "clocks": sampler.summary()}))
    return 0


KERIRAX_SIZES = {
    # parallel layers at the widths of HYBRID_SIZES with its latent attention, unit and experts, so many runs as the other
    # designs have layers (some layers run twice).  The Lufozen design (attention beside a state-space recurrence in looped
    # layers), the Tigitar hybrid (latent attention and experts) and the dense decoder are timed beside it
    "w2048": dict(width=2048, vocab=32256, attention=dict(heads=16, kv_heads=4, dim=128, vdim=128),
                  scan=dict(inner=4096, state=16, dt_rank=128, conv=4), q_rank=1024, runs=8),
    "w4096": dict(width=4096, vocab=32256, attention=dict(heads=32, kv_heads=8, dim=128, vdim=128),
                  scan=dict(inner=8192, state=16, dt_rank=256, conv=4), q_rank=1536, runs=4),
}


def kerirax_config(size):
    from fastllm_py_b200.config.kerirax import (AttentionConfig, DenseConfig, ExpertsConfig, KeriraxConfig, KeriraxLayerConfig,
                                                LatentConfig, LoopConfig, PairConfig, RotationConfig, SelectiveScanConfig)

    z, hz = KERIRAX_SIZES[size], HYBRID_SIZES[size]
    a, r, m = z["attention"], z["scan"], hz["latent"]
    pair = PairConfig(AttentionConfig(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["dim"] ** -0.5,
                                      RotationConfig(500000.0, a["dim"], 4.0)),
                      SelectiveScanConfig(r["inner"], r["state"], r["dt_rank"], r["conv"]), 0.7, 0.4)
    latent = LatentConfig(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], z["q_rank"],
                          (m["dim"] + m["rot_dim"]) ** -0.5, RotationConfig(10000.0, m["rot_dim"], None))
    dense, experts = DenseConfig(hz["dense_ff"]), ExpertsConfig(hz["experts"], hz["top"], hz["expert_ff"], 7.0)
    if z["runs"] == 8:
        kinds = [(pair, dense), (latent, experts), (pair, dense), (pair, experts), (latent, dense), (pair, dense)]
        loop = LoopConfig(1, 3, 2)
    else:
        kinds, loop = [(pair, dense), (latent, experts), (pair, dense)], LoopConfig(1, 2, 2)
    layers = tuple(KeriraxLayerConfig("parallel" if m is pair else "latent_attention", m, f) for m, f in kinds)
    return KeriraxConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-5, embedding_scale=8.0, logit_softcap=30.0, loop=loop,
                         layers=layers)


def _kerirax_run_sizes(layer, w):
    """(weight elements a token's mixer products touch, state floats per request, cache elements per token, attention FLOPs
    per query and key, state elements)."""
    from fastllm_py_b200.config.kerirax import LatentConfig

    m = layer.mixer
    if isinstance(m, LatentConfig):
        weights = w * (m.q_rank + m.kv_rank + m.rot_dim + m.heads * m.vdim) + m.q_rank * m.heads * (m.dim + m.rot_dim) + \
            m.kv_rank * m.heads * (m.dim + m.vdim)
        return weights, 0, m.kv_rank + m.rot_dim, 2 * m.heads * (2 * m.kv_rank + m.rot_dim), 0
    a, r = m.left, m.right
    weights = w * (a.heads * (a.dim + a.vdim + 1) + a.kv_heads * (a.dim + a.vdim) + 3 * r.inner) + \
        r.inner * (2 * r.dt_rank + 2 * r.state)
    return (weights, r.inner * (r.state + r.conv - 1), a.kv_heads * (a.dim + a.vdim), 2 * a.heads * (a.dim + a.vdim),
            r.inner * r.state)


def kerirax_decode_bytes(cfg, batch, context):
    """Bytes a decode step has to move: every run's weights in bfloat16 (of the experts those that the batch's tokens can
    reach), every request's states read and written in float, the cache rows that the attentions see."""
    from fastllm_py_b200.config.kerirax import ExpertsConfig

    w, total = cfg.width, 0
    for i, started in cfg.running_order():
        layer = cfg.layers[i]
        weights, state, cached, _, _ = _kerirax_run_sizes(layer, w)
        total += 2 * weights + batch * (2 * 4 * state + 2 * context * cached)
        if started is not None:
            total += 2 * 2 * w * w
        f = layer.mlp
        if isinstance(f, ExpertsConfig):
            total += 2 * (w * f.experts + min(f.experts, batch * f.top) * 3 * w * f.ff)
        elif f is not None:
            total += 2 * 3 * w * f.ff
    return total + 2 * w * cfg.vocab + 2 * batch * w


def kerirax_prefill_flops(cfg, tokens):
    """Matrix-product FLOPs of a prompt step (projections, feed-forwards, attention in latent space where it runs there, head)
    and 6 per state element and token of the recurrence."""
    from fastllm_py_b200.config.kerirax import ExpertsConfig

    w, total = cfg.width, 0
    for i, started in cfg.running_order():
        layer = cfg.layers[i]
        weights, _, _, attention, states = _kerirax_run_sizes(layer, w)
        total += 2 * tokens * weights + attention * (tokens * (tokens + 1) // 2) + 6 * tokens * states
        if started is not None:
            total += 2 * tokens * 2 * w * w
        f = layer.mlp
        if isinstance(f, ExpertsConfig):
            total += 2 * tokens * (w * f.experts + f.top * 3 * w * f.ff)
        elif f is not None:
            total += 2 * tokens * 3 * w * f.ff
    return total + 2 * w * cfg.vocab


def run_kerirax(args, warmup):
    """The Kerirax design beside the Lufozen design, the Tigitar hybrid and the dense decoder of equal width and number of layer
    runs, one JSON line: prompt steps of 512 and 2048 tokens and decode steps at batch 1 and 8 over 2048-token contexts, with
    each model's fraction of its own roofline (measured tensor peak for prompts, measured copy bandwidth for decode steps)."""
    import gc

    import torch

    from fastllm_py_b200 import LlamaConfig, Model

    pk = peaks()
    steps = max(8, min(args.steps, 32))
    out = {}
    sampler = ClockSampler().start()
    sampler.__enter__()
    for size in (args.size.split(",") if args.size else list(KERIRAX_SIZES)):
        z, hz = KERIRAX_SIZES[size], HYBRID_SIZES[size]
        llama = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                            num_layers=z["runs"], hidden_size=z["width"], vocab_size=z["vocab"], rope_theta=10000.0,
                            rms_norm_eps=1e-6, max_position_embeddings=4096, **hz["llama"])
        models = [("kerirax", kerirax_config(size), kerirax_prefill_flops, kerirax_decode_bytes),
                  ("lufozen", lufozen_config(size), lufozen_prefill_flops, lufozen_decode_bytes),
                  ("hybrid", hybrid_config(size), hybrid_prefill_flops, hybrid_decode_bytes),
                  ("dense", llama, prefill_flops, decode_bytes)]
        res = {}
        for name, cfg, flops_of, bytes_of in models:
            if args.only and name not in args.only.split(","):
                continue
            model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=8 * (CONTEXT + 256),
                                      max_requests=8, max_batched_tokens=2048, max_model_len=4096,
                                      cuda_graph=not args.no_graph)
            r = {"prompt_step": {}, "decode": {}}
            for t in (512, 2048):
                ms, _ = time_prefill(model, t, 8, 3)
                r["prompt_step"][str(t)] = {"ms": round(ms, 3), "value": round(t * 1000.0 / ms, 1),
                                            "frac": round(flops_of(cfg, t) / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for b in (1, 8):
                v, ms, launches, _ = time_decode(model, b, steps, warmup, CONTEXT)
                ctx = CONTEXT + warmup + (steps + 1) / 2
                r["decode"][f"{b}x{CONTEXT}"] = {"ms_per_step": round(ms, 3), "value": round(v, 1),
                                                 "launches_per_step": launches // steps,
                                                 "frac": round(bytes_of(cfg, b, ctx) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            res[name] = r
            del model
            gc.collect()
            torch.cuda.empty_cache()
        out[size] = res
    sampler.__exit__()
    print(json.dumps({
        "metric": "prompt and decode steps of the Kerirax design beside the Lufozen design, the Tigitar hybrid and the dense "
                  "decoder of equal size, bf16",
        "n_gpus": 1, "dtype": "bf16", "data": "synthetic", "impl": "ours", "steps": steps, "warmup": warmup,
        "config": {"sizes": {k: dict(KERIRAX_SIZES[k]) for k in out}, "page_size": 16,
                   "peaks": pk["source"], "hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"],
                   "cuda_graph": not args.no_graph},
        "sizes": out, "clocks": sampler.summary()}))
    return 0


def reference_cpu_path(ref_root, layers=1, context=256, decode_tokens=8):
    """fastllm-py's own NumPy model code (its CPU device, float32) timed at DeepSeek-LLM-7B layer
    sizes: `layers` of the 30 layers, one sequence (that path has no batch), a `context`-token
    prompt through Model.forward and `decode_tokens` greedy tokens one by one.  The package imports
    CuPy inside its functions; a stand-in module that maps the few names it uses onto NumPy lets
    the CPU path run where CuPy is absent (its GPU path cannot)."""
    import tempfile
    import types

    import numpy as np

    from fastllm_py_b200 import LlamaConfig
    from fastllm_py_b200.weights import write_model_folder

    if "cupy" not in sys.modules:
        cp = types.ModuleType("cupy")
        cp.ndarray = type("ndarray", (), {})
        cp.asnumpy = lambda x: np.asarray(x)
        cp.asarray = lambda x: np.asarray(x)
        cp.float32, cp.float16 = np.float32, np.float16
        sys.modules["cupy"] = cp
    sys.path.insert(0, str(ref_root))
    from fastllm_py import DeviceMap, Model

    cfg = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                      **dict(MODEL_7B, num_layers=layers))
    with tempfile.TemporaryDirectory() as tmp:
        folder = write_model_folder(cfg, Path(tmp) / "model", seed=0, std=0.02, norm_std=0.02)
        model = Model.load(str(folder), DeviceMap({"cpu": 1}), dtype="float32")
        ids = np.random.default_rng(7).integers(0, cfg.vocab_size, size=context).astype(np.int64)
        t0 = time.perf_counter()
        logits, kvs = model.forward(ids)
        prefill_s = time.perf_counter() - t0
        nxt = int(np.asarray(logits[-1]).argmax())
        times = []
        for _ in range(decode_tokens):
            t0 = time.perf_counter()
            logits, kvs = model.forward(np.asarray([nxt]), kvs)
            nxt = int(np.asarray(logits[-1]).argmax())
            times.append(time.perf_counter() - t0)
    return {"device": "cpu (NumPy path of the reference, float32)", "layers": layers,
            "layers_of_config": MODEL_7B["num_layers"], "batch": 1, "context": context,
            "prefill_tok_s": round(context / prefill_s, 1),
            "decode_tok_s": round(1.0 / statistics.median(times), 2)}


def run_reference(args):
    """The reference arm: codemk8/fastllm-py as installed under baseline/_ref, through its own API.
    Its GPU path is CuPy (RawKernel, cuBLAS through cupy): it is tried whenever `import cupy` works;
    where it does not, the line says so (and, with --reference-cpu, carries the timing of the
    reference's CPU path at one layer of the same sizes, for scale: no ratio is meant by it)."""
    ref_root = ROOT / "baseline" / "_ref"
    if not (ref_root / "fastllm_py").is_dir():
        print(json.dumps({"impl": "reference", "unavailable": "fastllm-py is not installed under baseline/_ref "
                          "(pip install --no-index --no-deps --target baseline/_ref of a copy of the reference)"}))
        return 0
    try:
        import cupy  # noqa: F401
        have_cupy = True
    except Exception as e:                                   # noqa: BLE001
        have_cupy, why = False, f"{type(e).__name__}: {e}"
    if not have_cupy:
        line = {"impl": "reference", "unavailable":
                "fastllm-py's GPU path needs CuPy (cupy-cuda12x), which cannot be imported here "
                f"({why}) and is not in the offline wheelhouse; the package itself installs with --no-deps"}
        if args.reference_cpu:
            try:
                line["cpu_path"] = reference_cpu_path(ref_root)
            except Exception as e:                           # noqa: BLE001
                line["cpu_path"] = {"failed": f"{type(e).__name__}: {e}"}
        print(json.dumps(line))
        return 0
    return run_reference_gpu(args, ref_root)


def run_reference_gpu(args, ref_root):
    """With CuPy at hand: the reference's own batched decoder (fastllm_py/batched.py:96-275) at the
    headline shape in float16 (it has no bfloat16), random weights written to a model folder."""
    import tempfile

    import numpy as np

    from fastllm_py_b200 import LlamaConfig
    from fastllm_py_b200.weights import write_model_folder

    sys.path.insert(0, str(ref_root))
    try:
        import cupy as cp
        from fastllm_py import DeviceMap, Model
        from fastllm_py.batched import BatchedDecoder

        layers = args.layers or MODEL_7B["num_layers"]
        cfg = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                          **dict(MODEL_7B, num_layers=layers))
        warmup = max(3, args.warmup)
        with tempfile.TemporaryDirectory() as tmp:
            folder = write_model_folder(cfg, Path(tmp) / "model", seed=0, std=0.02, norm_std=0.02)
            model = Model.load(str(folder), DeviceMap({"cuda:0": 1}), dtype="float16")
        rng = np.random.default_rng(8)
        prompts = [rng.integers(0, cfg.vocab_size, size=CONTEXT).astype(np.int64) for _ in range(args.batch)]
        dec = BatchedDecoder(model, args.batch, max_len=CONTEXT + warmup + args.steps + 8)
        dec.prime(prompts)
        tokens = np.zeros(args.batch, dtype=np.int64)
        for _ in range(warmup):
            dec.step(tokens)
        cp.cuda.Device().synchronize()
        start, stop = cp.cuda.Event(), cp.cuda.Event()
        start.record()
        for _ in range(args.steps):
            dec.step(tokens)
        stop.record()
        stop.synchronize()
        ms = cp.cuda.get_elapsed_time(start, stop) / args.steps
        print(json.dumps({"impl": "reference", "metric": "decode tok/s @ batch 8, 2048-token context, DeepSeek-LLM-7B",
                          "value": round(args.batch * 1000.0 / ms, 2), "unit": "tokens/s", "n_gpus": 1,
                          "steps": args.steps, "warmup": warmup, "ms_per_step": round(ms, 4),
                          "higher_is_better": True, "dtype": "fp16", "data": "synthetic",
                          "config": {"model": "DeepSeek-LLM-7B size, random weights", "global_batch": args.batch,
                                     "seq_len": CONTEXT, "layers": layers,
                                     "layers_of_config": MODEL_7B["num_layers"]}}))
    except Exception as e:                                   # noqa: BLE001
        print(json.dumps({"impl": "reference", "unavailable": f"the reference's GPU path failed: {type(e).__name__}: {e}"}))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=None,
                    help="run fewer layers of the same sizes (the line names both numbers)")
    ap.add_argument("--no-points", action="store_true", help="skip batch 1 / 64 and the prefill")
    ap.add_argument("--no-graph", action="store_true")
    ap.add_argument("--workload", default="decode", choices=["decode", "serve", "67b", "tables", "hybrid", "lasonex", "sakusun", "saberax", "lufozen",
                                                              "kerirax"],
                    help="decode: the headline line (DeepSeek-LLM-7B size); serve: continuous batching at "
                         "deepseek-coder-1.3b size; 67b: prompt and decode steps at deepseek-llm-67b size")
    ap.add_argument("--size", default="", help="hybrid, lasonex, sakusun, saberax, lufozen, kerirax: which sizes (w2048,w4096; default both)")
    ap.add_argument("--only", default="", help="lasonex, sakusun, saberax, lufozen, kerirax: which of the models timed side by side (the design's name, hybrid, dense, ...)")
    ap.add_argument("--requests", type=int, default=128, help="serve: how many requests")
    ap.add_argument("--rate", type=float, default=16.0, help="serve: mean arrivals a second")
    ap.add_argument("--reference-cpu", action="store_true",
                    help="--impl reference without CuPy: also time the reference's NumPy path (one layer, one sequence)")
    args = ap.parse_args()

    if args.impl == "reference":
        return run_reference(args)
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    warmup = max(3, args.warmup)
    if args.workload == "serve":
        return run_serving(args)
    if args.workload == "67b":
        return run_67b(args, warmup)
    if args.workload == "tables":
        return run_tables(args, warmup)
    if args.workload == "lasonex":
        return run_lasonex(args, warmup)
    if args.workload == "sakusun":
        return run_sakusun(args, warmup)
    if args.workload == "saberax":
        return run_saberax(args, warmup)
    if args.workload == "lufozen":
        return run_lufozen(args, warmup)
    if args.workload == "kerirax":
        return run_kerirax(args, warmup)
    if args.workload == "hybrid":
        return run_hybrid(args, warmup)
    args.layers = args.layers or MODEL_7B["num_layers"]

    import torch

    from fastllm_py_b200 import LlamaConfig, Model

    cfg = LlamaConfig(architecture="LlamaForCausalLM", rope_scaling=None, tie_word_embeddings=False,
                      **dict(MODEL_7B, num_layers=args.layers))
    pk = peaks()
    t_load = time.time()
    biggest = max(args.batch, 1 if args.no_points else 64)
    pool = biggest * (CONTEXT + warmup + args.steps + 64)
    model = Model.from_config(cfg, seed=0, dtype="bfloat16", page_size=16, max_tokens=pool,
                              max_requests=biggest, max_batched_tokens=PREFILL_TOKENS,
                              max_model_len=4096, cuda_graph=not args.no_graph)
    torch.cuda.synchronize()
    load_s = time.time() - t_load

    flops = prefill_flops(cfg, PREFILL_TOKENS)
    prefill_first = None
    if not args.no_points:
        # the prompt step once before the decode runs (the GPU has not yet reached its power cap) ...
        prefill_first = time_prefill(model, PREFILL_TOKENS, PREFILL_REPEATS, 3)
    value, ms, launches, clocks = time_decode(model, args.batch, args.steps, warmup, CONTEXT, True)
    mean_ctx = CONTEXT + warmup + (args.steps + 1) / 2
    nbytes = decode_bytes(cfg, args.batch, mean_ctx)
    achieved = nbytes / (ms * 1e-3) / 1e9
    # three passes of K steps each, the median reported: a pass of a quarter of a second now and then
    # catches a host hiccup of tens of milliseconds, which says nothing about the engine
    passes = sorted((time_e2e(model, args.batch, args.steps, warmup, CONTEXT) for _ in range(3)), key=lambda r: r[0])
    e2e, h2d, d2h = passes[1]
    line = {
        "metric": "decode tok/s @ batch 8, 2048-token context, DeepSeek-LLM-7B bf16",
        "value": round(value, 2), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps,
        "warmup": warmup, "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"model": "DeepSeek-LLM-7B size, random weights", "global_batch": args.batch,
                   "seq_len": CONTEXT, "parallelism": "single GPU", "layers": args.layers,
                   "layers_of_config": MODEL_7B["num_layers"], "hidden": cfg.hidden_size,
                   "heads": cfg.num_heads, "kv_heads": cfg.num_kv_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
                   "page_size": 16, "context_limit": 4096, "prefill_tokens": PREFILL_TOKENS,
                   "l2": "weights and cache exceed L2; no flush", "cuda_graph": not args.no_graph,
                   "peaks": pk["source"], "load_s": round(load_s, 1), "e2e_passes": 3},
        "e2e": {"value": round(e2e, 2), "unit": "tokens/s", "h2d_bytes_per_step": h2d,
                "d2h_bytes_per_step": d2h},
        "gpu_launches": launches,
        "clocks": clocks,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"],
                     "unit": "GB/s", "frac": round(achieved / pk["hbm_gbs"], 4)},
    }
    if not args.no_points:
        # ... and again after them, where a serving GPU sits: this is the figure reported as `ms`
        pms, pmean = time_prefill(model, PREFILL_TOKENS, PREFILL_REPEATS, 3)
        frac = lambda t: round(flops / (t * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)
        line["prefill"] = {"value": round(PREFILL_TOKENS * 1000.0 / pms, 1), "tokens": PREFILL_TOKENS,
                           "ms": round(pms, 3), "frac": frac(pms), "ms_mean": round(pmean, 3),
                           "repeats": PREFILL_REPEATS, "ms_before_decode": round(prefill_first[0], 3),
                           "ms_mean_before_decode": round(prefill_first[1], 3),
                           "frac_before_decode": frac(prefill_first[0]),
                           "frac_of_sustained": round(flops / (pms * 1e-3) / (pk["bf16_tflops_sustained"] * 1e12), 4)}
        points = {}
        for b in (1, 64):
            v, _, _, _ = time_decode(model, b, max(8, args.steps // 2), warmup, CONTEXT)
            points[f"decode_b{b}"] = round(v, 2)
        line["points"] = points
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
