#!/usr/bin/env python3
"""Decode and prefill throughput of the Llama-3.1-8B shape on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

Prints one JSON line.  A step is one decode step of a batch of 8 sequences with unequal
prompts (uniform in [128, 2048)) on a cache sized for 4096 tokens each; `value` is decoded
tokens per second measured with CUDA events around K steps after W warm-up steps (the loop of
K steps is repeated and the median repeat reported).  Before anything is timed the bfloat16
engine's tokens are compared with a float32 run at the same layer widths (`checked`).  The
same line carries: `e2e` (the same metric through one `LLM.generate` call, token ids in host lists
in and out, the last K of its W + K decode steps on the host clock), `prefill` (one 2,048-token prompt), `roofline` (bytes a decode step must
read / its time, against the measured HBM copy bandwidth), `points` (decode at batch 1
and 64, with their fractions of the HBM peak) and `workloads` (the Llama-2-7B shape at batch
16 and the Llama-3.2-1B shape at batch 64, each with its own bytes and fraction).  Weights are
random (N(0, 0.02)), token ids synthetic; every decode step reads gigabytes of weights and
cache, far more than the 126 MB L2, so no L2 flush is needed between iterations.  The metric definitions follow the reference's strict bench (timers around
forwards only, warm-ups first, fresh cache: src/bench_strict.cc:146-176).
"""
import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}
BATCH = 8
CONTEXT = 4096
PROMPT_RANGE = (128, 2048)
PREFILL_TOKENS = 2048


def load_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    peaks = dict(FALLBACK_PEAKS)
    if os.path.isfile(path):
        try:
            raw = json.load(open(path))
            flat = {}

            def walk(node):
                if isinstance(node, dict):
                    for k, v in node.items():
                        if isinstance(v, (int, float)):
                            flat.setdefault(k, float(v))
                        else:
                            walk(v)
            walk(raw)
            if "hbm_gbs" in flat:
                peaks["hbm_gbs"] = flat["hbm_gbs"]
                peaks["source"] = "measured"
            if "bf16_tflops" in flat:
                peaks["bf16_tflops"] = flat["bf16_tflops"]
            if "bf16_tflops_sustained" in flat:
                peaks["bf16_tflops_sustained"] = flat["bf16_tflops_sustained"]
        except (OSError, ValueError):
            pass
    return peaks


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index=0):
        self.samples = []      # (time of arrival, fields)
        self.proc = None
        self.index = index
        self.window = [None, None]

    def wait_for_first_line(self, limit=3.0):
        deadline = time.monotonic() + limit
        while self.proc is not None and not self.samples and time.monotonic() < deadline:
            time.sleep(0.01)

    def begin(self):
        """The timed region starts now: earlier samples are dropped."""
        self.window[0] = time.monotonic()

    def end(self):
        self.window[1] = time.monotonic()

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "50",
                 "-i", str(self.index)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) == 6:
                self.samples.append((time.monotonic(), parts))

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        clocks, reasons, top = [], set(), None
        lo, hi = self.window
        for at, (sm, mx, hw, hwt, swt, cap) in self.samples:
            # a line arrives up to one period after its reading
            if (lo is not None and at < lo + 0.05) or (hi is not None and at > hi + 0.05):
                continue
            try:
                clocks.append(int(float(sm)))
                top = int(float(mx))
            except ValueError:
                continue
            for name, flag in (("hw_slowdown", hw), ("hw_thermal_slowdown", hwt), ("sw_thermal_slowdown", swt),
                               ("sw_power_cap", cap)):
                if flag.lower().startswith("active"):
                    reasons.add(name)
        clocks.sort()
        return {"sm_mhz": clocks[len(clocks) // 2] if clocks else None, "sm_max_mhz": top,
                "reasons": sorted(reasons), "samples": len(clocks)}


SHAPES = {
    # BASELINE's configurations 3, 4 and 5: sizes as config.json keys, then the workload
    "llama31_8b": dict(
        config={"vocab_size": 128256, "hidden_size": 4096, "intermediate_size": 14336, "num_hidden_layers": 32,
                "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128,
                "max_position_embeddings": 131072, "rope_theta": 500000.0,
                "rope_scaling": {"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0,
                                 "high_freq_factor": 4.0, "original_max_position_embeddings": 8192},
                "rms_norm_eps": 1e-5, "tie_word_embeddings": False},
        batch=8, context=4096, prompts=(128, 2048)),
    "llama2_7b": dict(
        config={"vocab_size": 32000, "hidden_size": 4096, "intermediate_size": 11008, "num_hidden_layers": 32,
                "num_attention_heads": 32, "num_key_value_heads": 32, "head_dim": 128,
                "max_position_embeddings": 4096, "rope_theta": 10000.0, "rope_scaling": None,
                "rms_norm_eps": 1e-5, "tie_word_embeddings": False},
        batch=16, context=4096, prompts=(256, 1025), decode_steps=256),
    "llama32_1b": dict(
        config={"vocab_size": 128256, "hidden_size": 2048, "intermediate_size": 8192, "num_hidden_layers": 16,
                "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 64,
                "max_position_embeddings": 131072, "rope_theta": 500000.0,
                "rope_scaling": {"rope_type": "llama3", "factor": 32.0, "low_freq_factor": 1.0,
                                 "high_freq_factor": 4.0, "original_max_position_embeddings": 8192},
                "rms_norm_eps": 1e-5, "tie_word_embeddings": True},
        batch=64, context=8192, prompts=(64, 4097), decode_steps=128),
}


def shape_config(name, layers=None):
    import cpp_minilamma_b200 as ml
    raw = dict(SHAPES[name]["config"], architectures=["LlamaForCausalLM"], torch_dtype="bfloat16")
    if layers:
        raw["num_hidden_layers"] = layers
    return ml.config_from_dict(raw)


def llama31_8b(layers=None):
    return shape_config("llama31_8b", layers)


def prompts_for(batch, vocab, seed, prompt_range=PROMPT_RANGE):
    import numpy as np
    rng = np.random.RandomState(seed)
    lens = rng.randint(prompt_range[0], prompt_range[1], size=batch)
    return [[int(t) for t in rng.randint(0, vocab, size=n)] for n in lens]


def release_model(llm):
    """Give a model's memory back before the next one is built."""
    import gc
    import torch
    llm.engine.__dict__.clear()
    llm.__dict__.clear()
    gc.collect()
    torch.cuda.empty_cache()


def time_decode(llm, batch, steps, warmup, seed, sampler=None, prompt_range=PROMPT_RANGE, repeats=1, context=CONTEXT):
    """Prefill `batch` unequal prompts, then time `steps` decode steps (greedy sampling on
    the device included) with CUDA events, `repeats` times over on the same growing sequences.
    Returns (median ms per step, live context tokens at the middle of the timed steps, launches
    of this library's kernels per step, the times of all repeats, ms of the prompt step)."""
    import torch
    from cpp_minilamma_b200 import EngineBackend, SamplingParams, StepEntry
    from cpp_minilamma_b200.csrc import kernels as K
    engine = llm.engine
    backend = EngineBackend(engine, SamplingParams())
    prompts = prompts_for(batch, llm.config.vocab_size, seed, prompt_range)
    longest = max(len(p) for p in prompts)
    repeats = max(1, min(repeats, (context - longest - warmup - 2) // steps))
    slots = engine.acquire(batch)
    try:
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        begin.record()
        tokens = backend.step_and_sample([StepEntry(s, p, [len(p) - 1]) for s, p in zip(slots, prompts)],
                                         list(range(batch)), [0] * batch)
        end.record()
        torch.cuda.synchronize()
        prompt_ms = begin.elapsed_time(end)
        for i in range(warmup):
            tokens = backend.step_and_sample([StepEntry(s, [t], [0]) for s, t in zip(slots, tokens)],
                                             list(range(batch)), [i + 1] * batch)
        torch.cuda.synchronize()
        if sampler:
            sampler.wait_for_first_line()
            sampler.begin()
        launches_before = K.launches
        times = []
        done = warmup
        for _ in range(repeats):
            # as the generation loop runs it: step i + 1, fed on the device with the tokens of step i, is
            # enqueued before the host collects step i
            begin.record()
            ticket = backend.submit([StepEntry(s, [t], [0]) for s, t in zip(slots, tokens)], list(range(batch)),
                                    [done + 1] * batch)
            for i in range(steps):
                ahead = backend.submit_ahead(slots, list(range(batch)), [done + i + 2] * batch) if i + 1 < steps else None
                tokens = backend.collect(ticket)
                ticket = ahead
            end.record()
            torch.cuda.synchronize()
            times.append(begin.elapsed_time(end) / steps)
            done += steps
        if sampler:
            sampler.end()
        ordered = sorted(times)
        ms = ordered[len(ordered) // 2]
        live = sum(len(p) for p in prompts) + batch * (warmup + (repeats * steps) // 2)
        return ms, live, (K.launches - launches_before) / (steps * repeats), times, prompt_ms
    finally:
        for s in slots:
            engine.release(s)


def decode_bytes(llm, live_tokens):
    """Bytes a decode step has to read: every weight it uses once, and the cache of the live tokens."""
    return llm.model.step_weight_bytes() + llm.engine.cache.kv_bytes_per_token() * live_tokens


def check_against_float32(peaks_note=None):
    """Before anything is timed: the bfloat16 engine at the benchmark's layer widths and vocabulary (2 of the
    32 layers) generates greedily for a batch of 8 unequal prompts through `LLM.generate` (captured graphs,
    the device one step ahead), and a float32 run of the same weights scores those sequences.  Every
    generated token must be the float32 run's best token, or within 4 % of its largest |logit| of it
    (bfloat16 rounding moves near ties)."""
    import numpy as np
    import torch
    import cpp_minilamma_b200 as ml
    from cpp_minilamma_b200 import StepEntry
    cfg = shape_config("llama31_8b", layers=2)
    new_tokens = 6
    prompts = prompts_for(BATCH, cfg.vocab_size, seed=5, prompt_range=(128, 700))
    fast = ml.random_model(cfg, seed=0, dtype="bfloat16", max_tokens=BATCH * 1024, max_positions=1024, max_seqs=BATCH)
    generated = fast.generate(prompts, max_new_tokens=new_tokens, ignore_eos=True)
    release_model(fast)
    exact = ml.random_model(cfg, seed=0, dtype="float32", stored_as="bfloat16", max_tokens=2048, max_positions=1024,
                            max_seqs=2)
    worst = 0.0
    for prompt, tokens in zip(prompts, generated):
        assert len(tokens) == new_tokens
        slot, = exact.engine.acquire(1)
        whole = list(prompt) + tokens[:-1]
        want = list(range(len(prompt) - 1, len(whole)))
        logits = exact.engine.step([StepEntry(slot, whole, want)]).cpu().numpy()
        exact.engine.release(slot)
        for row, token in zip(logits, tokens):
            margin = float(row.max() - row[token]) / float(np.abs(row).max())
            worst = max(worst, margin)
            if margin > 0.04:
                raise AssertionError(f"bench check: the bfloat16 engine generated token {token}, which the float32 "
                                     f"run puts {margin:.3f} of its largest logit below its best token")
    release_model(exact)
    return {"checked": True, "check": f"8 prompts x {new_tokens} greedy tokens of the bfloat16 engine (2 layers, full widths "
                                       f"and vocabulary) against a float32 run of the same weights; worst margin {worst:.4f}"}


def time_workload(name, peaks, warmup, layers=None):
    """One of the further workloads: its batch of unequal prompts in one step, then all its decode steps,
    timed as the reference's strict bench times them (timers around the steps only, device sampling
    included; src/bench_strict.cc:146-176,200-209)."""
    import cpp_minilamma_b200 as ml
    spec = SHAPES[name]
    cfg = shape_config(name, layers)
    batch, steps, context = spec["batch"], spec["decode_steps"], spec["context"]
    budget = batch * (spec["prompts"][1] + warmup + steps + 64)
    llm = ml.random_model(cfg, seed=0, dtype="bfloat16", max_tokens=budget, max_positions=context, max_seqs=batch,
                          max_step_tokens=8192)
    ms, live, _, _, prompt_ms = time_decode(llm, batch, steps, warmup, seed=21, prompt_range=spec["prompts"],
                                            context=context)
    prompt_tokens = live - batch * (warmup + steps // 2)
    achieved = decode_bytes(llm, live) / (ms * 1e-3) / 1e9
    out = {"decode_tok_s": round(batch * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "batch": batch,
           "decode_steps": steps, "layers": cfg.num_hidden_layers, "layers_full": spec["config"]["num_hidden_layers"],
           "live_tokens": live, "gb_per_step": round(decode_bytes(llm, live) / 1e9, 3),
           "hbm_gbs": round(achieved, 1), "frac": round(achieved / peaks["hbm_gbs"], 4),
           "prefill_tok_s": round(prompt_tokens * 1000.0 / prompt_ms, 1), "prefill_tokens": prompt_tokens}
    release_model(llm)
    return out


def time_e2e(llm, batch, steps, warmup, seed):
    """Decoded tokens per second through LLM.generate, host token lists in, host lists out: one call that
    generates warmup + steps + 1 tokens per prompt; the host clock is read as each step's tokens arrive, and the
    last `steps` decode steps count (the `warmup` steps before them are the warm-up, as for the device-timed
    figure).  Also returned: the rate of the first `steps` decode steps, which follow the prompt step into the
    power cap and run slower."""
    prompts = prompts_for(batch, llm.config.vocab_size, seed)
    stats = {}
    llm.generate(prompts, max_new_tokens=warmup + steps + 1, ignore_eos=True, stats=stats)
    stamps = stats["step_stamps"]  # [0]: the prompt step's tokens, [k]: decode step k's
    if len(stamps) < warmup + steps + 1:
        raise RuntimeError(f"the generation made {len(stamps) - 1} decode steps, {warmup + steps} were asked for")
    timed = stamps[warmup + steps] - stamps[warmup]
    first = stamps[steps] - stamps[0]
    return batch * steps / timed, batch * steps / first


def time_prefill(llm, tokens, reps, warmup, seed, pause=0.0):
    """Mean time of one prompt step of `tokens` tokens (CUDA events around the engine's step call,
    host planning included).  `pause` seconds of idling before each timed step make it an isolated
    step, as a request meets it; without pauses the steps run back to back under the power cap."""
    import numpy as np
    import torch
    from cpp_minilamma_b200 import StepEntry
    rng = np.random.RandomState(seed)
    prompt = [int(t) for t in rng.randint(0, llm.config.vocab_size, size=tokens)]
    times = []
    for i in range(warmup + reps):
        slot, = llm.engine.acquire(1)
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        if pause and i >= warmup:
            time.sleep(pause)
        begin.record()
        llm.engine.step_borrowed([StepEntry(slot, prompt, [tokens - 1])])
        end.record()
        torch.cuda.synchronize()
        llm.engine.release(slot)
        if i >= warmup:
            times.append(begin.elapsed_time(end))
    return sum(times) / len(times)


def prefill_flops(cfg, tokens):
    d, hq, hk = cfg.head_dim, cfg.num_attention_heads, cfg.num_key_value_heads
    per_layer = 2 * tokens * cfg.hidden_size * ((hq + 2 * hk) * d + hq * d) \
        + 2 * tokens * cfg.hidden_size * cfg.intermediate_size * 3 \
        + 2 * hq * tokens * tokens * d  # causal: half of 4 T^2 d per head
    return cfg.num_hidden_layers * per_layer + 2 * cfg.hidden_size * cfg.vocab_size  # head on one row


def profile_region(args):
    """One eager step inside cudaProfilerStart/Stop, after warm-up steps of the same kind."""
    import numpy as np
    import torch
    import cpp_minilamma_b200 as ml
    from cpp_minilamma_b200 import StepEntry
    cfg = shape_config(args.shape, args.layers or 4)
    context = max(SHAPES[args.shape]["context"], args.context + 64)  # room for a longer --context than the workload's
    llm = ml.random_model(cfg, seed=0, dtype="bfloat16", max_tokens=(args.batch + 1) * context, max_positions=context,
                          max_seqs=args.batch + 2, max_step_tokens=8192)
    rng = np.random.RandomState(0)
    engine = llm.engine
    draw = lambda n: [int(t) for t in rng.randint(0, cfg.vocab_size, size=n)]
    if args.profile == "decode":
        slots = engine.acquire(args.batch)
        engine.step_borrowed([StepEntry(s, draw(args.context), [args.context - 1]) for s in slots])
        for _ in range(2):
            engine.step_borrowed([StepEntry(s, [5], [0]) for s in slots])
        step = lambda: engine.step_borrowed([StepEntry(s, [7], [0]) for s in slots])
    else:
        prompt = draw(PREFILL_TOKENS)
        slot, = engine.acquire(1)
        engine.step_borrowed([StepEntry(slot, prompt, [PREFILL_TOKENS - 1])])
        engine.release(slot)
        slot, = engine.acquire(1)
        step = lambda: engine.step_borrowed([StepEntry(slot, prompt, [PREFILL_TOKENS - 1])])
    torch.cuda.synchronize()
    torch.cuda.profiler.start()
    step()
    torch.cuda.synchronize()
    torch.cuda.profiler.stop()
    print(f"profiled one {args.profile} step: {args.shape}, {cfg.num_hidden_layers} layers, batch {args.batch}")
    return 0


# --------------------------------------------------------------------------------------------------- #
# --design kupirax: the Kupirax decoder beside the Llama decoder at equal sizes                         #
# --------------------------------------------------------------------------------------------------- #
DESIGN_SIZES = {
    # width, feed-forward and attention heads of the Llama-3.2-1B-like and Llama-3.1-8B-like layers; a group of
    # (chunked attention, retention, gated delta rule) layers, twice; vocabulary 32,000
    "w2048": dict(width=2048, ff=8192, vocab=32000, heads=16, kv_heads=4, chunk=1024, ret_heads=8, groups=2),
    "w4096": dict(width=4096, ff=14336, vocab=32000, heads=32, kv_heads=8, chunk=2048, ret_heads=16, groups=2),
}


def kupirax_config(size):
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    mlp = {"kind": "dense", "ff": s["ff"]}
    group = [
        {"type": "attention", "mlp": mlp,
         "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                   "mask": {"size": s["chunk"]},
                   "rot": {"base": 500000.0, "dims": 64,
                           "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}},
        {"type": "retention", "mlp": mlp,
         "mixer": {"heads": s["ret_heads"], "dim": 128, "vdim": 256, "rot": {"base": 10000.0, "dims": 128},
                   "decay": [1.0 - 2.0 ** (-5 - 4 * i / s["ret_heads"]) for i in range(s["ret_heads"])]}},
        {"type": "channel_delta", "mlp": mlp,
         "mixer": {"heads": s["heads"], "kv_heads": s["heads"], "dim": 128, "vdim": 128, "conv": 4,
                   "decay_rank": 64, "gate_rank": 64}},
    ]
    return ml.config_from_dict({"architecture": "Kupirax", "vocab": s["vocab"], "width": s["width"],
                                "norm": {"eps": 1e-6}, "layers": group * s["groups"], "torch_dtype": "bfloat16"})


def malulorn_config(size):
    """Three layers (attention with a sink, latent attention, attention with a sink) that run twice in a row, so
    six layer runs like the Llama decoder beside it; every token goes through 2 of 16 experts and a shared one, whose
    widths add up to the Llama decoder's feed-forward (equal work per token; the experts' total is 4.5 times that)."""
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    mlp = {"kind": "moe", "router": {"experts": 16, "top": 2}, "expert": {"ff": s["ff"] // 4}, "shared": {"ff": s["ff"] // 2}}
    sink = {"type": "attention", "mlp": mlp,
            "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                      "q_temp": {"coef": 0.1, "every": 1024}}}
    latent = {"type": "latent_attention", "mlp": mlp,
              "mixer": {"heads": s["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 192, "scale": 192 ** -0.5,
                        "rot": {"base": 500000.0, "dims": 64}}}
    return ml.config_from_dict({"architecture": "Malulorn", "vocab": s["vocab"], "width": s["width"],
                                "norm": {"eps": 1e-5}, "layers": [sink, latent, sink],
                                "loop": {"start": 0, "stop": 3, "times": s["groups"]}, "torch_dtype": "bfloat16"})


def malulorn_rooflines(size, tokens, batch, context, peaks):
    """As `design_rooflines`, for the kernels of the Malulorn decoder and their like in the Llama decoder."""
    s = DESIGN_SIZES[size]
    H, G, d, D, ff = s["heads"], s["kv_heads"], 128, s["width"], s["ff"]
    rank, row = 192, 256
    E, top, eff = 16, 2, ff // 4
    causal = tokens * (tokens + 1) // 2
    out = {}
    # prompt attention: the sink layers (d = dv = 128) and the latent layers (keys of 256, values of 192, one kv head)
    out["malulorn", "prefill", "attention_prefill"] = ("tensor", 2.0 * H * causal * 2 * d)
    out["malulorn", "prefill", "local_attention_mma"] = ("tensor", 2.0 * H * causal * (d + d + row + rank) / 2)  # mean of the two kinds
    out["llama", "prefill", "attention_prefill"] = ("tensor", 2.0 * H * causal * 2 * d)
    qkv = (H * d + 2 * G * d) * 2
    out["malulorn", "prefill", "local_attention_prepare"] = ("hbm", tokens * 2 * qkv)
    out["malulorn", "prefill", "latent_prepare"] = ("hbm", tokens * (H * 64 * 4 + row * 4 + rank * 2))
    out["llama", "prefill", "rope_cache_write"] = ("hbm", tokens * 2 * qkv)
    out["malulorn", "decode", "local_attention_prepare"] = ("hbm", batch * 2 * qkv)
    # single tokens: keys and values once (the latent layers read one row of 256 per position)
    sink_bytes, latent_bytes = batch * context * G * 2 * d * 2, batch * context * row * 2
    out["malulorn", "decode", "attention_decode"] = ("hbm", sink_bytes)
    out["malulorn", "decode", "local_attention_heads"] = ("hbm", (2 * sink_bytes + latent_bytes) / 3)  # if all three layers run here
    out["malulorn", "decode", "local_attention"] = ("hbm", (2 * sink_bytes + latent_bytes) / 3)
    out["llama", "decode", "attention_decode"] = ("hbm", sink_bytes)
    # the experts' products: FLOPs of the chosen experts in prompts; in decode steps every expert's weights once
    out["malulorn", "prefill", "moe_gate_up_mma"] = ("tensor", 2.0 * tokens * top * 2 * eff * D)
    out["malulorn", "prefill", "moe_down_mma"] = ("tensor", 2.0 * tokens * top * eff * D)
    touched = min(E, batch * top)
    out["malulorn", "decode", "moe_gate_up"] = ("hbm", touched * 2 * eff * D * 2)
    out["malulorn", "decode", "moe_down"] = ("hbm", touched * eff * D * 2)
    out["malulorn", "decode", "moe_gate_up_mma"] = ("hbm", touched * 2 * eff * D * 2)
    out["malulorn", "decode", "moe_down_mma"] = ("hbm", touched * eff * D * 2)
    for kind, n in (("prefill", tokens), ("decode", batch)):
        out["malulorn", kind, "moe_route"] = ("hbm", n * D * 2 + E * D * 4)
        out["malulorn", kind, "moe_combine"] = ("hbm", n * D * (top * 4 + 2 + 2))
        out["malulorn", kind, "layernorm"] = ("hbm", n * D * (4 + 4 + 2 + 2))
        out["llama", kind, "rmsnorm"] = ("hbm", n * D * (4 + 4 + 2 + 2))
        out["malulorn", kind, "heads_gate"] = ("hbm", n * H * d * 4)
    return out


def sopanex_config(size):
    """Six layers, each with attention (learned sink, values that are the keys, 64 of 128 dimensions rotated under a
    ramp) beside gated linear attention of half as many heads of 128, and 16 gelu experts of ff / 4 plus 2 pass-through
    experts, 3 per token, beside a gated shared expert of ff / 2: the Malulorn decoder's sizes (same width, heads,
    layer runs, expert count and widths), with the recurrent mixer on top."""
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    mlp = {"kind": "moe", "router": {"experts": 16, "top": 3, "identity": 2, "scale": 2.0}, "expert": {"ff": s["ff"] // 4},
           "shared": {"ff": s["ff"] // 2}}
    layer = {"type": "parallel", "mlp": mlp,
             "mixer": {"left_scale": 1.0, "right_scale": 1.0,
                       "left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                "rot": {"base": 500000.0, "dims": 64,
                                        "scaling": {"factor": 8.0, "original": 8192, "fast": 16.0, "slow": 1.0}}},
                       "right": {"heads": s["heads"] // 2, "dim": 128, "vdim": 128, "tau": 8.0, "decay_rank": 64}}}
    return ml.config_from_dict({"architecture": "Sopanex", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
                                "embedding": {"scale": 1.0, "bigram": {"buckets": 65521, "mul_prev": 33, "mul_cur": 5}},
                                "layers": [layer] * (3 * s["groups"]), "torch_dtype": "bfloat16"})


def sopanex_rooflines(size, tokens, batch, context, peaks):
    """As `design_rooflines`, for the kernels of the Sopanex decoder and their like in the Malulorn decoder (and, for
    the recurrent mixer, in the Kupirax decoder: `--design kupirax` measures those)."""
    s = DESIGN_SIZES[size]
    H, G, d, D, ff = s["heads"], s["kv_heads"], 128, s["width"], s["ff"]
    Hr, dr, dvr = s["heads"] // 2, 128, 128
    E, R, top, eff = 16, 18, 3, ff // 4
    causal = tokens * (tokens + 1) // 2
    out = {k: v for k, v in malulorn_rooflines(size, tokens, batch, context, peaks).items() if k[0] == "malulorn"}
    out["sopanex", "prefill", "attention_prefill"] = ("tensor", 2.0 * H * causal * 2 * d)
    qk = (H * d + G * d) * 2
    out["sopanex", "prefill", "local_attention_prepare"] = ("hbm", tokens * (qk + qk + G * d * 2))  # q, k rotated and v written
    out["sopanex", "decode", "local_attention_prepare"] = ("hbm", batch * (qk + qk + G * d * 2))
    out["sopanex", "decode", "attention_decode"] = ("hbm", batch * context * G * 2 * d * 2)
    out["sopanex", "prefill", "moe_gate_up_mma"] = ("tensor", 2.0 * tokens * top * (E / R) * eff * D)  # a share of the choices passes through
    out["sopanex", "prefill", "moe_down_mma"] = ("tensor", 2.0 * tokens * top * (E / R) * eff * D)
    touched = min(E, batch * top)
    out["sopanex", "decode", "moe_gate_up_mma"] = ("hbm", touched * eff * D * 2)
    out["sopanex", "decode", "moe_down_mma"] = ("hbm", touched * eff * D * 2)
    for kind, n, seqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        out["sopanex", kind, "moe_route"] = ("hbm", n * D * 2 + (R + 1) * D * 4)
        out["sopanex", kind, "moe_combine"] = ("hbm", n * D * (top * 4 + 2 + 2 + 2))
        out["sopanex", kind, "rmsnorm"] = ("hbm", n * D * (4 + 4 + 2 + 2 + 1))       # half of them add two deltas
        out["sopanex", kind, "heads_gate"] = ("hbm", n * H * d * 4)
        out["sopanex", kind, "embedding_pair"] = ("hbm", n * D * (2 + 2 + 4))
        out["sopanex", kind, "activation"] = ("hbm", n * (ff // 2) * 4)
        out["sopanex", kind, "state_scan (channel decay)"] = ("hbm", n * Hr * (3 * dr + 2 * dvr) * 4 + seqs * Hr * dr * dvr * 8)
        out["sopanex", kind, "channel_decay_prepare"] = ("hbm", n * Hr * ((2 * dr + dvr) * 2 + dr * 4 + (3 * dr + dvr) * 4))
        out["sopanex", kind, "head_norm_gate"] = ("hbm", n * Hr * dvr * (4 + 2 + 2))
    return out


def badolix_config(size):
    """Six layers: window attention (1,024 positions and the first 64 tokens, capped scores, 128 dimensions rotated at
    divided frequencies), window attention that reads the first layer's keys and values, latent attention (the Malulorn
    decoder's sizes, frequencies under a ramp), a state-space mixer (inner size 2 x width in heads of 64, states of 128,
    8 groups, 4 taps), window attention, latent attention; dense feed-forwards with biases and routed ones (4 of 16
    experts of ff / 4, chosen inside 2 of 4 groups: the dense layer's work per token) take turns."""
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    dense = {"kind": "dense", "ff": s["ff"]}
    moe = {"kind": "moe", "router": {"experts": 16, "top": 4, "groups": {"count": 4, "keep": 2}}, "expert": {"ff": s["ff"] // 4}}
    window = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
              "mask": {"size": 1024, "keep_first": 64}, "rot": {"base": 500000.0, "dims": 128, "scaling": {"factor": 8.0}}}
    latent = {"heads": s["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 192, "scale": 192 ** -0.5,
              "rot": {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 8192, "fast": 16.0, "slow": 1.0}}}
    ssm = {"heads": 2 * s["width"] // 64, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8}
    layers = [{"type": "attention", "mixer": window, "mlp": dense},
              {"type": "attention", "mixer": dict(window, kv_from=0), "mlp": moe},
              {"type": "latent_attention", "mixer": latent, "mlp": dense},
              {"type": "mamba2", "mixer": ssm, "mlp": moe},
              {"type": "attention", "mixer": window, "mlp": dense},
              {"type": "latent_attention", "mixer": latent, "mlp": moe}]
    return ml.config_from_dict({"architecture": "Badolix", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5},
                                "embedding": {"scale": 2.0}, "residual_mult": 0.7, "logit_scale": 0.5, "layers": layers,
                                "torch_dtype": "bfloat16"})


def badolix_rooflines(size, tokens, batch, context, peaks):
    """As `design_rooflines`, for the kernels of the Badolix decoder and their like in the Malulorn decoder."""
    s = DESIGN_SIZES[size]
    H, G, d, D, ff = s["heads"], s["kv_heads"], 128, s["width"], s["ff"]
    rank, row = 192, 256
    E, top, eff = 16, 4, ff // 4
    Hs, P, N, Gs, taps = 2 * D // 64, 64, 128, 8, 4
    inner = Hs * P
    out = {k: v for k, v in malulorn_rooflines(size, tokens, batch, context, peaks).items() if k[0] == "malulorn"}
    causal = tokens * (tokens + 1) // 2
    seen = sum(min(i + 1, 1024 + 64) for i in range(tokens))            # keys a prompt token sees: its window and the kept tokens
    out["badolix", "prefill", "local_attention_mma (window)"] = ("tensor", 2.0 * H * seen * 2 * d)
    out["badolix", "prefill", "attention_prefill"] = ("tensor", 2.0 * H * seen * 2 * d)
    out["badolix", "prefill", "local_attention_mma"] = ("tensor", 2.0 * H * causal * (row + rank))
    qkv = (H * d + 2 * G * d) * 2
    for kind, n, seqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        out["badolix", kind, "local_attention_prepare"] = ("hbm", n * (2 * qkv + 2 * H * d * 2) / 3)  # two layers of three write keys
        out["badolix", kind, "latent_prepare"] = ("hbm", n * (H * 64 * 4 + row * 4 + rank * 2))
        out["badolix", kind, "moe_route"] = ("hbm", n * D * 2 + E * D * 4)
        out["badolix", kind, "moe_combine"] = ("hbm", n * D * (top * 4 + 2))
        out["badolix", kind, "rmsnorm"] = ("hbm", n * D * (4 + 4 + 2 + 2))
        out["badolix", kind, "swiglu"] = ("hbm", n * ff * (4 + 2))
        out["badolix", kind, "add_bias"] = ("hbm", n * D * 4)
        # the state-space mixer: what a step must move at least - the projection's row, the float32 inputs and outputs
        # of the recurrence per token, and in a decode step the state once in and once out
        gn = Gs * N
        out["badolix", kind, "ssd_prepare"] = ("hbm", n * ((inner + 2 * gn + Hs) * 2 + (2 * inner + 2 * gn + Hs) * 4))
        out["badolix", kind, "state_scan (token decay)"] = ("hbm", n * (2 * inner + 2 * gn + Hs) * 4 + seqs * Hs * N * P * 8)
        out["badolix", kind, "gated_group_norm"] = ("hbm", n * inner * (4 + 4 + 2 + 2))
        out["badolix", kind, "conv_state_update"] = ("hbm", seqs * (taps - 1) * (inner + 2 * gn) * (2 + 4))
    visible = min(context, 1024 + 64)
    out["badolix", "decode", "local_attention_heads (window)"] = ("hbm", batch * visible * G * 2 * d * 2)
    out["badolix", "decode", "attention_decode"] = ("hbm", batch * visible * G * 2 * d * 2)
    out["badolix", "decode", "local_attention_heads"] = ("hbm", batch * context * row * 2)
    out["badolix", "prefill", "moe_gate_up_mma"] = ("tensor", 2.0 * tokens * top * 2 * eff * D)
    out["badolix", "prefill", "moe_down_mma"] = ("tensor", 2.0 * tokens * top * eff * D)
    touched = min(E, batch * top)
    out["badolix", "decode", "moe_gate_up_mma"] = ("hbm", touched * 2 * eff * D * 2)
    out["badolix", "decode", "moe_down_mma"] = ("hbm", touched * eff * D * 2)
    return out


def mefolorn_config(size):
    """Six layers: latent attention (queries through a latent of 3/8 of the width, 256 latent columns per position), mixed
    scores beside a linear recurrent unit (as wide as the model, in blocks of 256, 4 taps), the pair again, latent
    attention, the pair, latent attention; every attention under a window of 1,024 positions, a dense feed-forward
    beside every mixer."""
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    mlp = {"kind": "dense", "ff": s["ff"]}
    latent = {"type": "latent_attention", "mlp": mlp,
              "mixer": {"heads": s["heads"], "dim": 128, "vdim": 128, "q_rank": 3 * s["width"] // 8, "kv_rank": 256,
                        "scale": 128 ** -0.5, "mask": {"size": 1024}}}
    pair = {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                               "mask": {"size": 1024}, "rot": {"base": 500000.0, "dims": 128}},
                      "right": {"width": s["width"], "blocks": s["width"] // 256, "conv": 4},
                      "left_scale": 0.8, "right_scale": 1.2}}
    return ml.config_from_dict({"architecture": "Mefolorn", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5},
                                "embedding": {"scale": 2.0}, "layers": [latent, pair, pair, latent, pair, latent],
                                "torch_dtype": "bfloat16"})


def mefolorn_rooflines(size, tokens, batch, context, peaks):
    """As `design_rooflines`, for the kernels of the Mefolorn decoder and their like in the Badolix decoder."""
    s = DESIGN_SIZES[size]
    H, G, d, D, ff = s["heads"], s["kv_heads"], 128, s["width"], s["ff"]
    rank, q_rank, W, bs, taps = 256, 3 * D // 8, D, 256, 4
    out = {k: v for k, v in badolix_rooflines(size, tokens, batch, context, peaks).items() if k[0] == "badolix"}
    seen = sum(min(i + 1, 1024) for i in range(tokens))
    visible = min(context, 1024)
    out["mefolorn", "prefill", "mixed_attention_mma"] = ("tensor", 2.0 * seen * (H * 2 * d + H * H))
    out["mefolorn", "decode", "mixed_attention_single"] = ("hbm", batch * visible * G * 2 * d * 2)
    out["mefolorn", "prefill", "local_attention_mma"] = ("tensor", 2.0 * H * seen * 2 * rank)
    out["mefolorn", "decode", "local_attention_heads"] = ("hbm", batch * visible * rank * 2)
    qkv = (H * d + 2 * G * d) * 2
    for kind, n, seqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        out["mefolorn", kind, "tanh_norm"] = ("hbm", n * D * (4 + 4 + 2.5 * 2 + 2 * 2))  # half of them add three outputs
        out["mefolorn", kind, "local_attention_prepare"] = ("hbm", n * 2 * qkv)
        out["mefolorn", kind, "latent_prepare"] = ("hbm", n * (q_rank + rank) * 4)
        out["mefolorn", kind, "heads_gate"] = ("hbm", n * H * d * 4)
        out["mefolorn", kind, "swiglu"] = ("hbm", n * ff * (4 + 2))
        out["mefolorn", kind, "conv_state_update"] = ("hbm", seqs * (taps - 1) * W * (2 + 4))
    out["mefolorn", "prefill", "lru_gates"] = ("hbm", tokens * W * (2 + 8) + 2 * W * bs * 2)
    out["mefolorn", "prefill", "lru_scan"] = ("hbm", tokens * W * (8 + 2 + 2))
    out["mefolorn", "decode", "lru_gates (single tokens)"] = ("hbm", batch * W * (4 + 2 + 8 + 4 * (taps - 1)) + 2 * W * bs * 2)
    return out


def gopitar_config(size):
    """Six layers: the pair twice and the delta rule, twice over.  The pair: attention with query and key heads of 64 and
    value heads of 128 under a window of 1,024 behind a convolution of 3 taps, beside lightning attention with heads of
    128 x 128; the delta rule with heads of 128 x 128 and 4 taps; a dense feed-forward behind every mixer."""
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    mlp = {"kind": "dense", "ff": s["ff"]}
    R = s["ret_heads"]
    pair = {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 64, "vdim": 128, "conv": 3, "scale": 0.125,
                               "mask": {"size": 1024}, "rot": {"base": 500000.0, "dims": 32}},
                      "right": {"heads": R, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 4 * i / R) for i in range(R)]},
                      "left_scale": 0.7, "right_scale": 0.9}}
    delta = {"type": "delta", "mlp": mlp, "mixer": {"heads": s["heads"], "kv_heads": s["heads"], "dim": 128, "vdim": 128, "conv": 4}}
    return ml.config_from_dict({"architecture": "Gopitar", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5},
                                "embedding": {"scale": 2.0}, "logit_softcap": 50.0, "layers": [pair, pair, delta] * s["groups"],
                                "torch_dtype": "bfloat16"})


def gopitar_rooflines(size, tokens, batch, context, peaks):
    """As `design_rooflines`, for the kernels of the Gopitar decoder and their like in the Kupirax decoder."""
    s = DESIGN_SIZES[size]
    H, G, d, dv, R, D, ff = s["heads"], s["kv_heads"], 64, 128, s["ret_heads"], s["width"], s["ff"]
    e = 128  # rows and columns of every state
    out = {k: v for k, v in design_rooflines(size, tokens, batch, context, peaks).items() if k[0] == "kupirax"}
    seen = sum(min(i + 1, 1024) for i in range(tokens))
    visible = min(context, 1024)
    for name in ("attention_prefill", "local_attention_mma"):
        out["gopitar", "prefill", name] = ("tensor", 2.0 * H * seen * (d + dv))
    for name in ("attention_decode", "local_attention_heads"):
        out["gopitar", "decode", name] = ("hbm", batch * visible * G * (d + dv) * 2)
    qkv = (H * d + G * (d + dv)) * 2
    for kind, n, seqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        out["gopitar", kind, "conv_attention_prepare"] = ("hbm", n * 2 * qkv + (n * 4 * qkv if kind == "decode" else 0))
        out["gopitar", kind, "lightning_prepare"] = ("hbm", n * R * 3 * e * (2 + 4))
        out["gopitar", kind, "state_scan (retention)"] = ("hbm", n * R * 4 * e * 4 + seqs * R * e * e * 8)
        # the runs' matrices are not counted: what the recurrence must move is the same
        out["gopitar", kind, "state_chunks (head decay)"] = out["gopitar", kind, "state_scan (retention)"]
        out["gopitar", kind, "row_norm_gate"] = ("hbm", n * R * e * (4 + 2 + 2))
        conv = n * H * 3 * e * 2 * 3 * 4 if kind == "decode" else 0  # the convolution's state, in and out
        out["gopitar", kind, "delta_prepare"] = ("hbm", n * H * 3 * e * (2 + 4) + conv)
        out["gopitar", kind, "state_scan (delta rule, head decay)"] = ("hbm", n * H * 4 * e * 4 + seqs * H * e * e * 8)
        out["gopitar", kind, "state_chunks (delta rule)"] = out["gopitar", kind, "state_scan (delta rule, head decay)"]
        out["gopitar", kind, "head_norm_gate"] = ("hbm", n * H * e * (4 + 2 + 2))
        out["gopitar", kind, "heads_gate"] = ("hbm", n * H * dv * 4)
        for model in ("gopitar", "kupirax"):
            out[model, kind, "swiglu"] = ("hbm", n * ff * (4 + 2))
        for name in ("rmsnorm", "rmsnorm (normed delta)"):  # the stream in and out, the outputs that join it, the result
            out["gopitar", kind, name] = ("hbm", n * D * (8 + 2 + (4 if "delta" in name else 2)))
            out["kupirax", kind, name] = ("hbm", n * D * (8 + 2 + 4))
        out["gopitar", kind, "add_bias"] = ("hbm", n * D * 4)
        out["gopitar", kind, "softcap"] = ("hbm", seqs * s["vocab"] * 8)
    return out


def llama_like_config(size):
    import cpp_minilamma_b200 as ml
    s = DESIGN_SIZES[size]
    return ml.config_from_dict({
        "architectures": ["LlamaForCausalLM"], "torch_dtype": "bfloat16", "vocab_size": s["vocab"],
        "hidden_size": s["width"], "intermediate_size": s["ff"], "num_hidden_layers": 3 * s["groups"],
        "num_attention_heads": s["heads"], "num_key_value_heads": s["kv_heads"], "head_dim": 128,
        "max_position_embeddings": 8192, "rope_theta": 500000.0, "rope_scaling": None, "rms_norm_eps": 1e-6,
        "tie_word_embeddings": False})


def kernel_times_of_a_step(llm, entries_of):
    """Device time of every kernel of this library in one eager step on one stream (CUDA events around each launch),
    after two warm-up steps of the same kind: {kernel: (calls, ms)}."""
    from cpp_minilamma_b200.csrc import kernels as K
    from cpp_minilamma_b200.parts import branches
    import torch
    beside, branches.USE_SIDE_STREAMS = branches.USE_SIDE_STREAMS, False
    try:
        return _kernel_times_of_a_step(llm, entries_of, K, torch)
    finally:
        branches.USE_SIDE_STREAMS = beside


def _kernel_times_of_a_step(llm, entries_of, K, torch):
    for _ in range(2):
        slots, entries = entries_of()
        llm.engine.step_borrowed(entries)
        for slot in slots:
            llm.engine.release(slot)
    slots, entries = entries_of()
    torch.cuda.synchronize()
    with K.KernelTimes() as times:
        llm.engine.step_borrowed(entries)
    totals = times.totals()
    for slot in slots:
        llm.engine.release(slot)
    return totals


def design_rooflines(size, tokens, batch, context, peaks):
    """Algorithmic bytes (or FLOPs) per launch of the kernels that differ between the two decoders, at the sizes of
    `kernel_times_of_a_step`: {(model, kind of step, kernel): ("hbm" | "tensor", amount)}."""
    s = DESIGN_SIZES[size]
    H, G, d, dv, C = s["heads"], s["kv_heads"], 128, 128, s["chunk"]
    Hr, dr, dvr = s["ret_heads"], 128, 256
    out = {}
    seen = sum(min(i % C, i) + 1 for i in range(tokens))              # keys each prompt token sees in its chunk
    causal = tokens * (tokens + 1) // 2
    out["kupirax", "prefill", "local_attention_mma"] = ("tensor", 2.0 * H * seen * (d + dv))
    out["kupirax", "prefill", "attention_prefill"] = ("tensor", 2.0 * H * seen * (d + dv))
    out["llama", "prefill", "attention_prefill"] = ("tensor", 2.0 * H * causal * 2 * d)
    qkv = (H * d + G * d + G * dv) * 2
    out["kupirax", "prefill", "local_attention_prepare"] = ("hbm", tokens * (2 * qkv))
    out["llama", "prefill", "rope_cache_write"] = ("hbm", tokens * (2 * qkv))
    out["kupirax", "decode", "local_attention_prepare"] = ("hbm", batch * (2 * qkv))
    visible = min(context % C, context) + 1
    out["kupirax", "decode", "local_attention"] = ("hbm", batch * visible * G * (d + dv) * 2)
    out["kupirax", "decode", "attention_decode"] = ("hbm", batch * visible * G * (d + dv) * 2)
    out["llama", "decode", "attention_decode"] = ("hbm", batch * context * G * 2 * d * 2)
    # state mixers: what a step must move at least - the float32 inputs and outputs of the recurrence per token,
    # and in a decode step the state once in and once out
    for kind, n, seqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        ret_io = n * Hr * (2 * dr + 2 * dvr) * 4
        delta_io = n * H * (3 * d + 2 * dv + 1) * 4
        ret_state, delta_state = seqs * Hr * dr * dvr * 8, seqs * H * d * dv * 8
        out["kupirax", kind, "state_scan (retention)"] = ("hbm", ret_io + ret_state)
        out["kupirax", kind, "state_chunks (head decay)"] = ("hbm", ret_io + ret_state)
        out["kupirax", kind, "state_scan (delta rule)"] = ("hbm", delta_io + delta_state)
        out["kupirax", kind, "retention_prepare"] = ("hbm", n * Hr * (2 * dr + 2 * dvr) * 2 + n * Hr * (2 * dr + dvr) * 4)
        out["kupirax", kind, "delta_prepare"] = ("hbm", n * (H * (2 * d + dv) * 2 + H * d * 4) + n * H * (3 * d + dv + 1) * 4)
        out["kupirax", kind, "head_norm_gate"] = ("hbm", n * H * dv * (4 + 2 + 2))
    return out


def bench_design(args):
    """Prompt and decode throughput of the Kupirax or Malulorn decoder and of the Llama decoder (of the Sopanex or Badolix
    decoder and of the Malulorn decoder, the closest to them; of the Mefolorn decoder and of the Badolix decoder; of the
    Gopitar decoder and of the Kupirax decoder) at equal width, feed-forward, heads and layer count (random bfloat16 weights), and the device time of each of this library's kernels in one
    prompt step and one decode step of either, with the fraction of the measured peak it reaches."""
    import numpy as np
    import torch
    import cpp_minilamma_b200 as ml
    from cpp_minilamma_b200 import StepEntry
    peaks = load_peaks()
    warmup, steps = max(args.warmup, 3), max(min(args.steps, 64), 8)
    tokens, batch, context = PREFILL_TOKENS, 64, 1024
    design = args.design
    make_config = {"kupirax": kupirax_config, "malulorn": malulorn_config, "sopanex": sopanex_config,
                   "badolix": badolix_config, "mefolorn": mefolorn_config, "gopitar": gopitar_config}[design]
    rooflines = {"kupirax": design_rooflines, "malulorn": malulorn_rooflines, "sopanex": sopanex_rooflines,
                 "badolix": badolix_rooflines, "mefolorn": mefolorn_rooflines, "gopitar": gopitar_rooflines}[design]
    beside, beside_config = {"sopanex": ("malulorn", malulorn_config), "badolix": ("malulorn", malulorn_config),
                             "mefolorn": ("badolix", badolix_config),
                             "gopitar": ("kupirax", kupirax_config)}.get(design, ("llama", llama_like_config))
    result = {"design": design, "beside": beside, "dtype": "bf16", "data": "synthetic token ids, random-init weights",
              "prefill_tokens": tokens, "decode_prompts": "uniform[128,1024)", "steps": steps, "warmup": warmup,
              "peaks": {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "source": peaks["source"]},
              "sizes": {}}
    for size in ([args.size] if args.size else list(DESIGN_SIZES)):
        entry = {}
        expected = rooflines(size, tokens, batch, context, peaks)
        for model, cfg in ((design, make_config(size)), (beside, beside_config(size))):
            llm = ml.random_model(cfg, seed=0, dtype="bfloat16", max_tokens=batch * 1536 + 8192, max_positions=4096,
                                  max_seqs=batch, max_step_tokens=8192)
            numbers = {"layers": len(llm.model.spec.schedule), "parameters": llm.model.parameter_count()}
            ms = time_prefill(llm, tokens, reps=5, warmup=3, seed=3)
            numbers["prefill_tok_s"] = round(tokens * 1000.0 / ms, 1)
            numbers["prefill_ms"] = round(ms, 3)
            for b in (8, batch):
                d_ms, _, launches, _, _ = time_decode(llm, b, steps, warmup, seed=30 + b, prompt_range=(128, 1024),
                                                      repeats=3, context=4096)
                numbers[f"decode_b{b}_tok_s"] = round(b * 1000.0 / d_ms, 1)
                numbers[f"decode_b{b}_ms"] = round(d_ms, 4)
                numbers[f"decode_b{b}_launches"] = round(launches, 1)
            rng = np.random.RandomState(7)
            draw = lambda n: [int(t) for t in rng.randint(0, cfg.vocab_size, size=n)]

            def prompt_step():
                slot, = llm.engine.acquire(1)
                return [slot], [StepEntry(slot, draw(tokens), [tokens - 1])]

            kernels = {"prefill": kernel_times_of_a_step(llm, prompt_step)}
            slots = llm.engine.acquire(batch)
            llm.engine.step_borrowed([StepEntry(s, draw(context), [context - 1]) for s in slots])
            kernels["decode"] = kernel_times_of_a_step(llm, lambda: ([], [StepEntry(s, [5], [0]) for s in slots]))
            for s in slots:
                llm.engine.release(s)
            table = {}
            for kind, totals in kernels.items():
                for name, (calls, total_ms) in sorted(totals.items()):
                    row = {"calls": calls, "us_per_call": round(1000.0 * total_ms / calls, 2)}
                    table[f"{kind}: {name}"] = row
            entry[model] = numbers
            entry[model]["kernels"] = table
            for (m, kind, name), (bound, amount) in expected.items():
                if m != model:
                    continue
                # a kernel's launches may carry a suffix in brackets; a suffix with an entry of its own keeps that entry
                own = {f"{k2}: {n2}" for (m2, k2, n2) in expected if m2 == model}
                for key in [k for k in table if k == f"{kind}: {name}"
                            or (k.startswith(f"{kind}: {name} (") and k not in own)]:
                    us = table[key]["us_per_call"]
                    peak = peaks["hbm_gbs"] * 1e9 if bound == "hbm" else peaks["bf16_tflops"] * 1e12
                    table[key].update(bound=bound, frac=round(amount / (us * 1e-6) / peak, 4))
            release_model(llm)
        result["sizes"][size] = entry
    print(json.dumps(result))
    return 0


def main():
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=256)
    parser.add_argument("--warmup", type=int, default=8)
    parser.add_argument("--impl", default="ours", choices=["ours", "reference"])
    parser.add_argument("--layers", type=int, default=None, help="fewer layers than the model has (named in config)")
    parser.add_argument("--skip-points", action="store_true", help="leave out batch 1 and 64 and the further workloads")
    parser.add_argument("--skip-check", action="store_true", help="leave out the comparison with a float32 run")
    parser.add_argument("--profile", choices=["decode", "prefill"], default=None,
                        help="run one step of that kind between cudaProfilerStart/Stop (for ncu "
                             "--profile-from-start off) on a small case and exit; use with --layers")
    parser.add_argument("--shape", choices=sorted(SHAPES), default="llama31_8b", help="model shape of the --profile step")
    parser.add_argument("--batch", type=int, default=BATCH, help="batch of the --profile decode step")
    parser.add_argument("--context", type=int, default=1024, help="prompt length of the --profile decode step")
    parser.add_argument("--design", choices=["kupirax", "malulorn", "sopanex", "badolix", "mefolorn", "gopitar"], default=None,
                        help="instead of the default workload: prompt and decode throughput and kernel times of that "
                             "decoder beside the Llama decoder (sopanex, badolix: beside the Malulorn decoder; mefolorn: beside the Badolix decoder) at equal sizes")
    parser.add_argument("--size", choices=sorted(DESIGN_SIZES), default=None, help="one size of --design (default: all)")
    args = parser.parse_args()

    if args.impl == "reference":
        sys.path.insert(0, os.path.join(ROOT, "baseline"))
        import reference_arm
        return reference_arm.main(args)
    if args.gpus != 1:
        print(f"bench.py measures one GPU; --gpus {args.gpus} is not supported by this single-GPU library")
        return 2

    import torch
    import cpp_minilamma_b200 as ml
    if args.profile:
        return profile_region(args)
    if args.design:
        return bench_design(args)
    sampler = ClockSampler()
    sampler.start()  # nvidia-smi needs a moment before its first line: it runs through the set-up
    warmup = max(args.warmup, 3)
    steps = max(args.steps, 1)
    peaks = load_peaks()
    checked = {"checked": False, "check": "skipped"} if args.skip_check else check_against_float32()
    cfg = llama31_8b(args.layers)
    budget = 64 * (PROMPT_RANGE[1] + warmup + steps + 64)  # room for the batch-64 point
    llm = ml.random_model(cfg, seed=0, dtype="bfloat16", max_tokens=max(budget, BATCH * CONTEXT),
                          max_positions=CONTEXT, max_seqs=64, max_step_tokens=4096)
    # The prefill is one short step.  "ms" is the mean of isolated steps (half a second apart), the
    # condition of the burst GEMM figure it is held against; "ms_hot" is the same step back to back
    # after the decode loops, under the power cap, held against the sustained figure.
    prefill_ms = time_prefill(llm, PREFILL_TOKENS, reps=5, warmup=3, seed=3, pause=0.5)
    # the timed loop of exactly `steps` steps is repeated (at least 5 times and for at least 0.6 s, as far as the
    # context allows) and the median repeat is reported
    first_ms, _, _, _, _ = time_decode(llm, BATCH, steps, warmup, seed=1)
    repeats = max(5, min(60, int(600.0 / (first_ms * steps)) + 1))
    ms, live_tokens, launches, all_ms, _ = time_decode(llm, BATCH, steps, warmup, seed=1, sampler=sampler, repeats=repeats)
    clocks = sampler.summary()
    sampler.stop()
    value = BATCH * 1000.0 / ms
    achieved = decode_bytes(llm, live_tokens) / (ms * 1e-3) / 1e9

    e2e_value, e2e_after_prompt = time_e2e(llm, BATCH, steps, warmup, seed=2)
    # what a replayed decode step copies to the device: the captured step's index arrays and the parts' own lists
    # (counted from the buffer the engine copies; block-table rows ride along when a page is crossed)
    captured = [cap for key, cap in llm.engine.shared_decode_graphs()._captured.items() if key[0] == BATCH and cap.graph is not None]
    meta_ints = captured[0].updates_at if captured else 11 * BATCH
    d2h_ints = 2 * llm.engine.shared_sampler().rows  # the sampler's token ids and status words

    prefill_hot_ms = time_prefill(llm, PREFILL_TOKENS, reps=5, warmup=1, seed=3)
    flops = prefill_flops(cfg, PREFILL_TOKENS)
    points, workloads = {}, {}
    if not args.skip_points:
        for b in (1, 64):
            p_ms, p_live, _, _, _ = time_decode(llm, b, max(steps // 2, 8), warmup, seed=10 + b, repeats=5)
            points[f"decode_b{b}"] = round(b * 1000.0 / p_ms, 1)
            points[f"decode_b{b}_hbm_frac"] = round(decode_bytes(llm, p_live) / (p_ms * 1e-3) / 1e9 / peaks["hbm_gbs"], 4)
    release_model(llm)
    if not args.skip_points:
        for name in ("llama2_7b", "llama32_1b"):
            workloads[name] = time_workload(name, peaks, warmup, layers=None)

    line = {
        "metric": "decode tok/s at batch 8 (Llama-3.1-8B shape, random bf16 weights)",
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic token ids, random-init weights", "impl": "ours",
        "config": {"model": "Llama-3.1-8B shape", "layers": cfg.num_hidden_layers, "layers_full": 32,
                   "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads,
                   "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
                   "global_batch": BATCH, "seq_len": CONTEXT, "prompt_lens": "uniform[128,2048)",
                   "parallelism": "1 gpu", "l2": "inputs larger than L2 (15 GB of weights per step)",
                   "peaks": peaks["source"], "repeats": len(all_ms), "reported": "median repeat of `steps` steps"},
        "clocks": clocks,
        "e2e": {"value": round(e2e_value, 1), "unit": "tokens/s", "h2d_bytes_per_step": 4 * meta_ints,
                "d2h_bytes_per_step": 4 * d2h_ints, "warmup_steps": warmup,
                "first_steps_after_prompt": round(e2e_after_prompt, 1)},
        "gpu_launches": int(round(launches * steps)),
        "prefill": {"value": round(PREFILL_TOKENS * 1000.0 / prefill_ms, 1), "tokens": PREFILL_TOKENS,
                    "ms": round(prefill_ms, 3),
                    "frac": round(flops / (prefill_ms * 1e-3) / (peaks["bf16_tflops"] * 1e12), 4),
                    "ms_hot": round(prefill_hot_ms, 3),
                    "frac_hot": round(flops / (prefill_hot_ms * 1e-3) / (peaks["bf16_tflops_sustained"] * 1e12), 4),
                    "timing": "ms: 5 isolated steps 0.5 s apart; ms_hot: 5 steps back to back after the decode loops"},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / peaks["hbm_gbs"], 4)},
        "points": points,
        "workloads": workloads,
        "repeat_ms": [round(t, 4) for t in all_ms],
    }
    line.update(checked)
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
