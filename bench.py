#!/usr/bin/env python3
"""Decode and prefill throughput of the library on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch B] [--model 8b|14b|32b] [--impl ours|reference]
    python bench.py --design sanozen|gakenex|gazezen|biropel|dibesun|bimolix [--widths 2048,4096] [--layers 4]     (another record; see `design_comparison`)

A step is one decode step of the batch. The default run is the Qwen3-8B shape (every
layer size, all 36 layers) with random bfloat16 weights drawn on the device from a
seed, a batch of 8 sequences with 1,024-token prompts of uniform token ids, then 512
decoded tokens each. `--model 14b` and `--model 32b` run the other two shapes with their
batches of unequal prompts (16 prompts of 128 to 2,048 tokens, 8 prompts of 512 to 8,192
tokens; 256 steps). It prints ONE line of JSON:

* `value`: decoded tokens a second, timed on the device with CUDA events over exactly K
  steps after W warm-up steps (tokens selected and fed back on the device): the median
  of three measured repeats of the same prompts, whose token ids must be identical
  (the reference's protocol: benchmarks/README.md:27-35, benchmarks/cuda/run.py:48-49);
* `check`: what vouches for the timed work: the repeats' tokens were identical, and the
  first 16 tokens of the replayed graph are those of plain `Engine.step` calls fed with the
  same inputs (tokens that differ are counted, with the distance of the two candidates'
  logits: the graph may split a sequence's keys otherwise than a single step does, and
  bfloat16 rounding then reorders logits that lie closer together than it);
* `e2e`: the same through the Python entry point (`Engine.generate`): host token ids in
  and out; every step's tokens are read back to pinned host memory for the stop test
  while the next step, fed on the device, already runs;
* `prefill`: one 2,048-token prompt: tokens a second, milliseconds, and the fraction of
  the bfloat16 tensor-core peak its FLOPs reach;
* `roofline`: the decode step's bytes (every weight it uses once, plus the cache of the
  live sequences) over its time, against the measured HBM copy bandwidth;
* `points`: decode tokens a second at batch 1 and 64.

Every decode step reads about 16 GB of weights and cache, far more than the 126 MB L2, so
no L2 flush is needed between timed steps. Peaks come from MEASURED_PEAKS.json beside
this file when the driver wrote it. The reference arm cannot run here: the reference
does not build without its third-party submodules, which are empty in the mounted tree.
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_8B = {
    "architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3", "hidden_act": "silu",
    "num_hidden_layers": 36, "hidden_size": 4096, "num_attention_heads": 32, "num_key_value_heads": 8,
    "head_dim": 128, "intermediate_size": 12288, "vocab_size": 151936, "rope_theta": 1000000.0,
    "rms_norm_eps": 1e-6, "tie_word_embeddings": False, "max_position_embeddings": 40960, "attention_bias": False,
}
QWEN3_14B = dict(QWEN3_8B, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408)
QWEN3_32B = dict(QWEN3_8B, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, intermediate_size=25600)
# name -> (configuration, batch, (shortest, longest) prompt, decode steps): the benchmark's three shapes
MODELS = {
    "8b": ("Qwen3-8B shape", QWEN3_8B, 8, (1024, 1024), 512),
    "14b": ("Qwen3-14B shape", QWEN3_14B, 16, (128, 2048), 256),
    "32b": ("Qwen3-32B shape", QWEN3_32B, 8, (512, 8192), 256),
}
PREFILL_TOKENS = 2048
CHECKED_STEPS = 16
ROUNDING_DISTANCE = 2.5e-2   # of the largest logit: the bfloat16 bound of the benchmark-shape test
REPEATS = 3
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    try:
        with open(path) as handle:
            found = json.load(handle)
        hbm = float(found.get("hbm_gbs") or found.get("hbm_gb_s"))
        tflops = float(found.get("bf16_tflops"))
        sustained = float(found.get("bf16_tflops_sustained") or tflops)
        return {"hbm_gbs": hbm, "bf16_tflops": tflops, "bf16_tflops_sustained": sustained, "source": "measured"}
    except (OSError, ValueError, TypeError, KeyError):
        return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.lines, self.process, self.index = [], None, index

    def start(self):
        try:
            self.process = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.index)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.process = None

    def _read(self):
        for line in self.process.stdout:
            self.lines.append(line.strip())

    def stop(self) -> dict:
        if self.process is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.process.terminate()
        clocks, maxima, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in self.lines:
            fields = [field.strip() for field in line.split(",")]
            if len(fields) < 6 or not fields[0].isdigit():
                continue
            clocks.append(int(fields[0]))
            maxima.append(int(fields[1]))
            reasons.update(name for name, field in zip(names, fields[2:6]) if field.lower().startswith("active"))
        return {"sm_mhz": statistics.median(clocks) if clocks else None,
                "sm_max_mhz": max(maxima) if maxima else None, "reasons": sorted(reasons), "samples": len(clocks)}


def decode_bytes(config: dict, batch: int, context: float) -> float:
    """Bytes a decode step has to read: every weight it uses once (bfloat16), the
    embedding rows of the batch, and the keys and values of the live sequences."""
    hidden, inter, layers = config["hidden_size"], config["intermediate_size"], config["num_hidden_layers"]
    q = config["num_attention_heads"] * config["head_dim"]
    kv = config["num_key_value_heads"] * config["head_dim"]
    per_layer = hidden * (q + 2 * kv) + q * hidden + 3 * hidden * inter + 2 * hidden + 2 * config["head_dim"]
    weights = 2 * (layers * per_layer + config["vocab_size"] * hidden + hidden + batch * hidden)
    cache = 2 * layers * 2 * kv * context * batch
    return float(weights + cache)


def prefill_flops(config: dict, tokens: int) -> float:
    hidden, inter, layers = config["hidden_size"], config["intermediate_size"], config["num_hidden_layers"]
    q = config["num_attention_heads"] * config["head_dim"]
    kv = config["num_key_value_heads"] * config["head_dim"]
    linear = 2.0 * tokens * layers * (hidden * (q + 2 * kv) + q * hidden + 3 * hidden * inter)
    attention = layers * 4.0 * q * tokens * (tokens + 1) / 2
    head = 2.0 * config["vocab_size"] * hidden
    return linear + attention + head


def draw_prompts(vocab: int, batch: int, lengths, seed: int):
    """`batch` prompts of uniform token ids whose lengths are uniform in [lengths[0], lengths[1]]."""
    import numpy as np
    generator = np.random.default_rng(seed)
    sizes = [lengths[0]] * batch if lengths[0] == lengths[1] else generator.integers(lengths[0], lengths[1] + 1, size=batch)
    return [generator.integers(0, vocab, size=int(size)).tolist() for size in sizes]


def time_decode(engine, sampler, prompts, steps: int, warmup: int, clocks: bool, repeats: int = REPEATS,
                profile_steps: int = 0):
    """Device-timed decode, `repeats` times over: the prompts in one step, then `warmup` +
    `steps` replayed steps with tokens selected and fed back on the device, every step's
    tokens kept on the device. Returns the median repeat's measurements, the tokens of the
    first repeat and whether every repeat produced the same tokens."""
    import torch
    from kidi_b200 import StepBatch
    from kidi_b200.engine.decode_graph import DecodeSession

    batch = len(prompts)
    longest = max(len(prompt) for prompt in prompts) + warmup + steps + 1
    session = DecodeSession(engine, batch, sampler, longest=longest)
    history = torch.zeros((warmup + steps, batch), dtype=torch.int32, device=engine.device)
    runs, tokens_of_repeat, clock_record = [], [], None
    for repeat in range(repeats):
        slots = [engine.acquire() for _ in range(batch)]
        try:
            logits = engine.step(StepBatch(slots, prompts, None))
            first = sampler.select(logits).cpu().tolist()
            session.load(slots, first, [0.0] * batch, list(range(batch)), [1] * batch)
            session.reserve(warmup + steps)
            for step in range(warmup):
                session.launch()
                history[step].copy_(session.selected, non_blocking=True)
            torch.cuda.synchronize()
            sampler_thread = ClockSampler() if clocks and repeat == repeats - 1 else None
            if sampler_thread:
                sampler_thread.start()
                time.sleep(0.25)
            begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            begin.record()
            for step in range(steps):
                session.launch()
                history[warmup + step].copy_(session.selected, non_blocking=True)   # 4 bytes a sequence, on the device
            end.record()
            torch.cuda.synchronize()
            runs.append(begin.elapsed_time(end) / steps)
            if sampler_thread:
                clock_record = sampler_thread.stop()
            tokens_of_repeat.append([first] + history.cpu().tolist())
            if profile_steps and repeat == repeats - 1:  # a few more steps inside a profiler range
                session.reserve(profile_steps)
                torch.cuda.profiler.start()
                for _ in range(profile_steps):
                    session.launch()
                torch.cuda.synchronize()
                torch.cuda.profiler.stop()
        finally:
            for slot in slots:
                engine.release(slot)
    ms = statistics.median(runs)
    mean_prompt = sum(len(prompt) for prompt in prompts) / batch
    return {"ms_per_step": ms, "tokens_per_s": batch * 1e3 / ms, "ms_of_repeats": [round(run, 4) for run in runs],
            "kernels_per_step": session.kernels_per_step, "clocks": clock_record,
            "mean_context": mean_prompt + warmup + (steps + 1) / 2, "tokens": tokens_of_repeat[0],
            "repeats_identical": all(tokens == tokens_of_repeat[0] for tokens in tokens_of_repeat)}


def compare_with_plain_steps(engine, sampler, prompts, graph_tokens, steps: int):
    """The same prompts through `Engine.step`, one launch at a time and no graph, fed at every
    step with the tokens the replayed graph selected (so that one differing token does not set
    the two runs apart for good). Returns (tokens compared, tokens that differ, the largest
    distance between the two candidates' logits at a differing token, relative to the largest
    logit of its row). The two paths may split a sequence's keys differently (the graph fixes
    the split for the longest sequence it may hold), so bfloat16 rounding can reorder two logits
    that lie closer than that rounding; a fault would show as a large distance."""
    import torch
    from kidi_b200 import StepBatch
    slots = [engine.acquire() for _ in prompts]
    compared = differing = 0
    largest = 0.0
    try:
        logits = engine.step(StepBatch(slots, prompts, None))
        for step in range(steps + 1):
            chosen = sampler.select(logits).cpu().tolist()
            wanted = graph_tokens[step]
            for row, (mine, theirs) in enumerate(zip(chosen, wanted)):
                compared += 1
                if mine != theirs:
                    differing += 1
                    values = logits[row]
                    distance = float((values[mine] - values[theirs]).abs() / values.abs().max().clamp(min=1.0))
                    largest = max(largest, distance)
            if step < steps:
                logits = engine.step(StepBatch(slots, [[token] for token in wanted], None))
        return compared, differing, largest
    finally:
        for slot in slots:
            engine.release(slot)


def time_prefill(engine, seed: int, repeats: int = 5, profile: bool = False):
    import numpy as np
    import torch
    from kidi_b200 import StepBatch

    generator = np.random.default_rng(seed)
    prompt = generator.integers(0, engine.vocab_size, size=PREFILL_TOKENS).tolist()
    times = []
    for index in range(repeats + 2):
        slot = engine.acquire()
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        begin.record()
        engine.step(StepBatch([slot], [prompt], None))
        end.record()
        torch.cuda.synchronize()
        engine.release(slot)
        if index >= 2:  # two warm-up runs
            times.append(begin.elapsed_time(end))
    if profile:
        slot = engine.acquire()
        torch.cuda.profiler.start()
        engine.step(StepBatch([slot], [prompt], None))
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
        engine.release(slot)
    return statistics.median(times)


def time_end_to_end(engine, prompts, steps: int):
    """Decode tokens a second through `Engine.generate`: host token ids in and out. Returns
    the rate, the statistics and the generated tokens."""
    from kidi_b200.engine.generate import GenerationStats

    batch = len(prompts)
    engine.generate(prompts, max_new_tokens=steps + 1, ignore_eos=True, max_active=batch)   # captures the graph
    stats = GenerationStats()
    found = engine.generate(prompts, max_new_tokens=steps + 1, ignore_eos=True, max_active=batch, stats=stats)
    return batch * stats.decode_steps / (stats.decode_ns / 1e9), stats, found


# ---------------------------------------------------------------------------------------------- --design sanozen
def sanozen_shape(width: int, layers: int = 4) -> dict:
    """A Sanozen stack at the layer sizes of a model of `width`: heads of 128 (64 plain + 64 rotated query/key
    dimensions, values of 128), a latent of width / 8, query latents of 3 width / 8, recurrent heads of 128 x 128,
    dense feed-forwards of 4 width; latent attention and recurrence in turn, every other attention layer reading
    the cached rows of the one before it."""
    heads = width // 128
    attention = {"heads": heads, "dim": 64, "rot_dim": 64, "vdim": 128, "q_rank": 3 * width // 8,
                 "kv_rank": width // 8, "scale": 128 ** -0.5, "rot": {"base": 1000000.0, "dims": 64}}
    recurrent = {"heads": heads, "dim": 128, "vdim": 128}
    stack, source = [], None
    for index in range(layers):
        if index % 2 == 0:
            mixer = dict(attention)
            if source is not None:
                mixer["kv_from"], source = source, None
            else:
                source = index
            stack.append({"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": 4 * width}})
        else:
            stack.append({"type": "hgrn2", "mixer": dict(recurrent), "mlp": {"kind": "dense", "ff": 4 * width}})
    return {"architecture": "Sanozen", "vocab": 32768, "width": width, "embedding": {"scale": 1.0},
            "norm": {"eps": 1e-5}, "token_side": {"dim": 64}, "layers": stack, "max_positions": 8192}


def gakenex_shape(width: int, layers: int = 4) -> dict:
    """A Gakenex stack at the layer sizes of a model of `width`: heads with two maps of 64 and values of 128, a
    key/value head for four heads, four convolution taps, a window of 4,096 with eight kept tokens; dense
    feed-forwards of the Qwen3 layers' size in turn with routed ones (16 experts, two a token, each half that
    size, so that a token uses as many weights)."""
    heads = width // 128
    inter = (8 * width // 3 + 127) // 128 * 128
    mixer = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 64, "vdim": 128, "conv": 4, "diff": 0.5,
             "scale": 64 ** -0.5, "mask": {"size": 4096, "keep_first": 8}}
    stack = []
    for index in range(layers):
        mlp = {"kind": "dense", "ff": inter, "limit": 7.0} if index % 2 == 0 else \
            {"kind": "moe", "expert": {"ff": inter // 2}, "router": {"experts": 16, "top": 2}}
        stack.append({"type": "attention", "mixer": dict(mixer), "mlp": mlp})
    return {"architecture": "Gakenex", "vocab": 32768, "width": width, "max_positions": 8192, "norm": {"eps": 1e-5},
            "logit_softcap": 30.0, "layers": stack}


def gazezen_shape(width: int, layers: int = 4) -> dict:
    """A Gazezen stack at the layer sizes of a model of `width`: attention layers (heads of 128, a key/value head
    for four heads, half of a head rotated, a window of 4,096, sinks and head gates) in turn with latent
    attention layers (64 plain + 64 rotated query/key dimensions, values of 128, a latent of width / 8, stretched
    frequencies, the same window and gates); every layer's feed-forward routes over 16 plain gelu experts in four
    groups of which two are kept, two experts a token plus a shared one, each of half the Qwen3 layers'
    feed-forward size (a token uses as many feed-forward weights). No range of layers is run twice, so that both
    stacks run as many layers."""
    heads = width // 128
    inter = (8 * width // 3 + 127) // 128 * 128
    mlp = {"kind": "moe", "expert": {"ff": inter // 2}, "router": {"experts": 16, "top": 2, "groups": {"count": 4, "keep": 2}},
           "shared": {"ff": inter // 2}}
    attention = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "mask": {"size": 4096}, "rot": {"base": 10000.0, "dims": 64}}
    latent = {"heads": heads, "dim": 64, "rot_dim": 64, "vdim": 128, "kv_rank": width // 8, "scale": 128 ** -0.5,
              "mask": {"size": 4096}, "rot": {"base": 10000.0, "dims": 64, "scaling": {
                  "factor": 8.0, "original": 1024.0, "fast": 32.0, "slow": 1.0}}}
    stack = [{"type": "attention" if index % 2 == 0 else "latent_attention",
              "mixer": dict(attention if index % 2 == 0 else latent), "mlp": dict(mlp)} for index in range(layers)]
    return {"architecture": "Gazezen", "vocab": 32768, "width": width, "max_positions": 8192, "norm": {"eps": 1e-5},
            "logit_scale": 0.7, "layers": stack}


def biropel_shape(width: int, layers: int = 4) -> dict:
    """A Biropel stack at the layer sizes of a model of `width`, its kinds of layer in turn: an attention layer
    (heads of 128, a key/value head for four heads, half of a head rotated, a window of 4,096, biases, an element-wise
    gate), an attention layer that reads the keys and values of the one before it, attention with stretched
    frequencies and bounded scores (half the heads) beside a state-space mixer (heads of 64 values, inner width =
    width, a state of 128 rows, four taps), and attention with normalised queries and keys, a query temperature and
    bounded scores (half the heads, every earlier token visible) beside a matrix memory (heads of 128 x 128, half the
    heads). Squared-relu feed-forwards of 4 width (as many weights as the Qwen3 layers' gated ones); two lanes."""
    heads = width // 128
    groups = max(1, heads // 4)
    half, half_groups = max(1, heads // 2), max(1, heads // 8)
    mlp = {"kind": "dense", "ff": 4 * width}
    base = {"heads": heads, "kv_heads": groups, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 4096},
            "rot": {"base": 10000.0, "dims": 64}}
    stretched = {"heads": half, "kv_heads": half_groups, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "mask": {"size": 4096}, "softcap": 50.0, "rot": {"base": 100000.0, "dims": 128, "scaling": {
                     "factor": 8.0, "original": 1024.0, "fast": 32.0, "slow": 1.0}}}
    unrotated = {"heads": half, "kv_heads": half_groups, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0,
                 "q_temp": {"coef": 0.1, "every": 1024}}
    kinds = [
        lambda: {"type": "attention", "mixer": dict(base), "mlp": dict(mlp)},
        lambda source: {"type": "attention", "mixer": dict(base, kv_from=source), "mlp": dict(mlp)},
        lambda: {"type": "parallel", "mixer": {"left": dict(stretched), "right": {
            "heads": width // 64, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 8}}, "mlp": dict(mlp)},
        lambda: {"type": "parallel_2", "mixer": {"left": dict(unrotated), "right": {
            "heads": half, "dim": 128, "vdim": 128, "gate_cap": 20.0}}, "mlp": dict(mlp)},
    ]
    stack = []
    for index in range(layers):
        stack.append(kinds[1](index - 1) if index % 4 == 1 else kinds[index % 4]())
    return {"architecture": "Biropel", "vocab": 32768, "width": width, "max_positions": 8192, "norm": {"eps": 1e-5},
            "streams": 2, "layers": stack}


def dibesun_shape(width: int, layers: int = 4) -> dict:
    """A Dibesun stack at the layer sizes of a model of `width`: in every layer attention with sigmoid weights (half the
    heads, of 128, a key/value head for four heads, runs of 1,536 positions, bounded scores) beside linear attention (as
    many heads of 128 x 128); dense SiLU-gated feed-forwards of the Qwen3 layers' size in turn with sixteen routed
    experts of a quarter of it, two a token, plus a shared one of half of it (a token uses as many feed-forward
    weights); norms in eight parts."""
    heads = max(1, width // 256)
    inter = (8 * width // 3 + 127) // 128 * 128
    left = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
            "softcap": 50.0, "mask": {"size": 1536}}
    right = {"heads": heads, "dim": 128, "vdim": 128,
             "decay": [1.0 - 2.0 ** (-1.0 - 9.0 * index / max(1, heads - 1)) for index in range(heads)]}
    mixer = {"left": left, "right": right, "left_scale": 0.8, "right_scale": 0.6}
    dense = {"kind": "dense", "ff": inter}
    routed = {"kind": "moe", "expert": {"ff": inter // 4}, "router": {"experts": 16, "top": 2}, "shared": {"ff": inter // 2}}
    stack = [{"type": "parallel", "mixer": mixer, "mlp": dense if index % 2 == 0 else routed} for index in range(layers)]
    return {"architecture": "Dibesun", "vocab": 32768, "width": width, "max_positions": 8192,
            "norm": {"eps": 1e-5, "groups": 8}, "embedding": {"scale": 2.0}, "layers": stack}


def bimolix_shape(width: int, layers: int = 4) -> dict:
    """A Bimolix stack at the layer sizes of a model of `width`: retention (heads of 128 x 128, whole heads rotated) with a
    dense SiLU-gated feed-forward of the Qwen3 layers' size in turn with attention whose values are its keys (as many heads
    of 128, a key/value head for four heads, runs of 4,096 positions, 32 distance buckets up to 1,024) with sixteen routed
    experts of a quarter of that size in four groups of which two are kept, two experts a token, plus a shared one of half of
    it (a token uses as many feed-forward weights)."""
    heads = width // 128
    inter = (8 * width // 3 + 127) // 128 * 128
    retention = {"heads": heads, "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 128},
                 "decay": [1.0 - 2.0 ** (-2.0 - 8.0 * index / max(1, heads - 1)) for index in range(heads)]}
    attention = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "bias_max": 1024, "mask": {"size": 4096}}
    routed = {"kind": "moe", "expert": {"ff": inter // 4, "limit": 7.0},
              "router": {"experts": 16, "top": 2, "groups": {"count": 4, "keep": 2}, "scale": 1.5},
              "shared": {"ff": inter // 2, "limit": 7.0}}
    stack = [{"type": "retention", "mixer": retention, "mlp": {"kind": "dense", "ff": inter}} if index % 2 == 0 else
             {"type": "attention", "mixer": attention, "mlp": routed} for index in range(layers)]
    return {"architecture": "Bimolix", "vocab": 32768, "width": width, "max_positions": 8192, "norm": {"eps": 1e-5},
            "layers": stack}


DESIGN_SHAPES = {"sanozen": sanozen_shape, "gakenex": gakenex_shape, "gazezen": gazezen_shape, "biropel": biropel_shape,
                 "dibesun": dibesun_shape, "bimolix": bimolix_shape}


def qwen3_shape(width: int, layers: int = 4) -> dict:
    """The closest existing model at equal size: Qwen3 layers of the same width and head count (a key/value head for
    four heads) whose gated feed-forward has as many weights as the dense one of 4 width."""
    heads = width // 128
    return dict(QWEN3_8B, num_hidden_layers=layers, hidden_size=width, num_attention_heads=heads,
                num_key_value_heads=max(1, heads // 4), intermediate_size=(8 * width // 3 + 127) // 128 * 128,
                vocab_size=32768, max_position_embeddings=8192)


KERNEL_CLASSES = (
    ("products", ("gemm_", "library_mm", "library_bmm", "gemm_heads")),
    ("prompt attention", ("attention_prefill",)),
    ("decode attention", ("attention_decode", "latent_attention")),
    ("recurrence", ("gated_recurrence", "scalar_recurrence", "linear_attention", "retention")),
    ("stream norm", ("add_rmsnorm", "add_layernorm", "lanes_", "add_parts_norm")),
    ("activation", ("silu_gate", "poly_norm", "bounded_gate", "gelu", "relu_squared", "silu_columns")),
    ("experts through the choice", ("expert_slots",)),
)


def kernel_class(name: str, decode: bool = False) -> str:
    if name.startswith("diff_attention") or name == "attention":      # (`attention`: the general kernel)
        return "decode attention" if decode else "prompt attention"
    for label, prefixes in KERNEL_CLASSES:
        if name.startswith(prefixes):
            return label
    return "other row-wise kernels"


def timed_step(engine, slots, tokens, decode: bool = False) -> dict:
    """One `Engine.step` with every launch timed on the device: microseconds and launches per class of kernel."""
    from kidi_b200 import StepBatch
    from kidi_b200.kernels import ops
    with ops.time_launches() as timed:
        engine.step(StepBatch(slots, tokens, None))
    classes: dict = {}
    for name, microseconds in timed.spans():
        entry = classes.setdefault(kernel_class(name, decode), {"us": 0.0, "launches": 0, "kernels": {}})
        entry["us"] += microseconds
        entry["launches"] += 1
        kernel = entry["kernels"].setdefault(name.split(",")[0], [0, 0.0])
        kernel[0] += 1
        kernel[1] += microseconds
    for entry in classes.values():
        entry["us"] = round(entry["us"], 1)
        entry["kernels"] = {name: [count, round(us, 1)] for name, (count, us) in entry["kernels"].items()}
    return classes


def class_work(design: str, config: dict, rows: int, context: int, decode: bool) -> dict:
    """What each class of kernel has to do in one step, per the algorithm: ("flops" | "bytes", amount). Prompts:
    `rows` tokens of one sequence from position 0; decoding: `rows` sequences of `context` tokens."""
    work = {}
    if design == "qwen3":
        width, inter, layers = config["hidden_size"], config["intermediate_size"], config["num_hidden_layers"]
        heads, kv, hd = config["num_attention_heads"], config["num_key_value_heads"], config["head_dim"]
        weights = layers * (width * (heads + 2 * kv) * hd + heads * hd * width + 3 * width * inter) + config["vocab_size"] * width
        norms, act_width = 2 * layers + 1, layers * inter * 3          # gate and up read, the product written
        work["prompt attention"] = ("flops", layers * 4.0 * heads * hd * rows * (rows + 1) / 2)
        work["decode attention"] = ("bytes", layers * rows * context * kv * hd * 2 * 2.0)
    elif design == "gakenex":
        width, layers = config["width"], config["layers"]
        weights, norms, act_width, attention, cache, chosen = config["vocab"] * width, 2, 0, 0.0, 0.0, 0.0
        for layer in layers:
            m, mlp = layer["mixer"], layer["mlp"]
            heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            weights += width * (2 * (heads + groups) * dim + groups * vdim + heads * vdim) + heads * vdim * width
            norms += 1
            attention += 4.0 * heads * (dim + vdim) * rows * (rows + 1) / 2      # two maps: scores of dim, sums of vdim
            cache += rows * context * groups * (2 * dim + vdim) * 2.0
            if mlp["kind"] == "dense":
                weights += 3 * width * mlp["ff"]
                act_width += 3 * mlp["ff"]
            else:
                used = 3 * width * mlp["expert"]["ff"] * mlp["router"]["top"]        # per token
                if decode:     # each (row, choice) streams its expert's weights (rows * top <= experts here)
                    chosen += rows * used * 2.0
                else:
                    weights += used
                    act_width += 3 * mlp["expert"]["ff"] * mlp["router"]["top"]
        work["prompt attention"] = ("flops", attention)
        work["decode attention"] = ("bytes", cache)
        if decode:
            work["experts through the choice"] = ("bytes", chosen)
    elif design == "gazezen":
        width, layers = config["width"], config["layers"]
        weights, norms, act_width, attention, cache, chosen = config["vocab"] * width, 1, 0, 0.0, 0.0, 0.0
        for layer in layers:
            m, mlp = layer["mixer"], layer["mlp"]
            heads, vdim = m["heads"], m["vdim"]
            norms += 4 if mlp else 2
            if layer["type"] == "attention":
                groups, dim = m["kv_heads"], m["dim"]
                weights += width * (heads * dim + groups * (dim + vdim) + heads) + heads * vdim * width
                attention += 2.0 * heads * (dim + vdim) * rows * (rows + 1) / 2
                cache += rows * min(context, m["mask"]["size"]) * groups * (dim + vdim) * 2.0
            else:
                head, rank = m["dim"] + m["rot_dim"], m["kv_rank"]
                weights += width * (heads * head + rank + m["rot_dim"] + heads) + heads * (m["dim"] + vdim) * rank \
                    + heads * vdim * width
                attention += 4.0 * heads * head * rows * (rows + 1) / 2             # values padded to the key width
                cache += rows * min(context, m["mask"]["size"]) * (rank + m["rot_dim"]) * 2.0
            if mlp:
                router, ff, shared = mlp["router"], mlp["expert"]["ff"], (mlp.get("shared") or {}).get("ff", 0)
                weights += router["experts"] * width + 2 * width * shared
                used = 2 * width * ff * router["top"]                                # per token
                act_width += 2 * shared
                if decode:     # each (row, choice) streams its expert's weights (rows * top <= experts here)
                    chosen += rows * used * 2.0
                else:
                    weights += used
                    act_width += 2 * ff * router["top"]
        work["prompt attention"] = ("flops", attention)
        work["decode attention"] = ("bytes", cache)
        if decode:
            work["experts through the choice"] = ("bytes", chosen)
    elif design == "biropel":
        width, layers, lanes = config["width"], config["layers"], config.get("streams") or 1
        weights, norms, act_width, attention, cache, scan, stream = config["vocab"] * width, 0, 0, 0.0, 0.0, 0.0, 0.0
        sequences = rows if decode else 1
        for layer in layers:
            ff = layer["mlp"]["ff"] if layer["mlp"] else 0
            weights += 2 * width * ff
            act_width += 2 * ff                                      # read and written
            sublayers = 2 if ff else 1
            # a norm reads every lane and writes bfloat16 rows; an update reads the lanes and the result, writes the lanes
            stream += sublayers * rows * width * ((4 * lanes + 2) + (8 * lanes + 4.0))
            left = layer["mixer"] if layer["type"] == "attention" else layer["mixer"]["left"]
            heads, groups, dim, vdim = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
            own = 0 if "kv_from" in left else groups * (dim + vdim)
            gate = heads * vdim if layer["type"] == "attention" else 0
            weights += width * (heads * dim + own + gate) + heads * vdim * width
            attention += 2.0 * heads * (dim + vdim) * rows * (rows + 1) / 2
            reach = min(context, left["mask"]["size"]) if "mask" in left else context
            cache += rows * reach * groups * (dim + vdim) * 2.0
            right = layer["mixer"].get("right")
            if layer["type"] == "parallel":
                inner, span = right["heads"] * right["vdim"], right["groups"] * right["state"]
                weights += width * (2 * inner + 2 * span + right["heads"]) + inner * width
                scan += rows * (inner + 2 * span) * 2.0 + rows * inner * 4.0 \
                    + sequences * 2.0 * right["heads"] * right["state"] * right["vdim"] * 4
            elif layer["type"] == "parallel_2":
                keys, values = right["heads"] * right["dim"], right["heads"] * right["vdim"]
                weights += width * (2 * keys + 2 * values + 2 * right["heads"]) + values * width
                scan += rows * (2 * keys + values) * 2.0 + rows * (values + right["heads"]) * 4.0 \
                    + sequences * 2.0 * right["heads"] * right["dim"] * (right["vdim"] + 1) * 4
        work["prompt attention"] = ("flops", attention)
        work["decode attention"] = ("bytes", cache)
        work["recurrence"] = ("bytes", scan)
        norms = 2                                                     # the embedding's norm and the final one
    elif design == "dibesun":
        width, layers = config["width"], config["layers"]
        weights, norms, act_width, attention, cache, chosen, scan = config["vocab"] * width, 1, 0, 0.0, 0.0, 0.0, 0.0
        for layer in layers:
            left, right, mlp = layer["mixer"]["left"], layer["mixer"]["right"], layer["mlp"]
            heads, groups, dim, vdim, chunk = left["heads"], left["kv_heads"], left["dim"], left["vdim"], left["mask"]["size"]
            keys, values = right["heads"] * right["dim"], right["heads"] * right["vdim"]
            norms += 2
            weights += width * (heads * dim + groups * (dim + vdim) + 2 * keys + 2 * values) + (heads * vdim + values) * width
            act_width += 0 if decode else 2 * (2 * keys + values)        # decoding: in the product's epilogue
            whole, rest = divmod(rows, chunk)
            pairs = whole * chunk * (chunk + 1) / 2 + rest * (rest + 1) / 2
            attention += 2.0 * heads * (dim + vdim) * pairs
            cache += rows * ((context - 1) % chunk + 1) * groups * (dim + vdim) * 2.0
            scan += rows * (2 * keys + values) * 2.0 + rows * values * 4.0 \
                + (rows if decode else 1) * 2.0 * right["heads"] * right["dim"] * right["vdim"] * 4
            if mlp["kind"] == "dense":
                weights += 3 * width * mlp["ff"]
                act_width += 0 if decode else 3 * mlp["ff"]
                continue
            router, ff, shared = mlp["router"], mlp["expert"]["ff"], mlp["shared"]["ff"]
            weights += router["experts"] * width + 3 * width * shared
            used = 3 * width * ff * router["top"]                                    # per token
            act_width += 3 * shared
            if decode:         # each (row, choice) streams its expert's weights
                chosen += rows * used * 2.0
            else:
                weights += used
                act_width += 3 * ff * router["top"]
        work["prompt attention"] = ("flops", attention)
        work["decode attention"] = ("bytes", cache)
        work["recurrence"] = ("bytes", scan)
        if decode:
            work["experts through the choice"] = ("bytes", chosen)
    elif design == "bimolix":
        width, layers = config["width"], config["layers"]
        weights, norms, act_width, attention, cache, chosen, scan = config["vocab"] * width, 2, 0, 0.0, 0.0, 0.0, 0.0
        for layer in layers:
            m, mlp = layer["mixer"], layer["mlp"]
            heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
            norms += 2
            if layer["type"] == "retention":
                keys, values = heads * dim, heads * vdim
                weights += width * (2 * keys + 2 * values) + values * width
                # q, k, v and the gate read, the gated result written; the state read and written
                scan += rows * (2 * keys + 3 * values) * 2.0 + (rows if decode else 1) * 2.0 * heads * dim * vdim * 4
            else:
                groups, chunk = m["kv_heads"], m["mask"]["size"]
                weights += width * (2 * heads * dim + groups * dim) + heads * dim * width
                whole, rest = divmod(rows, chunk)
                attention += 4.0 * heads * dim * (whole * chunk * (chunk + 1) / 2 + rest * (rest + 1) / 2)
                cache += rows * ((context - 1) % chunk + 1) * groups * dim * 2.0         # a key is its value
            if mlp["kind"] == "dense":
                weights += 3 * width * mlp["ff"]
                act_width += 0 if decode else 3 * mlp["ff"]
                continue
            router, ff, shared = mlp["router"], mlp["expert"]["ff"], mlp["shared"]["ff"]
            weights += (router["experts"] + 1) * width + 3 * width * shared
            used = 3 * width * ff * router["top"]                                    # per token
            act_width += 0 if decode else 3 * shared                                 # (the routed gate: in the epilogue)
            if decode:         # each (row, choice) streams its expert's weights
                chosen += rows * used * 2.0
            else:
                weights += used
        work["prompt attention"] = ("flops", attention)
        work["decode attention"] = ("bytes", cache)
        work["recurrence"] = ("bytes", scan)
        if decode:
            work["experts through the choice"] = ("bytes", chosen)
    else:
        width, layers = config["width"], config["layers"]
        weights, norms, act_width, attention, cache, scan_flops, scan_bytes, state = config["vocab"] * width, 1, 0, 0.0, 0.0, 0.0, 0.0, 0.0
        for layer in layers:
            m, ff = layer["mixer"], layer["mlp"]["ff"] if layer["mlp"] else 0
            weights += 2 * width * ff + 2 * width * config["token_side"]["dim"]
            norms += 2 if ff else 1
            act_width += 2 * ff
            if layer["type"] == "latent_attention":
                head = m["dim"] + m["rot_dim"]
                weights += width * m["q_rank"] + m["q_rank"] * m["heads"] * head + m["heads"] * (m["dim"] + m["vdim"]) * m["kv_rank"] \
                    + m["heads"] * m["vdim"] * width + (0 if "kv_from" in m else width * (m["kv_rank"] + m["rot_dim"]))
                attention += 4.0 * m["heads"] * head * rows * (rows + 1) / 2       # values padded to the key width
                cache += rows * context * (m["kv_rank"] + m["rot_dim"]) * 2.0
            else:
                weights += width * m["heads"] * (2 * m["dim"] + m["vdim"]) + m["heads"] * m["vdim"] * width
                scan_flops += 4.0 * rows * m["heads"] * m["dim"] * m["vdim"]
                scan_bytes += rows * m["heads"] * (2 * m["dim"] + 2 * m["vdim"]) * 2.0
                state += 2.0 * m["heads"] * m["dim"] * m["vdim"] * 4
        work["prompt attention"] = ("flops", attention)
        work["decode attention"] = ("bytes", cache)
        work["recurrence"] = ("bytes", scan_bytes + (rows if decode else 1) * state)
    work["products"] = ("bytes", 2.0 * weights) if decode else ("flops", 2.0 * rows * weights)
    work["stream norm"] = ("bytes", norms * rows * width * (4 + 4 + 2 + 2.0) + (stream if design == "biropel" else 0.0))
    work["activation"] = ("bytes", rows * act_width * 2.0)
    if decode:
        work.pop("prompt attention")
    else:
        work.pop("decode attention")
    return work


def design_comparison(args) -> int:
    """`--design <one of DESIGN_SHAPES>`: prompts and decoding of a stack of that design beside Qwen3 layers
    of equal size, with every class of kernel against its roofline."""
    import torch
    from kidi_b200 import Engine
    from kidi_b200.sampling.sampler import Sampler

    peak = peaks()
    sampler = Sampler(args.seed)
    batch, context, steps = args.batch or 8, 1024, args.steps or 64
    sizes = []
    for width in [int(value) for value in args.widths.split(",")]:
        point = {"width": width}
        for design, shape in ((args.design, DESIGN_SHAPES[args.design](width, args.layers or 4)),
                              ("qwen3", qwen3_shape(width, args.layers or 4))):
            engine = Engine.from_config(shape, seed=args.seed, dtype="bfloat16", device="cuda:0",
                                        max_tokens=max(batch * (context + steps + 64 + args.warmup), 4096))
            from kidi_b200 import StepBatch
            prefill_ms = time_prefill(engine, args.seed)
            prompts = draw_prompts(engine.vocab_size, batch, (context, context), args.seed)
            run = time_decode(engine, sampler, prompts, steps, args.warmup, clocks=False, repeats=1)
            slot = engine.acquire()
            prompt = draw_prompts(engine.vocab_size, 1, (PREFILL_TOKENS, PREFILL_TOKENS), args.seed + 1)[0]
            engine.step(StepBatch([slot], [prompt], None))       # the same step once before: its buffers are allocated
            engine.release(slot)
            slot = engine.acquire()
            prompt_classes = timed_step(engine, [slot], [prompt])
            engine.release(slot)
            slots = [engine.acquire() for _ in range(batch)]
            engine.step(StepBatch(slots, prompts, None))
            engine.step(StepBatch(slots, [[1]] * batch, None))           # every decode kernel is built and configured
            decode_classes = timed_step(engine, slots, [[2]] * batch, decode=True)
            for used in slots:
                engine.release(used)
            for classes, decode in ((prompt_classes, False), (decode_classes, True)):
                work = class_work(design, shape, batch if decode else PREFILL_TOKENS, context + 2, decode)
                for label, entry in classes.items():
                    if label in work and entry["us"] > 0:
                        kind, amount = work[label]
                        rate = amount / (entry["us"] * 1e-6)
                        entry["roofline"] = kind
                        entry["frac"] = round(rate / (peak["bf16_tflops"] * 1e12 if kind == "flops" else peak["hbm_gbs"] * 1e9), 4)
            point[design] = {
                "prefill_tokens_per_s": round(PREFILL_TOKENS / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
                "decode_tokens_per_s": round(run["tokens_per_s"], 1), "decode_ms_per_step": round(run["ms_per_step"], 4),
                "decode_kernels_per_step": run["kernels_per_step"], "weight_bytes": engine.memory()["weight_bytes"],
                "prompt_kernels": prompt_classes, "decode_kernels": decode_classes}
            del engine
            torch.cuda.empty_cache()
        sizes.append(point)
    print(json.dumps({
        "metric": f"prefill and decode tokens/s of a {args.design.capitalize()} stack beside Qwen3 layers of equal size (bf16, "
                  f"{args.layers or 4} layers, one {PREFILL_TOKENS}-token prompt; batch {batch} decoding at {context} tokens)",
        "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": args.warmup, "dtype": "bf16", "impl": "ours",
        "data": "synthetic: random weights from a seed, uniform token ids", "peaks": peak, "sizes": sizes,
        "note": "kernel times: one step with a CUDA event behind every launch, queued behind a 20 ms head start so "
                "that the device never waits for the host; frac: the class's algorithmic FLOPs or bytes over its "
                "time, of the measured product peak or copy rate"}))
    return 0


def main() -> int:
    parser = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    parser.add_argument("--design", default="", choices=["", *sorted(DESIGN_SHAPES)],
                        help="a stack of one of these designs beside Qwen3 layers of equal size, kernel class by kernel class "
                             "(the default workload is left as it is)")
    parser.add_argument("--widths", default="2048,4096", help="model widths of --design runs")
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=0, help="timed decode steps (default: the model's: 512 / 256)")
    parser.add_argument("--warmup", type=int, default=8)
    parser.add_argument("--batch", type=int, default=0, help="sequences of the batch (default: the model's: 8 / 16 / 8)")
    parser.add_argument("--model", default="8b", choices=sorted(MODELS), help="which of the benchmark's shapes")
    parser.add_argument("--layers", type=int, default=0, help="fewer layers than the model has (0: all)")
    parser.add_argument("--impl", default="ours", choices=["ours", "reference"])
    parser.add_argument("--seed", type=int, default=0)
    parser.add_argument("--repeats", type=int, default=REPEATS, help="measured repeats of the decode run (median)")
    parser.add_argument("--skip-points", action="store_true", help="leave out batch 1 / 64 and prefill")
    parser.add_argument("--skip-e2e", action="store_true", help="leave out the end-to-end run (profiling)")
    parser.add_argument("--profile-steps", type=int, default=0,
                        help="run this many extra decode steps inside cudaProfilerStart/Stop")
    parser.add_argument("--profile-prefill", action="store_true",
                        help="run one extra 2,048-token prefill inside cudaProfilerStart/Stop")
    args = parser.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference does not build offline: its CMake stops at 'yaml-cpp is missing from "
                          "third_party' (empty submodules), and its Qwen3 is an INT8 bidirectional backbone "
                          "without cache, head or generation"}))
        return 0
    if args.design and args.gpus == 1:
        if args.warmup < 3:
            print("bench.py needs --warmup >= 3")
            return 2
        return design_comparison(args)
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this library is single-GPU by design (asked for {args.gpus})")
        return 2
    title, shape, default_batch, prompt_lengths, default_steps = MODELS[args.model]
    steps, batch = args.steps or default_steps, args.batch or default_batch
    if steps < 1 or args.warmup < 3 or args.repeats < 1:
        print("bench.py needs --steps >= 1, --warmup >= 3 and --repeats >= 1")
        return 2

    import torch
    from kidi_b200 import Engine
    from kidi_b200.sampling.sampler import Sampler

    config = dict(shape)
    full_layers = config["num_hidden_layers"]
    if args.layers:
        config["num_hidden_layers"] = args.layers
    points_of = () if args.skip_points or args.model != "8b" else (1, 64)
    per_sequence = -(-(prompt_lengths[1] + args.warmup + steps + 2) // 64) * 64
    budget = max(max([batch, *points_of]) * per_sequence, 4096)
    engine = Engine.from_config(config, seed=args.seed, dtype="bfloat16", device="cuda:0", max_tokens=budget)
    sampler = Sampler(args.seed)
    peak = peaks()

    prompts = draw_prompts(engine.vocab_size, batch, prompt_lengths, args.seed)
    main_run = time_decode(engine, sampler, prompts, steps, args.warmup, clocks=True, repeats=args.repeats,
                           profile_steps=args.profile_steps)
    # What vouches for the timed work: the same prompts through plain steps, without the graph.
    compared, mismatches, distance = compare_with_plain_steps(engine, sampler, prompts, main_run["tokens"],
                                                              min(CHECKED_STEPS, args.warmup + steps))
    check = {"repeats": args.repeats, "repeats_identical": main_run["repeats_identical"],
             "tokens_compared_with_plain_steps": compared, "token_mismatches": mismatches,
             "largest_logit_distance_at_a_mismatch": round(distance, 5), "allowed_distance": ROUNDING_DISTANCE,
             "ms_of_repeats": main_run["ms_of_repeats"]}
    if args.skip_e2e:
        from kidi_b200.engine.generate import GenerationStats
        e2e_value, e2e_stats = 0.0, GenerationStats()
    else:
        e2e_value, e2e_stats, generated = time_end_to_end(engine, prompts, steps)
        # The entry point's tokens are the device-timed run's: token n of a sequence is row n of its history.
        check["e2e_token_mismatches"] = sum(
            generated[b][n] != main_run["tokens"][n][b] for b in range(batch)
            for n in range(min(len(generated[b]), len(main_run["tokens"]))))
    if args.profile_prefill:
        time_prefill(engine, args.seed, repeats=1, profile=True)
    points, prefill = {}, None
    for size in points_of:
        run = time_decode(engine, sampler, draw_prompts(engine.vocab_size, size, prompt_lengths, args.seed + size),
                          min(steps, 128), args.warmup, clocks=False, repeats=args.repeats)
        points[f"decode_b{size}"] = round(run["tokens_per_s"], 1)
        check[f"decode_b{size}_repeats_identical"] = run["repeats_identical"]
    if not args.skip_points:
        prefill_ms = time_prefill(engine, args.seed)
        flops = prefill_flops(config, PREFILL_TOKENS)
        prefill = {"value": round(PREFILL_TOKENS / (prefill_ms / 1e3), 1), "unit": "tokens/s",
                   "tokens": PREFILL_TOKENS, "ms": round(prefill_ms, 3),
                   "frac": round(flops / (prefill_ms / 1e3) / (peak["bf16_tflops"] * 1e12), 4),
                   # `frac` is of the library product's burst rate; the timed prefills run back to back under the
                   # power cap, where that product itself settles at the sustained rate.
                   "frac_of_sustained": round(flops / (prefill_ms / 1e3) /
                                              (peak.get("bf16_tflops_sustained", peak["bf16_tflops"]) * 1e12), 4),
                   "tflops": round(flops / (prefill_ms / 1e3) / 1e12, 1)}

    achieved = decode_bytes(config, batch, main_run["mean_context"]) / (main_run["ms_per_step"] / 1e3) / 1e9
    shortest, longest = prompt_lengths
    prompt_words = f"{shortest}-token prompts" if shortest == longest else f"prompts of {shortest} to {longest} tokens"
    record = {
        "metric": f"decode tokens/s ({title}, bf16, batch {batch}, {prompt_words})",
        "value": round(main_run["tokens_per_s"], 1), "unit": "tokens/s", "n_gpus": 1,
        "steps": steps, "warmup": args.warmup, "ms_per_step": round(main_run["ms_per_step"], 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights N(0, 0.02) from a seed, uniform token ids", "impl": "ours",
        "config": {
            "model": title, "layers": config["num_hidden_layers"], "layers_of_model": full_layers,
            "hidden_size": config["hidden_size"], "heads": config["num_attention_heads"],
            "kv_heads": config["num_key_value_heads"], "head_dim": config["head_dim"],
            "intermediate_size": config["intermediate_size"], "vocab_size": config["vocab_size"],
            "rope_theta": config["rope_theta"], "rms_norm_eps": config["rms_norm_eps"],
            "tie_word_embeddings": False, "global_batch": batch,
            "prompt_tokens": shortest if shortest == longest else f"uniform in [{shortest}, {longest}]",
            "context_per_sequence": per_sequence if args.model != "8b" else 4096,
            "seq_len": int(main_run["mean_context"]), "parallelism": "single GPU",
            "l2": "no flush: a step reads far more than the 126 MB L2 holds", "peaks": peak["source"],
        },
        "clocks": main_run["clocks"],
        "checked": bool(main_run["repeats_identical"] and distance <= ROUNDING_DISTANCE), "check": check,
        "e2e": {"value": round(e2e_value, 1), "unit": "tokens/s",
                "h2d_bytes_per_step": round(e2e_stats.host_to_device_bytes / max(1, e2e_stats.decode_steps), 1),
                "d2h_bytes_per_step": 4 * batch, "steps": e2e_stats.decode_steps,
                "note": "a step's input tokens are its predecessor's output on the device; the host copies the "
                        "batch's tables up when decoding starts and reads every step's tokens back; decoding "
                        "starts right after the prompts, whose power draw leaves lowered clocks for the first "
                        "twenty steps or so (4.3, then 3.9 ms a step)"},
        "gpu_launches": main_run["kernels_per_step"] * steps,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peak["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / peak["hbm_gbs"], 4), "of": peak["source"]},
    }
    if prefill:
        record["prefill"] = prefill
    if points:
        record["points"] = points
    print(json.dumps(record))
    return 0


if __name__ == "__main__":
    sys.exit(main())
