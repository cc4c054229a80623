"""Benchmark of the engine on one B200: decode tokens a second at the Qwen3-8B shape.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]
    python bench.py --shape 14b --batch 16 --context 8192        decode at the Qwen3-14B shape
    python bench.py --shape 0.6b --continuous                    continuous batching at the Qwen3-0.6B shape

A "step" is one decode step: every live request gets its next token.  The default run has the
layer sizes of the Qwen3-8B shape with seeded random weights (bfloat16), a batch of 8 and a
context of 4,096 tokens: the timed steps are the last K before each request reaches 4,096
tokens.  One JSON line is printed:
  value      decoded tokens a second, timed on the device with CUDA events around the K steps
             (synthetic token ids, next token chosen by the arg-max kernel on the device);
  e2e        the same through the Python entry point (`EngineHandle`): every step copies the
             step's token ids from pinned host memory and reads the sampled tokens back;
  prefill    one prompt of 2,048 tokens in one step, with its fraction of the bf16 peak;
  roofline   bytes a decode step must read (every weight once and the live requests' cache)
             divided by its time, against the measured copy bandwidth;
  points     decode at batch 1 and batch 64, each with the same fraction of the copy bandwidth.
  prefill also carries `chunked_4x512_ms`: the same prompt in four steps of 512 tokens.
`--shape 14b` (40 layers, width 5120, 40 / 8 heads, feed-forward 17408) and `--shape 0.6b` (28 layers, width 1024,
16 / 8 heads, feed-forward 3072, tied head) run the same measurement at those sizes, with `--batch` and `--context`.
`--continuous` is the serving workload: 64 requests with seeded prompt lengths uniform in 16 to 2,048 tokens and 64
generated tokens each, through `EngineHandle` with prompts cut into portions under a budget of 512 tokens a step; its
line reports prompt and generated tokens a second, the mean step time and the share of steps that were replayed
from a recording.
Peaks come from MEASURED_PEAKS.json when the file exists.  The engine runs on one GPU; for
--gpus N > 1 a line says so and the exit code is 2.  The reference arm cannot run here (the
reference is a Rust workspace without a Python package, and supports no sm_100 device), so
`--impl reference` prints its `unavailable` line."""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_8B = dict(model_type="qwen3", architectures=["Qwen3ForCausalLM"], hidden_size=4096, intermediate_size=12288,
                num_hidden_layers=36, num_attention_heads=32, num_key_value_heads=8, head_dim=128, vocab_size=151936,
                max_position_embeddings=40960, rms_norm_eps=1e-6, rope_theta=1000000.0, tie_word_embeddings=False,
                hidden_act="silu", eos_token_id=151645)
QWEN3_06B = dict(QWEN3_8B, hidden_size=1024, intermediate_size=3072, num_hidden_layers=28, num_attention_heads=16,
                 num_key_value_heads=8, head_dim=128, tie_word_embeddings=True)
QWEN3_14B = dict(QWEN3_8B, hidden_size=5120, intermediate_size=17408, num_hidden_layers=40, num_attention_heads=40,
                 num_key_value_heads=8, head_dim=128)
SHAPES = {"8b": ("Qwen3-8B shape", QWEN3_8B), "0.6b": ("Qwen3-0.6B shape", QWEN3_06B), "14b": ("Qwen3-14B shape", QWEN3_14B)}
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def peaks() -> dict:
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            data = json.load(f)
        return {"hbm_gbs": float(data["hbm_gbs"]), "bf16_tflops": float(data["bf16_tflops"]), "source": "measured"}
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
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
        clocks, max_clock, reasons = [], None, set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for line in out.splitlines():
            parts = [p.strip() for p in line.split(",")]
            if len(parts) != 6:
                continue
            try:
                clocks.append(float(parts[0]))
                max_clock = float(parts[1])
            except ValueError:
                continue
            for name, value in zip(names, parts[2:]):
                if value.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": statistics.median(clocks) if clocks else None, "sm_max_mhz": max_clock,
                "reasons": sorted(reasons), "samples": len(clocks)}


def model_numbers(cfg: dict, layers: int) -> dict:
    """Weight bytes a decode step reads, cache bytes per context token, flops per prompt token."""
    h, i, v = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nq, nkv, d = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    per_layer = (nq + 2 * nkv) * d * h + h * nq * d + 2 * i * h + h * i
    return {"layer_params": per_layer, "head_params": v * h,
            "weight_bytes": 2 * (layers * per_layer + v * h),       # a tied head reads the embedding table: the same bytes
            "kv_bytes_per_token": layers * 2 * nkv * d * 2,
            "linear_flops_per_token": 2 * layers * per_layer,
            "attn_flops_per_pair": 4 * nq * d * layers}


def kernel_shares(torch, run) -> None:
    """Runs `run` under torch.profiler and prints, kernel by kernel, launches, the sum and the mean of their
    durations and the share of the sum (kernels that start under their predecessor overlap it, so the sum is more
    than the wall clock: compare shares)."""
    import collections

    from torch.profiler import ProfilerActivity, profile

    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        run()
        torch.cuda.synchronize()
    table = collections.defaultdict(lambda: [0, 0.0])
    for event in prof.events():
        if event.device_type.name == "CUDA":
            entry = table[event.name[:100]]
            entry[0] += 1
            entry[1] += event.device_time
    total = sum(t for _, t in table.values()) or 1.0
    print(f"kernels: {total / 1e3:.1f} ms in {sum(n for n, _ in table.values())} launches", file=sys.stderr)
    for name, (n, t) in sorted(table.items(), key=lambda kv: -kv[1][1])[:24]:
        print(f"{t / 1e3:9.2f} ms {100 * t / total:5.1f}% {n:7d} launches {t / n:8.1f} us  {name}", file=sys.stderr)


def continuous_run(args, torch, shape_name: str, cfg: dict, peak: dict) -> dict:
    """The serving workload of the 0.6B configuration: `--requests` requests (64) whose prompt lengths are drawn
    uniformly from 16 to 2,048 (seeded), `--output-tokens` generated tokens each (64), all submitted at once to
    `EngineHandle`; prompts are cut into portions under a budget of 512 tokens a step and run beside the decoded
    tokens of the requests that are further on.  A first wave of the same lengths (other tokens) runs untimed so
    that every kernel has been built and every step shape has been recorded once: the timed wave is the steady
    state of a server that has seen its traffic before."""
    import random

    from mini_rsglang_b200 import RuntimeConfig, SamplingParams
    from mini_rsglang_b200.engine import EngineHandle
    from mini_rsglang_b200.models import config_from_dict

    config = config_from_dict(cfg)
    requests, out_tokens, budget, page = args.requests, args.output_tokens, args.prefill_budget, 16
    rng = random.Random(20240611)
    lengths = [rng.randint(16, 2048) for _ in range(requests)]
    max_running = min(requests, args.max_running)
    max_seq_len = 2048 + out_tokens
    pages = max_running * (-(-max_seq_len // page) + 1) + 8
    limits = RuntimeConfig(max_seq_len=max_seq_len, page_size=page, prefill_budget=budget, max_running=max_running,
                           max_waiting=max(256, requests))
    engine = EngineHandle.from_random(config, seed=1, dtype="bfloat16", config=limits, num_pages=pages)
    runner = engine.runner
    params = SamplingParams(max_tokens=out_tokens, ignore_eos=True)

    def prompts(ns):
        return [[rng.randrange(cfg["vocab_size"]) for _ in range(n)] for n in ns]

    engine.generate_many(prompts(lengths), params)     # warm-up wave of the same lengths, untimed: every step shape is recorded
    work = prompts(lengths)
    torch.cuda.synchronize()
    steps0, recorded0, h2d0 = runner.steps, runner.recorded_steps, runner.h2d_bytes
    sampler = ClockSampler()
    sampler.start()
    t0 = time.perf_counter()
    results = engine.generate_many(work, params)
    torch.cuda.synchronize()
    elapsed = time.perf_counter() - t0
    clocks = sampler.stop()
    steps = runner.steps - steps0
    generated = sum(r.completion_tokens for r in results)
    prompt_tokens = sum(lengths)
    assert all(r.finish_reason == "length" and r.completion_tokens == out_tokens for r in results)
    recorded, h2d = runner.recorded_steps - recorded0, runner.h2d_bytes - h2d0
    if args.kernel_shares:
        kernel_shares(torch, lambda: engine.generate_many(prompts(lengths), params))
    engine.shutdown()
    total = prompt_tokens + generated
    return {
        "metric": f"continuous batching tok/s, {requests} requests of 16-2048 prompt tokens, {out_tokens} generated each ({shape_name})",
        "value": round(total / elapsed, 1), "unit": "tokens/s (prompt + generated)", "n_gpus": 1, "steps": steps, "warmup": 1,
        "ms_per_step": round(elapsed / steps * 1e3, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: seeded random weights, seeded prompt lengths, uniform random token ids",
        "prompt_tokens_per_s": round(prompt_tokens / elapsed, 1), "generated_tokens_per_s": round(generated / elapsed, 1),
        "prompt_tokens": prompt_tokens, "generated_tokens": generated, "elapsed_s": round(elapsed, 4),
        "recorded_step_share": round(recorded / max(steps, 1), 4),
        "h2d_bytes_per_step": h2d // max(steps, 1),
        "config": {"model": shape_name, "layers": cfg["num_hidden_layers"], "layers_of_shape": cfg["num_hidden_layers"],
                   "hidden": cfg["hidden_size"], "q_heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
                   "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
                   "tied_head": cfg["tie_word_embeddings"], "requests": requests, "max_running": max_running,
                   "prefill_budget": budget, "output_tokens": out_tokens, "page_size": page, "parallelism": "single GPU",
                   "timing": "wall clock around EngineHandle.generate_many, host tokens in and out", "peaks": peak["source"]},
        "clocks": clocks, "impl": "ours"}


HYBRID_SIZES = {
    # width, feed-forward, query / key heads of 128 (Niduvik: values of 128 too), layers; the recurrence has 2 * width / 64
    # heads of 64 with a state of 128 in 8 groups and 4 taps; the window is 1,024 with 4 kept tokens, the bias table 32 rows.
    "1b": dict(width=2048, ff=8192, heads=16, kv_heads=4, layers=8),
    "8b": dict(width=4096, ff=12288, heads=32, kv_heads=8, layers=8),
}


def hybrid_configs(size: dict, vocab: int = 32768):
    """Niduvik at these layer sizes (two attention layers, then two recurrent ones, and so on) and the Qwen3 of equal
    width, heads, feed-forward and depth."""
    w = size["width"]
    attention = {"type": "attention", "mlp": {"kind": "dense", "ff": size["ff"], "limit": 7.0},
                 "mixer": {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                           "softcap": 30.0, "bias_max": 4096.0, "bias_rows": 32, "v_mix": True, "mask": {"size": 1024, "keep_first": 4}}}
    recurrent = {"type": "mamba2", "mlp": {"kind": "dense", "ff": size["ff"], "limit": 7.0},
                 "mixer": {"heads": 2 * w // 64, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8}}
    layers = [attention if i % 4 < 2 else recurrent for i in range(size["layers"])]
    niduvik = {"architecture": "Niduvik", "vocab": vocab, "width": w, "norm": {"eps": 1e-6}, "layers": layers}
    qwen = dict(QWEN3_8B, hidden_size=w, intermediate_size=size["ff"], num_hidden_layers=size["layers"],
                num_attention_heads=size["heads"], num_key_value_heads=size["kv_heads"], head_dim=128, vocab_size=vocab,
                tie_word_embeddings=True, eos_token_id=1)
    return niduvik, qwen


def latent_configs(size: dict, vocab: int = 32768):
    """Satedra at these layer sizes: latent attention with a latent of 256 and a rotated part of 32 elements, heads of 64
    unrotated query/key and 64 value elements, a window of 1,024, every second layer reading the cache of the layer before
    it; the first layer's feed-forward dense, the others 32 experts of ff / 8 with 4 chosen, 2 identity experts and a shared
    expert of ff / 4.  Beside it the Qwen3 of equal width, heads and depth whose feed-forward is as wide as the experts a
    token passes (4 chosen + the shared one)."""
    w, ff = size["width"], size["ff"]
    rot = {"base": 1000000.0, "dims": 32, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    layers = []
    for i in range(size["layers"]):
        mixer = {"heads": size["heads"], "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256, "scale": 96 ** -0.5, "mask": {"size": 1024},
                 "rot": rot}
        if i % 2:
            mixer["kv_from"] = i - 1
        mlp = {"kind": "dense", "ff": ff} if i == 0 else {"kind": "moe", "expert": {"ff": ff // 8}, "shared": {"ff": ff // 4},
                                                          "router": {"experts": 32, "identity": 2, "top": 4, "scale": 2.0}}
        layers.append({"type": "latent_attention", "mixer": mixer, "mlp": mlp})
    satedra = {"architecture": "Satedra", "vocab": vocab, "width": w, "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": layers}
    qwen = dict(QWEN3_8B, hidden_size=w, intermediate_size=4 * (ff // 8) + ff // 4, num_hidden_layers=size["layers"],
                num_attention_heads=size["heads"], num_key_value_heads=size["kv_heads"], head_dim=128, vocab_size=vocab,
                tie_word_embeddings=False, eos_token_id=1)
    return satedra, qwen


def parallel_configs(size: dict, vocab: int = 32768):
    """Nubipel at these layer sizes (a delta-rule layer, a chunked attention, a latent attention, a delta-rule layer, and so
    on): attention heads of 128 in chunks of 1,024 positions with sinks; latent attention with heads of 64, a latent of 256
    for keys and values and one of width / 4 for the queries; the delta rule with width / 128 heads of 128 value elements,
    a quarter as many query/key heads of 128, 4 taps; every layer with the dense feed-forward beside its mixer.  Beside it
    Niduvik, the engine's other model of attention layers with a bounded sight next to recurrent layers, at equal width,
    heads, feed-forward and depth."""
    w = size["width"]
    mlp = {"kind": "dense", "ff": size["ff"]}
    attention = {"type": "attention", "mlp": mlp,
                 "mixer": {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024}}}
    latent = {"type": "latent_attention", "mlp": mlp,
              "mixer": {"heads": size["heads"], "dim": 64, "vdim": 64, "kv_rank": 256, "q_rank": w // 4, "scale": 64 ** -0.5}}
    delta = {"type": "delta", "mlp": mlp, "mixer": {"heads": w // 128, "kv_heads": max(w // 512, 1), "dim": 128, "vdim": 128, "conv": 4}}
    layers = [(delta, attention, latent, delta)[i % 4] for i in range(size["layers"])]
    nubipel = {"architecture": "Nubipel", "vocab": vocab, "width": w, "norm": {"eps": 1e-6}, "embedding": {"scale": w ** 0.5},
               "logit_scale": w ** -0.5, "logit_softcap": 30.0, "layers": layers}
    return nubipel, hybrid_configs(size, vocab)[0]


def looped_configs(size: dict, vocab: int = 32768):
    """Migenex at these layer sizes: six layers of which the third and fourth are passed twice (eight layer runs), layers with
    values taken from the keys (heads of 128, a window of 1,024, every value element gated) and a relu-gated feed-forward
    taking turns with layers that see everything (heads of 128, scores capped at 30) and route 4 of 32 ungated experts of
    ff / 8 beside a shared one of ff / 4; a table of 65,536 token pairs.  Beside it Satedra, the engine's other model of
    windowed attention with routed and shared experts, at equal width, heads, experts and depth."""
    w, ff = size["width"], size["ff"]
    rot = {"base": 1000000.0, "dims": 128}
    keyed = {"type": "attention_2", "mlp": {"kind": "dense", "ff": ff},
             "mixer": {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024},
                       "rot": rot}}
    routed = {"type": "attention", "mlp": {"kind": "moe", "expert": {"ff": ff // 8}, "shared": {"ff": ff // 4}, "router": {"experts": 32, "top": 4}},
              "mixer": {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                        "rot": rot}}
    runs = size["layers"]
    layers = [keyed if i % 2 == 0 else routed for i in range(runs - 2)]
    migenex = {"architecture": "Migenex", "vocab": vocab, "width": w, "norm": {"eps": 1e-6}, "residual_mult": 0.8,
               "embedding": {"scale": 1.0, "bigram": {"buckets": 65536, "mul_prev": 1000003, "mul_cur": 31}},
               "loop": {"start": 2, "stop": 4, "times": 2}, "layers": layers}
    return migenex, latent_configs(size, vocab)[0]


def recurrent_configs(size: dict, vocab: int = 32768):
    """Pisatar at these layer sizes: four layers (a retention, a channel-decayed delta rule, attention beside a matrix memory, a
    retention) that are run twice, the second four with the weights of the first and states of their own (eight layer runs).
    The retention has width / 128 heads of 128 query/key and 256 value elements; the delta rule width / 128 heads of 128 value
    elements, a quarter as many query/key heads of 128, 4 taps, thin products of 128; the attention heads of 128, rotated whole,
    and beside it width / 512 memory heads of 256 query/key and 512 value elements; every layer with the gated feed-forward
    beside its mixer.  Beside it Nubipel, the engine's other model of parallel branches with a delta rule, at equal width,
    heads, feed-forward and depth."""
    w = size["width"]
    mlp = {"kind": "dense", "ff": size["ff"]}
    heads = w // 128
    retention = {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": 128, "vdim": 256, "rot": {"base": 10000.0, "dims": 128},
                                                            "decay": [1.0 - 2.0 ** (-5.0 - 7.0 * i / heads) for i in range(heads)]}}
    delta = {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": max(w // 512, 1), "dim": 128, "vdim": 128, "conv": 4,
                                                            "decay_rank": 128, "gate_rank": 128}}
    both = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "rot": {"base": 500000.0, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}},
        "right": {"heads": w // 512, "dim": 256, "vdim": 512, "gate_cap": 15.0}, "left_scale": 0.7, "right_scale": 0.7}}
    first = (retention, delta, both, retention)
    layers = [first[i] if i < 4 else dict(first[i % 4], weights_of=i % 4) for i in range(size["layers"])]
    pisatar = {"architecture": "Pisatar", "vocab": vocab, "width": w, "norm": {"eps": 1e-6}, "layers": layers}
    return pisatar, parallel_configs(size, vocab)[0]


def passed_configs(size: dict, vocab: int = 32768):
    """Bilipel at these layer sizes: six layers of which the first two are passed twice (eight layer runs), gated linear attention
    (width / 128 heads of 128 query/key and 256 value elements, thin products of 16; in layers 0, 3 and 4), attention (heads of
    128, half of each rotated, sinks; layers 1 and 5) and latent attention (heads of 64 unrotated and 32 rotated query/key and 64
    value elements, a latent of 256, a window of 1,024, sinks; layer 2); the first layer's feed-forward dense, the others 32
    experts of ff / 8 with 4 chosen.  Beside it Satedra, the engine's other model of layer norms, latent attention and routed
    experts, at equal width, heads, experts and depth."""
    w, ff = size["width"], size["ff"]
    dense = {"kind": "dense", "ff": ff}
    routed = {"kind": "moe", "expert": {"ff": ff // 8}, "router": {"experts": 32, "top": 4}}
    recurrent = {"type": "gla", "mixer": {"heads": w // 128, "dim": 128, "vdim": 256, "tau": 16.0, "decay_rank": 16}}
    attention = {"type": "attention", "mixer": {
        "heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
        "rot": {"base": 1000000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    latent = {"type": "latent_attention", "mixer": {"heads": size["heads"], "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256, "scale": 96 ** -0.5,
                                                    "mask": {"size": 1024}, "rot": {"base": 1000000.0, "dims": 32}}}
    layers = [dict(recurrent, mlp=dense), dict(attention, mlp=routed), dict(latent, mlp=routed), dict(recurrent, mlp=routed),
              dict(recurrent, mlp=routed), dict(attention, mlp=routed)]
    bilipel = {"architecture": "Bilipel", "vocab": vocab, "width": w, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
               "loop": {"start": 0, "stop": 2, "times": 2}, "layers": layers}
    return bilipel, latent_configs(size, vocab)[0]


# design: (title, what stands beside it, the key of that model in the output, the two configurations)
DESIGNS = {"niduvik": ("Niduvik", "Qwen3 of equal width, heads, feed-forward and depth", "qwen3", hybrid_configs),
           "satedra": ("Satedra", "Qwen3 of equal width, heads and depth, its feed-forward as wide as the experts a token passes", "qwen3",
                       latent_configs),
           "nubipel": ("Nubipel", "Niduvik of equal width, heads, feed-forward and depth", "niduvik", parallel_configs),
           "migenex": ("Migenex", "Satedra of equal width, heads, experts and depth", "satedra", looped_configs),
           "pisatar": ("Pisatar", "Nubipel of equal width, heads, feed-forward and depth", "nubipel", recurrent_configs),
           "bilipel": ("Bilipel", "Satedra of equal width, heads, experts and depth", "satedra", passed_configs)}


def hybrid_run(args, torch, peak: dict) -> dict:
    """`--design NAME`: prefill of one prompt and decode steps of the design at layer sizes of real models, beside the
    engine's closest other model at equal sizes, both with seeded random weights in bfloat16, timed on the device; with --kernel-shares each
    model's kernels by their share of the device's time (standard error)."""
    from mini_rsglang_b200 import RuntimeConfig, kernels
    from mini_rsglang_b200.engine import EngineHandle, SequenceStep
    from mini_rsglang_b200.models import config_from_dict

    size = HYBRID_SIZES[args.size]
    context, batch, prompt_len = args.context, args.batch, args.prompt
    title, beside, beside_key, configs = DESIGNS[args.design]
    out = {"design": title, "beside": beside, "size": dict(size, name=args.size),
           "batch": batch, "context": context, "prompt": prompt_len, "dtype": "bf16", "data": "synthetic: seeded random weights",
           "peaks": peak}
    gen = torch.Generator().manual_seed(7)
    for name, raw in zip((args.design, beside_key), configs(size)):
        config = config_from_dict(raw)
        page = 16
        pages = batch * (-(-context // page)) + 2 * (-(-prompt_len // page)) + 8
        limits = RuntimeConfig(max_seq_len=max(context, prompt_len), page_size=page, prefill_budget=prompt_len, max_running=batch + 1)
        engine = EngineHandle.from_random(config, seed=1, dtype="bfloat16", config=limits, num_pages=pages)
        runner = engine.runner
        for entry in runner.storage.entries:
            for pages_of in (entry.k, entry.v):
                if pages_of is not None:
                    pages_of.normal_(0.0, 1.0)
        vocab = config.vocab_size

        def timed(fn, repeat):
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            start.record()
            for _ in range(repeat):
                fn()
            end.record()
            torch.cuda.synchronize()
            return start.elapsed_time(end)

        prompt = torch.randint(0, vocab, (prompt_len,), generator=gen).tolist()

        def prefill_once(request):
            runner.cache.open(request)
            runner.cache.extend(request, prompt_len)
            runner.forward([SequenceStep(request, prompt, 0, [prompt_len - 1])])
            torch.cuda.synchronize()
            runner.cache.close(request)

        samples = [timed(lambda r=r: prefill_once(10_000 + r), 1) for r in range(6)][3:]
        prefill_ms = statistics.median(samples)
        start_len = context - (args.warmup + args.steps) - (4 if args.kernel_shares else 0)      # the profiled step comes on top
        ids = list(range(20_000, 20_000 + batch))
        for r in ids:
            runner.cache.open(r)
            runner.cache.extend(r, start_len)
        picked = torch.empty(batch, dtype=torch.int32, device=runner.device)
        position = [start_len]

        def one_step():
            p = position[0]
            for r in ids:
                runner.cache.extend(r, p + 1)
            tokens = torch.randint(0, vocab, (batch,), generator=gen).tolist()
            logits = runner.forward([SequenceStep(r, [t], p, [0]) for r, t in zip(ids, tokens)])
            kernels.argmax(logits, picked)
            position[0] = p + 1

        timed(one_step, args.warmup)
        launches = kernels.launch_count
        decode_ms = timed(one_step, args.steps) / args.steps
        launches = (kernels.launch_count - launches) // args.steps
        if args.kernel_shares:
            print(f"--- {name}: one decode step at batch {batch}", file=sys.stderr)
            kernel_shares(torch, one_step)
            print(f"--- {name}: prefill of {prompt_len} tokens", file=sys.stderr)
            kernel_shares(torch, lambda: prefill_once(30_000))
        for r in ids:
            runner.cache.close(r)
        out[name] = {"prefill_tokens_per_s": round(prompt_len / prefill_ms * 1e3, 1), "prefill_ms": round(prefill_ms, 3),
                     "decode_tokens_per_s": round(batch / decode_ms * 1e3, 1), "decode_ms_per_step": round(decode_ms, 4),
                     "launches_per_decode_step": launches, "weight_bytes": runner.model.weight_bytes(),
                     "decode_weight_read_frac": round(runner.model.weight_bytes() / (decode_ms * 1e-3) / 1e9 / peak["hbm_gbs"], 4)}
        engine.shutdown()
        del engine, runner
        torch.cuda.empty_cache()
    return out


def main() -> int:
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=64)
    parser.add_argument("--warmup", type=int, default=8)
    parser.add_argument("--impl", choices=["ours", "reference"], default="ours")
    parser.add_argument("--shape", choices=sorted(SHAPES), default="8b", help="layer sizes: Qwen3-8B (the default line), 0.6B or 14B")
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--context", type=int, default=4096)
    parser.add_argument("--layers", type=int, default=0, help="fewer layers than the shape has (named in config); 0: all of them")
    parser.add_argument("--no-points", action="store_true", help="skip the batch-1 and batch-64 points")
    parser.add_argument("--no-e2e", action="store_true")
    parser.add_argument("--continuous", action="store_true", help="the continuous-batching workload instead of the decode measurement")
    parser.add_argument("--requests", type=int, default=64, help="--continuous: requests")
    parser.add_argument("--output-tokens", type=int, default=64, help="--continuous: generated tokens a request")
    parser.add_argument("--prefill-budget", type=int, default=512, help="--continuous: tokens a step")
    parser.add_argument("--max-running", type=int, default=64, help="--continuous: requests in flight at most")
    parser.add_argument("--design", choices=sorted(DESIGNS), help="that design beside the engine's closest other model at equal sizes (prefill and decode), instead of the default measurement")
    parser.add_argument("--size", choices=sorted(HYBRID_SIZES), default="1b", help="--design: layer sizes")
    parser.add_argument("--prompt", type=int, default=2048, help="--design: tokens of the prompt")
    parser.add_argument("--kernel-shares", action="store_true",
                        help="--continuous: after the timed wave, one more wave under torch.profiler; its kernels' shares of the "
                             "device's time go to standard error (not a timing)")
    args = parser.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference is a Rust workspace (no setup.py/pyproject.toml: pip cannot install it, "
                          "no cargo in the image) and its CUDA backend accepts only sm_80..sm_90"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported (run with --gpus 1)")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch

    from mini_rsglang_b200 import RuntimeConfig, SamplingParams, kernels
    from mini_rsglang_b200.engine import EngineHandle, GenerateRequest, SequenceStep, TokenIds
    from mini_rsglang_b200.models import config_from_dict

    torch.cuda.set_device(0)
    shape_name, shape = SHAPES[args.shape]
    full_layers = shape["num_hidden_layers"]
    layers = args.layers or full_layers
    cfg = dict(shape, num_hidden_layers=layers)
    peak = peaks()
    if args.design:
        print(json.dumps(hybrid_run(args, torch, peak)))
        return 0
    if args.continuous:
        print(json.dumps(continuous_run(args, torch, shape_name, cfg, peak)))
        return 0
    config = config_from_dict(cfg)
    numbers = model_numbers(cfg, layers)
    context, batch = args.context, args.batch
    default_line = args.shape == "8b"
    point_batches = [] if args.no_points or not default_line else [1, 64]
    max_batch = max([batch] + point_batches)
    page = 16
    pages = max_batch * (-(-context // page)) + 2 * (-(-2048 // page)) + 8
    limits = RuntimeConfig(max_seq_len=max(context, 2048), page_size=page, prefill_budget=2048, max_running=max_batch, max_waiting=256)
    engine = EngineHandle.from_random(config, seed=1, dtype="bfloat16", config=limits, num_pages=pages)
    runner = engine.runner
    for entry in runner.storage.entries:      # cache contents do not change the timing; avoid all-zero keys anyway
        entry.k.normal_(0.0, 1.0)
        entry.v.normal_(0.0, 1.0)
    gen = torch.Generator().manual_seed(7)

    def random_tokens(n):
        return torch.randint(0, cfg["vocab_size"], (n,), generator=gen).tolist()

    def timed(fn, repeat):
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        for _ in range(repeat):
            fn()
        end.record()
        torch.cuda.synchronize()
        return start.elapsed_time(end)

    # ---------------------------------------------------------------- prefill of 2,048 tokens: in one step, and in four of 512
    prefill_tokens = 2048
    prompt = random_tokens(prefill_tokens)

    def prefill_once(request, portion):
        runner.cache.open(request)
        for at in range(0, prefill_tokens, portion):
            runner.cache.extend(request, at + portion)
            runner.forward([SequenceStep(request, prompt[at:at + portion], at, [portion - 1] if at + portion == prefill_tokens else [])])

    def prefill_median(portion, first_id):
        samples = []
        for trial in range(3 + 3):
            ms = timed(lambda: prefill_once(first_id + trial, portion), 1)
            runner.cache.close(first_id + trial)
            if trial >= 3:
                samples.append(ms)
        return statistics.median(samples)

    prefill_time = prefill_median(prefill_tokens, 10_000)
    chunked_time = prefill_median(512, 11_000)
    prefill_flops = (prefill_tokens * numbers["linear_flops_per_token"]
                     + numbers["attn_flops_per_pair"] * prefill_tokens * (prefill_tokens + 1) // 2
                     + 2 * numbers["head_params"])
    prefill = {"value": round(prefill_tokens / prefill_time * 1e3, 1), "tokens": prefill_tokens,
               "ms": round(prefill_time, 3), "frac": round(prefill_flops / (prefill_time * 1e-3) / (peak["bf16_tflops"] * 1e12), 4),
               "flops": prefill_flops, "peak_tflops": peak["bf16_tflops"], "chunked_4x512_ms": round(chunked_time, 3),
               "chunked_4x512_value": round(prefill_tokens / chunked_time * 1e3, 1)}

    # ---------------------------------------------------------------- decode, timed on the device
    def decode_run(b, steps, warmup, sample_clocks=False):
        """b requests whose context ends at `context` after warmup + steps decode steps."""
        start_len = context - (warmup + steps)
        ids = list(range(20_000 + 1000 * b, 20_000 + 1000 * b + b))
        for r in ids:
            runner.cache.open(r)
            runner.cache.extend(r, start_len)
        picked = torch.empty(b, dtype=torch.int32, device=runner.device)
        position = [start_len]

        def one_step():
            p = position[0]
            for r in ids:
                runner.cache.extend(r, p + 1)
            tokens = random_tokens(b)
            logits = runner.forward([SequenceStep(r, [t], p, [0]) for r, t in zip(ids, tokens)])
            kernels.argmax(logits, picked)
            position[0] = p + 1

        timed(one_step, warmup)
        sampler = ClockSampler()
        if sample_clocks:
            sampler.start()
        launches_before = kernels.launch_count
        ms = timed(one_step, steps)
        launches = kernels.launch_count - launches_before
        clocks = sampler.stop() if sample_clocks else None
        for r in ids:
            runner.cache.close(r)
        mean_context = context - steps / 2
        return {"ms_per_step": ms / steps, "tokens_per_s": b * steps / ms * 1e3, "launches": launches,
                "clocks": clocks, "mean_context": mean_context}

    main_run = decode_run(batch, args.steps, args.warmup, sample_clocks=True)
    step_bytes = numbers["weight_bytes"] + batch * main_run["mean_context"] * numbers["kv_bytes_per_token"]
    achieved = step_bytes / (main_run["ms_per_step"] * 1e-3) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": peak["hbm_gbs"], "unit": "GB/s",
                "frac": round(achieved / peak["hbm_gbs"], 4), "bytes_per_step": int(step_bytes)}
    points = {}
    for b in point_batches:
        run = decode_run(b, max(args.steps // 2, 8), args.warmup)
        points[f"decode_b{b}"] = round(run["tokens_per_s"], 1)
        point_bytes = numbers["weight_bytes"] + b * run["mean_context"] * numbers["kv_bytes_per_token"]
        points[f"decode_b{b}_hbm_frac"] = round(point_bytes / (run["ms_per_step"] * 1e-3) / 1e9 / peak["hbm_gbs"], 4)

    # ---------------------------------------------------------------- the same through the Python entry point
    e2e = None
    if not args.no_e2e:
        total = args.warmup + args.steps
        # every request must still be live when the timing ends: the first one decodes while the others'
        # prompts are still running, a step for every 2,048 prompt tokens of the batch
        slack = batch * context // limits.prefill_budget + 16
        prompt_len = context - total - slack
        params = SamplingParams(max_tokens=total + slack, ignore_eos=True)
        streams = [engine.generate(GenerateRequest(TokenIds(random_tokens(prompt_len)), params)) for _ in range(batch)]
        while engine.scheduler.waiting() or any(engine.generated.get(s.request_id, 0) == 0 for s in streams):
            if not engine.run_step():                        # prompts, untimed
                raise RuntimeError("the scheduler went idle before every request had its first token")
            if len(engine.generated) < batch:
                raise RuntimeError("a request finished before the timing began; raise the slack")
        for _ in range(args.warmup):
            engine.run_step()
        torch.cuda.synchronize()
        h2d_before, steps_before = runner.h2d_bytes, runner.steps
        made_before = sum(engine.generated.values())
        t0 = time.perf_counter()
        for _ in range(args.steps):
            engine.run_step()
        torch.cuda.synchronize()
        elapsed = time.perf_counter() - t0
        made = sum(engine.generated.values()) - made_before
        timed_steps = runner.steps - steps_before
        e2e = {"value": round(made / elapsed, 1), "unit": "tokens/s", "tokens": made,
               "h2d_bytes_per_step": (runner.h2d_bytes - h2d_before) // max(timed_steps, 1),
               "d2h_bytes_per_step": 4 * batch, "ms_per_step": round(elapsed / args.steps * 1e3, 3)}
        engine.shutdown()

    line = {
        "metric": f"decode tok/s at batch {batch}, context {context} ({shape_name})", "value": round(main_run["tokens_per_s"], 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(main_run["ms_per_step"], 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic: seeded random weights, uniform random token ids",
        "config": {"model": shape_name, "layers": layers, "layers_of_shape": full_layers,
                   "hidden": cfg["hidden_size"], "q_heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
                   "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"], "global_batch": batch,
                   "seq_len": context, "page_size": page, "parallelism": "single GPU",
                   "l2": "inputs larger than L2 (weights read every step)", "peaks": peak["source"]},
        "clocks": main_run["clocks"], "e2e": e2e, "gpu_launches": main_run["launches"],
        "prefill": prefill, "roofline": roofline, "points": points, "impl": "ours",
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
