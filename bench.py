"""Decode and prefill throughput of the engine on one B200, Llama 3.2 1B shape, random weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--impl ours|reference]
                    [--only all|decode|prefill] [--shape 3b|8b] [--per-kernel [--per-kernel-out FILE]]

A "step" is one decode step of the whole batch (captured forward + sampling). The default run
is the Llama 3.2 1B benchmark configuration in bfloat16 with a batch of 8, 512-token prompts and a 4096-token
context limit. It prints ONE JSON line: `value` is decoded tokens per second over K timed steps
(CUDA events, after W warm-up steps); `e2e` is the same through `generate()` with host tokens
in and out every step; `prefill` is one 2,048-token prompt; `roofline` compares the decode
step with the bytes it must read (every weight once + the live requests' cache) at the measured
HBM bandwidth; `points` gives decode at batch 1 and 64; `shapes` holds the two larger workloads
(Llama 3.2 3B shape: 16 requests of unequal prompts through `generate()`; Llama 3.1 8B shape:
a 2,048-token prefill and decode at batch 64 after 1,024-token prompts), each with the number of
layers it ran and the number the shape has. Weights (2.5 GB and more) are far larger than
L2, so every step streams them from HBM; no extra L2 flush is needed (stated in `config`).

`--impl reference` runs the unmodified reference engine on the same workload (baseline/reference_arm.py).
`--shape 3b|8b` runs only that workload at full depth (or `--layers L`). `--per-kernel` times every
kernel of the eager decode step (batch 1, 8, 64) and of the 2,048-token prefill with CUDA events and
prints one table each: time, bytes, FLOPs and the fraction of the measured peak they amount to.
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

METRIC = "decode tok/s at batch 1/8/64; prefill tok/s at 2,048 tokens (Llama 3.2 1B)"

_LLAMA3 = {"rope_type": "llama3", "factor": 32.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
           "original_max_position_embeddings": 8192}
_COMMON = {
    "architectures": ["LlamaForCausalLM"], "model_type": "llama", "vocab_size": 128256, "rope_theta": 500000.0,
    "rms_norm_eps": 1e-5, "max_position_embeddings": 131072, "hidden_act": "silu", "attention_bias": False,
    "mlp_bias": False, "bos_token_id": 128000, "eos_token_id": 128001, "torch_dtype": "bfloat16",
}
# the benchmark configuration: the Llama 3.2 1B shape
CONFIG_1B = dict(_COMMON, num_hidden_layers=16, hidden_size=2048, num_attention_heads=32, num_key_value_heads=8,
                 head_dim=64, intermediate_size=8192, rope_scaling=_LLAMA3, tie_word_embeddings=True)
# the two larger shapes of the benchmark set
CONFIG_3B = dict(_COMMON, num_hidden_layers=28, hidden_size=3072, num_attention_heads=24, num_key_value_heads=8,
                 head_dim=128, intermediate_size=8192, rope_scaling=_LLAMA3, tie_word_embeddings=True)
CONFIG_8B = dict(_COMMON, num_hidden_layers=32, hidden_size=4096, num_attention_heads=32, num_key_value_heads=8,
                 head_dim=128, intermediate_size=14336, rope_scaling=dict(_LLAMA3, factor=8.0),
                 tie_word_embeddings=False)
CONTEXT = 4096
PROMPT_LEN = 512
PREFILL_TOKENS = 2048
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                p = json.load(f)
            return {"hbm_gbs": float(p["hbm_gbs"]), "bf16_tflops": float(p["bf16_tflops"]), "source": "measured"}
        except (OSError, ValueError, KeyError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while timed work runs."""
    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.samples = []
        self.proc = None
        self.index = index

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.index)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 6:
                self.samples.append(parts)

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        clocks, max_clocks, reasons = [], [], set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for s in self.samples:
            try:
                clocks.append(int(float(s[0])))
                max_clocks.append(int(float(s[1])))
            except ValueError:
                continue
            for name, val in zip(names, s[2:6]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        clocks.sort()
        return {"sm_mhz": clocks[len(clocks) // 2] if clocks else None,
                "sm_max_mhz": max(max_clocks) if max_clocks else None, "reasons": sorted(reasons),
                "samples": len(clocks)}


def make_model_folder(cfg: dict, n_layers: int, seed: int, tag: str) -> str:
    from llm_infer_engine_b200 import write_random_model
    from llm_infer_engine_b200.weights import scratch_folder
    cfg = dict(cfg)
    cfg["num_hidden_layers"] = n_layers
    folder = scratch_folder(f"llmie_bench_{tag}_")          # deleted at exit: these folders are gigabytes
    t0 = time.time()
    write_random_model(cfg, folder, seed=seed, std=0.02)
    print(f"[bench] wrote a random {n_layers}-layer {tag} model folder in {time.time() - t0:.1f}s", file=sys.stderr)
    return folder


def drop_folder(folder: str) -> None:
    import shutil
    shutil.rmtree(folder, ignore_errors=True)


def random_prompts(lengths, vocab: int, seed: int):
    import torch
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (int(n),), generator=g).tolist() for n in lengths]


def time_decode(engine, batch: int, prompt_len: int, steps: int, warmup: int, seed: int):
    """Device time of `steps` decode steps of `batch` sequences after prompts of `prompt_len` tokens.
    Returns (seconds, mean context length over the timed steps, launches of this library's kernels)."""
    import torch
    from llm_infer_engine_b200.engine.engine import bucket_for
    from llm_infer_engine_b200.kernels import ops
    cache = engine.cache
    prompts = random_prompts([prompt_len] * batch, engine.vocab_size, seed)
    slots = [engine.open() for _ in range(batch)]
    try:
        logits = engine.step(slots, prompts, "last")
        sampled = torch.empty(batch, dtype=torch.int32, device=engine.device)
        ops.sample(logits, sampled)
        graph = engine.decode_graph(bucket_for(batch), prompt_len + warmup + steps + 1)
        graph.set_lanes(slots)
        graph.tokens[:batch].copy_(sampled)

        def one_step():
            for s in slots:
                cache.reserve(s, cache.lengths[s] + 1)
            out = graph.replay()
            for s in slots:
                cache.note_appended(s, cache.lengths[s] + 1, device_updated=True)
            ops.sample(out[:batch], graph.tokens)      # greedy; feeds the next step on the device

        for _ in range(warmup):
            one_step()
        torch.cuda.synchronize()
        ctx0 = cache.lengths[slots[0]]
        launches0 = ops.LAUNCHES
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        for _ in range(steps):
            one_step()
        end.record()
        torch.cuda.synchronize()
        seconds = start.elapsed_time(end) / 1e3
        mean_ctx = ctx0 + (steps + 1) / 2.0
        return seconds, mean_ctx, ops.LAUNCHES - launches0
    finally:
        for s in slots:
            engine.close(s)


def time_prefill(engine, n_tokens: int, warmup: int, reps: int, seed: int):
    """Median time of a one-prompt step: host token ids in, logits of the last row on the device."""
    import torch
    prompt = random_prompts([n_tokens], engine.vocab_size, seed)[0]
    times = []
    for i in range(warmup + reps):
        slot = engine.open()
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        engine.step([slot], [prompt], "last")
        end.record()
        torch.cuda.synchronize()
        engine.close(slot)
        if i >= warmup:
            times.append(start.elapsed_time(end) / 1e3)
    times.sort()
    return times[len(times) // 2]


def prefill_flops(cfg: dict, n_layers: int, lengths) -> float:
    """GEMM and causal-attention FLOPs of a prompt step over sequences of these lengths; the head runs on the
    last row of each."""
    d, ff, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    hq, hkv, hd = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    per_token = 2 * (d * (hq + 2 * hkv) * hd + hq * hd * d + 3 * d * ff)
    total = 0.0
    for T in lengths:
        total += n_layers * per_token * T + 2 * d * V
        total += n_layers * 4 * hq * hd * (T * (T + 1) / 2)      # causal QK^T and PV
    return total


def e2e_decode(engine, batch: int, steps: int, seed: int):
    """Decoded tokens per second through generate(): host prompts in, host tokens out every step."""
    from llm_infer_engine_b200 import GenerationStats, SamplingParams, generate
    prompts = random_prompts([PROMPT_LEN] * batch, engine.vocab_size, seed)
    generate(engine, prompts[:batch], max_new_tokens=8, stop_ids=[])            # warm-up: graphs, pools
    stats = GenerationStats()
    generate(engine, prompts, max_new_tokens=steps + 1, sampling=SamplingParams(), stop_ids=[], stats=stats)
    return stats.decode_tokens / stats.decode_seconds, stats


def workload_config(args, n_layers: int, pk: dict) -> dict:
    """The `config` of the JSON line: the workload and every layer size, the same for both arms."""
    c = CONFIG_1B
    return {
        "model": "Llama-3.2-1B shape", "global_batch": args.batch, "seq_len": CONTEXT, "parallelism": "single GPU",
        "layers": n_layers, "layers_full": c["num_hidden_layers"], "hidden_size": c["hidden_size"],
        "heads": c["num_attention_heads"], "kv_heads": c["num_key_value_heads"], "head_dim": c["head_dim"],
        "intermediate_size": c["intermediate_size"], "vocab_size": c["vocab_size"], "prompt_len": PROMPT_LEN,
        "new_tokens": args.steps, "prefill_tokens": PREFILL_TOKENS, "sampling": "greedy",
        "l2": "weights 2.5 GB per step >> 126 MB L2, no flush needed", "peaks": pk["source"],
    }


# ------------------------------------------------------------------------------------------ larger shapes
def run_3b(n_layers: int, pk: dict, new_tokens: int = 256) -> dict:
    """Llama 3.2 3B shape: 16 requests with prompt lengths uniform in [128, 2048] start together (one ragged
    prompt step), each generates `new_tokens`; through generate(), host tokens in and out."""
    import torch
    from llm_infer_engine_b200 import Engine, GenerationStats, generate
    cfg = CONFIG_3B
    folder = make_model_folder(cfg, n_layers, seed=3, tag="3b")
    g = torch.Generator().manual_seed(33)
    lens = [int(x) for x in torch.randint(128, 2049, (16,), generator=g)]
    total = sum((n + new_tokens + 64) // 64 * 64 for n in lens)
    engine = Engine(folder, dtype="bfloat16", device=0, max_batch=16, max_seq_len=CONTEXT, max_tokens=total)
    drop_folder(folder)
    prompts = random_prompts(lens, engine.vocab_size, seed=34)
    # warm-up with the same lengths: the sequences outgrow a captured step's length bucket on the way (2,048 to
    # 4,096), and capturing the next one belongs to start-up, not to the steps that are timed
    generate(engine, prompts, max_new_tokens=new_tokens, stop_ids=[])
    # three timed runs, the median of each figure: the prompt step is a single eager step of 18 thousand tokens
    # and its time scatters from run to run
    runs = []
    for _ in range(3):
        st = GenerationStats()
        generate(engine, prompts, max_new_tokens=new_tokens, stop_ids=[], stats=st)
        runs.append(st)
    print("[bench] 3B runs: prefill ms " + ", ".join(f"{r.prefill_seconds * 1e3:.1f}" for r in runs) + "; decode ms/step "
          + ", ".join(f"{r.decode_seconds / r.decode_steps * 1e3:.3f}" for r in runs), file=sys.stderr)
    stats = sorted(runs, key=lambda r: r.decode_seconds)[1]
    stats.prefill_seconds = sorted(r.prefill_seconds for r in runs)[1]
    steps = stats.decode_steps
    mean_keys = sum(lens) + 16 * (steps + 1) / 2.0                               # keys all 16 hold, mean over the steps
    step_bytes = engine.weight_bytes_per_step() + engine.kv_bytes_per_token() * mean_keys
    achieved = step_bytes / (stats.decode_seconds / steps) / 1e9
    flops = prefill_flops(cfg, n_layers, lens)
    out = {
        "model": "Llama-3.2-3B shape", "layers": n_layers, "layers_full": cfg["num_hidden_layers"],
        "requests": 16, "prompt_tokens": sum(lens), "new_tokens": new_tokens,
        "decode_tok_s": round(stats.decode_tokens / stats.decode_seconds, 1),
        "decode_ms_per_step": round(stats.decode_seconds / steps * 1e3, 4),
        "decode_gbs": round(achieved, 1), "decode_frac_hbm": round(achieved / pk["hbm_gbs"], 4),
        "prefill_tok_s": round(stats.prefill_tokens / stats.prefill_seconds, 1),
        "prefill_ms": round(stats.prefill_seconds * 1e3, 3),
        "prefill_frac_bf16": round(flops / stats.prefill_seconds / (pk["bf16_tflops"] * 1e12), 4),
        "path": "generate(): host tokens in and out every step", "timed_runs": 3,
    }
    del engine
    torch.cuda.empty_cache()
    return out


def run_8b(n_layers: int, pk: dict, steps: int, warmup: int) -> dict:
    """Llama 3.1 8B shape: one 2,048-token prefill; decode at batch 64 after 1,024-token prompts. The cache is
    sized by need (64 sequences of 1,024 + the decoded tokens), not for 64 x 8,192."""
    import torch
    from llm_infer_engine_b200 import Engine
    cfg = CONFIG_8B
    folder = make_model_folder(cfg, n_layers, seed=4, tag="8b")
    prompt_len, batch = 1024, 64
    per_seq = (prompt_len + steps + warmup + 64 + 63) // 64 * 64
    engine = Engine(folder, dtype="bfloat16", device=0, max_batch=batch, max_seq_len=8192, max_tokens=batch * per_seq)
    drop_folder(folder)
    sec, mean_ctx, _ = time_decode(engine, batch, prompt_len, steps, warmup, seed=44)
    step_bytes = engine.weight_bytes_per_step() + engine.kv_bytes_per_token() * mean_ctx * batch
    achieved = step_bytes / (sec / steps) / 1e9
    prefill_s = time_prefill(engine, PREFILL_TOKENS, warmup=3, reps=3, seed=45)
    flops = prefill_flops(cfg, n_layers, [PREFILL_TOKENS])
    out = {
        "model": "Llama-3.1-8B shape", "layers": n_layers, "layers_full": cfg["num_hidden_layers"],
        "decode_batch": batch, "prompt_len": prompt_len, "new_tokens": steps,
        "decode_tok_s": round(batch * steps / sec, 1), "decode_ms_per_step": round(sec / steps * 1e3, 4),
        "decode_gbs": round(achieved, 1), "decode_frac_hbm": round(achieved / pk["hbm_gbs"], 4),
        "prefill_tokens": PREFILL_TOKENS, "prefill_tok_s": round(PREFILL_TOKENS / prefill_s, 1),
        "prefill_ms": round(prefill_s * 1e3, 3),
        "prefill_frac_bf16": round(flops / prefill_s / (pk["bf16_tflops"] * 1e12), 4),
    }
    del engine
    torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------ per-kernel report
def kernel_table(rows, n_steps: int, pk: dict, title: str) -> str:
    """Markdown table of a KernelTimer's rows, per step: microseconds, share, bytes -> GB/s and the fraction of
    the measured copy bandwidth, FLOPs -> TFLOP/s and the fraction of the measured bf16 GEMM rate."""
    total = sum(r["us"] for r in rows) or 1.0
    lines = [f"### {title}", "",
             "| stage | kernel | launches/step | us/step | share | MB/step | GB/s | of HBM peak | GFLOP/step | TFLOP/s | "
             "of bf16 peak |", "|---|---|---|---|---|---|---|---|---|---|---|"]
    for r in sorted(rows, key=lambda r: -r["us"]):
        us = r["us"] / n_steps
        sec = us * 1e-6
        gbs = r["bytes"] / n_steps / sec / 1e9 if sec > 0 else 0.0
        tf = r["flops"] / n_steps / sec / 1e12 if sec > 0 else 0.0
        lines.append(f"| {r['stage']} | {r['kernel']} | {r['launches'] / n_steps:.0f} | {us:.1f} | "
                     f"{100 * r['us'] / total:.1f} % | {r['bytes'] / n_steps / 1e6:.2f} | {gbs:.0f} | "
                     f"{100 * gbs / pk['hbm_gbs']:.1f} % | {r['flops'] / n_steps / 1e9:.2f} | {tf:.1f} | "
                     f"{100 * tf / pk['bf16_tflops']:.1f} % |")
    lines.append(f"| | **sum** | {sum(r['launches'] for r in rows) / n_steps:.0f} | {total / n_steps:.1f} | | "
                 f"{sum(r['bytes'] for r in rows) / n_steps / 1e6:.2f} | | | "
                 f"{sum(r['flops'] for r in rows) / n_steps / 1e9:.2f} | | |")
    return "\n".join(lines) + "\n"


def run_per_kernel(args, engine, pk: dict) -> str:
    """Times every kernel of the EAGER step with CUDA events (no graph, no overlap between kernels, so the sum
    is above the captured step's time). Peaks are the measured ones."""
    import torch
    from llm_infer_engine_b200.kernels import ops, trace
    n_layers = engine.config.num_hidden_layers
    parts = [f"Per-kernel times, Llama 3.2 1B shape, {n_layers} layers, bfloat16, eager steps bracketed by CUDA events "
             f"(peaks: {pk['hbm_gbs']:.0f} GB/s, {pk['bf16_tflops']:.0f} TFLOP/s, {pk['source']}).\n"]
    n_steps = 8
    for batch in (1, 8, 64):
        prompts = random_prompts([PROMPT_LEN] * batch, engine.vocab_size, seed=10 + batch)
        slots = [engine.open() for _ in range(batch)]
        logits = engine.step(slots, prompts, "last")
        tokens = torch.empty(batch, dtype=torch.int32, device=engine.device)
        ops.sample(logits, tokens)
        for _ in range(3):                                  # warm-up, untimed
            logits = engine.step(slots, [[t] for t in tokens.tolist()], "last")
            ops.sample(logits, tokens)
        with trace.timing() as timer:
            for _ in range(n_steps):
                logits = engine.step(slots, [[t] for t in tokens.tolist()], "last")
                trace.push("Sample")
                ops.sample(logits, tokens)
                trace.pop()
            rows = timer.table()
        for s in slots:
            engine.close(s)
        parts.append(kernel_table(rows, n_steps, pk, f"decode, batch {batch}, context {PROMPT_LEN + 4}..{PROMPT_LEN + 4 + n_steps}"))
    prompt = random_prompts([PREFILL_TOKENS], engine.vocab_size, seed=99)[0]
    for i in range(3):
        slot = engine.open()
        engine.step([slot], [prompt], "last")
        engine.close(slot)
    with trace.timing() as timer:
        for _ in range(3):
            slot = engine.open()
            engine.step([slot], [prompt], "last")
            engine.close(slot)
        rows = timer.table()
    parts.append(kernel_table(rows, 3, pk, f"prefill, one prompt of {PREFILL_TOKENS} tokens"))
    return "\n".join(parts)


# ------------------------------------------------------------------------------------------ two designs side by side
def zemivik_config(width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, n_layers: int,
                   window: int, keep_first: int) -> dict:
    """A Zemivik configuration with a Llama shape's layer sizes (window 0 = no mask: every earlier token)."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
             "v_mix": True, "mask": {"size": window, "keep_first": keep_first} if window else None}
    return {"architecture": "Zemivik", "vocab": vocab, "width": width, "max_positions": CONTEXT,
            "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5},
            "layers": [{"type": "attention", "mixer": dict(mixer), "mlp": {"kind": "dense", "ff": ff}}
                       for _ in range(n_layers)]}


def dofipel_config(width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, n_layers: int,
                   window: int) -> dict:
    """A Dofipel configuration with a Llama shape's layer sizes. Layers cycle through its four kinds: windowed
    attention + gated feed-forward, latent attention + routed experts, latent attention that reads the layer
    before's latent + gated feed-forward, windowed attention + routed experts. The routed feed-forward's active
    width (3 of 16 experts of ff / 4, plus a shared expert of ff / 4) equals the dense one's; the latent is
    4 head sizes wide with a rotated part of half a head size."""
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
            "softcap": 30.0, "bias_max": 2048, "mask": {"size": window} if window else None}
    rot = head_dim // 2
    latent = {"heads": heads, "dim": head_dim, "rot_dim": rot, "vdim": head_dim, "kv_rank": 4 * head_dim,
              "scale": (head_dim + rot) ** -0.5, "rot": {"base": 10000.0, "dims": rot}}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "router": {"experts": 16, "top": 3}, "expert": {"ff": ff // 4}, "shared": {"ff": ff // 4}}
    layers = []
    for i in range(n_layers):
        kind = i % 4
        if kind == 0:
            layers.append({"type": "attention", "mixer": dict(attn), "mlp": dense})
        elif kind == 1:
            layers.append({"type": "latent_attention", "mixer": dict(latent), "mlp": moe})
        elif kind == 2:
            layers.append({"type": "latent_attention", "mixer": dict(latent, kv_from=i - 1), "mlp": dense})
        else:
            layers.append({"type": "attention", "mixer": dict(attn), "mlp": moe})
    return {"architecture": "Dofipel", "vocab": vocab, "width": width, "logit_scale": 1.0, "norm": {"eps": 1e-6},
            "layers": layers}


def ganupel_config(width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, n_layers: int,
                   window: int) -> dict:
    """A Ganupel configuration with a Llama shape's layer sizes. Layers cycle through four kinds: the two mixers
    side by side (sigmoid-weight attention over a window, and a gated linear recurrence with as many heads, half
    a head size of gate channels and a head size of value channels) + dense feed-forward, the same + routed experts,
    a recurrent unit as wide as the model (one block per head) + routed experts, the two mixers + routed experts.
    The routed feed-forward's active width (4 of 16 experts of ff / 4, beside 4 outputs that return the input)
    is at most the dense one's."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
            "rot": {"base": 10000.0, "dims": head_dim}, "mask": {"size": window} if window else None}
    right = {"heads": heads, "dim": head_dim // 2, "vdim": head_dim}
    both = {"left": left, "right": right, "left_scale": 1.0, "right_scale": 1.0}
    unit = {"width": width, "blocks": heads, "conv": 4}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "router": {"experts": 16, "identity": 4, "top": 4, "scale": 1.0}, "expert": {"ff": ff // 4}}
    layers = []
    for i in range(n_layers):
        kind = i % 4
        if kind == 2:
            layers.append({"type": "rglru", "mixer": dict(unit), "mlp": moe})
        else:
            layers.append({"type": "parallel", "mixer": json.loads(json.dumps(both)), "mlp": dense if kind == 0 else moe})
    return {"architecture": "Ganupel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers}


def burinex_config(width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, n_layers: int,
                   window: int) -> dict:
    """A Burinex configuration with a Llama shape's layer sizes. Layers cycle through four kinds: latent attention
    (queries through a latent of 6 head sizes, a cached latent of 4 head sizes with a rotated part of half a head size,
    YaRN-scaled rotation, a window, a learned sink), grouped-query attention with a query temperature, a sink and a gate
    per head, linear attention with a decay per head (as many heads, a head size of key and of value channels), and the
    grouped-query attention again. Every layer has the routed feed-forward: 3 of 16 experts of ff / 4 under a sigmoid
    router whose weights multiply the experts' input, plus a shared expert of ff / 4 (the active width of the dense
    feed-forward of the shape)."""
    rot = head_dim // 2
    latent = {"heads": heads, "dim": head_dim, "rot_dim": rot, "vdim": head_dim, "kv_rank": 4 * head_dim,
              "q_rank": 6 * head_dim, "scale": (head_dim + rot) ** -0.5, "mask": {"size": window} if window else None,
              "rot": {"base": 10000.0, "dims": rot,
                      "scaling": {"factor": 8.0, "original": 2048, "fast": 16.0, "slow": 2.0}}}
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
            "q_temp": {"coef": 0.25, "every": 256}}
    linear = {"heads": heads, "dim": head_dim, "vdim": head_dim,
              "decay": [1.0 - 2.0 ** (-1.0 - 7.0 * h / max(heads - 1, 1)) for h in range(heads)]}
    moe = {"kind": "moe", "router": {"experts": 16, "top": 3}, "expert": {"ff": ff // 4}, "shared": {"ff": ff // 4}}
    kinds = [("latent_attention", latent), ("attention", attn), ("lightning", linear), ("attention", attn)]
    layers = [{"type": kinds[i % 4][0], "mixer": json.loads(json.dumps(kinds[i % 4][1])), "mlp": dict(moe)}
              for i in range(n_layers)]
    return {"architecture": "Burinex", "vocab": vocab, "width": width, "postln_alpha": 2.0, "logit_softcap": 50.0,
            "norm": {"eps": 1e-6}, "layers": layers}


def rogizen_config(width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, n_layers: int,
                   chunk: int) -> dict:
    """A Rogizen configuration with a Llama shape's layer sizes. Layers cycle through four kinds: attention in chunks (4
    taps, whole heads rotated with YaRN-scaled frequencies) + feed-forward, a state space layer (twice the width inside,
    heads of 64 columns over 128 state rows, one group, 4 taps) + feed-forward, the same without a feed-forward, attention
    + feed-forward. All layers form the loop, of one pass, so that as many layers run as in the other design."""
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "conv": 4, "scale": head_dim ** -0.5,
            "mask": {"size": chunk} if chunk else None,
            "rot": {"base": 10000.0, "dims": head_dim,
                    "scaling": {"factor": 8.0, "original": 2048, "fast": 16.0, "slow": 2.0}}}
    ssm = {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1, "conv": 4}
    dense = {"kind": "dense", "ff": ff}
    kinds = [("attention", attn, dense), ("mamba2", ssm, dense), ("mamba2", ssm, None), ("attention", attn, dense)]
    layers = [{"type": k, "mixer": json.loads(json.dumps(m)), "mlp": f} for k, m, f in (kinds[i % 4] for i in range(n_layers))]
    return {"architecture": "Rogizen", "vocab": vocab, "width": width, "embedding": {"scale": width ** 0.5},
            "logit_softcap": 30.0, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": n_layers, "times": 1},
            "layers": layers}


def selinex_config(width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, n_layers: int,
                   window: int) -> dict:
    """A Selinex configuration with a Llama shape's layer sizes. Layers cycle through four kinds: window attention with a
    gate per head beside gated linear attention (as many heads, half a head size of key channels and a head size of value
    channels) + dense feed-forward, rotated window attention beside time mixing (as many heads of a head size) + routed
    experts, the gated delta rule (as many heads, a head size of key and of value channels, 4 taps) + routed experts, the
    first pair again + routed experts. The routed feed-forward uses 4 of 16 experts of ff / 4, from two of four groups (the
    active width of the dense one). The loop holds all layers and runs once, so that as many layers run as in the other
    design."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
            "mask": {"size": window} if window else None}
    first = {"left": left, "right": {"heads": heads, "dim": head_dim // 2, "vdim": head_dim, "tau": 16.0},
             "left_scale": 0.5, "right_scale": 0.5}
    second = {"left": dict(left, rot={"base": 10000.0, "dims": head_dim}), "right": {"heads": heads, "dim": head_dim}}
    delta = {"heads": heads, "kv_heads": heads, "dim": head_dim, "vdim": head_dim, "conv": 4}
    dense = {"kind": "dense", "ff": ff, "limit": 7.0}
    moe = {"kind": "moe", "router": {"experts": 16, "top": 4, "groups": {"count": 4, "keep": 2}}, "expert": {"ff": ff // 4}}
    kinds = [("parallel", first, dense), ("parallel_2", second, moe), ("delta", delta, moe), ("parallel", first, moe)]
    layers = [{"type": k, "mixer": json.loads(json.dumps(m)), "mlp": f} for k, m, f in (kinds[i % 4] for i in range(n_layers))]
    return {"architecture": "Selinex", "vocab": vocab, "width": width, "residual_mult": 0.5, "norm": {"eps": 1e-6},
            "loop": {"start": 0, "stop": n_layers, "times": 1}, "layers": layers}


def step_tables(engine, pk: dict, title: str, batch: int = 8) -> str:
    """Per-kernel tables (eager steps, CUDA events) of a decode step at `batch` sequences and of a 2,048-token
    prompt."""
    import torch
    from llm_infer_engine_b200.kernels import ops, trace
    n_steps = 8
    prompts = random_prompts([PROMPT_LEN] * batch, engine.vocab_size, seed=10 + batch)
    slots = [engine.open() for _ in range(batch)]
    logits = engine.step(slots, prompts, "last")
    tokens = torch.empty(batch, dtype=torch.int32, device=engine.device)
    ops.sample(logits, tokens)
    for _ in range(3):
        logits = engine.step(slots, [[t] for t in tokens.tolist()], "last")
        ops.sample(logits, tokens)
    with trace.timing() as timer:
        for _ in range(n_steps):
            logits = engine.step(slots, [[t] for t in tokens.tolist()], "last")
            ops.sample(logits, tokens)
        rows = timer.table()
    for s_ in slots:
        engine.close(s_)
    parts = [kernel_table(rows, n_steps, pk, f"{title}: decode, batch {batch}, context about {PROMPT_LEN + 8}")]
    prompt = random_prompts([PREFILL_TOKENS], engine.vocab_size, seed=99)[0]
    for _ in range(3):
        slot = engine.open()
        engine.step([slot], [prompt], "last")
        engine.close(slot)
    with trace.timing() as timer:
        for _ in range(3):
            slot = engine.open()
            engine.step([slot], [prompt], "last")
            engine.close(slot)
        rows = timer.table()
    parts.append(kernel_table(rows, 3, pk, f"{title}: prefill, one prompt of {PREFILL_TOKENS} tokens"))
    return "\n".join(parts)


def run_designs(args, pk: dict, which: str = "Zemivik") -> str:
    """Zemivik (or, with which="Dofipel", Dofipel with a window of 1,024) beside Llama at equal layer sizes, or, with
    which="Ganupel" or "Burinex", that design beside Dofipel, or, with which="Rogizen" or "Selinex", that design beside
    Ganupel (random weights, bfloat16): decode throughput at batch 1, 8 and 64
    after 512-token prompts (captured steps, device time), prefill throughput of one 2,048-token prompt, and the
    per-kernel tables of both. Zemivik once without a mask (the attention work of Llama's) and once with a window
    of 1,024 tokens that keeps the first four. The shared vocabulary is kept small so that the layers, not the
    head, are what is compared."""
    import torch
    from llm_infer_engine_b200 import Engine, write_random_model
    from llm_infer_engine_b200.weights import scratch_folder
    n_layers = args.layers or 4
    vocab = 32000
    shapes = [("1B layer sizes", CONFIG_1B), ("8B layer sizes", CONFIG_8B)]
    steps = min(args.steps, 64)
    beside = {"Ganupel": "Dofipel", "Burinex": "Dofipel", "Rogizen": "Ganupel", "Selinex": "Ganupel"}.get(which, "Llama")
    lines = [f"{which} beside {beside} at equal layer sizes, {n_layers} layers, vocabulary {vocab}, bfloat16, random weights "
             f"(peaks: {pk['hbm_gbs']:.0f} GB/s, {pk['bf16_tflops']:.0f} TFLOP/s, {pk['source']}).", "",
             "| layer sizes | design | decode b1 tok/s | ms/step | decode b8 tok/s | ms/step | decode b64 tok/s | ms/step | "
             f"prefill {PREFILL_TOKENS} tok/s | ms |", "|---|---|---|---|---|---|---|---|---|---|"]
    tables = []
    for name, base in shapes:
        d, hq, hkv, hd, ff = (base["hidden_size"], base["num_attention_heads"], base["num_key_value_heads"],
                              base["head_dim"], base["intermediate_size"])
        llama = dict(base, vocab_size=vocab, num_hidden_layers=n_layers, tie_word_embeddings=False, bos_token_id=1,
                     eos_token_id=2)
        designs = [("Llama", llama),
                   ("Zemivik, no mask", zemivik_config(d, hq, hkv, hd, ff, vocab, n_layers, 0, 0)),
                   ("Zemivik, window 1024 + 4", zemivik_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024, 4))]
        if which == "Dofipel":
            designs = [("Llama", llama),
                       ("Dofipel, window 1024", dofipel_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024))]
        if which == "Ganupel":
            designs = [("Dofipel, window 1024", dofipel_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024)),
                       ("Ganupel, window 1024", ganupel_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024))]
        if which == "Burinex":
            designs = [("Dofipel, window 1024", dofipel_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024)),
                       ("Burinex, window 1024", burinex_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024))]
        if which == "Rogizen":
            designs = [("Ganupel, window 1024", ganupel_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024)),
                       ("Rogizen, chunks of 1024", rogizen_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024))]
        if which == "Selinex":
            designs = [("Ganupel, window 1024", ganupel_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024)),
                       ("Selinex, window 1024", selinex_config(d, hq, hkv, hd, ff, vocab, n_layers, 1024))]
        for design, cfg in designs:
            folder = scratch_folder("llmie_bench_design_")
            write_random_model(cfg, folder, seed=3, std=0.02)
            per_seq = PROMPT_LEN + steps + args.warmup + 64
            engine = Engine(folder, dtype="bfloat16", device=0, max_batch=64, max_seq_len=CONTEXT,
                            max_tokens=max(64 * ((per_seq + 63) // 64 * 64), PREFILL_TOKENS + 64), cuda_graph=True)
            drop_folder(folder)
            cells = []
            for batch in (1, 8, 64):
                sec, _, _ = time_decode(engine, batch, PROMPT_LEN, steps, max(args.warmup, 3), seed=batch)
                cells += [f"{batch * steps / sec:,.0f}", f"{1e3 * sec / steps:.3f}"]
            t = time_prefill(engine, PREFILL_TOKENS, warmup=3, reps=5, seed=7)
            cells += [f"{PREFILL_TOKENS / t:,.0f}", f"{1e3 * t:.2f}"]
            lines.append(f"| {name} | {design} | " + " | ".join(cells) + " |")
            print(f"[bench] {name} / {design}: {cells}", file=sys.stderr)
            if design != "Zemivik, no mask":
                engine.use_cuda_graph = False
                tables.append(step_tables(engine, pk, f"{name}, {design}"))
            del engine
            torch.cuda.empty_cache()
    return "\n".join(lines) + "\n\n" + "\n".join(tables)


# ------------------------------------------------------------------------------------------ attention kernels alone
def attention_sweep(heads: int, kv_heads: int, head_dim: int, pk: dict) -> str:
    """The two attention kernels alone, at several batch sizes and context lengths, against the measured peaks:
    the one-token kernel by the cache bytes it has to read, the prompt kernel by its FLOPs. Every case is 16
    launches in one CUDA graph over caches that rotate through more than the L2 holds; CUDA events around two
    replays."""
    import torch
    from llm_infer_engine_b200.kernels import ops
    dev, P = "cuda", 64
    ops.set_pdl(False)                      # a launch may not start while the one before it runs: these are kernel times

    def timed(call, n=16):
        for i in range(3):
            call(i)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for i in range(n):
                call(i)
        g.replay()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        g.replay()
        g.replay()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) * 1e3 / (2 * n)

    lines = [f"Attention kernels alone, {heads} query / {kv_heads} KV heads of {head_dim}, bfloat16 "
             f"(peaks: {pk['hbm_gbs']:.0f} GB/s, {pk['bf16_tflops']:.0f} TFLOP/s, {pk['source']}).", "",
             "### one token a sequence (`attention_decode_mma` with rotation and cache write inside)", "",
             "| batch | context | MB of cache read | us | GB/s | of HBM peak |", "|---|---|---|---|---|---|"]
    gen = torch.Generator(device=dev).manual_seed(0)
    for batch, ctx in [(1, 512), (8, 512), (32, 512), (64, 512), (128, 512), (64, 1024), (16, 1200), (8, 3500),
                       (64, 3500)]:
        pages_per = (ctx + 16 + P - 1) // P
        nbytes = batch * ctx * kv_heads * head_dim * 2 * 2
        copies = max(2, int(300e6 // nbytes) + 1)
        ks = [torch.randn(batch * pages_per + 1, kv_heads, P, head_dim, device=dev, generator=gen).to(torch.bfloat16)
              for _ in range(copies)]
        vs = [torch.randn(batch * pages_per + 1, kv_heads, P, head_dim, device=dev, generator=gen).to(torch.bfloat16)
              for _ in range(copies)]
        table = torch.randperm(batch * pages_per, device=dev, generator=gen).to(torch.int32).view(batch, pages_per)
        qkv = torch.randn(batch, (heads + 2 * kv_heads) * head_dim, device=dev, generator=gen).to(torch.bfloat16)
        out = torch.empty(batch, heads * head_dim, dtype=torch.bfloat16, device=dev)
        rope = torch.randn(ctx + 64, head_dim // 2, 2, device=dev, generator=gen)
        slots = torch.arange(batch, device=dev, dtype=torch.int32)
        lens = torch.full((batch,), ctx, device=dev, dtype=torch.int32)
        pages = ops.attention_decode_mma_pages(batch, heads, kv_heads, ctx)
        n_runs = ((ctx + 63) // 64 + pages - 1) // pages
        counters = torch.zeros(ops.decode_counter_ints(batch, heads, kv_heads) + 64, dtype=torch.int32, device=dev)
        scratch = torch.empty(max(1, ops.decode_scratch_floats(batch, heads, head_dim, n_runs)), dtype=torch.float32,
                              device=dev)
        us = timed(lambda i: ops.attention_decode_mma_rope(
            qkv, ks[i % copies], vs[i % copies], out, rope, slots, lens, table.contiguous(), P, heads, kv_heads,
            head_dim, head_dim ** -0.5, 0, pages, n_runs, True, counters=counters, scratch=scratch))
        gbs = nbytes / us / 1e3
        lines.append(f"| {batch} | {ctx} | {nbytes / 1e6:.1f} | {us:.1f} | {gbs:.0f} | {100 * gbs / pk['hbm_gbs']:.0f} % |")
        del ks, vs
    lines += ["", "### prompts (`attention_prefill_tc`, causal, from position 0)", "",
              "| prompts | tokens each | GFLOP | us | TFLOP/s | of bf16 peak |", "|---|---|---|---|---|---|"]
    for n_seqs, T in [(8, 512), (3, 1000), (1, 2048), (1, 4096), (1, 8192), (4, 2048)]:
        pages_per = (T + P - 1) // P
        k = torch.randn(n_seqs * pages_per + 1, kv_heads, P, head_dim, device=dev, generator=gen).to(torch.bfloat16)
        v = torch.randn(n_seqs * pages_per + 1, kv_heads, P, head_dim, device=dev, generator=gen).to(torch.bfloat16)
        table = torch.arange(n_seqs * pages_per, device=dev, dtype=torch.int32).view(n_seqs, pages_per).contiguous()
        q = torch.randn(n_seqs * T, heads * head_dim, device=dev, generator=gen).to(torch.bfloat16)
        out = torch.empty_like(q)
        cu = torch.arange(0, (n_seqs + 1) * T, T, device=dev, dtype=torch.int32)
        slots = torch.arange(n_seqs, device=dev, dtype=torch.int32)
        start = torch.zeros(n_seqs, device=dev, dtype=torch.int32)
        us = timed(lambda i: ops.attention_prefill_tc(q, k, v, out, cu, slots, start, table, P, n_seqs, T, heads,
                                                      kv_heads, head_dim, head_dim ** -0.5, 0), n=8)
        ops.check_tc_status(dev)
        flops = n_seqs * 4.0 * heads * head_dim * (T * (T + 1) / 2)
        tf = flops / us / 1e6
        lines.append(f"| {n_seqs} | {T} | {flops / 1e9:.1f} | {us:.1f} | {tf:.0f} | {100 * tf / pk['bf16_tflops']:.0f} % |")
        del k, v, q, out
    ops.set_pdl(True)
    return "\n".join(lines)


# ------------------------------------------------------------------------------------------ the two arms
def run_ours(args):
    import torch
    if not torch.cuda.is_available():
        print(json.dumps({"metric": METRIC, "error": "no CUDA device"}))
        return 1
    from llm_infer_engine_b200 import Engine
    pk = peaks()
    if args.attention_sweep:
        text = attention_sweep(args.heads, args.kv_heads, args.head_dim, pk)
        print(text)
        if args.per_kernel_out:
            with open(args.per_kernel_out, "w", encoding="utf-8") as f:
                f.write(text + "\n")
        return 0
    if args.designs or args.dofipel or args.ganupel or args.burinex or args.rogizen or args.selinex:
        text = run_designs(args, pk, "Selinex" if args.selinex else "Rogizen" if args.rogizen else "Burinex" if args.burinex else "Ganupel" if args.ganupel
                           else "Dofipel" if args.dofipel else "Zemivik")
        print(text)
        if args.per_kernel_out:
            with open(args.per_kernel_out, "w", encoding="utf-8") as f:
                f.write(text + "\n")
        return 0
    if args.shape:                                          # one of the larger workloads alone, at full depth
        cfg = CONFIG_3B if args.shape == "3b" else CONFIG_8B
        n = args.layers or cfg["num_hidden_layers"]
        out = run_3b(n, pk) if args.shape == "3b" else run_8b(n, pk, args.steps, args.warmup)
        print(json.dumps({"metric": METRIC, "impl": "ours", "dtype": "bf16", "shape": out}))
        return 0
    full_layers = CONFIG_1B["num_hidden_layers"]
    n_layers = args.layers or full_layers
    folder = make_model_folder(CONFIG_1B, n_layers, seed=2, tag="1b")
    max_batch = max(64, args.batch)
    per_seq = PROMPT_LEN + args.steps + args.warmup + 64
    engine = Engine(folder, dtype="bfloat16", device=0, max_batch=max_batch, max_seq_len=CONTEXT,
                    max_tokens=max(max_batch * ((per_seq + 63) // 64 * 64), PREFILL_TOKENS + 64), cuda_graph=True)
    drop_folder(folder)
    if args.per_kernel:
        text = run_per_kernel(args, engine, pk)
        if args.per_kernel_out:
            with open(args.per_kernel_out, "w") as f:
                f.write(text)
        print(text, file=sys.stderr)
    sampler = ClockSampler(0)
    sampler.start()
    results = {}
    launches = 0
    batches = (args.batch, 1, 64) if args.only == "all" else ((args.batch,) if args.only == "decode" else ())
    for batch in batches:
        if batch in results:
            continue
        sec, mean_ctx, n_launch = time_decode(engine, batch, PROMPT_LEN, args.steps, args.warmup, seed=10 + batch)
        results[batch] = (sec, mean_ctx)
        if batch == args.batch:
            launches = n_launch
    prefill_s = None
    if args.only in ("all", "prefill"):
        prefill_s = time_prefill(engine, PREFILL_TOKENS, warmup=max(3, min(args.warmup, 5)),
                                 reps=5 if args.only == "all" else 2, seed=99)
    e2e_tps = None
    if args.only == "all":
        e2e_tps, stats = e2e_decode(engine, args.batch, args.steps, seed=10 + args.batch)
    sampler.stop()

    flops = prefill_flops(CONFIG_1B, n_layers, [PREFILL_TOKENS])
    out = {
        "metric": METRIC, "value": None, "unit": "tokens/s", "n_gpus": 1, "steps": args.steps,
        "warmup": args.warmup, "ms_per_step": None, "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random weights N(0,0.02), "
        "uniform-random token ids", "impl": "ours",
        "config": workload_config(args, n_layers, pk),
        "impl_notes": {"path": "generate() / captured one-token steps", "head": "tied to the embedding"},
        "gpu_launches": int(launches),
    }
    if args.batch in results:
        sec, mean_ctx = results[args.batch]
        step_bytes = engine.weight_bytes_per_step() + engine.kv_bytes_per_token() * mean_ctx * args.batch
        achieved = step_bytes / (sec / args.steps) / 1e9
        out["value"] = round(args.batch * args.steps / sec, 1)
        out["ms_per_step"] = round(sec / args.steps * 1e3, 4)
        out["roofline"] = {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                           "frac": round(achieved / pk["hbm_gbs"], 4)}
    if e2e_tps is not None:
        out["e2e"] = {"value": round(e2e_tps, 1), "unit": "tokens/s", "h2d_bytes_per_step": 4 * args.batch,
                      "d2h_bytes_per_step": 4 * args.batch}
    if prefill_s is not None:
        out["prefill"] = {"value": round(PREFILL_TOKENS / prefill_s, 1), "tokens": PREFILL_TOKENS,
                          "ms": round(prefill_s * 1e3, 3),
                          "frac": round(flops / prefill_s / (pk["bf16_tflops"] * 1e12), 4)}
    if 1 in results and 64 in results:
        out["points"] = {f"decode_b{b}": round(b * args.steps / results[b][0], 1) for b in (1, 64)}
    out["clocks"] = sampler.summary()
    if args.only == "all" and not args.layers and not args.no_shapes:
        del engine
        torch.cuda.empty_cache()
        # the larger shapes: the 3B one at full depth, the 8B one at half depth (its folder of random weights
        # would be 16 GB; both numbers are in the record)
        out["shapes"] = {"llama_3b_ragged16": run_3b(CONFIG_3B["num_hidden_layers"], pk),
                         "llama_8b_b64": run_8b(CONFIG_8B["num_hidden_layers"] // 2, pk, min(args.steps, 64), 5)}
    print(json.dumps(out))
    return 0


def run_reference(args):
    """The unmodified reference on the same workload (baseline/reference_arm.py): the same JSON keys, with
    `"impl": "reference"`. Whatever stops it is reported with its own text in an `unavailable` line."""
    sys.path.insert(0, os.path.join(ROOT, "baseline"))
    try:
        import torch
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device")
        import reference_arm
        n_layers = args.layers or CONFIG_1B["num_hidden_layers"]
        arm = reference_arm.ReferenceArm(CONFIG_1B, n_layers, CONTEXT)
        pk = peaks()
        arm.compile_pass(args.batch, PROMPT_LEN)
        sampler = ClockSampler(0)
        sampler.start()
        sec, mean_ctx = arm.decode(args.batch, PROMPT_LEN, args.steps, args.warmup, seed=10 + args.batch,
                                   host_io=False)
        points = {}
        prefill_s = e2e_sec = None
        if args.only == "all":
            e2e_sec, _ = arm.decode(args.batch, PROMPT_LEN, args.steps, args.warmup, seed=10 + args.batch,
                                    host_io=True)
            for b in (1, 64):
                arm.compile_pass(b, PROMPT_LEN)
                s_b, _ = arm.decode(b, PROMPT_LEN, args.steps, args.warmup, seed=10 + b, host_io=True)
                points[f"decode_b{b}"] = round(b * args.steps / s_b, 1)
            s_g, _ = arm.decode(1, PROMPT_LEN, args.steps, args.warmup, seed=11, host_io=True, graph=True)
            points["decode_b1_graph"] = round(args.steps / s_g, 1)
            prefill_s = arm.prefill(PREFILL_TOKENS, warmup=3, reps=5, seed=99)
        sampler.stop()
    except Exception as exc:                                   # noqa: BLE001 - the reason goes into the line
        text = " ".join(f"{type(exc).__name__}: {exc}".split())[:400]
        print(json.dumps({"impl": "reference", "unavailable": text}))
        return 0
    step_bytes = arm.weight_bytes_per_step() + arm.kv_bytes_per_token() * mean_ctx * args.batch
    achieved = step_bytes / (sec / args.steps) / 1e9
    out = {
        "metric": METRIC, "value": round(args.batch * args.steps / sec, 1), "unit": "tokens/s", "n_gpus": 1,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(sec / args.steps * 1e3, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: the reference's own random initialisation, uniform-random token ids",
        "impl": "reference", "config": workload_config(args, n_layers, pk),
        "impl_notes": {"path": "Llama3.forward + KVCache + sample, eager (its graph runner serves batch 1 only: "
                               "points.decode_b1_graph)", "head": "separate output matrix (its random mode)"},
        "gpu_launches": 0,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
    }
    if e2e_sec is not None:
        out["e2e"] = {"value": round(args.batch * args.steps / e2e_sec, 1), "unit": "tokens/s",
                      "h2d_bytes_per_step": 8 * args.batch, "d2h_bytes_per_step": 8 * args.batch}
    if prefill_s is not None:
        flops = prefill_flops(CONFIG_1B, n_layers, [PREFILL_TOKENS])
        out["prefill"] = {"value": round(PREFILL_TOKENS / prefill_s, 1), "tokens": PREFILL_TOKENS,
                          "ms": round(prefill_s * 1e3, 3),
                          "frac": round(flops / prefill_s / (pk["bf16_tflops"] * 1e12), 4)}
    if points:
        out["points"] = points
    out["clocks"] = sampler.summary()
    print(json.dumps(out))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--prompt-len", type=int, default=512,
                    help="tokens every sequence holds before decoding starts (the benchmark's 512; up to the context)")
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration (0 = all)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--only", default="all", choices=["all", "decode", "prefill"],
                    help="measure only one part (for short profiler captures); the JSON line then lacks the rest")
    ap.add_argument("--shape", default="", choices=["", "3b", "8b"],
                    help="run only the Llama 3.2 3B or Llama 3.1 8B workload, at full depth unless --layers is given")
    ap.add_argument("--no-shapes", action="store_true", help="leave the 3B and 8B workloads out of the default run")
    ap.add_argument("--per-kernel", action="store_true",
                    help="also time every kernel of the eager steps and print the tables (stderr)")
    ap.add_argument("--per-kernel-out", default="", help="write the per-kernel tables to this file as well")
    ap.add_argument("--attention-sweep", action="store_true",
                    help="time the two attention kernels alone at several batch sizes and contexts; prints a table")
    ap.add_argument("--designs", action="store_true",
                    help="Zemivik beside Llama at equal layer sizes: decode and prefill throughput and per-kernel tables "
                         "(prints markdown; --layers sets the depth, default 4)")
    ap.add_argument("--dofipel", action="store_true",
                    help="the same comparison for Dofipel (windowed and latent attention, gated and routed "
                         "feed-forwards) beside Llama")
    ap.add_argument("--ganupel", action="store_true",
                    help="the same comparison for Ganupel (sigmoid-weight attention beside a gated linear recurrence, "
                         "recurrent units, PolyNorm and routed feed-forwards) beside Dofipel, the closest design")
    ap.add_argument("--burinex", action="store_true",
                    help="the same comparison for Burinex (post-norm layers; latent attention with a query latent, a "
                         "window and a learned sink; gated attention with a query temperature; linear attention with a "
                         "decay per head; routed experts weighted on their input) beside Dofipel, the closest design")
    ap.add_argument("--rogizen", action="store_true",
                    help="the same comparison for Rogizen (attention in chunks behind a short convolution, state space "
                         "layers, the embedding mixed into the stream) beside Ganupel, the closest design")
    ap.add_argument("--selinex", action="store_true",
                    help="the same comparison for Selinex (norms in front of and behind every branch; window attention "
                         "beside gated linear attention or time mixing, gated delta rule layers, a router over groups of "
                         "experts) beside Ganupel, the closest design")
    ap.add_argument("--heads", type=int, default=32, help="query heads of --attention-sweep")
    ap.add_argument("--kv-heads", type=int, default=8, help="KV heads of --attention-sweep")
    ap.add_argument("--head-dim", type=int, default=64, choices=[64, 128], help="head size of --attention-sweep")
    args = ap.parse_args()
    if args.gpus != 1:
        print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    global PROMPT_LEN
    PROMPT_LEN = max(1, min(args.prompt_len, CONTEXT - args.steps - max(args.warmup, 3) - 8))
    if args.impl == "reference":
        return run_reference(args)
    if args.warmup < 3:
        args.warmup = 3
    return run_ours(args)


if __name__ == "__main__":
    sys.exit(main())
