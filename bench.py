"""Decode and prefill throughput of the Llama-3.1-8B shape on one B200, random weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--layers L] [--impl ours|reference]
                    [--no-points] [--no-breakdown]

Prints ONE JSON line.  A "step" is one decode step of the whole batch.  ``value`` is decoded
tokens a second timed on the device (CUDA events around K steps, after W warm-up steps);
``e2e`` is the same through the Python entry point (``Local.generate``: host token ids in,
host token ids out every step); ``prefill`` is one 2,048-token prompt; ``roofline`` sets the
decode step's mandatory bytes (every weight once, the live requests' cache once) against the
measured copy bandwidth.  ``points`` adds decoding at batch 1 and 64 (device-timed and end to
end) and two more workloads of other shapes: the Llama-2-13B shape (one kv head a head) with
16 prompts of unequal lengths, and the Llama-3.2-3B shape (tied head) at batch 64 sampled at
temperature 1.0 through the entry point, and the two tiny workloads on the device and on the
library's plain C++ twin on the host (the CPU baseline).  ``classes`` times every kernel class of one decode
step and one prompt step launch by launch and sets each against its own bytes or operations.
``checked`` says that the tokens of the end-to-end run equal those of the same prompts
stepped without captured graphs; the line is not printed otherwise.  Every decode step
streams all weights (16 GB), far more than the 126 MB L2, so nothing is flushed between
iterations.

The reference (Harshil089/Borrowed-Compute) is a Rust workspace; no Rust toolchain exists
here, so ``--impl reference`` reports itself unavailable.
"""

from __future__ import annotations

import argparse
import gc
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)


def _llama3_scaling(factor: float) -> dict:
    return {"rope_type": "llama3", "factor": factor, "low_freq_factor": 1.0, "high_freq_factor": 4.0, "original_max_position_embeddings": 8192}


# The headline: the Llama-3.1-8B shape.
CONFIG_8B = {
    "architectures": ["LlamaForCausalLM"], "num_hidden_layers": 32, "hidden_size": 4096, "num_attention_heads": 32,
    "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 14336, "vocab_size": 128256, "rope_theta": 500000.0,
    "rope_scaling": _llama3_scaling(8.0), "rms_norm_eps": 1e-5, "tie_word_embeddings": False, "max_position_embeddings": 8192,
}
# The Llama-2-13B shape: every head has a kv head of its own.
CONFIG_13B = {
    "architectures": ["LlamaForCausalLM"], "num_hidden_layers": 40, "hidden_size": 5120, "num_attention_heads": 40,
    "num_key_value_heads": 40, "head_dim": 128, "intermediate_size": 13824, "vocab_size": 32000, "rope_theta": 10000.0,
    "rms_norm_eps": 1e-5, "tie_word_embeddings": False, "max_position_embeddings": 4096,
}
# The Llama-3.2-3B shape: the head is the embedding table.
CONFIG_3B = {
    "architectures": ["LlamaForCausalLM"], "num_hidden_layers": 28, "hidden_size": 3072, "num_attention_heads": 24,
    "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 8192, "vocab_size": 128256, "rope_theta": 500000.0,
    "rope_scaling": _llama3_scaling(32.0), "rms_norm_eps": 1e-5, "tie_word_embeddings": True, "max_position_embeddings": 16384,
}
# The two tiny configurations, which differ in every size and option; their workloads are timed
# against the library's plain C++ twin on the host.
CONFIG_TINY_A = {
    "architectures": ["LlamaForCausalLM"], "num_hidden_layers": 2, "hidden_size": 64, "num_attention_heads": 4, "num_key_value_heads": 2,
    "intermediate_size": 176, "vocab_size": 256, "rope_theta": 10000.0, "rms_norm_eps": 1e-5, "tie_word_embeddings": False,
    "max_position_embeddings": 128,
}
CONFIG_TINY_B = {
    "architectures": ["LlamaForCausalLM"], "num_hidden_layers": 3, "hidden_size": 96, "num_attention_heads": 4, "num_key_value_heads": 1,
    "head_dim": 32, "intermediate_size": 256, "vocab_size": 320, "rope_theta": 500000.0,
    "rope_scaling": {"rope_type": "llama3", "factor": 4.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0, "original_max_position_embeddings": 64},
    "rms_norm_eps": 1e-6, "tie_word_embeddings": True, "max_position_embeddings": 256,
}
CONTEXT = 8192
PROMPT = 2048
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


E2E_SETTLE_PASSES = 24   # decode passes after a prompt before the end-to-end clock starts (see end_to_end)


def peaks() -> dict:
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            d = json.load(f)
        out = {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
        if "bf16_tflops_sustained" in d:
            out["bf16_tflops_sustained"] = float(d["bf16_tflops_sustained"])
        return out
    except (OSError, KeyError, ValueError, TypeError):
        return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""

    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.lines, self.proc, self.thread = [], None, None

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=lambda: self.lines.extend(self.proc.stdout), daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
            self.thread.join(timeout=5)

    def summary(self):
        mhz, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in self.lines:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) < 6:
                continue
            try:
                mhz.append(int(parts[0]))
                mx = max(mx, int(parts[1]))
            except ValueError:
                continue
            for name, val in zip(names, parts[2:6]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        if not mhz:
            return None
        return {"sm_mhz": int(statistics.median(mhz)), "sm_max_mhz": mx, "reasons": sorted(reasons), "samples": len(mhz)}


# ------------------------------------------------------------------------ bytes and operations
def model_numbers(cfg: dict, layers: int) -> dict:
    E, H, G, D, F, V = (cfg["hidden_size"], cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"],
                        cfg["intermediate_size"], cfg["vocab_size"])
    qkv, o, gate_up, down = E * (H + 2 * G) * D, H * D * E, 2 * E * F, E * F
    return {"qkv": qkv, "o": o, "gate_up": gate_up, "down": down, "layer_params": qkv + o + gate_up + down, "head_params": V * E,
            "norm_params": (2 * layers + 1) * E, "kv_bytes_per_token": layers * 2 * G * D * 2, "E": E, "H": H, "G": G, "D": D, "F": F, "V": V}


def decode_bytes(cfg, layers, batch, cached_tokens) -> float:
    """What a decode step has to read: every weight it uses once (a tied head is the
    embedding table, read once as the head), the norms, the batch's embedding rows, and
    the cache of the live requests (``cached_tokens`` positions in all)."""
    n = model_numbers(cfg, layers)
    weights = 2.0 * (layers * n["layer_params"] + n["head_params"]) + 4.0 * n["norm_params"] + 2.0 * batch * n["E"]
    return weights + float(cached_tokens) * n["kv_bytes_per_token"]


def prefill_flops(cfg, layers, lengths) -> float:
    """Operations of one prompt step over sequences of ``lengths`` tokens, scores at each one's last token."""
    n = model_numbers(cfg, layers)
    tokens = sum(lengths)
    linear = 2.0 * tokens * layers * n["layer_params"]
    attention = sum(layers * 2.0 * 2.0 * n["H"] * n["D"] * t * (t + 1) / 2.0 for t in lengths)
    return linear + attention + 2.0 * n["head_params"] * len(lengths)


def class_costs(cfg, layers, batch, cached_tokens, prompt_tokens) -> dict:
    """What each kernel class of a decode step has to move (bytes) and of a one-sequence
    prompt step has to compute (operations; bytes for the classes that only move data)."""
    n = model_numbers(cfg, layers)
    E, H, G, D, F, V = n["E"], n["H"], n["G"], n["D"], n["F"], n["V"]
    B, T = batch, prompt_tokens
    qkv_w = (H + 2 * G) * D
    decode = {
        "embedding": B * E * 6.0,
        "norm": (2 * layers + 1) * (B * E * 6.0 + E * 4.0),
        "qkv product": layers * (2.0 * n["qkv"] + 2.0 * B * (E + qkv_w)),
        "attention": float(cached_tokens) * n["kv_bytes_per_token"] + layers * 2.0 * B * (qkv_w + H * D),
        "output product": layers * (2.0 * n["o"] + B * (2.0 * H * D + 8.0 * E)),
        "gate/up product": layers * (2.0 * n["gate_up"] + 2.0 * B * (E + F)),
        "down product": layers * (2.0 * n["down"] + B * (2.0 * F + 8.0 * E)),
        "head product": 2.0 * n["head_params"] + B * (2.0 * E + 4.0 * V),
        "sampling": B * V * 4.0,
    }
    prefill = {
        "embedding": ("bytes", T * E * 6.0),
        "norm": ("bytes", 2 * layers * T * E * 6.0 + E * 6.0),
        "qkv product": ("flops", layers * 2.0 * T * n["qkv"]),
        "rotary + append": ("bytes", layers * 2.0 * T * (2.0 * (H + G) * D + 2.0 * G * D + 2.0 * G * D)),
        "attention": ("flops", layers * 4.0 * H * D * T * (T + 1) / 2.0),
        "output product": ("flops", layers * 2.0 * T * n["o"]),
        "gate/up product": ("flops", layers * 2.0 * T * n["gate_up"]),
        "down product": ("flops", layers * 2.0 * T * n["down"]),
        "head product": ("bytes", 2.0 * n["head_params"]),
    }
    return {"decode": decode, "prefill": prefill}


# ------------------------------------------------------------------------------- measuring
def free_device_memory():
    import torch

    gc.collect()
    torch.cuda.empty_cache()


def timed_decode(eng, prompts, steps, warmup, rng, vocab, sample_clocks=False, prompts_a_step=8):
    """Device time of ``steps`` decode steps of the given sequences after their prompts.
    Returns also the prompt step's time when all prompts go in one step."""
    import torch

    from borrowed_compute_b200 import Sampling, ops
    from borrowed_compute_b200.engine import StepEntry
    from borrowed_compute_b200.sampling import RowSampler

    batch = len(prompts)
    slots = [eng.acquire() for _ in range(batch)]
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for i in range(0, batch, prompts_a_step):   # prompts in steps of a few, to bound activation memory
        eng.step([StepEntry(s, p, want=()) for s, p in zip(slots[i:i + prompts_a_step], prompts[i:i + prompts_a_step])])
    b.record()
    sampler = RowSampler(eng.rt.device, batch)
    sampler.set_rows([Sampling()] * batch)
    steps_t = torch.zeros(batch, dtype=torch.int32, device=eng.rt.device)
    toks = [[int(t) for t in rng.integers(0, vocab, batch)] for _ in range(steps + warmup)]

    def one(i):
        scores = eng.step([StepEntry(s, (toks[i][j],), want=(0,)) for j, s in enumerate(slots)], borrow_scores=True)
        sampler.sample(scores, steps_t)

    for i in range(warmup):
        one(i)
    torch.cuda.synchronize()
    prompt_ms = a.elapsed_time(b)
    before = ops.launches
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    clocks = ClockSampler() if sample_clocks else None
    if clocks:
        clocks.__enter__()
        time.sleep(0.3)
    torch.cuda.synchronize()
    start.record()
    for i in range(warmup, warmup + steps):
        one(i)
    stop.record()
    torch.cuda.synchronize()
    if clocks:
        time.sleep(0.2)
        clocks.__exit__()
    ms = start.elapsed_time(stop)
    cached = sum(len(p) for p in prompts) + batch * (warmup + steps / 2.0)     # positions the live requests hold, mid-run
    for s in slots:
        eng.release(s)
    eng.raise_on_kernel_error()
    return {"ms_per_step": ms / steps, "tok_s": batch * steps / (ms / 1000.0), "cached_tokens": cached, "prompt_ms": prompt_ms,
            "clocks": clocks.summary() if clocks else None, "eager_launches": ops.launches - before}


def breakdown(eng, cfg, layers, batch, pk, rng):
    """Every kernel class of one decode step (``batch`` sequences after 2,048-token prompts)
    and of one 2,048-token prompt step, launch by launch, against its own bytes or operations."""
    from borrowed_compute_b200 import Sampling
    from borrowed_compute_b200.engine import StepEntry, StepProfile
    from borrowed_compute_b200.sampling import RowSampler
    import torch

    vocab = cfg["vocab_size"]
    slots = [eng.acquire() for _ in range(batch)]
    prompts = [[int(t) for t in rng.integers(0, vocab, PROMPT)] for _ in range(batch)]
    for i in range(0, batch, 8):
        eng.step([StepEntry(s, p, want=()) for s, p in zip(slots[i:i + 8], prompts[i:i + 8])])
    sampler = RowSampler(eng.rt.device, batch)
    sampler.set_rows([Sampling()] * batch)
    steps_t = torch.zeros(batch, dtype=torch.int32, device=eng.rt.device)

    def one():
        scores = eng.step([StepEntry(s, (int(rng.integers(0, vocab)),), want=(0,)) for s in slots])
        sampler.sample(scores, steps_t)

    reps = 5
    with StepProfile(eng) as warm:
        one()
    with StepProfile(eng) as prof:
        for _ in range(reps):
            one()
    decode = prof.classes(reps)
    for s in slots:
        eng.release(s)
    slot = eng.acquire()
    p = prompts[0]
    with StepProfile(eng) as warm:   # noqa: F841
        eng.step([StepEntry(slot, p, want=(PROMPT - 1,))])
    eng.rollback(slot, 0)
    with StepProfile(eng) as prof:
        for _ in range(3):
            eng.step([StepEntry(slot, p, want=(PROMPT - 1,))])
            eng.rollback(slot, 0)
    prefill = prof.classes(3)
    eng.release(slot)
    costs = class_costs(cfg, layers, batch, batch * (PROMPT + 3), PROMPT)
    out = {"decode": {}, "prefill": {}, "how": "eager steps, CUDA events around every launch (no overlap between launches): shares, not a step's time"}
    for cls, m in sorted(decode.items(), key=lambda kv: -kv[1]["us"]):
        row = {"us": round(m["us"], 1), "launches": round(m["launches"], 1)}
        if cls in costs["decode"]:
            gbs = costs["decode"][cls] / (m["us"] * 1e-6) / 1e9
            row.update({"bytes": int(costs["decode"][cls]), "gb_s": round(gbs, 1), "frac": round(gbs / pk["hbm_gbs"], 3)})
        out["decode"][cls] = row
    for cls, m in sorted(prefill.items(), key=lambda kv: -kv[1]["us"]):
        row = {"us": round(m["us"], 1), "launches": round(m["launches"], 1)}
        if cls in costs["prefill"]:
            kind, amount = costs["prefill"][cls]
            if kind == "flops":
                tf = amount / (m["us"] * 1e-6) / 1e12
                row.update({"flops": float(amount), "tflops": round(tf, 1), "frac": round(tf / pk["bf16_tflops"], 3)})
            else:
                gbs = amount / (m["us"] * 1e-6) / 1e9
                row.update({"bytes": int(amount), "gb_s": round(gbs, 1), "frac": round(gbs / pk["hbm_gbs"], 3)})
        out["prefill"][cls] = row
    out["decode_sum_us"] = round(sum(m["us"] for m in decode.values()), 1)
    out["prefill_sum_us"] = round(sum(m["us"] for m in prefill.values()), 1)
    return out


def bench_tiny(rng) -> dict:
    """The two tiny workloads (float32): a batch of 3 prompts of 5 / 17 / 1 tokens and 8 greedy
    steps; a batch of 4 prompts of 1 / 9 / 33 / 70 tokens and 16 steps at temperature 0.8,
    top_p 0.9.  Through the entry point on the device, and through the plain C++ twin on the
    host (which recomputes the whole sequence every step): the twin's time is the CPU baseline,
    and its tokens must be the engine's."""
    import torch

    from borrowed_compute_b200 import Local, Sampling, twin
    from borrowed_compute_b200.weights import random_tensors

    out = {}
    for name, cfg, lengths, new, sampling in (("tiny_a", CONFIG_TINY_A, (5, 17, 1), 8, Sampling()),
                                              ("tiny_b", CONFIG_TINY_B, (1, 9, 33, 70), 16, Sampling(temperature=0.8, top_p=0.9, seed=1234567))):
        model = Local.random(cfg, seed=1, dtype="float32", max_tokens=1024, max_slots=4, max_seq=cfg["max_position_embeddings"])
        weights = {k: v.float().cpu().numpy() for k, v in random_tensors(model.engine.model.expected_tensors(), 1, torch.float32, "cuda").items()}
        host = twin.TwinLlama(cfg, weights)
        prompts = [[int(t) for t in rng.integers(0, cfg["vocab_size"], n)] for n in lengths]
        model.generate(prompts, new, sampling, stop_ids=())                      # first-use set-up outside the timed call
        started = time.perf_counter()
        got, _ = model.generate(prompts, new, sampling, stop_ids=())
        engine_ms = 1000.0 * (time.perf_counter() - started)
        started = time.perf_counter()
        want = [host.generate(p, new, sampling.temperature, sampling.top_p, sampling.seed) for p in prompts]
        twin_ms = 1000.0 * (time.perf_counter() - started)
        if got != want:
            raise AssertionError(f"bench: {name}: the engine generated {got}, the plain C++ twin {want}")
        out[f"{name}_engine_ms"], out[f"{name}_cpu_twin_ms"] = round(engine_ms, 2), round(twin_ms, 2)
        del model
    free_device_memory()
    return out


def bench_13b(pk, rng) -> dict:
    """The Llama-2-13B shape: 16 prompts of unequal lengths (uniform in 64 .. 2,048, seeded)
    in ONE ragged prompt step, then 128 decode steps, device-timed."""
    from borrowed_compute_b200 import Local

    cfg, layers = CONFIG_13B, CONFIG_13B["num_hidden_layers"]
    lengths = [int(n) for n in rng.integers(64, 2049, 16)]
    steps, warmup = 128, 4
    max_tokens = sum(-(-(n + steps + warmup + 8) // 64) * 64 for n in lengths)
    model = Local.random(cfg, seed=0, dtype="bfloat16", max_tokens=max_tokens, max_slots=16, max_seq=cfg["max_position_embeddings"])
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab_size"], n)] for n in lengths]
    r = timed_decode(model.engine, prompts, steps, warmup, rng, cfg["vocab_size"], prompts_a_step=16)
    need = decode_bytes(cfg, layers, 16, r["cached_tokens"])
    gbs = need / (r["ms_per_step"] / 1000.0) / 1e9
    flops = prefill_flops(cfg, layers, lengths)
    out = {"llama2_13b_mha_decode_b16": round(r["tok_s"], 1), "llama2_13b_mha_ms_per_step": round(r["ms_per_step"], 4),
           "llama2_13b_mha_bytes_per_step": int(need), "llama2_13b_mha_hbm_frac": round(gbs / pk["hbm_gbs"], 4),
           "llama2_13b_mha_prompt_tokens": sum(lengths), "llama2_13b_mha_prefill_tok_s": round(sum(lengths) / (r["prompt_ms"] / 1000.0), 1),
           "llama2_13b_mha_prefill_frac": round(flops / (r["prompt_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4)}
    del model
    free_device_memory()
    return out


def bench_long(pk, rng, layers=0) -> dict:
    """The 8B shape with one sequence of 32,000 tokens (the context that Llama-3.1 is made
    for is 131,072): the prompt in ONE step, then 64 decode steps, device-timed.  At this
    length a decode step reads 4 GB of keys and values beside the 16 GB of weights, and the
    prompt's work is half attention."""
    from borrowed_compute_b200 import Local

    layers = layers or CONFIG_8B["num_hidden_layers"]
    cfg = dict(CONFIG_8B, max_position_embeddings=32768, num_hidden_layers=layers)
    length, steps, warmup = 32000, 64, 4
    model = Local.random(cfg, seed=0, dtype="bfloat16", max_tokens=32768, max_slots=1, max_seq=32768)
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab_size"], length)]]
    r = timed_decode(model.engine, prompts, steps, warmup, rng, cfg["vocab_size"], prompts_a_step=1)
    need = decode_bytes(cfg, layers, 1, r["cached_tokens"])
    flops = prefill_flops(cfg, layers, [length])
    out = {"decode_b1_ctx32k_layers": layers, "decode_b1_ctx32k": round(r["tok_s"], 1), "decode_b1_ctx32k_ms_per_step": round(r["ms_per_step"], 4),
           "decode_b1_ctx32k_hbm_frac": round(need / (r["ms_per_step"] / 1000.0) / 1e9 / pk["hbm_gbs"], 4),
           "prefill_32k_tok_s": round(length / (r["prompt_ms"] / 1000.0), 1),
           "prefill_32k_frac": round(flops / (r["prompt_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4)}
    del model
    free_device_memory()
    return out


def bench_3b(pk, rng) -> dict:
    """The Llama-3.2-3B shape (tied head): 64 prompts of 1,024 tokens, then 512 tokens each
    sampled at temperature 1.0, through the entry point (the sampler runs every step)."""
    from borrowed_compute_b200 import Local, Sampling

    cfg, layers = CONFIG_3B, CONFIG_3B["num_hidden_layers"]
    batch, prompt, new = 64, 1024, 512
    model = Local.random(cfg, seed=0, dtype="bfloat16", max_tokens=batch * (-(-(prompt + new + 8) // 64) * 64), max_slots=batch,
                         max_seq=prompt + new + 8)
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab_size"], prompt)] for _ in range(batch)]
    model.generate(prompts[:2], 4, Sampling(temperature=1.0, seed=1), stop_ids=())      # first-use set-up outside the timed call
    out, stats = model.generate(prompts, new, Sampling(temperature=1.0, top_p=1.0, seed=7), stop_ids=())
    assert all(len(o) == new for o in out)
    tok_s = stats.decode_tokens_per_second
    ms = 1000.0 * batch / tok_s
    need = decode_bytes(cfg, layers, batch, batch * (prompt + new / 2.0))
    res = {"llama32_3b_sampled_e2e_b64": round(tok_s, 1), "llama32_3b_sampled_ms_per_step": round(ms, 4),
           "llama32_3b_sampled_bytes_per_step": int(need), "llama32_3b_sampled_hbm_frac": round(need / (ms / 1000.0) / 1e9 / pk["hbm_gbs"], 4),
           "llama32_3b_prefill_tok_s": round(batch * prompt / (stats.first_token_ms / 1000.0), 1)}
    del model
    free_device_memory()
    return res


# ------------------------------------------------------------------- the second architecture
def fegidra_config(width, heads, kv_heads, dim, vdim, chunk, delta_heads, delta_dim, rank, ff, vocab, layers):
    """``layers`` layers of the Fegidra design, delta-rule and attention layers in turn."""
    out = []
    for i in range(layers):
        if i % 2 == 0:
            mixer, kind = {"heads": delta_heads, "dim": delta_dim, "decay_rank": rank}, "general_delta"
        else:
            mixer, kind = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
                           "rot": {"dims": dim // 2, "base": 500000.0}, "scale": 1.0 / dim ** 0.5}, "attention"
        out.append({"type": kind, "mixer": mixer, "mlp": {"ff": ff, "kind": "dense"}})
    return {"architecture": "Fegidra", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "canon": {"taps": 4}, "layers": out}


def llama_like(width, heads, kv_heads, dim, ff, vocab, layers):
    return {"architectures": ["LlamaForCausalLM"], "num_hidden_layers": layers, "hidden_size": width, "num_attention_heads": heads,
            "num_key_value_heads": kv_heads, "head_dim": dim, "intermediate_size": ff, "vocab_size": vocab, "rope_theta": 500000.0,
            "rms_norm_eps": 1e-5, "tie_word_embeddings": False, "max_position_embeddings": 8192}


FEGIDRA_SIZES = {
    # the width, heads and feed-forward of the 8B shape; delta heads of 64 channels; chunks of 1,024 positions
    "wide": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, chunk=1024, delta_heads=64, delta_dim=64, rank=64, ff=14336, vocab=32000),
    # a 2,048-wide model with values half as wide as keys
    "mid": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=64, chunk=512, delta_heads=32, delta_dim=64, rank=32, ff=8192, vocab=32000),
}


def fegidra_costs(c, layers, batch, ctx_len, T) -> dict:
    """What each kernel class of the Fegidra model has to move in a decode step (bytes) and to compute in a
    prompt step of T tokens (operations, or bytes where it only moves data), summed over the model's layers.
    Half of the layers are delta-rule layers, half attention layers."""
    E, H, G, D, DV, C = c["width"], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["chunk"]
    HD, rank, F, V = c["delta_heads"] * c["delta_dim"], c["rank"], c["ff"], c["vocab"]
    nd, na, B = (layers + 1) // 2, layers // 2, batch
    n_in, n_qkv = 5 * HD + rank, H * D + G * D + G * DV
    seen_decode = min(ctx_len % C + 1, ctx_len + 1)                     # keys a decoded row reads
    seen_prefill = sum(min(t % C, t) + 1 for t in range(T))            # (query, key) pairs of a prompt
    state = c["delta_heads"] * c["delta_dim"] ** 2 * 4.0
    decode = {
        "norm": (2 * layers + 1) * (B * E * 6.0 + E * 4.0),
        "short convolution": layers * B * E * 2.0 * (2 + 2 * 3),
        "delta projections": nd * (2.0 * n_in * E + B * (2.0 * E + 4.0 * n_in)),
        "delta rule": nd * B * (2.0 * state + 4.0 * (n_in + 5 * HD) + 2.0 * HD),
        "qkv product": na * (2.0 * n_qkv * E + B * (2.0 * E + 4.0 * n_qkv)),
        "rotary + append": na * B * (4.0 * n_qkv + 2.0 * n_qkv),
        "attention": na * B * (seen_decode * G * (D + DV) * 2.0 + 2.0 * H * (D + DV)),
        "output product": nd * (2.0 * HD * E + B * (2.0 * HD + 8.0 * E)) + na * (2.0 * H * DV * E + B * (2.0 * H * DV + 8.0 * E)),
        "up product": layers * (2.0 * E * F + B * (2.0 * E + 4.0 * F)),
        "activation": layers * B * F * 6.0,
        "down product": layers * (2.0 * E * F + B * (2.0 * F + 8.0 * E)),
        "head product": 2.0 * V * E + B * (2.0 * E + 4.0 * V),
    }
    prefill = {
        "norm": ("bytes", 2 * layers * T * E * 6.0),
        "short convolution": ("bytes", layers * T * E * 4.0),
        "delta projections": ("flops", nd * 2.0 * T * n_in * E),
        # a step of the recurrence: two sums over the old state and its update, 11 operations a state element
        "delta rule": ("flops32", nd * T * c["delta_heads"] * c["delta_dim"] ** 2 * 11.0),
        "qkv product": ("flops", na * 2.0 * T * n_qkv * E),
        "rotary + append": ("bytes", na * T * (4.0 * n_qkv + 2.0 * n_qkv)),
        "attention": ("flops", na * 2.0 * H * (D + DV) * seen_prefill),
        "output product": ("flops", nd * 2.0 * T * HD * E + na * 2.0 * T * H * DV * E),
        "up product": ("flops", layers * 2.0 * T * E * F),
        "activation": ("bytes", layers * T * F * 6.0),
        "down product": ("flops", layers * 2.0 * T * E * F),
    }
    return {"decode": decode, "prefill": prefill}


def _against(costs, measured, pk, fp32_tflops):
    out = {}
    for cls, m in sorted(measured.items(), key=lambda kv: -kv[1]["us"]):
        row = {"us": round(m["us"], 1), "launches": round(m["launches"], 1)}
        cost = costs.get(cls)
        if cost is not None:
            kind, amount = cost if isinstance(cost, tuple) else ("bytes", cost)
            rate = amount / (m["us"] * 1e-6)
            if kind == "bytes":
                row.update({"gb_s": round(rate / 1e9, 1), "frac": round(rate / 1e9 / pk["hbm_gbs"], 3), "of": "copy rate"})
            elif kind == "flops":
                row.update({"tflops": round(rate / 1e12, 1), "frac": round(rate / 1e12 / pk["bf16_tflops"], 3), "of": "bf16 product rate"})
            else:
                row.update({"tflops": round(rate / 1e12, 2), "frac": round(rate / 1e12 / fp32_tflops, 3), "of": "float32 CUDA-core rate"})
        out[cls] = row
    return out


def _bench_models(configs, costs_of, vocab, out, pk, rng, fp32_tflops, batch, prompt, steps, warmup, prepare=None):
    """For each (name, config): decode steps of ``batch`` sequences after prompts of ``prompt`` tokens, one prompt alone,
    all prompts in one step, and every kernel class launch by launch against ``costs_of(name, config)``.  ``prepare(name, engine)``
    runs once on every fresh engine."""
    import torch

    from borrowed_compute_b200.engine import Engine, StepEntry, StepProfile

    for name, cfg in configs.items():
        eng = Engine.from_random(cfg, seed=1, max_tokens=batch * (prompt + 256), max_slots=batch, max_seq=prompt + 256)
        if prepare is not None:
            prepare(name, eng)
        prompts = [[int(t) for t in rng.integers(0, vocab, prompt)] for _ in range(batch)]
        # the step of all prompts once untimed (a kernel's first launch loads it), then timed inside timed_decode
        warm = [eng.acquire() for _ in range(batch)]
        eng.step([StepEntry(s, p, want=()) for s, p in zip(warm, prompts)])
        for s in warm:
            eng.release(s)
        torch.cuda.synchronize()
        res = timed_decode(eng, prompts, steps, warmup, rng, vocab, prompts_a_step=batch)
        # one prompt alone, timed on the device over three runs after a warm-up
        slot = eng.acquire()
        times = []
        for i in range(4):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            eng.step([StepEntry(slot, prompts[0], want=(prompt - 1,))])
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b))
            eng.rollback(slot, 0)
        prompt_ms = statistics.median(times[1:])
        # every class, launch by launch
        slots = [slot] + [eng.acquire() for _ in range(batch - 1)]
        eng.step([StepEntry(s, p, want=()) for s, p in zip(slots, prompts)])
        one = lambda: eng.step([StepEntry(s, (int(rng.integers(0, vocab)),), want=(0,)) for s in slots])   # noqa: E731
        with StepProfile(eng):
            one()
        with StepProfile(eng) as prof:
            for _ in range(3):
                one()
        decode_classes = prof.classes(3)
        for s in slots:
            eng.release(s)
        slot = eng.acquire()
        with StepProfile(eng):
            eng.step([StepEntry(slot, prompts[0], want=(prompt - 1,))])
        eng.rollback(slot, 0)
        with StepProfile(eng) as prof:
            eng.step([StepEntry(slot, prompts[0], want=(prompt - 1,))])
        prefill_classes = prof.classes(1)
        eng.release(slot)
        eng.raise_on_kernel_error()
        costs = costs_of(name, cfg)
        out[name] = {
            "decode_ms_per_step": round(res["ms_per_step"], 4), "decode_tok_s": round(res["tok_s"], 1),
            "prompt_ms": round(prompt_ms, 3), "prompt_tok_s": round(prompt / (prompt_ms / 1000.0), 1),
            "batch_prompt_tok_s": round(batch * prompt / (res["prompt_ms"] / 1000.0), 1),
            "weight_bytes": eng.weight_bytes(),
            "decode_classes": _against(costs["decode"], decode_classes, pk, fp32_tflops),
            "prefill_classes": _against(costs["prefill"], prefill_classes, pk, fp32_tflops),
        }
        del eng
        free_device_memory()
    return out


# 128 float32 lanes an SM, one fused multiply-add a clock each, at the clock the part sustains (nominal 1.965 GHz)
FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12


def bench_fegidra(pk, rng, size="wide", layers=4, batch=8, prompt=PROMPT, steps=32, warmup=4) -> dict:
    """Prompt and decode throughput of a Fegidra model of ``layers`` layers at sizes that resemble a real model's
    layers (random weights), beside a Llama model of the same width, heads, feed-forward width, vocabulary and
    depth, and every kernel class of both against its own bytes or operations (eager steps, events around
    every launch).  Inputs exceed the L2: a step reads hundreds of MB of weights."""
    c = FEGIDRA_SIZES[size]
    configs = {"fegidra": fegidra_config(layers=layers, **c),
               "llama": llama_like(c["width"], c["heads"], c["kv_heads"], c["dim"], c["ff"], c["vocab"], layers)}
    out = {"size": size, "sizes": c, "layers": layers, "batch": batch, "prompt": prompt,
           "between": "weights of a step exceed the L2", "peaks": pk, "fp32_cuda_core_tflops_nominal": round(FP32_TFLOPS, 1)}

    def costs_of(name, cfg):
        return fegidra_costs(c, layers, batch, prompt + 2, prompt) if name == "fegidra" else class_costs(cfg, layers, batch, batch * (prompt + 2), prompt)

    return _bench_models(configs, costs_of, c["vocab"], out, pk, rng, FP32_TFLOPS, batch, prompt, steps, warmup)


# -------------------------------------------------------------------- the third architecture
def pozirax_config(width, heads, kv_heads, dim, vdim, window, ssm_heads, ssm_vdim, state, groups, gla_heads, gla_dim, gla_vdim, rank, experts,
                   top, ff, shared, vocab, layers):
    """``layers`` layers of the Pozirax design: gated-linear-attention layers and layers of sliding-window attention beside a
    state-space mixer in turn, each with routed experts and a shared expert."""
    out = []
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared}}
    for i in range(layers):
        if i % 2 == 0:
            mixer, kind = {"heads": gla_heads, "dim": gla_dim, "vdim": gla_vdim, "tau": 16.0, "rank": rank}, "gla"
        else:
            left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": {"dims": dim, "base": 1e6},
                    "scale": 1.0 / dim ** 0.5}
            right = {"heads": ssm_heads, "vdim": ssm_vdim, "state": state, "groups": groups, "norm_groups": groups, "conv": 4}
            mixer, kind = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}, "parallel"
        out.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Pozirax", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "logit_softcap": 30.0,
            "layers": out}


POZIRAX_SIZES = {
    # the width and attention heads of the 8B shape; 32 experts of 2,048 of which a row uses 4, and a shared expert of 4,096
    "wide": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, window=1024, ssm_heads=64, ssm_vdim=64, state=128, groups=8,
                 gla_heads=16, gla_dim=128, gla_vdim=256, rank=16, experts=32, top=4, ff=2048, shared=4096, vocab=32000),
    # a 2,048-wide model: 64 experts of 1,408 of which a row uses 6, and a shared expert of 2,816
    "mid": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=64, window=512, ssm_heads=32, ssm_vdim=64, state=64, groups=4,
                gla_heads=8, gla_dim=128, gla_vdim=256, rank=16, experts=64, top=6, ff=1408, shared=2816, vocab=32000),
}


def pozirax_costs(c, layers, batch, ctx_len, T) -> dict:
    """What each kernel class of the Pozirax model has to move in a decode step (bytes) and to compute in a prompt step of T
    tokens (operations, or bytes where it only moves data), summed over the model's layers.  Even layers are gated linear
    attention, odd ones attention beside a state-space mixer."""
    E, H, G, D, DV, W, V = c["width"], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["window"], c["vocab"]
    Hs, Ps, N, Gs = c["ssm_heads"], c["ssm_vdim"], c["state"], c["groups"]
    Hg, Dg, Pg, rank = c["gla_heads"], c["gla_dim"], c["gla_vdim"], c["rank"]
    X, k, f, fs = c["experts"], c["top"], c["ff"], c["shared"]
    ng, np_, B = (layers + 1) // 2, layers // 2, batch
    inner, conv = Hs * Ps, Hs * Ps + 2 * Gs * N
    n_gla, n_ssm, n_qkv = 2 * Hg * Dg + 2 * Hg * Pg + rank, 2 * inner + 2 * Gs * N + Hs, H * D + G * D + G * DV
    state_g, state_s = Hg * Dg * Pg * 4.0, Hs * N * Ps * 4.0
    seen_decode = min(ctx_len + 1, W)
    seen_prefill = sum(min(t + 1, W) for t in range(T))
    touched = X * (1.0 - (1.0 - k / X) ** B)                          # experts that a step of B rows reads, on average
    decode = {
        "norm": (layers + 1) * (B * E * 6.0 + E * 4.0),
        "recurrence projections": ng * (2.0 * n_gla * E + B * (2.0 * E + 4.0 * n_gla)) + np_ * (2.0 * n_ssm * E + B * (2.0 * E + 4.0 * n_ssm)),
        "recurrence set-up": ng * (4.0 * rank * Hg * Dg + B * 4.0 * (rank + Hg * Dg)) + np_ * B * 4.0 * (2 * conv + 6 * conv + 3 * Hs),
        "recurrence": ng * B * (2.0 * state_g + 4.0 * (3 * Hg * Dg + 2 * Hg * Pg)) + np_ * B * (2.0 * state_s + 4.0 * (2 * conv + 2 * Hs)),
        "gated norm": (ng * Hg * Pg + np_ * inner) * B * 10.0,
        "qkv product": np_ * (2.0 * n_qkv * E + B * (2.0 * E + 4.0 * n_qkv)),
        "rotary + append": np_ * B * 6.0 * n_qkv,
        "attention": np_ * B * (seen_decode * G * (D + DV) * 2.0 + 2.0 * H * (D + DV)),
        "output product": ng * (2.0 * Hg * Pg * E + B * (2.0 * Hg * Pg + 8.0 * E)) + np_ * (2.0 * (H * DV + inner) * E + B * (2.0 * (H * DV + inner) + 16.0 * E)),
        "routing": layers * (4.0 * X * E + B * (2.0 * E + 8.0 * k)),
        "expert sort": layers * B * k * 16.0,
        "expert gather": layers * B * k * E * 4.0,
        "expert sum": layers * (B * k * E * 4.0 + B * E * 8.0),
        "expert product": layers * (touched * 3.0 * f * E * 2.0 + B * k * (2.0 * E + 4.0 * f + 4.0 * E)),
        "gate/up product": layers * (4.0 * fs * E + B * (2.0 * E + 2.0 * fs)),
        "down product": layers * (2.0 * fs * E + B * (2.0 * fs + 8.0 * E)),
        "head product": 2.0 * V * E + B * (2.0 * E + 4.0 * V),
    }
    prefill = {
        "norm": ("bytes", layers * T * E * 6.0),
        "recurrence projections": ("flops", 2.0 * T * E * (ng * n_gla + np_ * n_ssm)),
        "recurrence set-up": ("bytes", ng * T * 4.0 * (rank + Hg * Dg) + np_ * T * 4.0 * (2 * conv + 3 * Hs)),
        # a step of the recurrence: the update and the output, two fused multiply-adds a state element
        "recurrence": ("flops32", T * 4.0 * (ng * Hg * Dg * Pg + np_ * Hs * N * Ps)),
        "gated norm": ("bytes", (ng * Hg * Pg + np_ * inner) * T * 10.0),
        "qkv product": ("flops", np_ * 2.0 * T * n_qkv * E),
        "rotary + append": ("bytes", np_ * T * 6.0 * n_qkv),
        "attention": ("flops", np_ * 2.0 * H * (D + DV) * seen_prefill),
        "output product": ("flops", 2.0 * T * E * (ng * Hg * Pg + np_ * (H * DV + inner))),
        "routing": ("flops32", layers * 2.0 * T * X * E),
        "expert sort": ("bytes", layers * T * k * 16.0),
        "expert gather": ("bytes", layers * T * k * E * 4.0),
        "expert sum": ("bytes", layers * T * (k * E * 4.0 + E * 8.0)),
        "expert product": ("flops", layers * 2.0 * T * k * 3.0 * f * E),
        "gate/up product": ("flops", layers * 4.0 * T * fs * E),
        "down product": ("flops", layers * 2.0 * T * fs * E),
    }
    return {"decode": decode, "prefill": prefill}


def bench_pozirax(pk, rng, size="wide", layers=4, batch=8, prompt=PROMPT, steps=32, warmup=4) -> dict:
    """Prompt and decode throughput of a Pozirax model of ``layers`` layers at sizes that resemble a real model's layers
    (random weights), beside a Fegidra model, the closest of the other designs (recurrent and attention layers in turn,
    parallel blocks), of the same width, attention heads, vocabulary and depth, whose dense feed-forward is as wide as the
    experts a row uses; every kernel class of both against its own bytes or operations."""
    c = POZIRAX_SIZES[size]
    active = c["top"] * c["ff"] + c["shared"]
    f = dict(width=c["width"], heads=c["heads"], kv_heads=c["kv_heads"], dim=c["dim"], vdim=c["vdim"], chunk=c["window"],
             delta_heads=c["width"] // 64, delta_dim=64, rank=64, ff=active, vocab=c["vocab"])
    configs = {"pozirax": pozirax_config(layers=layers, **c), "fegidra": fegidra_config(layers=layers, **f)}
    out = {"size": size, "sizes": c, "beside": f, "layers": layers, "batch": batch, "prompt": prompt,
           "between": "weights of a step exceed the L2", "peaks": pk, "fp32_cuda_core_tflops_nominal": round(FP32_TFLOPS, 1)}

    def costs_of(name, cfg):
        return pozirax_costs(c, layers, batch, prompt + 2, prompt) if name == "pozirax" else fegidra_costs(f, layers, batch, prompt + 2, prompt)

    return _bench_models(configs, costs_of, c["vocab"], out, pk, rng, FP32_TFLOPS, batch, prompt, steps, warmup)


# ------------------------------------------------------------------- the fourth architecture
FUDELORN_SIZES = {
    # the width, heads and feed-forward of the 8B shape: latents of 512 (queries 1,536), keys of 64 plain and 64 rotated values on
    # the layers that rotate and 128 plain ones on the windowed layers; 32 experts of 3,072 of which a row uses 4, a shared one of 2,048
    "wide": dict(width=4096, heads=32, dim=64, rot=64, wdim=128, vdim=128, q_rank=1536, kv_rank=512, window=1024, ff=14336, experts=32, top=4,
                 expert_ff=3072, shared=2048, vocab=32000),
    # a 2,048-wide model: latents of 256, values half as wide as keys
    "mid": dict(width=2048, heads=16, dim=64, rot=32, wdim=128, vdim=64, q_rank=768, kv_rank=256, window=512, ff=8192, experts=16, top=2,
                expert_ff=3072, shared=2048, vocab=32000),
}


def fudelorn_config(width, heads, dim, rot, wdim, vdim, q_rank, kv_rank, window, ff, experts, top, expert_ff, shared, vocab, layers):
    """Layers in turn: a windowed mixer without positions and a dense feed-forward, then a rotating mixer over every earlier
    position with experts named by the token; every second rotating layer reads the first one's cache."""
    out, owner = [], None
    for i in range(layers):
        if i % 2 == 0:
            mixer = {"heads": heads, "dim": wdim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": window}, "scale": wdim ** -0.5}
            out.append({"type": "latent_attention_2", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}})
            continue
        mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": (dim + rot) ** -0.5,
                 "rot": {"base": 500000.0, "dims": rot, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
        if owner is not None:
            mixer["kv_from"] = owner
        else:
            owner = i
        out.append({"type": "latent_attention", "mixer": mixer,
                    "mlp": {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}})
    return {"architecture": "Fudelorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": out}


def fudelorn_costs(c, layers, batch, ctx_len, T) -> dict:
    """What each kernel class of the Fudelorn model has to move in a decode step (bytes) and to compute in a prompt step of T
    tokens (operations, or bytes where it only moves data), summed over the model's layers.  A decode step reads a position's
    latent once for all heads; a prompt step expands what it sees into every head's keys and values."""
    E, H, DV, QR, R, W, V = c["width"], c["heads"], c["vdim"], c["q_rank"], c["kv_rank"], c["window"], c["vocab"]
    X, k, f, fs, F, B = c["experts"], c["top"], c["expert_ff"], c["shared"], c["ff"], batch
    kinds = []                                            # (plain key width, rotated width, down projection rows, window) of every layer
    for i in range(layers):
        own = i % 2 == 0 or i == 1
        rot, d = (0, c["wdim"]) if i % 2 == 0 else (c["rot"], c["dim"])
        kinds.append((d, rot, QR + H + (R + rot if own else 0), W if i % 2 == 0 else 0))
    nd, nm = (layers + 1) // 2, layers // 2               # layers with a dense feed-forward, with experts
    touched = X * (1.0 - (1.0 - k / X) ** B)
    decode = {cls: 0.0 for cls in ("latent down product", "latent norm + append", "query up product", "latent query", "attention", "latent values")}
    prefill = {cls: 0.0 for cls in ("latent down product", "latent norm + append", "query up product", "latent query", "latent keys and values",
                                    "key and value up product", "attention", "latent values")}
    for d, rot, P, w in kinds:
        seen = min(ctx_len + 1, w) if w else ctx_len + 1
        decode["latent down product"] += 2.0 * P * E + B * (2.0 * E + 4.0 * P)
        decode["latent norm + append"] += B * (4.0 * P + 2.0 * QR + 4.0 * H + 2.0 * (R + rot))
        decode["query up product"] += 2.0 * H * (d + rot) * QR + B * (2.0 * QR + 4.0 * H * (d + rot))
        decode["latent query"] += 2.0 * H * d * R + B * (4.0 * H * (d + rot) + 2.0 * H * (R + rot))
        decode["attention"] += B * (seen * (R + rot) * 2.0 + 2.0 * H * (R + rot) + 2.0 * H * R)
        decode["latent values"] += 2.0 * H * DV * R + B * (2.0 * H * R + 4.0 * H + 2.0 * H * DV)
        pairs = sum(min(t + 1, w) if w else t + 1 for t in range(T))
        pages = -(-T // 64)
        prefill["latent down product"] += 2.0 * T * P * E
        prefill["latent norm + append"] += T * (4.0 * P + 2.0 * QR + 4.0 * H + 2.0 * (R + rot))
        prefill["query up product"] += 2.0 * T * H * (d + rot) * QR
        prefill["latent query"] += T * H * (d + rot) * 6.0                                   # the heads' queries rotated and rounded
        prefill["latent keys and values"] += pages * 64 * (4.0 * (R + rot) + 4.0 * H * (d + DV) + 2.0 * H * rot)
        prefill["key and value up product"] += 2.0 * pages * 64 * H * (d + DV) * R
        prefill["attention"] += 2.0 * H * (d + rot + DV) * pairs
        prefill["latent values"] += T * H * DV * 4.0
    decode.update({
        "norm": layers * 2 * (B * E * 6.0 + E * 4.0 + B * E * 12.0 + E * 4.0) + B * E * 6.0,
        "output product": layers * (2.0 * H * DV * E + B * (2.0 * H * DV + 8.0 * E)),
        "up product": nd * (2.0 * E * F + B * (2.0 * E + 2.0 * F)) + nm * (2.0 * E * fs + B * (2.0 * E + 2.0 * fs)),     # relu^2 in its epilogue
        "down product": nd * (2.0 * E * F + B * (2.0 * F + 8.0 * E)) + nm * (2.0 * E * fs + B * (2.0 * fs + 8.0 * E)),
        "routing": nm * B * k * 12.0,
        "expert sort": nm * B * k * 16.0,
        "expert gather": nm * B * k * E * 4.0,
        "expert sum": nm * (B * k * E * 4.0 + B * E * 8.0),
        "expert product": nm * (touched * 2.0 * f * E * 2.0 + B * k * (2.0 * E + 4.0 * f + 4.0 * E)),
        "gated sum": nm * (B * E * 14.0 + E * 2.0),
        "head product": 2.0 * V * E + B * (2.0 * E + 4.0 * V),
    })
    prefill = {cls: ("bytes" if cls in ("latent norm + append", "latent query", "latent keys and values", "latent values") else "flops", v)
               for cls, v in prefill.items()}
    prefill.update({
        "norm": ("bytes", layers * 2 * T * E * 18.0),
        "output product": ("flops", layers * 2.0 * T * H * DV * E),
        "up product": ("flops", 2.0 * T * E * (nd * F + nm * fs)),
        "down product": ("flops", 2.0 * T * E * (nd * F + nm * fs)),
        "routing": ("bytes", nm * T * k * 12.0),
        "expert sort": ("bytes", nm * T * k * 16.0),
        "expert gather": ("bytes", nm * T * k * E * 4.0),
        "expert sum": ("bytes", nm * T * (k * E * 4.0 + E * 8.0)),
        "expert product": ("flops", nm * 2.0 * T * k * 2.0 * f * E),
        "gated sum": ("bytes", nm * T * E * 14.0),
    })
    return {"decode": decode, "prefill": prefill}


def bench_fudelorn(pk, rng, size="wide", layers=4, batch=8, prompt=PROMPT, steps=32, warmup=4) -> dict:
    """Prompt and decode throughput of a Fudelorn model of ``layers`` layers at sizes that resemble a real model's layers
    (random weights), beside a Llama model, the closest of the other designs (softmax attention over a paged cache and a
    dense feed-forward), of the same width, heads, feed-forward width, vocabulary and depth; every kernel class of both
    against its own bytes or operations."""
    c = FUDELORN_SIZES[size]
    configs = {"fudelorn": fudelorn_config(layers=layers, **c),
               "llama": llama_like(c["width"], c["heads"], max(1, c["heads"] // 4), 128, c["ff"], c["vocab"], layers)}
    out = {"size": size, "sizes": c, "layers": layers, "batch": batch, "prompt": prompt,
           "between": "weights of a step exceed the L2", "peaks": pk, "fp32_cuda_core_tflops_nominal": round(FP32_TFLOPS, 1)}

    def costs_of(name, cfg):
        return fudelorn_costs(c, layers, batch, prompt + 2, prompt) if name == "fudelorn" else class_costs(cfg, layers, batch, batch * (prompt + 2), prompt)

    return _bench_models(configs, costs_of, c["vocab"], out, pk, rng, FP32_TFLOPS, batch, prompt, steps, warmup)


def logirax_config(width, heads, dim, rot, wdim, vdim, q_rank, kv_rank, window, ff, experts, top, expert_ff, shared, vocab, layers):
    """Layers in turn: attention whose heads talk (a quarter as many kv heads, heads of ``wdim``, half of their dimensions turning,
    a window that keeps the first four positions) with a dense feed-forward whose gate is clipped, then latent attention with a
    sink and routed experts plus a shared one."""
    out = []
    for i in range(layers):
        if i % 2 == 0:
            mixer = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": wdim, "vdim": wdim, "scale": wdim ** -0.5, "softcap": 30.0,
                     "mask": {"size": window, "keep_first": 4}, "rot": {"base": 10000.0, "dims": wdim // 2}}
            out.append({"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}})
            continue
        mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": (dim + rot) ** -0.5,
                 "rot": {"base": 500000.0, "dims": rot}}
        out.append({"type": "latent_attention", "mixer": mixer,
                    "mlp": {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top, "scale": 1.5}, "shared": {"ff": shared}}})
    return {"architecture": "Logirax", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "logit_scale": 1.0, "layers": out}


def logirax_costs(c, layers, batch, ctx_len, T) -> dict:
    """What each kernel class of the Logirax model has to move in a decode step (bytes) and to compute in a prompt step of T tokens
    (operations, or bytes where it only moves data), summed over the model's layers.  The latent layers' classes are Fudelorn's
    (a rotating layer that keeps its own cache); the talking layers read, a row, at most a window and the kept positions of two
    planes (keys, and the keys as projected), and mix heads * heads raw scores a (row, position) on the CUDA cores."""
    E, H, DV, QR, R, W, V = c["width"], c["heads"], c["vdim"], c["q_rank"], c["kv_rank"], c["window"], c["vocab"]
    X, k, f, fs, F, B = c["experts"], c["top"], c["expert_ff"], c["shared"], c["ff"], batch
    D, G = c["wdim"], max(1, c["heads"] // 4)
    d, rot = c["dim"], c["rot"]
    nt, nl = (layers + 1) // 2, layers // 2               # talking layers (dense feed-forward), latent layers (experts)
    touched = X * (1.0 - (1.0 - k / X) ** B)
    P = QR + H + R + rot                                  # rows of the latent layers' fused down projection
    Pt = (2 * H + G) * D                                  # rows of the talking layers' fused projection [q | k | gate]
    seen_t = min(ctx_len + 1, W + 4)
    seen_l = ctx_len + 1
    pairs_t = sum(min(t + 1, W + 4) for t in range(T))
    pairs_l = T * (T + 1) / 2.0
    pages = -(-T // 64)
    decode = {
        "qkv product": nt * (2.0 * Pt * E + B * (2.0 * E + 4.0 * Pt)),
        "talk prepare": nt * B * (4.0 * Pt + 2.0 * H * D + 4.0 * G * D + 4.0 * H * D),
        "talking attention": nt * B * (seen_t * G * D * 4.0 + 2.0 * H * D + 4.0 * H * D + 2.0 * H * D),
        "bias": nt * B * E * 8.0,
        "latent down product": nl * (2.0 * P * E + B * (2.0 * E + 4.0 * P)),
        "latent norm + append": nl * B * (4.0 * P + 2.0 * QR + 4.0 * H + 2.0 * (R + rot)),
        "query up product": nl * (2.0 * H * (d + rot) * QR + B * (2.0 * QR + 4.0 * H * (d + rot))),
        "latent query": nl * (2.0 * H * d * R + B * (4.0 * H * (d + rot) + 2.0 * H * (R + rot))),
        "attention": nl * B * (seen_l * (R + rot) * 2.0 + 2.0 * H * (R + rot) + 2.0 * H * R),
        "latent values": nl * (2.0 * H * DV * R + B * (2.0 * H * R + 4.0 * H + 2.0 * H * DV)),
        "norm": layers * 2 * (B * E * 6.0 + E * 4.0 + B * E * 12.0 + E * 4.0) + B * E * 6.0,
        "output product": nt * (2.0 * H * D * E + B * (2.0 * H * D + 8.0 * E)) + nl * (2.0 * H * DV * E + B * (2.0 * H * DV + 8.0 * E)),
        "gate/up product": nt * (4.0 * E * F + B * (2.0 * E + 2.0 * F)) + nl * (4.0 * E * fs + B * (2.0 * E + 2.0 * fs)),
        "down product": nt * (2.0 * E * F + B * (2.0 * F + 8.0 * E)) + nl * (2.0 * E * fs + B * (2.0 * fs + 8.0 * E)),
        "routing": nl * (X * E * 4.0 + B * (2.0 * E + X * 4.0 + k * 8.0)),
        "expert sort": nl * B * k * 16.0,
        "expert gather": nl * B * k * E * 4.0,
        "expert sum": nl * (B * k * E * 4.0 + B * E * 8.0),
        "expert product": nl * (touched * 3.0 * f * E * 2.0 + B * k * (2.0 * E + 4.0 * f + 4.0 * E)),
        "head product": 2.0 * V * E + B * (2.0 * E + 4.0 * V),
    }
    prefill = {
        "qkv product": ("flops", nt * 2.0 * T * Pt * E),
        "talk prepare": ("bytes", nt * T * (4.0 * Pt + 2.0 * H * D + 4.0 * G * D + 4.0 * H * D)),
        # tensor-core operations (scores and values); the mix of heads * heads raw scores a pair is CUDA-core work on top of it
        "talking attention": ("flops", nt * 4.0 * H * D * pairs_t),
        "bias": ("bytes", nt * T * E * 8.0),
        "short convolution": ("bytes", layers * T * E * 4.0),
        "latent down product": ("flops", nl * 2.0 * T * P * E),
        "latent norm + append": ("bytes", nl * T * (4.0 * P + 2.0 * QR + 4.0 * H + 2.0 * (R + rot))),
        "query up product": ("flops", nl * 2.0 * T * H * (d + rot) * QR),
        "latent query": ("bytes", nl * T * H * (d + rot) * 6.0),
        "latent keys and values": ("bytes", nl * pages * 64 * (4.0 * (R + rot) + 4.0 * H * (d + DV) + 2.0 * H * rot)),
        "key and value up product": ("flops", nl * 2.0 * pages * 64 * H * (d + DV) * R),
        "attention": ("flops", nl * 2.0 * H * (d + rot + DV) * pairs_l),
        "latent values": ("bytes", nl * T * H * DV * 4.0),
        "norm": ("bytes", layers * 2 * T * E * 18.0),
        "output product": ("flops", 2.0 * T * E * (nt * H * D + nl * H * DV)),
        "gate/up product": ("flops", 4.0 * T * E * (nt * F + nl * fs)),
        "down product": ("flops", 2.0 * T * E * (nt * F + nl * fs)),
        "routing": ("bytes", nl * T * (2.0 * E + X * 4.0 + k * 8.0)),
        "expert sort": ("bytes", nl * T * k * 16.0),
        "expert gather": ("bytes", nl * T * k * E * 4.0),
        "expert sum": ("bytes", nl * T * (k * E * 4.0 + E * 8.0)),
        "expert product": ("flops", nl * 2.0 * T * k * 3.0 * f * E),
    }
    return {"decode": decode, "prefill": prefill}


def bench_logirax(pk, rng, size="wide", layers=4, batch=8, prompt=PROMPT, steps=32, warmup=4) -> dict:
    """Prompt and decode throughput of a Logirax model of ``layers`` layers at sizes that resemble a real model's layers (random
    weights), beside a Fudelorn model, the closest of the other designs (sandwich blocks, latent attention, experts), of the same
    width, heads, latents, feed-forward widths, vocabulary and depth; every kernel class of both against its own bytes or operations."""
    c = FUDELORN_SIZES[size]
    configs = {"logirax": logirax_config(layers=layers, **c), "fudelorn": fudelorn_config(layers=layers, **c)}
    out = {"size": size, "sizes": c, "layers": layers, "batch": batch, "prompt": prompt,
           "between": "weights of a step exceed the L2", "peaks": pk, "fp32_cuda_core_tflops_nominal": round(FP32_TFLOPS, 1)}

    def costs_of(name, cfg):
        return (logirax_costs if name == "logirax" else fudelorn_costs)(c, layers, batch, prompt + 2, prompt)

    return _bench_models(configs, costs_of, c["vocab"], out, pk, rng, FP32_TFLOPS, batch, prompt, steps, warmup)


# -------------------------------------------------------------------- the sixth architecture
DURATAR_SIZES = {
    # the width, projections and feed-forward of the 8B shape: 32 heads of two maps of 64 on values of 128, delta heads and lightning heads that
    # fill the width, four streams
    "wide": dict(width=4096, heads=32, kv_heads=8, dim=64, vdim=128, window=1024, keep=4, delta_heads=64, delta_dim=64, delta_vdim=64, rank=64,
                 light_heads=32, light_dim=128, light_vdim=128, ff=14336, streams=4, vocab=32000),
    # a 2,048-wide model, values as wide as a map
    "mid": dict(width=2048, heads=16, kv_heads=4, dim=64, vdim=64, window=512, keep=4, delta_heads=32, delta_dim=64, delta_vdim=64, rank=32,
                light_heads=16, light_dim=128, light_vdim=128, ff=8192, streams=4, vocab=32000),
}


def duratar_config(width, heads, kv_heads, dim, vdim, window, keep, delta_heads, delta_dim, delta_vdim, rank, light_heads, light_dim, light_vdim, ff, streams,
                   vocab, layers):
    """``layers`` layers of the Duratar design in turns of four: the delta rule, attention, lightning, attention over the first one's keys and values."""
    out = []
    for i in range(layers):
        attention = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep}, "diff": 0.4,
                     "rot": {"dims": dim // 2, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}, "scale": 1.0 / dim ** 0.5}
        if i % 4 == 0:
            mixer, kind = {"heads": delta_heads, "kv_heads": delta_heads, "dim": delta_dim, "vdim": delta_vdim, "conv": 4, "decay_rank": rank, "gate_rank": rank}, "channel_delta"
        elif i % 4 == 2:
            mixer, kind = {"heads": light_heads, "dim": light_dim, "vdim": light_vdim, "decay": [1.0 - 2.0 ** (-3 - 6 * h / light_heads) for h in range(light_heads)]}, "lightning"
        else:
            mixer, kind = dict(attention, kv_from=i - 2) if i % 4 == 3 else attention, "attention"
        out.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Duratar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": 1e-5}, "layers": out}


def duratar_costs(c, layers, batch, ctx_len, T) -> dict:
    """What each kernel class of the Duratar model has to move in a decode step (bytes) and to compute in a prompt step of T tokens
    (operations, or bytes where it only moves data), summed over the model's layers."""
    E, H, G, D, DV, W, K, S, F, V, B = (c["width"], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["window"], c["keep"], c["streams"], c["ff"], c["vocab"], batch)
    Hd, Dd, Pd, rank, Hl, Dl, Pl = c["delta_heads"], c["delta_dim"], c["delta_vdim"], c["rank"], c["light_heads"], c["light_dim"], c["light_vdim"]
    nd, nl = sum(i % 4 == 0 for i in range(layers)), sum(i % 4 == 2 for i in range(layers))
    na, nq = sum(i % 4 == 1 for i in range(layers)), sum(i % 4 == 3 for i in range(layers))
    ch = 2 * Hd * Dd + Hd * Pd
    n_d, n_l, n_q = ch + 2 * rank + Hd, 2 * Hl * Dl + 2 * Hl * Pl, 2 * H * D
    n_qkv = n_q + 2 * G * D + G * DV
    seen = lambda t: min(t + 1, W) + max(0, min(K, t + 1 - W))                                                       # noqa: E731
    seen_decode, seen_prefill = seen(ctx_len), sum(seen(t) for t in range(T))
    state_d, state_l = Hd * Dd * Pd * 4.0, Hl * Dl * Pl * 4.0
    mul = lambda n, k, out: 2.0 * n * k + B * (2.0 * k + out * n)                                                    # noqa: E731
    row = E * (8.0 * S + 8.0 + 2.0)                                # streams read and written, a result read and cleared, a normed row written
    decode = {
        "streams + norm": (2 * layers + 1) * B * row, "delta projections": nd * mul(n_d, E, 4.0), "recurrence set-up": nd * B * ch * 4.0 * (2 + 2 * 3),
        "delta rule": nd * (B * (2.0 * state_d + 4.0 * n_d + 2.0 * Hd * Pd) + 2.0 * rank * Hd * (Dd + Pd)),
        "recurrence projections": nl * mul(n_l, E, 4.0), "recurrence": nl * B * (2.0 * state_l + 4.0 * (2 * Hl * Dl + 2 * Hl * Pl)),
        "gated norm": nl * B * Hl * Pl * 10.0, "qkv product": na * mul(n_qkv, E, 4.0), "query product": nq * mul(n_q, E, 4.0),
        "rotary + append": (na * n_qkv + nq * n_q) * B * 6.0,
        "attention": (na + nq) * B * (seen_decode * G * (2 * D + DV) * 2.0 + 2.0 * H * (2 * D + DV)),
        "output product": nd * mul(E, Hd * Pd, 8.0) + nl * mul(E, Hl * Pl, 8.0) + (na + nq) * mul(E, H * DV, 8.0),
        "up product": layers * mul(F, E, 2.0), "down product": layers * mul(E, F, 8.0), "head product": mul(V, E, 4.0),
    }
    prefill = {
        "streams + norm": ("bytes", 2 * layers * T * row), "delta projections": ("flops", nd * 2.0 * T * n_d * E), "recurrence set-up": ("bytes", nd * T * ch * 8.0),
        "low-rank split": ("bytes", nd * T * 2 * rank * 8.0), "low-rank product": ("bytes", nd * T * Hd * (Dd + Pd) * 4.0),
        # a step of the recurrence: decay, two sums over the state and its update, 7 operations a state element
        "delta rule": ("flops32", nd * T * Hd * Dd * Pd * 7.0), "recurrence projections": ("flops", nl * 2.0 * T * n_l * E),
        "recurrence": ("flops32", nl * T * 4.0 * Hl * Dl * Pl), "gated norm": ("bytes", (nl * Hl * Pl + nd * Hd * Pd) * T * 10.0),
        "qkv product": ("flops", na * 2.0 * T * n_qkv * E), "query product": ("flops", nq * 2.0 * T * n_q * E), "rotary + append": ("bytes", (na * n_qkv + nq * n_q) * T * 6.0),
        "attention": ("flops", (na + nq) * 2.0 * H * 2 * (D + DV) * seen_prefill),
        "output product": ("flops", 2.0 * T * E * (nd * Hd * Pd + nl * Hl * Pl + (na + nq) * H * DV)),
        "up product": ("flops", layers * 2.0 * T * E * F), "down product": ("flops", layers * 2.0 * T * E * F),
    }
    return {"decode": decode, "prefill": prefill}


def bench_duratar(pk, rng, size="wide", layers=4, batch=8, prompt=PROMPT, steps=32, warmup=4) -> dict:
    """Prompt and decode throughput of a Duratar model of ``layers`` layers at sizes that resemble a real model's layers (random weights),
    beside a Fegidra model, the closest of the other designs (delta-rule and masked attention layers in turn, dense feed-forwards without a
    gate), of the same width, projections, feed-forward, vocabulary and depth; every kernel class of both against its own bytes or operations."""
    c = DURATAR_SIZES[size]
    f = dict(width=c["width"], heads=c["heads"], kv_heads=c["kv_heads"], dim=2 * c["dim"], vdim=c["vdim"], chunk=c["window"], delta_heads=c["delta_heads"],
             delta_dim=c["delta_dim"], rank=c["rank"], ff=c["ff"], vocab=c["vocab"])
    configs = {"duratar": duratar_config(layers=layers, **c), "fegidra": fegidra_config(layers=layers, **f)}
    out = {"size": size, "sizes": c, "beside": f, "layers": layers, "batch": batch, "prompt": prompt,
           "between": "weights of a step exceed the L2", "peaks": pk, "fp32_cuda_core_tflops_nominal": round(FP32_TFLOPS, 1)}

    def costs_of(name, cfg):
        return duratar_costs(c, layers, batch, prompt + 2, prompt) if name == "duratar" else fegidra_costs(f, layers, batch, prompt + 2, prompt)

    return _bench_models(configs, costs_of, c["vocab"], out, pk, rng, FP32_TFLOPS, batch, prompt, steps, warmup)


# ------------------------------------------------------------------ the seventh architecture
KODULIX_SIZES = {
    # the width and heads of the 8B shape; 32 experts of 2,048 of which a row uses 4, beside 8 identity experts, in 4 groups of which 2
    # are kept, and a shared expert of 4,096; 32 buckets of distances up to 128
    "wide": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, rows=32, reach=128, experts=32, top=4, identity=8, groups=4, keep=2, ff=2048,
                 shared=4096, vocab=32000),
    # a 2,048-wide model: values half as wide as keys, 64 experts of 1,408 of which a row uses 6, distances up to 1,024
    "mid": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=64, rows=64, reach=1024, experts=64, top=6, identity=16, groups=8, keep=4, ff=1408,
                shared=2816, vocab=32000),
}


def kodulix_config(width, heads, kv_heads, dim, vdim, rows, reach, experts, top, identity, groups, keep, ff, shared, vocab, layers):
    """``layers`` layers of the Kodulix design: attention with biases by distance, experts in groups beside identity experts."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.0 / dim ** 0.5, "bias_rows": rows, "bias_max": reach,
             "q_temp": {"coef": 0.1, "every": 1024}}
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": 7.0}, "shared": {"ff": shared, "limit": 7.0},
           "router": {"experts": experts, "top": top, "identity": identity, "groups": {"count": groups, "keep": keep}}}
    return {"architecture": "Kodulix", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "logit_scale": 1.0,
            "embedding": {"bigram": {"buckets": vocab, "mul_prev": 31, "mul_cur": 7}}, "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}] * layers}


def kodulix_costs(c, layers, batch, ctx_len, T) -> dict:
    """What each kernel class of the Kodulix model has to move in a decode step (bytes) and to compute in a prompt step of T tokens
    (operations, or bytes where it only moves data), summed over the model's layers.  c["counted"] tells how many of a row's choices
    are experts with matrices, in a decode step and in a prompt, and how many of these experts a decode step touches a layer: counted in
    steps of the model that is timed, since its random routers favour some experts."""
    E, H, G, D, DV, V = c["width"], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["vocab"]
    X, XI, f, fs, B = c["experts"], c["experts"] + c["identity"], c["ff"], c["shared"], batch
    n_qkv, top = H * D + G * D + G * DV, c["top"]
    k, k_prompt, touched = c["counted"]
    pairs = T * (T + 1) / 2.0
    decode = {
        "embedding": B * E * 8.0,
        # a result read and cleared, the stream read and written, a rounded row written: twice a layer
        "norm": 2 * layers * (B * E * 18.0 + E * 4.0) + B * E * 6.0,
        "qkv product": layers * (2.0 * n_qkv * E + B * (2.0 * E + 4.0 * n_qkv)),
        "rotary + append": layers * B * 6.0 * n_qkv,
        "attention": layers * B * ((ctx_len + 1) * G * (D + DV) * 2.0 + 2.0 * H * (D + DV)),
        "output product": layers * (2.0 * H * DV * E + B * (2.0 * H * DV + 8.0 * E)),
        "routing": layers * (4.0 * XI * E + B * (2.0 * E + 8.0 * top)),
        "expert sort": layers * B * top * 16.0,
        "expert gather": layers * B * k * E * 4.0,
        "expert sum": layers * B * (k * E * 4.0 + E * 10.0),
        "expert product": layers * (touched * 3.0 * f * E * 2.0 + B * k * (2.0 * E + 4.0 * f + 4.0 * E)),
        "gate/up product": layers * (4.0 * fs * E + B * (2.0 * E + 2.0 * fs)),
        "down product": layers * (2.0 * fs * E + B * (2.0 * fs + 8.0 * E)),
        "head product": 2.0 * V * E + B * (2.0 * E + 4.0 * V),
    }
    prefill = {
        "embedding": ("bytes", T * E * 8.0),
        "norm": ("bytes", 2 * layers * T * E * 18.0),
        "qkv product": ("flops", layers * 2.0 * T * n_qkv * E),
        "rotary + append": ("bytes", layers * T * 6.0 * n_qkv),
        "attention": ("flops", layers * 2.0 * H * (D + DV) * pairs),
        "output product": ("flops", layers * 2.0 * T * E * H * DV),
        "routing": ("flops32", layers * 2.0 * T * XI * E),
        "expert sort": ("bytes", layers * T * top * 16.0),
        "expert gather": ("bytes", layers * T * k_prompt * E * 4.0),
        "expert sum": ("bytes", layers * T * (k_prompt * E * 4.0 + E * 10.0)),
        "expert product": ("flops", layers * 2.0 * T * k_prompt * 3.0 * f * E),
        "gate/up product": ("flops", layers * 4.0 * T * fs * E),
        "down product": ("flops", layers * 2.0 * T * fs * E),
    }
    return {"decode": decode, "prefill": prefill}


def bench_kodulix(pk, rng, size="wide", layers=4, batch=8, prompt=PROMPT, steps=32, warmup=4) -> dict:
    """Prompt and decode throughput of a Kodulix model of ``layers`` layers at sizes that resemble a real model's layers (random weights),
    beside a Pozirax model, the closest of the other designs (attention with normed heads, routed experts plus a shared one), and a Llama
    model (attention over every earlier position), both of the same width, attention heads, vocabulary and depth; the Pozirax model's
    experts are as many and as wide, the Llama model's feed-forward as wide as the experts a row uses.  Every kernel class of the three
    against its own bytes or operations."""
    c = dict(KODULIX_SIZES[size])
    same = {k: c[k] for k in ("width", "heads", "kv_heads", "dim", "vdim", "experts", "top", "ff", "shared", "vocab")}
    z = dict(POZIRAX_SIZES[size], **same)
    configs = {"kodulix": kodulix_config(layers=layers, **KODULIX_SIZES[size]), "pozirax": pozirax_config(layers=layers, **z),
               "llama": llama_like(c["width"], c["heads"], c["kv_heads"], c["dim"], c["top"] * c["ff"] + c["shared"], c["vocab"], layers)}
    out = {"size": size, "sizes": KODULIX_SIZES[size], "beside": z, "layers": layers, "batch": batch, "prompt": prompt,
           "between": "weights of a step exceed the L2", "peaks": pk, "fp32_cuda_core_tflops_nominal": round(FP32_TFLOPS, 1)}

    def prepare(name, eng):
        """Embedded rows as large as the sinusoids beside them (else every row routes alike), and a count of what the experts get."""
        if name != "kodulix":
            return
        from borrowed_compute_b200 import ops
        from borrowed_compute_b200.engine import StepEntry

        eng.model.embedding.weight.mul_(50.0)
        chosen, plain = [], ops.moe_combine_identity
        ops.moe_combine_identity = lambda y, choice, *rest: (chosen.append(choice.cpu().numpy()), plain(y, choice, *rest))
        eng.use_graphs = False
        slots = [eng.acquire() for _ in range(batch)]
        for _ in range(2):
            chosen.clear()
            tokens = [[int(t) for t in rng.integers(0, c["vocab"], 64)] for _ in slots]
            eng.step([StepEntry(s, t, want=()) for s, t in zip(slots, tokens)])
            k_prompt = sum((x < c["experts"]).sum() / x.shape[0] for x in chosen) / len(chosen)
        k, touched, reps = 0.0, 0.0, 8
        for _ in range(reps):
            chosen.clear()
            eng.step([StepEntry(s, (int(rng.integers(0, c["vocab"])),), want=(0,)) for s in slots])
            k += sum((x < c["experts"]).sum() / x.shape[0] for x in chosen) / len(chosen) / reps
            touched += sum(len(set(x[x < c["experts"]].tolist())) for x in chosen) / len(chosen) / reps
        for s in slots:
            eng.release(s)
        ops.moe_combine_identity, eng.use_graphs = plain, True
        c["counted"] = (float(k), float(k_prompt), float(touched))
        out["counted"] = {"experts_a_row": round(float(k), 2), "experts_a_row_prompt": round(float(k_prompt), 2), "experts_touched_a_step": round(float(touched), 2)}

    def costs_of(name, cfg):
        if name == "llama":
            return class_costs(cfg, layers, batch, batch * (prompt + 2), prompt)
        return (kodulix_costs if name == "kodulix" else pozirax_costs)(c if name == "kodulix" else z, layers, batch, prompt + 2, prompt)

    return _bench_models(configs, costs_of, c["vocab"], out, pk, rng, FP32_TFLOPS, batch, prompt, steps, warmup, prepare)


def run_ours(args) -> dict:
    import numpy as np
    import torch

    from borrowed_compute_b200 import Local, Sampling, ops
    from borrowed_compute_b200.engine import StepEntry
    from borrowed_compute_b200.engine import engine as engine_module

    global PROMPT
    PROMPT = args.prompt
    cfg = dict(CONFIG_8B)
    full_layers = cfg["num_hidden_layers"]
    cfg["num_hidden_layers"] = args.layers or full_layers
    layers = cfg["num_hidden_layers"]
    vocab = cfg["vocab_size"]
    pk = peaks()
    rng = np.random.default_rng(0)
    biggest = max(args.batch, 64 if not args.no_points else args.batch)
    new_tokens = max(args.warmup, E2E_SETTLE_PASSES) + args.steps + 8
    max_tokens = biggest * (-(-(PROMPT + new_tokens + 64) // 64) * 64)
    model = Local.random(cfg, seed=0, dtype="bfloat16", max_tokens=max_tokens, max_slots=biggest, max_seq=CONTEXT)
    eng = model.engine
    torch.cuda.synchronize()

    def prompts(batch):
        return [[int(t) for t in rng.integers(0, vocab, PROMPT)] for _ in range(batch)]

    # --- the headline: decode at the requested batch, timed on the device
    main = timed_decode(eng, prompts(args.batch), args.steps, args.warmup, rng, vocab, sample_clocks=True)
    # kernels a step: count them on one eager (uncaptured) step
    eng.use_graphs = False
    s = eng.acquire()
    eng.step([StepEntry(s, [1, 2, 3], want=())])
    before = ops.launches
    eng.step([StepEntry(s, (5,), want=(0,))])
    launches_per_step = ops.launches - before + 2   # + the two kernels of greedy sampling
    eng.release(s)
    eng.use_graphs = True

    need = decode_bytes(cfg, layers, args.batch, main["cached_tokens"])
    achieved = need / (main["ms_per_step"] / 1000.0) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                "frac": round(achieved / pk["hbm_gbs"], 4), "bytes_per_step": int(need), "peak_source": pk["source"]}

    # --- prefill of 2,048 tokens (one prompt, scores at its last token)
    slot = eng.acquire()
    p = prompts(1)[0]
    for _ in range(2):
        eng.step([StepEntry(slot, p, want=(PROMPT - 1,))])
        eng.rollback(slot, 0)
    torch.cuda.synchronize()
    times = []
    for _ in range(3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        eng.step([StepEntry(slot, p, want=(PROMPT - 1,))])
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
        eng.rollback(slot, 0)
    eng.release(slot)
    pms = min(times)
    flops = prefill_flops(cfg, layers, [PROMPT])
    prefill = {"value": round(PROMPT / (pms / 1000.0), 1), "tokens": PROMPT, "ms": round(pms, 3),
               "frac": round(flops / (pms / 1000.0) / (pk["bf16_tflops"] * 1e12), 4), "tflops": round(flops / (pms / 1000.0) / 1e12, 1)}
    if "bf16_tflops_sustained" in pk:   # what the same library product holds for seconds under the power cap, beside the burst figure above
        prefill["frac_of_sustained"] = round(flops / (pms / 1000.0) / (pk["bf16_tflops_sustained"] * 1e12), 4)

    # --- end to end through the Python entry point: host ids in, host ids out, every step.
    # Passes that are not timed, then exactly K passes, timed on the host from the arrival of one
    # pass's ids to that of the K-th pass after it.  The untimed passes are W, but at least 24:
    # after the prompt burst (which runs into the power cap) the part takes 11 to 19 decode steps
    # to raise its clocks again, and a generation goes on straight from its prompt, so a timed
    # region that began after 3 passes would time that recovery, not decoding.  (The device-timed
    # figure above is taken after a host pause of 0.3 s, during which the clocks recover at once.)
    def end_to_end(batch, steps, warmup):
        warmup = max(warmup, E2E_SETTLE_PASSES)
        ps = prompts(batch)
        traffic = engine_module.TRAFFIC
        arrived = []
        seen = {"h2d": 0, "d2h": 0}

        def on_token(i, tok):
            if i == 0:
                arrived.append(time.perf_counter())
                if len(arrived) == warmup + 1:
                    seen["h2d"], seen["d2h"] = traffic["h2d_decode"], traffic["d2h_decode"]

        out, stats = model.generate(ps, warmup + steps + 1, Sampling(), on_token=on_token, stop_ids=())
        seconds = arrived[warmup + steps] - arrived[warmup]
        per_step = float(steps)
        return {"prompts": ps, "out": out, "stats": stats, "tok_s": batch * steps / seconds, "ms_per_step": 1000.0 * seconds / steps, "warmup": warmup,
                "h2d": (traffic["h2d_decode"] - seen["h2d"]) / per_step, "d2h": (traffic["d2h_decode"] - seen["d2h"]) / per_step}

    r = end_to_end(args.batch, args.steps, args.warmup)
    ps, out, stats = r["prompts"], r["out"], r["stats"]
    e2e = {"value": round(r["tok_s"], 1), "unit": "tokens/s", "h2d_bytes_per_step": int(round(r["h2d"])),
           "d2h_bytes_per_step": int(round(r["d2h"])), "ms_per_step": round(r["ms_per_step"], 4), "generated": stats.generated,
           "passes": stats.passes, "untimed_passes": r["warmup"], "first_token_ms": round(stats.first_token_ms, 1),
           "of_device_timed": round(r["tok_s"] / main["tok_s"], 4)}
    # --- the check: the same prompts stepped launch by launch (no captured graph, no step begun ahead) give the same tokens
    eng.use_graphs = False
    plain_out, _ = model.generate(ps, r["warmup"] + args.steps + 1, Sampling(), stop_ids=())
    eng.use_graphs = True
    if plain_out != out:
        bad = next(i for i, (x, y) in enumerate(zip(out, plain_out)) if x != y)
        raise AssertionError(f"bench: sequence {bad} generated {out[bad][:8]}... through captured steps and {plain_out[bad][:8]}... step by step")
    if len({tuple(o) for o in out}) < len(out) or any(not 0 <= t < vocab for o in out for t in o):
        raise AssertionError("bench: the generated sequences are not distinct sequences of token ids")

    classes = None if args.no_breakdown else breakdown(eng, cfg, layers, args.batch, pk, rng)

    points = {}
    if not args.no_points:
        for b in (1, 64):
            r = timed_decode(eng, prompts(b), max(16, args.steps // 2), max(3, args.warmup // 2), rng, vocab)
            points[f"decode_b{b}"] = round(r["tok_s"], 1)
            need_b = decode_bytes(cfg, layers, b, r["cached_tokens"])
            points[f"decode_b{b}_hbm_frac"] = round(need_b / (r["ms_per_step"] / 1000.0) / 1e9 / pk["hbm_gbs"], 4)
            e = end_to_end(b, max(16, args.steps // 2), max(3, args.warmup // 2))
            points[f"e2e_b{b}"] = round(e["tok_s"], 1)
            points[f"e2e_b{b}_of_device_timed"] = round(e["tok_s"] / r["tok_s"], 4)
    del model, eng
    free_device_memory()
    if not args.no_points and not args.layers:
        points.update(bench_long(pk, rng))
        points.update(bench_13b(pk, rng))
        points.update(bench_3b(pk, rng))
        points.update(bench_tiny(rng))

    config = {"model": "llama-3.1-8b-shape", "layers": layers, "layers_full": full_layers, "hidden": cfg["hidden_size"],
              "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
              "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"], "global_batch": args.batch,
              "seq_len": CONTEXT, "prompt_len": PROMPT, "parallelism": "single-gpu", "l2": "inputs larger than L2 (16 GB of weights a step)"}
    line = {
        "metric": "decode tokens/s (Llama-3.1-8B shape, bf16, batch %d, 2,048-token prompts)" % args.batch,
        "value": round(main["tok_s"], 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(main["ms_per_step"], 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: seeded uniform token ids, random N(0,0.02) weights", "config": config,
        "clocks": main["clocks"], "e2e": e2e, "gpu_launches": launches_per_step * args.steps, "launches_per_step": launches_per_step,
        "prefill": prefill, "roofline": roofline, "points": points, "checked": True, "impl": "ours",
    }
    if classes is not None:
        line["classes"] = classes
    return line


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--prompt", type=int, default=PROMPT, help="prompt tokens before the timed decode steps")
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration has (0: all)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-points", action="store_true", help="skip batch 1 and 64 and the two other shapes")
    ap.add_argument("--no-breakdown", action="store_true", help="skip the per-class timing of one decode and one prompt step")
    ap.add_argument("--point", default="", choices=["", "long", "13b", "3b", "tiny", "fegidra", "pozirax", "fudelorn", "logirax", "duratar", "kodulix"],
                    help="run one of the further workloads alone and print its figures (not the default run's one JSON line)")
    ap.add_argument("--size", default="wide", choices=sorted(FEGIDRA_SIZES), help="with --point fegidra, pozirax, fudelorn, logirax, duratar or kodulix: which sizes")
    args = ap.parse_args()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": "the reference is a Rust workspace (no setup.py or pyproject) "
                          "and no Rust toolchain is installed: it can be neither pip-installed nor built here"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures one GPU; --gpus {args.gpus} is not supported (this library does not use several GPUs)")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.point:
        import numpy as np

        rng = np.random.default_rng(0)
        one = {"long": lambda: bench_long(peaks(), rng, args.layers), "13b": lambda: bench_13b(peaks(), rng), "3b": lambda: bench_3b(peaks(), rng),
               "tiny": lambda: bench_tiny(rng),
               "fegidra": lambda: bench_fegidra(peaks(), rng, args.size, args.layers or 4, args.batch, args.prompt, min(args.steps, 32), args.warmup),
               "pozirax": lambda: bench_pozirax(peaks(), rng, args.size, args.layers or 4, args.batch, args.prompt, min(args.steps, 32), args.warmup),
               "fudelorn": lambda: bench_fudelorn(peaks(), rng, args.size, args.layers or 4, args.batch, args.prompt, min(args.steps, 32), args.warmup),
               "logirax": lambda: bench_logirax(peaks(), rng, args.size, args.layers or 4, args.batch, args.prompt, min(args.steps, 32), args.warmup),
               "duratar": lambda: bench_duratar(peaks(), rng, args.size, args.layers or 4, args.batch, args.prompt, min(args.steps, 32), args.warmup),
               "kodulix": lambda: bench_kodulix(peaks(), rng, args.size, args.layers or 4, args.batch, args.prompt, min(args.steps, 32), args.warmup)}[args.point]
        print(json.dumps({"point": args.point, **one()}))
        return 0
    print(json.dumps(run_ours(args)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
