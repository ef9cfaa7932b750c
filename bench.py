#!/usr/bin/env python3
"""Decode and prefill throughput of alpacca_b200 on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference] [--shape 1b|7b|8b]

Workloads (layer sizes, prompts and sampling as the benchmark configurations name them; random
bfloat16 weights N(0, 0.02), seeded uniform-random token ids):

  1b (default)  Llama-3.2-1B sizes, context 4096.  8 sequences, each prefilled with 512 tokens, then
                K greedy decode steps (256 unless --steps says otherwise).  Also one prompt of 2,048
                tokens (`prefill`) and decode at batch 1 and 64 (`points`).
  7b            Llama-2-7B sizes.  8 prompts with lengths uniform in [16, 1024], then 128 greedy steps.
  8b            Llama-3.1-8B sizes.  64 prompts with lengths uniform in [128, 2048], then 256 steps at
                temperature 1.0 with a seeded generator; the cache holds 4,096 tokens per sequence.

A "step" is one decode step of the whole batch.  `value` is decoded tokens per second, timed on the
device with CUDA events around exactly K steps replayed from the engine's CUDA graph (a step's sampled
token is the next step's input, on the device).  `e2e` is the same workload through the Python entry
point (`alpacca_b200.api.generate`): token ids in from host lists, token ids out to host lists, with
the per-step host traffic that serving has.  `prefill` is the 2,048-token prompt (1b) or the
workload's own unequal batch of prompts in one step (7b, 8b); `roofline` divides the bytes a decode
step must read (all weights once, plus the cache of the live requests) by the step time.  Every step
streams more bytes than the L2 holds, so nothing is flushed between timed iterations.  The default run
(1b) also times the decode of the 7b and 8b workloads, each in a child process, with their own numbers of
steps: `points.decode_7b_b8`, `points.decode_8b_b64` and `other_workloads` (--no-other-workloads leaves
them out).

`--impl reference` runs the same workload through the unmodified reference (a CPU engine for one
sequence at a time: it takes the sequences one after another) and prints the same line.

`--design lefatar` leaves the workload above alone and measures the Lefatar decoder (matrix-memory and
latent-attention layers, dense and routed feed-forwards) beside the Llama decoder of the same width, depth and
dense feed-forward: one prompt of 2,048 tokens and decode at batch 8 from 512-token prompts, at two sizes.
`--design buguzen` does the same for the Buguzen decoder (linear attention with a fixed decay, attention with
two score maps, attention over its own keys, token inputs, two layers that run twice).
`--design sazepel` does the same for the Sazepel decoder (retention; attention with mixed heads beside a retention;
routed gated experts in every layer), beside the Lefatar decoder (the framework's other decoder with routed experts
and a matrix state per head) and the Llama decoder.
`--design mavidra` does the same for the Mavidra decoder (gated linear attention; latent attention with a window, one
layer reading another's cache; attention with a sink beside the gated delta rule; routed gated experts with sigmoid
scores in every layer; layer norms around every sub-layer), beside the Sazepel decoder (the closest: recurrent mixers,
two mixers side by side, routed gated experts of the same sizes, norms around every sub-layer), the Lefatar decoder
(the same latent-attention kernels) and the Llama decoder.
`--design ponusun` does the same for the Ponusun decoder (attention with a window and a penalty on distance, every second
layer reading the keys of the layer before; experts chosen by token id beside a shared one; norms on the sub-layers'
outputs, an input convolution and an average over depth in every layer), beside the Sazepel decoder (routed gated
experts of the same sizes), the Buguzen decoder (attention with a window and a query/key norm) and the Llama decoder.
`--design nagavik` does the same for the Nagavik decoder (state-space mixers, every fourth layer attention with bounded scores
and a slope per head; ungated experts chosen by sigmoid scores beside a shared one; norms around every sub-layer), beside the
Mavidra decoder (the closest: recurrences with decays that depend on the token, short convolutions, a sink attention, experts
with sigmoid scores, norms around every sub-layer), the Ponusun decoder (the same experts' kernels with gates, attention with
a penalty on distance) and the Llama decoder.

One JSON line goes to standard output.  With --gpus N > 1 it prints a line that says so and exits
with 2: this library runs on one GPU.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

LLAMA3_SCALING = {"rope_type": "llama3", "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                  "original_max_position_embeddings": 8192}
# No stop token is configured: with random weights a sequence must not end by chance.
SHAPES = {
    "1b": {
        "name": "Llama-3.2-1B shape",
        "config": {"architectures": ["LlamaForCausalLM"], "num_hidden_layers": 16, "hidden_size": 2048,
                   "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 64, "intermediate_size": 8192,
                   "vocab_size": 128256, "max_position_embeddings": 131072, "rms_norm_eps": 1e-5,
                   "rope_theta": 500000.0, "rope_pairing": "neox", "rope_scaling": dict(LLAMA3_SCALING, factor=32.0),
                   "tie_word_embeddings": True, "hidden_act": "silu", "bos_token_id": 128000},
        "context": 4096, "batch": 8, "prompt_lengths": (512, 512), "steps": 256, "temperature": 0.0,
        "prefill_tokens": 2048, "points": (1, 64),
    },
    "7b": {
        "name": "Llama-2-7B shape",
        "config": {"architectures": ["LlamaForCausalLM"], "num_hidden_layers": 32, "hidden_size": 4096,
                   "num_attention_heads": 32, "num_key_value_heads": 32, "head_dim": 128, "intermediate_size": 11008,
                   "vocab_size": 32000, "max_position_embeddings": 4096, "rms_norm_eps": 1e-5,
                   "rope_theta": 10000.0, "rope_pairing": "neox", "rope_scaling": None,
                   "tie_word_embeddings": False, "hidden_act": "silu", "bos_token_id": 1},
        "context": 4096, "batch": 8, "prompt_lengths": (16, 1024), "steps": 128, "temperature": 0.0,
        "prefill_tokens": None, "points": (),
    },
    "8b": {
        "name": "Llama-3.1-8B shape",
        "config": {"architectures": ["LlamaForCausalLM"], "num_hidden_layers": 32, "hidden_size": 4096,
                   "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 14336,
                   "vocab_size": 128256, "max_position_embeddings": 131072, "rms_norm_eps": 1e-5,
                   "rope_theta": 500000.0, "rope_pairing": "neox", "rope_scaling": dict(LLAMA3_SCALING, factor=8.0),
                   "tie_word_embeddings": False, "hidden_act": "silu", "bos_token_id": 128000},
        "context": 4096, "batch": 64, "prompt_lengths": (128, 2048), "steps": 256, "temperature": 1.0,
        "prefill_tokens": None, "points": (),
    },
}
SAMPLING_SEED = 1234
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def peaks():
    p = ROOT / "MEASURED_PEAKS.json"
    if p.is_file():
        try:
            d = json.loads(p.read_text())
            return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
        except (ValueError, KeyError):
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


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
        time.sleep(0.15)
        self.proc.terminate()
        out, _ = self.proc.communicate(timeout=10)
        mhz, top, reasons = [], None, set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for line in out.splitlines():
            f = [x.strip() for x in line.split(",")]
            if len(f) < 6 or not f[0].isdigit():
                continue
            mhz.append(int(f[0]))
            top = int(f[1])
            reasons |= {n for n, v in zip(names, f[2:6]) if v.lower().startswith("active")}
        return {"sm_mhz": statistics.median(mhz) if mhz else None, "sm_max_mhz": top, "reasons": sorted(reasons)}


def workload_prompts(shape, batch, seed):
    """`batch` prompts of the workload: lengths uniform in the shape's range, uniform-random token ids."""
    import random
    rng = random.Random(seed)
    lo, hi = shape["prompt_lengths"]
    vocab = shape["config"]["vocab_size"]
    lengths = [rng.randint(lo, hi) for _ in range(batch)]
    return [[rng.randrange(vocab) for _ in range(n)] for n in lengths]


def sampler_params(shape):
    from alpacca_b200.sampling import SamplerParams
    if shape["temperature"] <= 0:
        return SamplerParams.greedy()
    # plain temperature sampling over the whole vocabulary, seeded
    return SamplerParams(temperature=shape["temperature"], top_k=0, top_p=1.0, repeat_penalty=1.0, seed=SAMPLING_SEED)


def model_bytes(model) -> int:
    """Bytes of every weight a decode step reads once (a tied embedding table counts once: it is the head;
    an untied one is read by rows only and does not count)."""
    seen, total = set(), 0
    head_is_table = model.decoder.spec.head.tied_to is not None
    stack = [model.decoder]
    while stack:
        part = stack.pop()
        stack.extend(part.children())
        if type(part).__name__ == "RotaryEncoding" or (type(part).__name__ == "TokenEmbedding" and not head_is_table):
            continue
        for v in vars(part).values():
            if hasattr(v, "data_ptr") and hasattr(v, "element_size") and v.is_cuda and v.dim() >= 1:
                if v.data_ptr() not in seen and v.dtype.is_floating_point:
                    seen.add(v.data_ptr())
                    total += v.numel() * v.element_size()
    return total


def prefill_flops(cfg, lengths) -> float:
    """Floating-point operations of one step that runs prompts of these lengths whole and asks for the
    logits of each prompt's last token."""
    E, H, K, D = cfg["hidden_size"], cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    F, L, V = cfg["intermediate_size"], cfg["num_hidden_layers"], cfg["vocab_size"]
    per_token = 2.0 * (E * (H + 2 * K) * D + H * D * E + 3 * E * F)
    attention = sum(2.0 * 2.0 * H * D * T * (T + 1) / 2.0 for T in lengths)
    return L * (sum(lengths) * per_token + attention) + len(lengths) * 2.0 * V * E


def start_batch(model, shape, batch, seed):
    """Prefills the workload's prompts in one step, samples their first tokens; returns what the decoder needs."""
    from alpacca_b200.engine.step import StepEntry
    from alpacca_b200.sampling import DeviceSampler
    eng = model.engine
    prompts = workload_prompts(shape, batch, seed)
    slots = [eng.alloc_slot() for _ in prompts]
    sampler = DeviceSampler(sampler_params(shape), eng.device)
    states = [sampler.new_state(i, p) for i, p in enumerate(prompts)]
    logits = eng.step([StepEntry(s, p, [len(p) - 1]) for s, p in zip(slots, prompts)])
    first = sampler.sample(logits, states)
    decoder = model.decoder_for(sampler)
    return slots, decoder, [(s, t, st) for s, t, st in zip(slots, first, states)]


def measure_decode(model, shape, batch, steps, warmup, seed=0):
    """Device-timed decode: (tokens per second, ms per step, mean tokens held per step, kernels per step)."""
    import torch
    from alpacca_b200 import ops
    slots, decoder, live = start_batch(model, shape, batch, seed)
    try:
        warm = max(warmup, 3)
        # the pages of the whole run are reserved first, so that the warm-up steps and the timed
        # steps have the same batch shape (and the capture of its graph falls into the warm-up)
        model.engine.cache.reserve([(s, warm + steps) for s in slots])
        decoder.run(live, warm)
        before = ops.launches
        torch.cuda.synchronize()
        t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        held0 = sum(model.engine.length(s) for s in slots)
        t0.record()
        decoder.run(live, steps)
        t1.record()
        torch.cuda.synchronize()
        ops.check_tc_status()
        ms = t0.elapsed_time(t1)
        eager_launches = ops.launches - before
        per_step = getattr(decoder, "kernels_per_step", None) or (eager_launches // max(steps, 1))
        # step i reads the held0 + i * batch tokens cached so far (and appends one per sequence)
        measure_decode.last_held = held0 + batch * (steps - 1) / 2.0
        return batch * steps / (ms / 1e3), ms / steps, measure_decode.last_held, per_step
    finally:
        for s in slots:
            model.engine.free_slot(s)


def measure_e2e(model, shape, batch, steps, seed=1):
    """The same decode through the Python entry point: host token lists in, host token lists out."""
    from alpacca_b200.api import generate
    prompts = workload_prompts(shape, batch, seed)
    params = sampler_params(shape)
    generate(model, prompts, params, n_predict=8, stop_token_ids=[])     # warm-up (graphs)
    res = generate(model, prompts, params, n_predict=steps + 1, stop_token_ids=[])
    tokens = sum(r.tokens - 1 for r in res)            # the first token of each comes from the prompt step
    seconds = max(r.seconds for r in res)
    return tokens / seconds, seconds


def measure_prefill(model, prompts, runs=5):
    """Median device time (ms) of one step that runs `prompts` whole."""
    import numpy as np
    import torch
    from alpacca_b200.engine.step import StepEntry
    eng = model.engine
    prompts = [np.asarray(p, dtype=np.int32) for p in prompts]     # token ids as arrays, as a tokenizer hands them over
    times = []
    for i in range(runs + 2):
        slots = [eng.alloc_slot() for _ in prompts]
        torch.cuda.synchronize()
        t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        t0.record()
        eng.step([StepEntry(s, p, [len(p) - 1]) for s, p in zip(slots, prompts)])
        t1.record()
        eng.wait()
        for s in slots:
            eng.free_slot(s)
        if i >= 2:
            times.append(t0.elapsed_time(t1))
    return statistics.median(times)


def other_workload(name: str, timeout: float = 240.0) -> dict:
    """`python bench.py --shape NAME --only decode` in a child process; its short line, or why there is none."""
    cmd = [sys.executable, str(Path(__file__).resolve()), "--shape", name, "--only", "decode"]
    try:
        out = subprocess.run(cmd, capture_output=True, text=True, timeout=timeout)
    except subprocess.TimeoutExpired:
        return {"unavailable": f"no result within {timeout:.0f} s"}
    lines = [ln for ln in out.stdout.splitlines() if ln.startswith("{")]
    if out.returncode != 0 or not lines:
        tail = (out.stderr or out.stdout).strip().splitlines()[-1:] or [""]
        return {"unavailable": f"exit code {out.returncode}: {tail[0][:200]}"}
    d = json.loads(lines[-1])
    return {k: d[k] for k in ("batch", "tok_s", "ms_per_step", "gb_s", "of_hbm_peak", "steps") if k in d}


def flat_config(shape, cfg, layers_full, batch, steps, weights, kv_per_token, prompts):
    lens = [len(p) for p in prompts]
    lo, hi = shape["prompt_lengths"]
    return {"model": shape["name"], "layers": cfg["num_hidden_layers"], "layers_of_config": layers_full,
            "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"],
            "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
            "ffn": cfg["intermediate_size"], "vocab": cfg["vocab_size"], "global_batch": batch,
            "prompt_len": lo if lo == hi else f"uniform in [{lo}, {hi}], seeded (sum {sum(lens)})",
            "seq_len": shape["context"], "decode_steps": steps,
            "sampling": "greedy" if shape["temperature"] <= 0 else f"temperature {shape['temperature']}, seeded",
            "parallelism": "single GPU", "l2": "inputs larger than L2 (no flush)",
            "weight_bytes": weights, "kv_bytes_per_token": kv_per_token}


def metric_name(shape, batch):
    lo, hi = shape["prompt_lengths"]
    prompt = f"{lo}-token prompts" if lo == hi else f"prompts of {lo} to {hi} tokens"
    return f"decode tok/s at batch {batch} ({shape['name']}, {prompt}, context {shape['context']})"


def run_ours(args):
    import torch
    from alpacca_b200.api import Model

    assert torch.cuda.is_available(), "bench.py needs a CUDA device"
    torch.cuda.set_device(0)
    pk = peaks()
    shape = dict(SHAPES[args.shape])
    if args.only == "decode" and args.prompt_len:
        shape["prompt_lengths"] = (args.prompt_len, args.prompt_len)
        # room for the prompt, the warm-up steps and the timed steps in every slot
        shape["context"] = max(shape["context"], args.prompt_len + max(args.warmup, 3) + (args.steps or shape["steps"]) + 1)
    if args.only == "prefill" and args.prefill_tokens:
        shape["prefill_tokens"] = args.prefill_tokens
        shape["context"] = max(shape["context"], args.prefill_tokens)
    cfg = dict(shape["config"])
    layers_full = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    batch = args.batch or shape["batch"]
    if args.only == "prefill" and args.prefill_tokens and not args.batch:
        batch = 1           # one prompt: the cache is sized for it alone
    steps = args.steps or shape["steps"]
    biggest = max([batch, *shape["points"]]) if args.only == "all" else batch
    model = Model.random(cfg, seed=0, n_ctx=shape["context"], dtype="bfloat16", max_batch=biggest)
    weights = model_bytes(model)
    kv_per_token = sum(g.bytes_per_token for g in model.engine.cache.kv_groups)

    if args.only == "decode":
        tps, ms_step, _, kernels = measure_decode(model, shape, batch, steps, args.warmup)
        held = measure_decode.last_held
        gbs = (weights + held * kv_per_token) / (ms_step / 1e3) / 1e9
        print(json.dumps({"only": "decode", "shape": args.shape, "batch": batch, "steps": steps, "tok_s": round(tps, 1),
                          "ms_per_step": round(ms_step, 4), "kernels_per_step": kernels,
                          "tokens_held": int(held), "gb_s": round(gbs, 1), "of_hbm_peak": round(gbs / pk["hbm_gbs"], 3)}))
        return 0
    if shape["prefill_tokens"]:
        pre_prompts = workload_prompts(dict(shape, prompt_lengths=(shape["prefill_tokens"],) * 2), 1, seed=2)
    else:
        pre_prompts = workload_prompts(shape, batch, seed=0)        # the prompts that the decode run starts from
    if args.only == "prefill":
        pre_ms = measure_prefill(model, pre_prompts, runs=max(args.steps, 1))
        fl = prefill_flops(cfg, [len(p) for p in pre_prompts])
        print(json.dumps({"only": "prefill", "shape": args.shape, "tokens": sum(map(len, pre_prompts)),
                          "ms": round(pre_ms, 3), "tok_s": round(sum(map(len, pre_prompts)) / (pre_ms / 1e3), 1),
                          "of_bf16_peak": round(fl / (pre_ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4)}))
        return 0

    clocks = ClockSampler()
    clocks.start()
    tps, ms_step, held_mean, kernels = measure_decode(model, shape, batch, steps, args.warmup)
    clock_info = clocks.stop()

    e2e_tps, _ = measure_e2e(model, shape, batch, steps)
    # the points: at least 64 timed steps after at least 16 untimed ones, so that a short run's figure
    # is not that of the few milliseconds after the prompt step (which runs into the power cap at batch 64)
    points = {}
    for b in shape["points"]:
        points[f"decode_b{b}"] = round(measure_decode(model, shape, b, max(steps, 64), max(args.warmup, 16),
                                                      seed=10 + b)[0], 1)
    pre_ms = measure_prefill(model, pre_prompts)
    pre_tokens = sum(map(len, pre_prompts))
    flops = prefill_flops(cfg, [len(p) for p in pre_prompts])

    # the other two workloads of the benchmark, each in a process of its own (its own memory, and a
    # failure there leaves this line whole): device-timed decode with its share of the HBM peak
    others = {}
    if args.shape == "1b" and not args.no_other_workloads and not args.layers:
        del model
        torch.cuda.empty_cache()
        for other in ("7b", "8b"):
            others[other] = other_workload(other)
            if "tok_s" in others[other]:
                points[f"decode_{other}_b{others[other]['batch']}"] = others[other]["tok_s"]

    step_bytes = weights + held_mean * kv_per_token
    achieved = step_bytes / (ms_step / 1e3) / 1e9
    from alpacca_b200.engine.decode import bucket_rows
    rows = bucket_rows(batch)
    line = {
        "metric": metric_name(shape, batch),
        "value": round(tps, 1), "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": max(args.warmup, 3),
        "ms_per_step": round(ms_step, 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: uniform-random token ids, random-init weights N(0, 0.02)",
        "impl": "ours",
        "config": flat_config(shape, cfg, layers_full, batch, steps, weights, kv_per_token,
                              workload_prompts(shape, batch, seed=0)),
        "e2e": {"value": round(e2e_tps, 1), "unit": "tok/s", "h2d_bytes_per_step": 4 * rows,
                "d2h_bytes_per_step": 4 * rows},
        "gpu_launches": int(kernels * steps),
        "prefill": {"value": round(pre_tokens / (pre_ms / 1e3), 1), "tokens": pre_tokens,
                    "ms": round(pre_ms, 3), "frac": round(flops / (pre_ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "peaks": pk["source"],
                     "bytes_per_step": int(step_bytes)},
        "points": points,
        "clocks": clock_info,
    }
    if others:
        line["other_workloads"] = others
    print(json.dumps(line), flush=True)
    return 0


# ---------------------------------------------------------------------------------------------
# the reference arm

def write_reference_model(gguf, np, path, cfg, context):
    """An F32 GGUF of `cfg`'s layer sizes with random weights N(0, 0.02), written with the reference's own writer."""
    E, H, K, D = cfg["hidden_size"], cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    F, V, L = cfg["intermediate_size"], cfg["vocab_size"], cfg["num_hidden_layers"]
    w = gguf.GGUFWriter(path, "llama")
    for key, typ, val in (("general.name", gguf.T_STRING, "bench"), ("llama.context_length", gguf.T_UINT32, context),
                          ("llama.embedding_length", gguf.T_UINT32, E), ("llama.block_count", gguf.T_UINT32, L),
                          ("llama.feed_forward_length", gguf.T_UINT32, F),
                          ("llama.attention.head_count", gguf.T_UINT32, H),
                          ("llama.attention.head_count_kv", gguf.T_UINT32, K),
                          ("llama.attention.layer_norm_rms_epsilon", gguf.T_FLOAT32, cfg["rms_norm_eps"]),
                          ("llama.rope.dimension_count", gguf.T_UINT32, D), ("llama.vocab_size", gguf.T_UINT32, V),
                          ("llama.rope.freq_base", gguf.T_FLOAT32, cfg["rope_theta"]),
                          ("tokenizer.ggml.model", gguf.T_STRING, "llama")):
        w.add(key, typ, val)
    w.add_array("tokenizer.ggml.tokens", gguf.T_STRING, [f"t{i}" for i in range(V)])
    w.add_array("tokenizer.ggml.scores", gguf.T_FLOAT32, [0.0] * V)
    w.add_array("tokenizer.ggml.token_type", gguf.T_INT32, [1] * V)
    rng = np.random.default_rng(0)

    def mat(name, shape):
        n = int(np.prod(shape))
        w.add_raw_tensor(name, shape, "F32", (rng.standard_normal(n, dtype=np.float32) * 0.02).tobytes())

    ones = np.ones(E, np.float32).tobytes()
    mat("token_embd.weight", (E, V))
    for i in range(L):
        p = f"blk.{i}."
        w.add_raw_tensor(p + "attn_norm.weight", (E,), "F32", ones)
        mat(p + "attn_q.weight", (E, H * D))
        mat(p + "attn_k.weight", (E, K * D))
        mat(p + "attn_v.weight", (E, K * D))
        mat(p + "attn_output.weight", (H * D, E))
        w.add_raw_tensor(p + "ffn_norm.weight", (E,), "F32", ones)
        mat(p + "ffn_gate.weight", (E, F))
        mat(p + "ffn_up.weight", (E, F))
        mat(p + "ffn_down.weight", (F, E))
    w.add_raw_tensor("output_norm.weight", (E,), "F32", ones)
    if not cfg.get("tie_word_embeddings"):
        mat("output.weight", (E, V))
    w.write()


def run_reference(args):
    """The unmodified reference (installed into baseline/_ref) through its own public API.

    It is a CPU engine for one sequence at a time and has no batch: it takes the workload's sequences
    one after another (`reset`, `prefill`, then the decode loop), which is how its user serves several
    requests.  `value` is decoded tokens over the time of the hand-timed `forward` + `sample` loop,
    `e2e` the same through its own generation loop (`alpacca.chat.generate`, whose clock starts after
    the prompt), `prefill` one prompt of 2,048 tokens.
    """
    ref = ROOT / "baseline" / "_ref"
    if not (ref / "alpacca" / "model.py").is_file():
        print(json.dumps({"impl": "reference", "unavailable": "baseline/_ref holds no installed reference "
                          "(pip install --no-index --no-build-isolation --target baseline/_ref <the reference's source tree>)"}))
        return 0
    sys.path.insert(0, str(ref))
    try:
        import numpy as np
        from alpacca import chat, gguf
        from alpacca.model import Model
        from alpacca.sample import Sampler, SamplerParams
    except Exception as e:  # noqa: BLE001
        print(json.dumps({"impl": "reference", "unavailable": f"reference does not import: {e}"}))
        return 0
    import tempfile
    shape = SHAPES[args.shape]
    if args.shape != "1b":
        print(json.dumps({"impl": "reference", "unavailable": f"the reference arm runs the 1b workload only "
                          f"(float32 weights of the {args.shape} sizes on the host and minutes per prompt)"}))
        return 0
    cfg = dict(shape["config"])
    layers_full = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    batch = args.batch or shape["batch"]
    steps = min(args.steps or shape["steps"], 32)
    warm = max(args.warmup, 3)
    prompts = workload_prompts(shape, batch, seed=0)
    greedy = dict(temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0, seed=1)
    with tempfile.TemporaryDirectory() as tmp:
        path = os.path.join(tmp, "bench.gguf")
        write_reference_model(gguf, np, path, cfg, shape["context"])
        model = Model.load(path, n_ctx=shape["context"], progress=False)
        # the timed loop by hand: prompt, warm-up steps, then `steps` steps, for each sequence in turn
        decode_s = 0.0
        per_seq = []
        for prompt in prompts:
            model.reset()
            sampler = Sampler(SamplerParams(**greedy))
            logits = model.prefill(prompt)
            for _ in range(warm):
                logits = model.forward(sampler.sample(logits))
            t0 = time.perf_counter()
            for _ in range(steps):
                logits = model.forward(sampler.sample(logits))
            per_seq.append(time.perf_counter() - t0)
            decode_s += per_seq[-1]
        # the same through the reference's own generation loop
        e2e_tokens, e2e_s = 0, 0.0
        for prompt in prompts:
            model.reset()
            res = chat.generate(model, list(prompt), SamplerParams(**greedy), n_predict=steps + 1)
            e2e_tokens += res.tokens - 1           # the first token comes from the prompt step
            e2e_s += res.seconds
        model.reset()
        long_prompt = workload_prompts(dict(shape, prompt_lengths=(shape["prefill_tokens"],) * 2), 1, seed=2)[0]
        t0 = time.perf_counter()
        model.prefill(long_prompt)
        prefill_s = time.perf_counter() - t0
    lo, _ = shape["prompt_lengths"]
    print(json.dumps({
        "metric": metric_name(shape, batch), "impl": "reference",
        "value": round(batch * steps / decode_s, 2), "unit": "tok/s", "n_gpus": args.gpus,
        "device": "cpu (the reference has no GPU path)", "steps": steps, "warmup": warm,
        "ms_per_step": round(decode_s / steps * 1e3, 2), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "fp32 (the reference has no reduced-precision dense path)",
        "data": "synthetic: uniform-random token ids, random-init weights N(0, 0.02)",
        "config": {"model": shape["name"], "layers": cfg["num_hidden_layers"], "layers_of_config": layers_full,
                   "global_batch": batch, "prompt_len": lo, "seq_len": shape["context"], "decode_steps": steps,
                   "sampling": "greedy", "parallelism": "CPU; the sequences of the batch one after another (the "
                   "reference has no batch and no GPU path)"},
        "e2e": {"value": round(e2e_tokens / e2e_s, 2), "unit": "tok/s", "h2d_bytes_per_step": 0,
                "d2h_bytes_per_step": 0, "through": "alpacca.chat.generate"},
        "gpu_launches": 0,
        "points": {"decode_b1": round(steps / per_seq[0], 2)},
        "prefill": {"value": round(len(long_prompt) / prefill_s, 1), "tokens": len(long_prompt),
                    "ms": round(prefill_s * 1e3, 1)}}))
    return 0


# ---------------------------------------------------------------------------------------------------------
# --design lefatar | buguzen | sazepel | mavidra | ponusun | nagavik: that decoder beside the Llama decoder of the same width, depth and dense
# feed-forward, at sizes that resemble a real model's layers (random weights).

def _lefatar_layers(E, mlstm, latent, dense_ff, moe, n_layers):
    """The pattern (memory + dense, memory + experts, latent attention + dense, memory + experts), repeated."""
    dense = {"kind": "dense", "ff": dense_ff}
    pattern = [{"type": "mlstm", "mixer": mlstm, "mlp": dense}, {"type": "mlstm", "mixer": mlstm, "mlp": moe},
               {"type": "latent_attention", "mixer": latent, "mlp": dense}, {"type": "mlstm", "mixer": mlstm, "mlp": moe}]
    return [pattern[i % 4] for i in range(n_layers)]


def _moe(ff, experts, top, count, keep):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "scale": 1.0, "groups": {"count": count, "keep": keep}}}


DESIGN_SIZES = {
    "w1024": {"width": 1024, "layers": 8, "vocab": 32000, "dense_ff": 2816, "heads": 16, "kv_heads": 4, "head_dim": 64,
              "mlstm": {"heads": 4, "dim": 128, "vdim": 256, "gate_cap": 12.0},
              "latent": {"heads": 16, "dim": 64, "rot_dim": 32, "vdim": 64, "q_rank": 384, "kv_rank": 224,
                         "scale": 96 ** -0.5, "rot": {"base": 10000.0, "dims": 32}},
              "moe": _moe(704, 8, 2, 2, 1),
              "buguzen": {"lin_heads": 8, "lin_dim": 128, "lin_vdim": 128, "diff_heads": 8, "diff_dim": 64, "window": 1024,
                          "side": 64}},
    "w2048": {"width": 2048, "layers": 8, "vocab": 32000, "dense_ff": 5632, "heads": 16, "kv_heads": 4, "head_dim": 128,
              "mlstm": {"heads": 8, "dim": 128, "vdim": 256, "gate_cap": 12.0},
              "latent": {"heads": 16, "dim": 128, "rot_dim": 32, "vdim": 128, "q_rank": 768, "kv_rank": 224,
                         "scale": 160 ** -0.5, "rot": {"base": 10000.0, "dims": 32}},
              "moe": _moe(1408, 16, 4, 4, 2),
              "buguzen": {"lin_heads": 16, "lin_dim": 128, "lin_vdim": 128, "diff_heads": 16, "diff_dim": 64, "window": 1024,
                          "side": 128}},
}


def _decays(heads):
    """A decay per head between 1 - 2^-3 and 1 - 2^-9: short and long memories side by side."""
    return [1.0 - 2.0 ** -(3.0 + 6.0 * h / max(heads - 1, 1)) for h in range(heads)]


def _buguzen_config(z):
    """Six layers in the pattern (linear attention, attention with two maps, attention over its keys), each with a
    dense feed-forward and a token input; layers 2 and 3 run twice: eight layer runs, as the Llama decoder beside it."""
    b = z["buguzen"]
    dense = {"kind": "dense", "ff": z["dense_ff"]}
    lightning = {"type": "lightning", "mlp": dense,
                 "mixer": {"heads": b["lin_heads"], "dim": b["lin_dim"], "vdim": b["lin_vdim"], "decay": _decays(b["lin_heads"])}}
    diff = {"type": "attention", "mlp": dense,
            "mixer": {"heads": b["diff_heads"], "kv_heads": z["kv_heads"], "dim": b["diff_dim"], "vdim": 2 * b["diff_dim"],
                      "scale": b["diff_dim"] ** -0.5, "diff": 0.2, "mask": {"size": b["window"]},
                      "rot": {"base": 100000.0, "dims": b["diff_dim"] // 2, "scaling": {"factor": 2.0}}}}
    keys = {"type": "attention_2", "mlp": dense,
            "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["head_dim"], "scale": z["head_dim"] ** -0.5,
                      "mask": {"size": b["window"]},
                      "rot": {"base": 250000.0, "dims": z["head_dim"] // 2,
                              "scaling": {"factor": 16.0, "low": 1.0, "high": 8.0, "original": 2048}}}}
    return {"architecture": "Buguzen", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [lightning, diff, keys, lightning, diff, keys], "loop": {"start": 2, "stop": 4, "times": 2},
            "token_side": {"dim": b["side"]}}


def _sazepel_config(z):
    """Eight layers in the pattern (attention with mixed heads beside a retention, retention), every layer with routed
    gated experts of the size of the Lefatar decoder's beside it."""
    rt = z["moe"]["router"]
    mlp = {"kind": "moe", "expert": dict(z["moe"]["expert"]), "router": {"experts": rt["experts"], "top": rt["top"]}}
    lin = z["buguzen"]

    def ret(heads):
        return {"heads": heads, "dim": lin["lin_dim"], "vdim": lin["lin_vdim"], "decay": _decays(heads),
                "rot": {"base": 1e6, "dims": lin["lin_dim"]}}
    left = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["head_dim"], "vdim": z["head_dim"],
            "scale": z["head_dim"] ** -0.5}
    pair = [{"type": "parallel", "mixer": {"left": left, "right": ret(lin["lin_heads"] // 2)}, "mlp": mlp},
            {"type": "retention", "mixer": ret(lin["lin_heads"]), "mlp": mlp}]
    return {"architecture": "Sazepel", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "logit_scale": 1.0, "layers": [pair[i % 2] for i in range(z["layers"])]}


def _mavidra_config(z):
    """Eight layers in the pattern (gated linear attention, latent attention, attention beside the delta rule, gated
    linear attention), the second latent-attention layer reading the first one's cache; every layer with routed gated
    experts of the size of the Sazepel and Lefatar decoders' beside it."""
    rt = z["moe"]["router"]
    mlp = {"kind": "moe", "expert": dict(z["moe"]["expert"]),
           "router": {"experts": rt["experts"], "top": rt["top"], "groups": dict(rt["groups"])}}
    lin = z["buguzen"]
    gla = {"type": "gla", "mlp": mlp, "mixer": {"heads": lin["lin_heads"], "dim": lin["lin_dim"], "vdim": lin["lin_vdim"],
                                                "tau": 16.0, "rank": z["width"] // 16}}
    lat = {k: v for k, v in z["latent"].items()}
    lat["mask"] = {"size": lin["window"]}
    left = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["head_dim"], "vdim": z["head_dim"],
            "scale": z["head_dim"] ** -0.5, "rot": {"base": 500000.0, "dims": z["head_dim"] // 2}}
    right = {"heads": lin["lin_heads"] // 2, "kv_heads": lin["lin_heads"] // 4, "dim": lin["lin_dim"], "vdim": lin["lin_vdim"],
             "conv": 4}
    par = {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": right, "left_scale": 1.0, "right_scale": 1.0}}
    layers = [gla, {"type": "latent_attention", "mixer": lat, "mlp": mlp}, par, gla, gla,
              {"type": "latent_attention", "mixer": dict(lat, kv_from=1, mask={"size": lin["window"] // 2}), "mlp": mlp}, par, gla]
    return {"architecture": "Mavidra", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "embedding": {"scale": 8.0, "bigram": {"buckets": 65521, "mul_prev": 257, "mul_cur": 31}},
            "layers": layers[:z["layers"]]}


def _ponusun_config(z):
    """Eight layers of attention with a window, every second one reading the keys of the layer before with half the window;
    a dense feed-forward in the first layer, then experts of the size of the other decoders' beside a shared one of twice
    that size."""
    rt = z["moe"]["router"]
    ff = z["moe"]["expert"]["ff"]
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": rt["experts"], "top": rt["top"]}, "shared": {"ff": 2 * ff}}
    window = z["buguzen"]["window"]
    layers = []
    for i in range(z["layers"]):
        mx = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["head_dim"], "vdim": z["head_dim"],
              "scale": z["head_dim"] ** -0.5, "mask": {"size": window if i % 2 == 0 else window // 2}}
        if i % 2:
            mx["kv_from"] = i - 1
        layers.append({"type": "attention", "mixer": mx, "mlp": moe if i else {"kind": "dense", "ff": z["dense_ff"]}})
    return {"architecture": "Ponusun", "vocab": z["vocab"], "width": z["width"], "max_positions": 8192, "norm": {"eps": 1e-6},
            "canon": {"taps": 4}, "logit_softcap": 30.0, "layers": layers}


def _nagavik_config(z):
    """Eight layers, every fourth one attention with bounded scores and slopes, the others state-space mixers of twice the
    width; a dense feed-forward in the first layer, then ungated experts of the inner size of the other decoders' beside a
    shared one of twice that size."""
    rt = z["moe"]["router"]
    ff = z["moe"]["expert"]["ff"]
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": rt["experts"], "top": rt["top"]}, "shared": {"ff": 2 * ff}}
    ssm = {"type": "mamba2", "mixer": {"heads": z["width"] // 32, "vdim": 64, "state": 128, "groups": 4, "conv": 4, "norm_groups": 4}}
    att = {"type": "attention", "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["head_dim"], "vdim": z["head_dim"],
                                          "scale": z["head_dim"] ** -0.5, "softcap": 16.0}}
    layers = [dict(att if i % 4 == 3 else ssm, mlp=moe if i else {"kind": "dense", "ff": z["dense_ff"]}) for i in range(z["layers"])]
    return {"architecture": "Nagavik", "vocab": z["vocab"], "width": z["width"], "max_positions": 8192, "norm": {"eps": 1e-6},
            "embedding": {"scale": 4.0}, "logit_softcap": 40.0, "layers": layers}


def design_configs(size, design="lefatar"):
    z = DESIGN_SIZES[size]
    llama = {"architectures": ["LlamaForCausalLM"], "num_hidden_layers": z["layers"], "hidden_size": z["width"],
             "num_attention_heads": z["heads"], "num_key_value_heads": z["kv_heads"], "head_dim": z["head_dim"],
             "intermediate_size": z["dense_ff"], "vocab_size": z["vocab"], "max_position_embeddings": 8192,
             "rms_norm_eps": 1e-6, "rope_theta": 10000.0, "rope_pairing": "neox", "tie_word_embeddings": False,
             "hidden_act": "silu"}
    if design == "buguzen":
        return {"buguzen": _buguzen_config(z), "llama": llama}
    lefatar = {"architecture": "Lefatar", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
               "layers": _lefatar_layers(z["width"], z["mlstm"], z["latent"], z["dense_ff"], z["moe"], z["layers"])}
    if design == "sazepel":
        return {"sazepel": _sazepel_config(z), "lefatar": lefatar, "llama": llama}
    if design == "mavidra":
        return {"mavidra": _mavidra_config(z), "sazepel": _sazepel_config(z), "lefatar": lefatar, "llama": llama}
    if design == "ponusun":
        return {"ponusun": _ponusun_config(z), "sazepel": _sazepel_config(z), "buguzen": _buguzen_config(z), "llama": llama}
    if design == "nagavik":
        return {"nagavik": _nagavik_config(z), "mavidra": _mavidra_config(z), "ponusun": _ponusun_config(z), "llama": llama}
    return {"lefatar": lefatar, "llama": llama}


def op_table(model, entries):
    """{operation: [launches, microseconds]} of one step issued launch by launch."""
    from alpacca_b200 import ops
    with ops.timers() as t:
        model.engine.step(entries)
    return {k: [n, round(us, 1)] for k, (n, us) in sorted(t.totals().items(), key=lambda kv: -kv[1][1])}


def run_design(args):
    import torch
    from alpacca_b200.api import Model
    from alpacca_b200.engine.step import StepEntry

    assert torch.cuda.is_available(), "bench.py needs a CUDA device"
    torch.cuda.set_device(0)
    pk = peaks()
    batch, prompt_len, prefill_tokens = args.batch or 8, args.prompt_len or 512, args.prefill_tokens or 2048
    steps = args.steps or 64
    out = {"design": args.design, "batch": batch, "prompt_len": prompt_len, "prefill_tokens": prefill_tokens,
           "decode_steps": steps, "dtype": "bf16", "data": "synthetic: uniform-random token ids, random-init weights",
           "peaks": pk, "sizes": {}}
    for size in ([args.size] if args.size else sorted(DESIGN_SIZES)):
        row = {}
        for name, cfg in design_configs(size, args.design).items():
            vocab = cfg.get("vocab") or cfg["vocab_size"]
            shape = {"config": {"vocab_size": vocab}, "prompt_lengths": (prompt_len, prompt_len), "temperature": 0.0}
            context = max(prefill_tokens, prompt_len + steps + max(args.warmup, 3) + 2)
            model = Model.random(cfg, seed=0, n_ctx=context, dtype="bfloat16", max_batch=batch)
            weights = model_bytes(model)
            long_prompt = workload_prompts(dict(shape, prompt_lengths=(prefill_tokens, prefill_tokens)), 1, 7)
            ms = measure_prefill(model, long_prompt)
            tps, ms_step, held, kernels = measure_decode(model, shape, batch, steps, args.warmup)
            kv = sum(g.bytes_per_token for g in model.engine.cache.kv_groups)
            state = sum(g.state[:, 0].numel() * 4 for g in model.engine.cache.state_groups)     # per sequence
            step_bytes = weights + held * kv + 2 * batch * state
            res = {"parameters_m": round(model.decoder.n_params() / 1e6, 1), "weight_bytes": weights,
                   "prefill": {"tok_s": round(prefill_tokens / (ms / 1e3), 1), "ms": round(ms, 3)},
                   "decode": {"tok_s": round(tps, 1), "ms_per_step": round(ms_step, 4), "kernels_per_step": kernels,
                              "bytes_per_step": int(step_bytes),
                              "of_hbm_peak": round(step_bytes / (ms_step / 1e3) / 1e9 / pk["hbm_gbs"], 3)}}
            if args.ops:
                eng = model.engine
                s = eng.alloc_slot()
                res["prefill_ops_us"] = op_table(model, [StepEntry(s, long_prompt[0], [prefill_tokens - 1])])
                eng.free_slot(s)
                slots = [eng.alloc_slot() for _ in range(batch)]
                prompts = workload_prompts(shape, batch, 3)
                eng.step([StepEntry(a, q, []) for a, q in zip(slots, prompts)])
                res["decode_ops_us"] = op_table(model, [StepEntry(a, [1], [0]) for a in slots])
                for a in slots:
                    eng.free_slot(a)
            row[name] = res
            del model
            torch.cuda.empty_cache()
        out["sizes"][size] = row
    print(json.dumps(out))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=0, help="decode steps to time (0: the workload's own number)")
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--shape", default="1b", choices=sorted(SHAPES), help="which benchmark workload")
    ap.add_argument("--batch", type=int, default=0, help="another batch size than the workload's (0: its own)")
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration (0: all)")
    ap.add_argument("--only", default="all", choices=["all", "decode", "prefill"],
                    help="measure one part only and print a short line (for profiling runs)")
    ap.add_argument("--no-other-workloads", action="store_true",
                    help="the default run also times the decode of the 7b and 8b workloads (in child processes, "
                         "into `points` and `other_workloads`); this leaves them out")
    ap.add_argument("--prompt-len", type=int, default=0,
                    help="with --only decode: equal prompts of this many tokens instead of the workload's")
    ap.add_argument("--prefill-tokens", type=int, default=0,
                    help="with --only prefill: one prompt of this many tokens instead of the workload's")
    ap.add_argument("--design", default="", choices=["", "lefatar", "buguzen", "sazepel", "mavidra", "ponusun", "nagavik"],
                    help="instead of the benchmark workload: prefill and decode throughput of this design beside the "
                         "Llama decoder of the same width and depth (random weights), one JSON line")
    ap.add_argument("--size", default="", choices=[""] + sorted(DESIGN_SIZES), help="with --design: one size only")
    ap.add_argument("--ops", action="store_true", help="with --design: device time per kind of operation as well")
    args = ap.parse_args()
    n = int(os.environ.get("WORLD_SIZE", args.gpus))
    if args.gpus > 1 or n > 1:
        if int(os.environ.get("RANK", "0")) == 0:
            print(json.dumps({"impl": args.impl, "n_gpus": max(args.gpus, n),
                              "unsupported": "alpacca_b200 is a single-GPU library; bench.py runs with --gpus 1 only"}))
        return 2
    if args.design:
        return run_design(args)
    return run_reference(args) if args.impl == "reference" else run_ours(args)


if __name__ == "__main__":
    raise SystemExit(main())
