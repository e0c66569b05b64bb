#!/usr/bin/env python3
"""Decode and prefill throughput of rllm_b200 on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference] [--no-workloads]

Prints ONE JSON line.

Headline (Llama-3.2-1B shape, bfloat16, random weights): a batch of 8 sequences, each holding a 2,048-token
prompt, decodes greedily; a "step" is one decode step.  After W warm-up steps exactly K steps are timed
(K = 256 by default: the sequences then go from 2,048 to 2,304 tokens).  ``value`` is decoded tokens per
second timed on the device with CUDA events around K steps that stay on the device (graph replay, argmax,
next-token feed-back), the median of three such runs; SETTLE_STEPS further untimed steps come before the W warm-up steps of every
device-timed point (``config.settle_steps``: the first steps behind the prompts run slower than the rest).  ``e2e`` is the same metric through the Python entry point (``LLM.step``): host token
ids in, pinned-memory copy of the step's inputs to the device, sampled tokens read back to the host, every
step, timed by the host's clock between two device synchronisations.  ``points`` holds the same two figures
at batch 1 and 64, and device-timed decoding at the full context of 4,096 tokens.  ``prefill`` is one
2,048-token prompt as one step, device-timed as a burst after ``prefill_idle_s`` seconds of rest (its ``frac`` is
against the burst peak of the library's product).  ``roofline`` is the decode step against the measured copy bandwidth: the
bytes it has to read (every weight once, the keys and values of the live requests) over its time.

``workloads`` holds two serving runs through ``LLM.add_request`` / ``LLM.step`` with continuous batching:
the Llama-3.2-3B shape (32 requests, prompts of 128 to 4,096 tokens, at most 4,096 tokens a step, 128 tokens
each at temperature 0.8) and the Llama-3.1-8B shape (16 requests that share a 1,024-token prefix, 512-token
portions beside decoded tokens, 256 greedy tokens, prefix caching on), after the reference's synthetic
workload generator (crates/rllm-bench/src/workload.rs:74-90).  Each gives wall time, generated and prompt
tokens per second, preemptions, prefix-hit tokens, steps launched ahead, and the fraction of the roofline:
the sum over the steps that ran of max(flops / peak flops, bytes / peak bandwidth), over the wall time.

``library_standin`` is not the reference (which cannot be built here): it is the same model shape written
with PyTorch's library operators only, timed the same way, so that the figures above have something
beside the roofline to stand against.

Weights are random (N(0, 0.02), seed 0), token ids uniform random: synthetic data, as in the reference's own
workloads.  No flush of L2 is needed between steps: every step reads all weights (2.5 GB and more) and the
live KV cache, far more than the 126 MB of L2.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)


def llama(layers, hidden, heads, kv_heads, head_dim, inter, factor, tied):
    return {
        "architectures": ["LlamaForCausalLM"], "model_type": "llama", "num_hidden_layers": layers,
        "hidden_size": hidden, "num_attention_heads": heads, "num_key_value_heads": kv_heads, "head_dim": head_dim,
        "intermediate_size": inter, "vocab_size": 128256, "rope_theta": 500000.0,
        "rope_scaling": {"rope_type": "llama3", "factor": factor, "low_freq_factor": 1.0,
                         "high_freq_factor": 4.0, "original_max_position_embeddings": 8192},
        "max_position_embeddings": 131072, "rms_norm_eps": 1e-5, "tie_word_embeddings": tied,
        "hidden_act": "silu", "torch_dtype": "bfloat16", "bos_token_id": 128000, "eos_token_id": 128001,
    }


LLAMA_1B = llama(16, 2048, 32, 8, 64, 8192, 32.0, True)
LLAMA_3B = llama(28, 3072, 24, 8, 128, 8192, 32.0, True)
LLAMA_8B = llama(32, 4096, 32, 8, 128, 14336, 8.0, False)
CONTEXT_LEN = 4096
PROMPT_LEN = 2048
DECODE_TOKENS = 256
BLOCK_SIZE = 16
PREFILL_TOKENS = 2048
PREFILL_IDLE_S = 1.5       # the GPU rests this long before the prefill point's burst (see there)
SETTLE_STEPS = 48          # untimed decode steps of a device-timed point before its warm-up steps (see device_point)


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        with open(path) as f:
            p = json.load(f)
        return {"hbm_gbs": float(p["hbm_gbs"]), "bf16_tflops": float(p["bf16_tflops"]), "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while it runs."""

    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.time(), line.strip()))

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()

    def summary(self, windows):
        sm, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for t, line in self.samples:
            if not any(a <= t <= b for a, b in windows):
                continue
            parts = [p.strip() for p in line.split(",")]
            try:
                sm.append(int(parts[0]))
                mx = max(mx, int(parts[1]))
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, parts[2:]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(sm)}


# -- what a step has to read and to compute ---------------------------------------------------------------
def layer_param_count(c, layers):
    h, i, d = c["hidden_size"], c["intermediate_size"], c["head_dim"]
    nq, nkv = c["num_attention_heads"], c["num_key_value_heads"]
    per_layer = h * (nq + 2 * nkv) * d + nq * d * h + 3 * h * i
    return per_layer * layers


def kv_bytes_per_token(c, layers):
    return layers * 2 * c["num_key_value_heads"] * c["head_dim"] * 2


def prefill_flops(c, layers, T):
    linear = 2 * T * layer_param_count(c, layers) + 2 * c["hidden_size"] * c["vocab_size"]
    attn = layers * 4 * c["head_dim"] * c["num_attention_heads"] * T * (T + 1) // 2
    return linear + attn


def decode_bytes(c, layers, batch, ctx_mid):
    weights = 2 * (layer_param_count(c, layers) + c["hidden_size"] * c["vocab_size"])
    return weights + batch * ctx_mid * kv_bytes_per_token(c, layers)


def step_floor_seconds(c, layers, scheduled, pk):
    """The least time a step of these (start, tokens, wants logits) entries can take: the larger of its
    flops over the tensor peak and the bytes it must read over the copy bandwidth."""
    tokens = sum(n for _, n, _ in scheduled)
    rows = sum(1 for _, _, w in scheduled if w)
    flops = 2 * tokens * layer_param_count(c, layers) + 2 * rows * c["hidden_size"] * c["vocab_size"]
    nbytes = 2 * (layer_param_count(c, layers) + c["hidden_size"] * c["vocab_size"])
    for start, n, _ in scheduled:
        # token i of the portion sees start + i + 1 keys; the keys are read once per portion
        flops += layers * 4 * c["head_dim"] * c["num_attention_heads"] * (n * start + n * (n + 1) // 2)
        nbytes += (start + n) * kv_bytes_per_token(c, layers)
    return max(flops / (pk["bf16_tflops"] * 1e12), nbytes / (pk["hbm_gbs"] * 1e9))


def write_config(cfg):
    d = tempfile.mkdtemp(prefix="rllm_bench_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    return d


# -- a serving workload through the entry point -------------------------------------------------------------
def run_workload(cfg, prompts, params, pk, windows, warm_prompts, **llm_kw):
    """All requests are added at once and stepped until none is left.  A workload of the same shape with
    other tokens (``warm_prompts``) runs once untimed first (graphs are captured, libraries warmed, and
    nothing of the timed prompts is in the prefix cache), then the workload itself three times, each timed
    by the host's clock with the prefix cache emptied in between; the pass with the median wall time is
    reported."""
    import torch

    from rllm_b200 import LLM
    layers = cfg["num_hidden_layers"]
    t0 = time.time()
    llm = LLM(write_config(cfg), dtype="bf16", random_weights=True, seed=0, draw_on_device=True,
              block_size=BLOCK_SIZE, **llm_kw)
    load_s = time.time() - t0
    eng = llm.engine
    results = []
    for timed in (False, True, True, True):
        before = dict(eng.stats())
        floor = 0.0
        n_out = n_prompt_steps = 0
        prompt_tokens = prompt_time = 0.0
        torch.cuda.synchronize()
        a_wall = time.time()
        a = time.perf_counter()
        for p, sp in zip(prompts if timed else warm_prompts, params):
            llm.add_request(p, sp)
        while llm.has_work():
            t_step = time.perf_counter()
            outs = llm.step()
            sched = eng.last_schedule
            n_out += len(outs)
            if sched is not None and sched.scheduled:
                floor += step_floor_seconds(cfg, layers, [(s.start, s.num_tokens, s.want_logits)
                                                          for s in sched.scheduled], pk)
                if sched.num_prefill_tokens:
                    # a step with prompt tokens is never launched ahead: its host time is its own
                    torch.cuda.synchronize()
                    prompt_time += time.perf_counter() - t_step
                    prompt_tokens += sched.num_prefill_tokens
                    n_prompt_steps += 1
        torch.cuda.synchronize()
        wall = time.perf_counter() - a
        eng.runner.check_errors()
        if timed:
            windows.append((a_wall, time.time()))
            st = eng.stats()
            results.append({
                "wall_s": round(wall, 4), "requests": len(prompts), "generated_tokens": n_out,
                "prompt_tokens": sum(len(p) for p in prompts),
                "output_tok_s": round(n_out / wall, 1),
                "total_tok_s": round((n_out + prompt_tokens) / wall, 1),
                "prefill_tok_s": round(prompt_tokens / prompt_time, 1) if prompt_time else None,
                "prompt_tokens_computed": int(prompt_tokens), "steps": st["num_steps"] - before["num_steps"],
                "steps_with_prompt_tokens": n_prompt_steps,
                "preemptions": st["num_preemptions"] - before["num_preemptions"],
                "prefix_hit_tokens": st["prefix_hit_tokens"] - before["prefix_hit_tokens"],
                "steps_launched_ahead": st["num_steps_ahead"] - before["num_steps_ahead"],
                "roofline_frac": round(floor / wall, 4), "cache_pages": eng.num_pages[0],
                "layers": layers, "load_s": round(load_s, 1),
            })
            # the prompts of this pass must not be found in the prefix cache by the next one
            if eng.cache.prefix_caching:
                eng.cache.reset_prefix_cache()
    results.sort(key=lambda r: r["wall_s"])
    result = dict(results[len(results) // 2], timed_passes=len(results),
                  wall_s_all=" ".join(str(r["wall_s"]) for r in results))
    del llm, eng
    import gc
    gc.collect()
    torch.cuda.empty_cache()
    return result


# -- a stand-in for the missing reference arm: the same model through library operators only --------------
def library_standin(cfg, batches, prompt_len, steps, warm, windows):
    """The reference cannot be built here (no Rust toolchain), so nothing of this engine can be compared with
    it.  This is NOT the reference: it is the same Llama shape written with PyTorch's library operators
    alone (torch.mm -> cuBLAS, scaled_dot_product_attention, rms_norm, silu), random weights, a contiguous
    key/value cache of exactly the context (no paging, no scheduler), greedy decoding captured in one CUDA
    graph a batch size, timed with CUDA events like ``value``.  It says what stock library kernels reach on
    this GPU for the same arithmetic; none of this engine's code runs in it."""
    import torch
    import torch.nn.functional as F
    dev = torch.device("cuda:0")
    L, H, I = cfg["num_hidden_layers"], cfg["hidden_size"], cfg["intermediate_size"]
    nq, nkv, d, V = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"], cfg["vocab_size"]
    eps = cfg["rms_norm_eps"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *shape: (torch.randn(*shape, generator=g, device=dev) * 0.02).bfloat16()
    emb = rnd(V, H)
    layers = [dict(qkv=rnd((nq + 2 * nkv) * d, H), o=rnd(H, nq * d), gu=rnd(2 * I, H), down=rnd(H, I),
                   n1=torch.ones(H, device=dev, dtype=torch.bfloat16), n2=torch.ones(H, device=dev, dtype=torch.bfloat16))
              for _ in range(L)]
    nf = torch.ones(H, device=dev, dtype=torch.bfloat16)
    inv = 1.0 / (cfg["rope_theta"] ** (torch.arange(0, d, 2, device=dev, dtype=torch.float32) / d))

    def rope(x, pos):                                  # x [B, T, heads, d], pos [B, T]
        ang = pos[..., None].float() * inv
        cos, sin = ang.cos()[:, :, None, :], ang.sin()[:, :, None, :]
        a, b = x[..., : d // 2].float(), x[..., d // 2:].float()
        return torch.cat([a * cos - b * sin, b * cos + a * sin], dim=-1).to(x.dtype)

    def forward(ids, pos, kc, vc, causal):
        """ids, pos [B, T]; kc, vc: per layer [B, nkv, C, d]; the T tokens sit at positions pos."""
        B, T = ids.shape
        x = emb[ids]
        for w, k_l, v_l in zip(layers, kc, vc):
            h = F.rms_norm(x, (H,), w["n1"], eps)
            qkv = (h.view(B * T, H) @ w["qkv"].t()).view(B, T, nq + 2 * nkv, d)
            q, k, v = rope(qkv[:, :, :nq], pos), rope(qkv[:, :, nq:nq + nkv], pos), qkv[:, :, nq + nkv:]
            idx = pos[:, None, :, None].expand(B, nkv, T, d)
            k_l.scatter_(2, idx, k.transpose(1, 2))
            v_l.scatter_(2, idx, v.transpose(1, 2))
            if causal:
                att = F.scaled_dot_product_attention(q.transpose(1, 2), k.transpose(1, 2), v.transpose(1, 2),
                                                     is_causal=True, enable_gqa=True)
            else:
                att = F.scaled_dot_product_attention(q.transpose(1, 2), k_l, v_l, enable_gqa=True)
            x = x + (att.transpose(1, 2).reshape(B * T, nq * d) @ w["o"].t()).view(B, T, H)
            h = F.rms_norm(x, (H,), w["n2"], eps)
            gu = h.view(B * T, H) @ w["gu"].t()
            x = x + ((F.silu(gu[:, :I]) * gu[:, I:]) @ w["down"].t()).view(B, T, H)
        last = F.rms_norm(x[:, -1], (H,), nf, eps)
        return (last @ emb.t()).float().argmax(dim=-1)

    out = {"what": "PyTorch library operators only (cuBLAS, SDPA), contiguous cache, CUDA graph; not the reference"}
    with torch.no_grad():
        for B in batches:
            C = prompt_len + warm + steps                 # the cache holds exactly what the run needs
            kc = [torch.randn(B, nkv, C, d, device=dev).bfloat16() for _ in range(L)]
            vc = [torch.randn(B, nkv, C, d, device=dev).bfloat16() for _ in range(L)]
            ids = torch.randint(0, V, (B, 1), device=dev)
            pos = torch.full((B, 1), prompt_len, device=dev, dtype=torch.long)

            def step():
                nxt = forward(ids, pos, kc, vc, causal=False)
                ids.copy_(nxt[:, None])
            # every step attends over the whole cache (a few more keys than the engine's sequences hold on
            # average: C against prompt_len + warm + steps / 2)
            side = torch.cuda.Stream()
            with torch.cuda.stream(side):
                for _ in range(3):
                    step()
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                step()
            for _ in range(warm):
                graph.replay()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a = time.time()
            e0.record()
            for _ in range(steps):
                graph.replay()
            e1.record()
            torch.cuda.synchronize()
            windows.append((a, time.time()))
            out[f"decode_b{B}"] = round(B * steps / (e0.elapsed_time(e1) / 1e3), 1)
            del kc, vc, graph
            torch.cuda.empty_cache()
        T = PREFILL_TOKENS
        kc = [torch.zeros(1, nkv, T, d, device=dev, dtype=torch.bfloat16) for _ in range(L)]
        vc = [torch.zeros(1, nkv, T, d, device=dev, dtype=torch.bfloat16) for _ in range(L)]
        ids = torch.randint(0, V, (1, T), device=dev)
        pos = torch.arange(T, device=dev)[None]
        for _ in range(3):
            forward(ids, pos, kc, vc, causal=True)
        evs = [torch.cuda.Event(enable_timing=True) for _ in range(6)]
        torch.cuda.synchronize()
        a = time.time()
        for i in range(5):
            evs[i].record()
            forward(ids, pos, kc, vc, causal=True)
        evs[5].record()
        torch.cuda.synchronize()
        windows.append((a, time.time()))
        ms = min(evs[i].elapsed_time(evs[i + 1]) for i in range(5))
        out["prefill_tok_s"] = round(T / (ms / 1e3), 1)
        out["prefill_ms"] = round(ms, 3)
    del emb, layers, kc, vc
    torch.cuda.empty_cache()
    return out


def workload_3b(pk, windows):
    """32 requests, prompts uniform in [128, 4096], at most 4,096 tokens a step with
    chunked prefill, 128 tokens each at temperature 0.8, context 8,192."""
    import numpy as np

    from rllm_b200 import SamplingParams
    rng = np.random.default_rng(3)
    lengths = rng.integers(128, 4097, size=32)
    prompts = [[int(t) for t in rng.integers(0, 128256, size=int(n))] for n in lengths]
    warm = [[int(t) for t in rng.integers(0, 128256, size=int(n))] for n in lengths]
    params = [SamplingParams(temperature=0.8, seed=1000 + i, max_tokens=128, ignore_eos=True) for i in range(32)]
    return run_workload(LLAMA_3B, prompts, params, pk, windows, warm, max_model_len=8192, max_num_seqs=32,
                        max_num_batched_tokens=4096, long_prefill_token_threshold=4096,
                        enable_prefix_caching=False)


def workload_8b(pk, windows):
    """16 requests that share a 1,024-token prefix, followed by suffixes of 256 to
    2,048 tokens of their own; 512-token portions beside decoded tokens; 256 greedy tokens each; context 8,192;
    prefix caching on."""
    import numpy as np

    from rllm_b200 import SamplingParams
    rng = np.random.default_rng(4)
    lengths = rng.integers(256, 2049, size=16)
    shared, shared_warm = ([int(t) for t in rng.integers(0, 128256, size=1024)] for _ in range(2))
    prompts = [shared + [int(t) for t in rng.integers(0, 128256, size=int(n))] for n in lengths]
    warm = [shared_warm + [int(t) for t in rng.integers(0, 128256, size=int(n))] for n in lengths]
    params = [SamplingParams(temperature=0.0, max_tokens=256, ignore_eos=True) for _ in range(16)]
    return run_workload(LLAMA_8B, prompts, params, pk, windows, warm, max_model_len=8192, max_num_seqs=16,
                        max_num_batched_tokens=4096, long_prefill_token_threshold=512,
                        enable_prefix_caching=True)


# -- two designs side by side: Fasulix and the Llama of equal size ------------------------------------------
def fasulix(layers, width, heads, dim, rot, vdim, q_rank, kv_rank, gru, experts, top, ff, window, vocab):
    """layers of the pattern [latent attention with sink, minGRU, windowed latent attention, minGRU]."""
    def latent(kind):
        m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "rot": {"base": 500000.0, "dims": rot}, "scale": (dim + rot) ** -0.5}
        if kind == "latent_attention_2":
            m["mask"] = {"size": window}
        return m
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": 7.0}, "router": {"experts": experts, "top": top}}
    kinds = ["latent_attention", "mingru", "latent_attention_2", "mingru"]
    return {"architecture": "Fasulix", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "max_positions": 8192,
            "layers": [{"type": kinds[i % 4], "mlp": mlp,
                        "mixer": {"width": gru} if kinds[i % 4] == "mingru" else latent(kinds[i % 4])}
                       for i in range(layers)]}


def fevolorn(layers, width, streams, lheads, ldim, lvdim, heads, kv_heads, dim, vdim, window, inner, state, dt_rank,
             experts, top, ff, shared, dense, vocab):
    """layers of the pattern [lightning + dense, parallel + experts, lightning + experts, parallel + experts]."""
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": 2.0},
           "shared": {"ff": shared}}
    lightning = {"heads": lheads, "dim": ldim, "vdim": lvdim,
                 "decay": [1.0 - 2.0 ** (-5.0 - 3.0 * h / max(1, lheads - 1)) for h in range(lheads)]}
    parallel = {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5,
                         "mask": {"size": window}},
                "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": 4}}
    kinds = ["lightning", "parallel", "lightning", "parallel"]
    return {"architecture": "Fevolorn", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0}, "max_positions": 8192,
            "layers": [{"type": kinds[i % 4], "mixer": lightning if kinds[i % 4] == "lightning" else parallel,
                        "mlp": {"kind": "dense", "ff": dense} if i % 4 == 0 else moe} for i in range(layers)]}


# (name, Fasulix sizes, the Llama beside it: same width, layers, heads and vocabulary, head size dim + rot,
#  an intermediate size of top * ff, so that a token multiplies as many feed-forward weights)
DESIGN_SIZES = [
    ("w1024", dict(layers=4, width=1024, heads=8, dim=64, rot=32, vdim=64, q_rank=384, kv_rank=256, gru=1024,
                   experts=16, top=2, ff=1024, window=512, vocab=32768),
     dict(layers=4, hidden=1024, heads=16, kv_heads=4, head_dim=64, inter=2048)),
    ("w2048", dict(layers=4, width=2048, heads=16, dim=128, rot=64, vdim=128, q_rank=768, kv_rank=512, gru=2048,
                   experts=32, top=4, ff=1024, window=1024, vocab=32768),
     dict(layers=4, hidden=2048, heads=16, kv_heads=4, head_dim=128, inter=4096)),
]


# Fevolorn beside Fasulix (the closest design: recurrences, windowed attention and routed experts in one stack) of
# equal width, layers, vocabulary, experts and expert width, and the Llama of that width.  w1024 keeps the
# design's own head shape (values twice as wide as keys), w2048 has keys and values of one size.
FEVOLORN_SIZES = {
    "w1024": dict(layers=4, width=1024, streams=4, lheads=8, ldim=64, lvdim=128, heads=16, kv_heads=4, dim=64,
                  vdim=128, window=512, inner=2048, state=16, dt_rank=64, experts=16, top=2, ff=1024, shared=1024,
                  dense=2048, vocab=32768),
    "w2048": dict(layers=4, width=2048, streams=4, lheads=16, ldim=128, lvdim=128, heads=16, kv_heads=4, dim=128,
                  vdim=128, window=1024, inner=4096, state=16, dt_rank=128, experts=32, top=4, ff=1024, shared=2048,
                  dense=4096, vocab=32768),
}


def munupel(layers, width, heads, kv_heads, dim, window, keep, chunk, cap, ff, vocab):
    """layers of the pattern [window with kept first tokens and sinks, chunked with capped scores and biases]:
    parallel-residual layers of one layer norm, gated attention and a dense feed-forward."""
    rot = {"base": 1000000.0, "dims": dim // 2}
    win = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
           "mask": {"size": window, "keep_first": keep}, "rot": rot}
    chk = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "softcap": cap,
           "mask": {"size": chunk},
           "rot": dict(rot, scaling={"factor": 8.0, "original": 2048, "fast": 16.0, "slow": 2.0})}
    return {"architecture": "Munupel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "max_positions": 8192,
            "layers": [{"type": "attention_2" if i % 2 == 0 else "attention", "mixer": win if i % 2 == 0 else chk,
                        "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)]}


# Munupel beside the Llama (the closest design: grouped-query attention over pages, a SiLU-gated dense
# feed-forward) of equal width, layers, heads, head size, feed-forward width and vocabulary.  The Llama sees
# every earlier key; Munupel's layers see a window beside four kept tokens, or their chunk.
MUNUPEL_SIZES = {
    "w1024": dict(layers=4, width=1024, heads=16, kv_heads=4, dim=64, window=512, keep=4, chunk=1024, cap=50.0,
                  ff=2048, vocab=32768),
    "w2048": dict(layers=4, width=2048, heads=16, kv_heads=4, dim=128, window=1024, keep=4, chunk=1024, cap=50.0,
                  ff=4096, vocab=32768),
}


def tibelix(layers, width, mheads, mdim, mvdim, heads, kv_heads, dim, lheads, ldim, lrot, lvdim, q_rank, kv_rank,
            experts, top, groups, keep, ff, shared, dense, vocab):
    """layers of the pattern [mLSTM + dense, attention + experts, latent attention + experts, attention that
    reads the second layer's keys and values + experts]: sandwich layers (a norm before and after each sublayer)."""
    moe = {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
           "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
           "q_temp": {"coef": 0.4, "every": 128}}
    lat = {"heads": lheads, "dim": ldim, "rot_dim": lrot, "vdim": lvdim, "q_rank": q_rank, "kv_rank": kv_rank,
           "scale": (ldim + lrot) ** -0.5,
           "rot": {"base": 500000.0, "dims": lrot, "scaling": {"factor": 4.0, "original": 4096, "fast": 16.0, "slow": 2.0}}}
    out = []
    for i in range(layers):
        k = i % 4
        if k == 0:
            out.append({"type": "mlstm", "mixer": {"heads": mheads, "dim": mdim, "vdim": mvdim, "gate_cap": 12.0},
                        "mlp": {"kind": "dense", "ff": dense}})
        elif k == 2:
            out.append({"type": "latent_attention", "mixer": lat, "mlp": moe})
        else:
            out.append({"type": "attention", "mixer": dict(att, kv_from=i - 2) if k == 3 else att, "mlp": moe})
    return {"architecture": "Tibelix", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "max_positions": 8192,
            "layers": out}


# Tibelix beside Fasulix (the closest design: latent attention, a recurrence with state slots and routed experts
# in layers with a norm before and after each sublayer) of equal width, layers, vocabulary, experts and expert
# width, and the Llama of that width.
TIBELIX_SIZES = {
    "w1024": dict(layers=4, width=1024, mheads=8, mdim=64, mvdim=128, heads=16, kv_heads=4, dim=64, lheads=8, ldim=64,
                  lrot=32, lvdim=64, q_rank=384, kv_rank=256, experts=16, top=2, groups=4, keep=2, ff=1024, shared=1024,
                  dense=2048, vocab=32768),
    "w2048": dict(layers=4, width=2048, mheads=8, mdim=128, mvdim=256, heads=16, kv_heads=4, dim=128, lheads=16,
                  ldim=128, lrot=64, lvdim=128, q_rank=768, kv_rank=512, experts=32, top=4, groups=8, keep=4, ff=1024,
                  shared=2048, dense=4096, vocab=32768),
}


def biranex(layers, width, dheads, ddim, dvdim, rank, heads, kv_heads, dim, window, sheads, sdim, state, groups, ff, vocab):
    """layers of the pattern [gated delta rule, parallel (windowed attention beside a state-space recurrence) +
    dense]: post-norm layers.  ``rank`` is not written: the random weights draw the low-rank pairs with the head's size."""
    assert rank == ddim
    delta = {"heads": dheads, "kv_heads": dheads, "dim": ddim, "vdim": dvdim, "conv": 4}
    par = {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
                    "mask": {"size": window}, "rot": {"base": 500000.0, "dims": dim // 2, "scaling": {"factor": 4.0}}},
           "left_scale": 0.9, "right_scale": 0.6,
           "right": {"heads": sheads, "vdim": sdim, "state": state, "groups": groups, "conv": 4, "norm_groups": groups}}
    return {"architecture": "Biranex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 0.8,
            "max_positions": 8192,
            "layers": [{"type": "channel_delta", "mixer": delta, "mlp": None} if i % 2 == 0 else
                       {"type": "parallel", "mixer": par, "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)]}


# Biranex beside Fevolorn (the closest design: linear-attention layers with a matrix state, and windowed attention
# beside a state-space recurrence) of equal width, layers, vocabulary, attention and matrix-state sizes, and the
# Llama of that width.  The state-space part has eight times Fevolorn's state a channel (128 against 16).
BIRANEX_SIZES = {
    "w1024": dict(layers=4, width=1024, dheads=8, ddim=64, dvdim=128, rank=64, heads=16, kv_heads=4, dim=64, window=512,
                  sheads=32, sdim=64, state=128, groups=1, ff=2048, vocab=32768),
    "w2048": dict(layers=4, width=2048, dheads=16, ddim=128, dvdim=128, rank=128, heads=16, kv_heads=4, dim=128,
                  window=1024, sheads=64, sdim=64, state=128, groups=2, ff=4096, vocab=32768),
}


def bikovik(layers, width, sheads, sdim, svdim, heads, kv_heads, dim, window, keep, ff, vocab):
    """layers of the pattern [hgrn2, attention, retention, attention], each with a clamped dense feed-forward."""
    rot = {"base": 500000.0, "dims": dim // 2}
    state = {"heads": sheads, "dim": sdim, "vdim": svdim}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "rot": rot, "v_mix": True,
           "mask": {"size": window, "keep_first": keep}}
    ret = dict(state, decay=[1.0 - 2.0 ** -(5 + 4.0 * h / sheads) for h in range(sheads)], rot={"base": 10000.0, "dims": sdim})
    kinds = [("hgrn2", state), ("attention", att), ("retention", ret), ("attention", att)]
    return {"architecture": "Bikovik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 2.0},
            "logit_softcap": 20.0, "max_positions": 8192,
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}}
                       for i in range(layers)]}


# Bikovik beside Biranex (the closest dense design: layers with a matrix state, and windowed attention) of equal width,
# layers, vocabulary, attention and matrix-state sizes, and the Llama of that width.
BIKOVIK_SIZES = {
    "w1024": dict(layers=4, width=1024, sheads=8, sdim=64, svdim=128, heads=16, kv_heads=4, dim=64, window=512, keep=4,
                  ff=2048, vocab=32768),
    "w2048": dict(layers=4, width=2048, sheads=16, sdim=128, svdim=128, heads=16, kv_heads=4, dim=128, window=1024, keep=4,
                  ff=4096, vocab=32768),
}


def compare_designs(args):
    """Prefill and decode throughput of Fasulix at sizes that resemble a real model's layers (random weights)
    beside the Llama of equal size, through the same step function; and, from one eager prefill step and one
    eager decode step of each, the device time of every kernel of the step by entry point, with what the
    kernel has to move or multiply at the least, as a fraction of the measured peaks."""
    import numpy as np
    import torch

    from rllm_b200 import LLM
    from rllm_b200.engine.runner import StepEntry
    from rllm_b200.kernels import ops

    pk = peaks()
    T, B, CTX, K, W = args.prompt_len, args.batch, args.prompt_len, min(args.steps, 64), max(3, args.warmup)
    clocks = ClockSampler()
    clocks.start()
    windows, rows = [], []
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def roofline(name, a, kw, shape):
        """(flops, bytes) a call has to do at the least, from its arguments; None: not modelled."""
        S, ctx, Tn = shape["seqs"], shape["ctx"], shape["tokens"]
        pairs = sum(min(p + 1, shape.get("window") or p + 1) for p in range(ctx - Tn // S, ctx)) * S

        def seen(window, keep, chunk):
            """(query-key pairs, keys that have to be read) of the step under a mask."""
            def lo(p):
                a = max(0, p - window + 1) if window else 0
                return max(a, p // chunk * chunk) if chunk else a
            first = ctx - Tn // S
            vis = sum(p + 1 - lo(p) + min(keep if window else 0, lo(p)) for p in range(first, ctx)) * S
            return vis, S * (ctx - lo(first) + min(keep if window else 0, lo(first)))
        if name == "latent_attention_mma":
            q, heads, dk, dv, window = a[0], a[8], a[9], a[10], a[11]
            vis = sum(min(p + 1, window or p + 1) for p in range(ctx - Tn // S, ctx)) * S
            keys = S * min(ctx, (window or ctx) + Tn // S)
            return 2.0 * (dk + dv) * heads * vis, 2.0 * (keys * dk + q.numel() + a[1].numel())
        if name in ("attention_prefill_tcgen05", "attention_prefill_bf16", "attention_decode_bf16"):
            nq, nkv, d, window = (a[11], a[12], a[13], a[14]) if name != "attention_decode_bf16" else \
                (a[9], a[10], a[11], a[12])
            vis, keys = seen(window, kw.get("keep_first", 0), kw.get("chunk", 0))
            return 4.0 * d * nq * vis, 2.0 * (2 * keys * nkv * d + 2 * Tn * nq * d)
        if name == "layernorm":
            extra = len(kw.get("deltas", ())) * 2.0 + (4.0 if kw.get("writeback") else 0.0)
            return 0.0, a[4].numel() * (4.0 + 2.0 + extra)
        if name == "add_rows":
            return 0.0, a[0].numel() * (8.0 + 2.0 * len(a[1]))
        if name == "add_row_bias":
            return 0.0, a[0].numel() * 4.0
        if name == "moe_experts":
            h, ids, wgu = a[0], a[1], a[2]
            E, F2, H = wgu.shape
            P = ids.numel()
            used = min(E, P)
            return 2.0 * 3 * H * (F2 // 2) * P, 2.0 * (used * 3 * H * (F2 // 2) + h.numel() + P * (H + F2))
        if name == "head_gemm":
            M, heads, Kd = a[0].shape
            N = a[2].shape[2]
            return 2.0 * M * heads * Kd * N, 2.0 * (a[0].numel() + a[1].numel() + M * heads * N)
        if name == "mingru_scan":
            return 0.0, 2.0 * (a[0].numel() + a[7].numel())
        if name == "lightning_scan":
            heads, d, dv = a[4].shape[1:]
            return 0.0, a[0].shape[0] * heads * (4.0 * d + 2.0 * dv + 4.0 * dv) + 8.0 * S * heads * d * dv
        if name == "selective_scan":
            return 0.0, a[0].numel() * 10.0 + 8.0 * S * a[9].shape[1] * a[9].shape[2]
        if name == "causal_conv":
            return 0.0, a[0].numel() * 4.0
        if name == "streams_read":
            return 0.0, a[0].numel() * 4.0 + a[0][0].numel() * 2.0
        if name == "streams_write":
            return 0.0, a[0].numel() * 8.0 + a[0][0].numel() * 4.0
        if name in ("head_norm_kv_write", "act_mul", "act", "sigmoid_gate"):
            return 0.0, 4.0 * a[0].numel()
        if name == "mlstm_scan":
            heads, d, dv = a[12], a[13], a[14]
            # q, k, v in, o out (float32), the gates; the state once in and once out per sequence
            return 4.0 * a[0].shape[0] * heads * d * dv, a[0].shape[0] * heads * (4.0 * d + 2.0 * dv + 4.0 * dv + 8.0) + \
                8.0 * S * heads * (d * dv + d + 1)
        if name == "postnorm_add":
            terms = 1 if isinstance(a[1], torch.Tensor) else 2
            return 0.0, a[0].numel() * (8.0 + 2.0 + 2.0 * terms)
        if name == "ssd_scan":
            heads, n, p = a[9], a[11], a[12]
            # x, B, C and the steps in, y out (float32); the state once in and once out per sequence
            return 4.0 * a[0].shape[0] * heads * n * p, 2.0 * a[0].numel() + 4.0 * a[0].shape[0] * heads * (p + 1) + \
                8.0 * S * heads * n * p
        if name == "silu_gated_group_rmsnorm":
            return 0.0, 8.0 * a[0].numel()
        if name == "channel_delta_step":
            heads, d, dv = a[12], a[14], a[15]
            # the second low-rank products' weights and beta's, the token's rows; the state in and out
            return 0.0, 2.0 * (a[0].numel() + sum(a[3][k].numel() for k in ("b", "a2", "g2"))) + 8.0 * S * heads * d * dv
        if name == "channel_delta_scan":
            heads, d, dv = a[10], a[12], a[13]
            # the convolutions' results, the decays' steps and beta in, o out (float32); the state in and out
            return 6.0 * a[0].shape[0] * heads * d * dv, 2.0 * a[0].numel() + 4.0 * (a[1].numel() + a[2].numel()) + \
                4.0 * a[0].shape[0] * heads * dv + 8.0 * S * heads * d * dv
        if name == "linear_state_scan":
            heads, d, dv = a[1].shape[1:]
            # a token's projections in, its results out; the state in and out
            return 4.0 * a[0].shape[0] * heads * d * dv, 2.0 * a[0].numel() + 2.0 * a[0].shape[0] * heads * dv + \
                8.0 * S * heads * d * dv
        if name in ("shared_key_attention_tcgen05", "shared_key_attention_mma"):
            nq, nkv, dv, window, keep = a[9:14] if name == "shared_key_attention_mma" else a[10:15]
            dk = a[2].shape[3] // nkv
            vis, keys = seen(window, keep, 0)
            # the heads' scores, their mixture, the values: less than what is issued (every head against the whole row)
            return 2.0 * (dk + nq + dv) * nq * vis, 2.0 * (keys * nkv * (dk + dv) + Tn * nq * (dk + dv))
        if name == "talking_prep":
            return 0.0, 2.0 * (a[0].numel() + Tn * (a[10] + 1) * a[8].shape[3] + Tn * a[9].shape[3])
        if name == "dyt":
            return 0.0, a[4].numel() * (8.0 if kw.get("delta") is None else 14.0)
        if name == "softcap_rows":
            return 0.0, 8.0 * a[0].numel()
        if name == "head_gated_rmsnorm":
            return 0.0, 8.0 * a[0].numel()
        if name in ("rms_mean2", "gated_rmsnorm"):
            return 0.0, 6.0 * a[0].numel()
        if name == "attention_simt_kv":
            dk, dv, nq, nkv, window = a[3].shape[3], a[4].shape[3], a[8], a[9], a[10]
            vis, keys = seen(window, kw.get("keep_first", 0), kw.get("chunk", 0))
            return 2.0 * (dk + dv) * nq * vis, 2.0 * (keys * nkv * (dk + dv) + Tn * nq * (dk + dv))
        if name == "gated_postnorm_add":
            return 0.0, 8.0 * a[0].numel() + 2.0 * (a[2].numel() + (2 * a[3].numel() if a[3] is not None else a[0].numel()))
        if name == "depth_average":
            return 0.0, 4.0 * a[1] * a[0][0].numel() + 6.0 * a[0][0].numel()
        if name == "rmsnorm":
            return 0.0, a[3].numel() * 10.0
        if name == "silu_mul":
            return 0.0, a[1].numel() * 6.0
        if name in ("latent_prep", "latent_q_rot", "moe_route", "rope_kv_write"):
            return 0.0, 4.0 * a[0].numel()
        if name in ("gemm_tcgen05", "gemm_small_m", "gemm_small_m_rstd", "gemm_small_m_residual"):
            x, w = (a[0], a[1]) if name != "gemm_small_m_rstd" else (a[0], a[3])
            rows_out = w.shape[0] // 2 if (len(a) > 3 and a[-1] == "silu_mul") else w.shape[0]
            return 2.0 * x.shape[0] * x.shape[1] * w.shape[0], 2.0 * (x.numel() + w.numel() + x.shape[0] * rows_out)
        return None

    def kernel_table(runner, entries, shape):
        """One eager step with CUDA events around every entry point of ``ops`` (L2 flushed before the step)."""
        names = [n for n in dir(ops) if callable(getattr(ops, n)) and n in (
            "latent_attention_mma", "attention_prefill_tcgen05", "attention_prefill_bf16", "attention_decode_bf16",
            "moe_experts", "moe_route", "head_gemm", "mingru_scan", "gated_postnorm_add", "depth_average", "rmsnorm",
            "silu_mul", "latent_prep", "latent_q_rot", "rope_kv_write", "gemm_small_m", "moe_choose", "gemm_small_m_residual",
            "gemm_small_m_rstd", "gemm_tcgen05", "embedding", "lightning_scan", "selective_scan", "causal_conv",
            "streams_read", "streams_write", "head_norm_kv_write", "attention_simt_kv", "rms_mean2", "gated_rmsnorm",
            "act_mul", "moe_choose_sigmoid", "weighted_slot_sum", "layernorm", "add_rows", "add_row_bias", "mlstm_scan",
            "head_gated_rmsnorm", "act", "sigmoid_gate", "postnorm_add", "ssd_scan", "silu_gated_group_rmsnorm",
            "channel_delta_scan", "channel_delta_step", "activation_rows", "linear_state_scan", "talking_prep", "dyt",
            "shared_key_attention_tcgen05", "shared_key_attention_mma", "softcap_rows")]
        saved, log = {}, []

        def wrap(name, fn):
            def timed(*a, **kw):
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                out = fn(*a, **kw)
                e1.record()
                log.append((name, e0, e1, roofline(name, a, kw, shape)))
                return out
            return timed
        mm = torch.mm

        def timed_mm(x, w, **kw):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            out = mm(x, w, **kw)
            e1.record()
            log.append(("library_mm", e0, e1, (2.0 * x.shape[0] * x.shape[1] * w.shape[1],
                                               2.0 * (x.numel() + w.numel() + x.shape[0] * w.shape[1]))))
            return out
        for n in names:
            saved[n] = getattr(ops, n)
            setattr(ops, n, wrap(n, saved[n]))
        torch.mm = timed_mm
        was = runner.capture_graphs
        runner.capture_graphs = False
        try:
            runner.step(entries)               # every kernel of the step has run once (module loading, first-call setup)
            torch.cuda.synchronize()
            log.clear()
            flush.zero_()
            runner.step(entries)
            torch.cuda.synchronize()
        finally:
            runner.capture_graphs = was
            torch.mm = mm
            for n, f in saved.items():
                setattr(ops, n, f)
        agg = {}
        for name, e0, e1, need in log:
            ms = e0.elapsed_time(e1)
            a = agg.setdefault(name, [0, 0.0, 0.0, 0.0])
            a[0] += 1
            a[1] += ms
            if need is not None:
                a[2] += need[0]
                a[3] += need[1]
        out = {}
        for name, (n, ms, fl, by) in sorted(agg.items(), key=lambda kv: -kv[1][1]):
            floor_ms = max(fl / (pk["bf16_tflops"] * 1e12), by / (pk["hbm_gbs"] * 1e9)) * 1e3
            out[name] = {"calls": n, "ms": round(ms, 4), "of_roofline": round(floor_ms / ms, 3) if floor_ms else None,
                         "bound": "compute" if fl / (pk["bf16_tflops"] * 1e12) > by / (pk["hbm_gbs"] * 1e9) else "memory"}
        return out

    def measure(label, cfg):
        d = write_config(cfg)
        pages = (B + 1) * (-(-(CTX + K + W + 8) // BLOCK_SIZE) + 2) + 64
        llm = LLM(d, dtype="bf16", max_model_len=CTX + K + W + 8, max_num_seqs=B + 1, max_num_batched_tokens=8192,
                  long_prefill_token_threshold=8192, block_size=BLOCK_SIZE, num_gpu_blocks=pages,
                  enable_prefix_caching=False, random_weights=True, seed=0, draw_on_device=True)
        eng, runner = llm.engine, llm.engine.runner
        vocab = eng.model.spec.vocab_size
        rng = np.random.default_rng(0)
        toks = lambda n: [int(t) for t in rng.integers(0, vocab, size=n)]
        # prefill: whole prompts of T tokens, one a step, timed on the device
        ms_all = []
        a = time.time()
        for i in range(W + 5):
            eng.cache.admit("p")
            assert eng.cache.ensure("p", 0, T)
            entries = [StepEntry("p", toks(T), 0, [T - 1])]
            flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            runner.step(entries)
            e1.record()
            torch.cuda.synchronize()
            if i >= W:
                ms_all.append(e0.elapsed_time(e1))
            if i == W + 4:
                eng.cache.free("p")
                eng.cache.admit("p")
                assert eng.cache.ensure("p", 0, T)
                table_p = kernel_table(runner, [StepEntry("p", toks(T), 0, [T - 1])],
                                       {"seqs": 1, "ctx": T, "tokens": T})
            eng.cache.free("p")
        prefill_ms = sorted(ms_all)[len(ms_all) // 2]
        # decode: B sequences that hold CTX tokens each
        ids = [f"d{i}" for i in range(B)]
        for i in ids:
            eng.cache.admit(i)
            assert eng.cache.ensure(i, 0, CTX + K + W + 2)
        per = max(1, 8192 // CTX)
        for x in range(0, B, per):
            runner.step([StepEntry(i, toks(CTX), 0, []) for i in ids[x:x + per]])
        entries = [StepEntry(i, toks(1), CTX, [0]) for i in ids]
        table_d = kernel_table(runner, entries, {"seqs": B, "ctx": CTX + 1, "tokens": B})
        entries = [StepEntry(i, toks(1), CTX + 1, [0]) for i in ids]
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        runner.greedy_decode_run(entries, W + K, timing=(W, e0, e1))
        torch.cuda.synchronize()
        windows.append((a, time.time()))
        decode_ms = e0.elapsed_time(e1) / K
        runner.check_errors()
        for i in ids:
            eng.cache.free(i)
        res = {"design": label, "weights_gb": round(eng.model.num_weight_bytes() / 1e9, 3),
               "prefill_tok_s": round(T / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
               "decode_tok_s": round(B / (decode_ms / 1e3), 1), "decode_ms_per_step": round(decode_ms, 4),
               "kernels_prefill": table_p, "kernels_decode": table_d}
        del llm, eng, runner
        torch.cuda.empty_cache()
        return res

    for name, fx, ll in DESIGN_SIZES:
        if args.design_size and name != args.design_size:
            continue
        row = {"size": name}
        if args.design == "fevolorn":
            row["fevolorn"] = measure("fevolorn", fevolorn(**FEVOLORN_SIZES[name]))
        if args.design == "tibelix":
            row["tibelix"] = measure("tibelix", tibelix(**TIBELIX_SIZES[name]))
        if args.design == "biranex":
            row["biranex"] = measure("biranex", biranex(**BIRANEX_SIZES[name]))
            row["fevolorn"] = measure("fevolorn", fevolorn(**FEVOLORN_SIZES[name]))
        elif args.design == "bikovik":
            row["bikovik"] = measure("bikovik", bikovik(**BIKOVIK_SIZES[name]))
            row["biranex"] = measure("biranex", biranex(**BIRANEX_SIZES[name]))
        elif args.design == "munupel":
            row["munupel"] = measure("munupel", munupel(**MUNUPEL_SIZES[name]))
        else:
            row["fasulix"] = measure("fasulix", fasulix(**fx))
        cfg = llama(ll["layers"], ll["hidden"], ll["heads"], ll["kv_heads"], ll["head_dim"], ll["inter"], 32.0, True)
        cfg["vocab_size"] = fx["vocab"]
        row["llama"] = measure("llama", cfg)
        rows.append(row)
    clocks.stop()
    print(json.dumps({"metric": "%s_vs_llama_step_throughput" % args.design, "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16",
                      "data": "synthetic", "prompt_len": T, "decode_batch": B, "decode_context": CTX,
                      "timing": "CUDA events; prefill: median of 5 steps after warm-up, 256 MiB written between steps; "
                                "decode: %d graph steps on the device" % K,
                      "peaks": pk, "clocks": clocks.summary(windows), "sizes": rows}))
    return 0


def main():
    global SETTLE_STEPS
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=DECODE_TOKENS)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the model has (stated in config)")
    ap.add_argument("--prompt-len", type=int, default=PROMPT_LEN)
    ap.add_argument("--no-points", action="store_true", help="skip the other batch sizes and contexts")
    ap.add_argument("--no-workloads", action="store_true", help="skip the 3B and 8B serving workloads")
    ap.add_argument("--no-standin", action="store_true", help="skip the library-operator stand-in")
    ap.add_argument("--settle-steps", type=int, default=SETTLE_STEPS,
                    help="untimed decode steps of a device-timed point before its warm-up steps (0 for a short capture under a profiler)")
    ap.add_argument("--design", default=None, choices=["bikovik", "biranex", "fasulix", "fevolorn", "munupel", "tibelix"],
                    help="instead of the default workload: this design beside the Llama of equal size (prefill and "
                         "decode throughput, kernels against their rooflines)")
    ap.add_argument("--design-size", default=None, help="only this entry of the design comparison's sizes")
    args = ap.parse_args()
    SETTLE_STEPS = max(0, args.settle_steps)
    if args.design:
        return compare_designs(args)

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "rLLM is a Rust workspace (cargo, Candle and ~300 crates); no Rust toolchain and no "
                          "network here, and its paged CUDA path does not compile (paged_attention.cu:409)"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not measured")
        return 2
    K, W = args.steps, max(3, args.warmup)
    if args.prompt_len + K + W + SETTLE_STEPS + 4 > CONTEXT_LEN:
        print(f"bench.py: a prompt of {args.prompt_len} tokens and {K} + {W} steps do not fit the context of {CONTEXT_LEN}")
        return 2

    import numpy as np
    import torch

    from rllm_b200 import LLM, SamplingParams
    from rllm_b200.engine.runner import StepEntry
    from rllm_b200.kernels import ops

    cfg = dict(LLAMA_1B)
    layers = args.layers or cfg["num_hidden_layers"]
    cfg["num_hidden_layers"] = layers
    model_dir = write_config(cfg)
    max_batch = args.batch if args.no_points else max(args.batch, 64)
    pages = max_batch * (-(-CONTEXT_LEN // BLOCK_SIZE) + 2) + -(-PREFILL_TOKENS // BLOCK_SIZE) + 64
    t0 = time.time()
    llm = LLM(model_dir, dtype="bf16", max_model_len=CONTEXT_LEN, max_num_seqs=max_batch,
              max_num_batched_tokens=8192, long_prefill_token_threshold=8192, block_size=BLOCK_SIZE,
              num_gpu_blocks=pages, enable_prefix_caching=False, random_weights=True, seed=0,
              draw_on_device=True)
    load_s = time.time() - t0
    eng, runner = llm.engine, llm.engine.runner
    rng = np.random.default_rng(0)
    pk = peaks()
    clocks = ClockSampler()
    clocks.start()
    windows = []

    def e2e_point(batch, prompt_len, steps, warm):
        """Through ``LLM.step``: tokens a second, ms a step, bytes to and from the device a step."""
        prompts = [[int(t) for t in rng.integers(0, cfg["vocab_size"], size=prompt_len)] for _ in range(batch)]
        # no request may end inside the timed steps (those whose prompts are computed first decode a few
        # tokens while the others' prompts are still being computed)
        sp = SamplingParams(temperature=0.0, max_tokens=CONTEXT_LEN - prompt_len, ignore_eos=True)
        ids = [llm.add_request(p, sp) for p in prompts]
        while any(eng.scheduler.requests[i].num_computed < prompt_len for i in ids):
            llm.step()                                         # the prompts
        for _ in range(warm):
            llm.step()
        torch.cuda.synchronize()
        h2d0 = sum(g.h2d_bytes for g in runner.graphs.values())
        a = time.time()
        t_a = time.perf_counter()
        n_tok = 0
        for _ in range(steps):
            n_tok += len(llm.step())
        torch.cuda.synchronize()
        dt = time.perf_counter() - t_a
        windows.append((a, time.time()))
        assert n_tok == batch * steps, (n_tok, batch, steps)
        # host -> device: the step's positions, lengths and block tables from pinned memory, on the steps
        # where a block table changed (the token ids of a decode step are the step before's samples and
        # stay on the device); device -> host: the sampled tokens, every step, and the error words
        h2d = sum(g.h2d_bytes for g in runner.graphs.values()) - h2d0
        for i in ids:
            llm.abort_request(i)
        return {"value": n_tok / dt, "unit": "tok/s", "h2d_bytes_per_step": int(h2d / steps),
                "d2h_bytes_per_step": int(batch * 4 + 1), "ms_per_step": 1e3 * dt / steps}

    def device_point(batch, prompt_len, steps, warm):
        """(tokens a second, ms a step) timed on the device around ``steps`` steps that stay there, every
        sequence holding ``prompt_len`` tokens when they begin.  The step function is driven directly.
        SETTLE_STEPS more untimed steps come before the ``warm`` ones: right behind the prompts (tens of
        milliseconds at the power cap) the first decode steps run 3 to 6 % slower than the rest."""
        warm += SETTLE_STEPS
        ids = [f"dev{i}" for i in range(batch)]
        for i in ids:
            eng.cache.admit(i)
            assert eng.cache.ensure(i, 0, prompt_len + steps + warm + 1)
        per_step = max(1, 8192 // prompt_len)
        for a in range(0, batch, per_step):                    # the prompts, some at a time
            runner.step([StepEntry(i, [int(t) for t in rng.integers(0, cfg["vocab_size"], size=prompt_len)], 0, [])
                         for i in ids[a:a + per_step]])
        entries = [StepEntry(i, [int(rng.integers(0, cfg["vocab_size"]))], prompt_len, [0]) for i in ids]
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a = time.time()
        runner.greedy_decode_run(entries, warm + steps, timing=(warm, ev0, ev1))
        torch.cuda.synchronize()
        windows.append((a, time.time()))
        ms = ev0.elapsed_time(ev1)
        runner.check_errors()
        for i in ids:
            eng.cache.free(i)
        return batch * steps / (ms / 1e3), ms / steps

    def frac(batch, ms, ctx_mid):
        return decode_bytes(cfg, layers, batch, ctx_mid) / (ms / 1e3) / 1e9 / pk["hbm_gbs"]

    P = args.prompt_len
    ctx_mid = P + SETTLE_STEPS + W + K // 2
    e2e = e2e_point(args.batch, P, K, W)
    # three such runs, each with requests and pages of its own (where the pages lie moves the step by a few
    # per cent); the median is reported
    runs = sorted((device_point(args.batch, P, K, W) for _ in range(3)), key=lambda r: r[1])
    value, ms_step = runs[1]
    points = {}
    if not args.no_points:
        for b in (1, 64):
            pv, pms = device_point(b, P, K, W)
            pe = e2e_point(b, P, K, W)
            points[f"decode_b{b}"] = round(pv, 1)
            points[f"decode_b{b}_e2e"] = round(pe["value"], 1)
            points[f"decode_b{b}_hbm_frac"] = round(frac(b, pms, ctx_mid), 4)
        # the whole context of the configuration: sequences that end the run with 4,096 tokens
        k4 = min(K, 64)
        for b in (1, 8, 64):
            pv, pms = device_point(b, CONTEXT_LEN - (k4 + W + SETTLE_STEPS) - 4, k4, W)      # ends with 4,092 tokens
            points[f"decode_b{b}_ctx4096"] = round(pv, 1)
            points[f"decode_b{b}_ctx4096_hbm_frac"] = round(frac(b, pms, CONTEXT_LEN - 4 - k4 // 2), 4)

    # prefill of one 2,048-token prompt, device-timed
    eng.cache.admit("prefill")
    assert eng.cache.ensure("prefill", 0, PREFILL_TOKENS)
    ptoks = [int(t) for t in rng.integers(0, cfg["vocab_size"], size=PREFILL_TOKENS)]
    entry = [StepEntry("prefill", ptoks, 0, [PREFILL_TOKENS - 1])]
    for _ in range(3):
        runner.step(entry)
    n0 = ops.LAUNCHES[0]
    torch.cuda.synchronize()
    # A burst, like the peak it is divided by: the GPU rests PREFILL_IDLE_S first (right behind other work the
    # same prefill takes 4.5 to 4.9 ms instead of 4.4 under the power cap, and its time then says more about
    # what ran before it than about the prefill), then two more untimed repetitions.
    time.sleep(PREFILL_IDLE_S)
    for _ in range(2):
        runner.step(entry)
    torch.cuda.synchronize()
    n0 = ops.LAUNCHES[0]
    reps = 5
    evs = [torch.cuda.Event(enable_timing=True) for _ in range(reps + 1)]
    a = time.time()
    for i in range(reps):
        evs[i].record()
        runner.step(entry)
    evs[reps].record()
    torch.cuda.synchronize()
    windows.append((a, time.time()))
    prefill_launches = (ops.LAUNCHES[0] - n0) // reps
    p_ms = min(evs[i].elapsed_time(evs[i + 1]) for i in range(reps))
    eng.cache.free("prefill")
    pf = prefill_flops(cfg, layers, PREFILL_TOKENS)
    prefill = {"value": round(PREFILL_TOKENS / (p_ms / 1e3), 1), "tokens": PREFILL_TOKENS, "ms": round(p_ms, 3),
               "frac": round(pf / (p_ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4)}

    # own kernel launches of one decode step, counted on an eager step of the same shape
    eng.cache.admit("count")
    assert eng.cache.ensure("count", 0, 8)
    was = runner.capture_graphs
    runner.capture_graphs = False
    n0 = ops.LAUNCHES[0]
    runner.step([StepEntry("count", [1], 0, [0])])
    per_step = ops.LAUNCHES[0] - n0 + 2                        # + argmax and the feed-back kernel
    runner.capture_graphs = was
    eng.cache.free("count")
    torch.cuda.synchronize()

    workloads = {}
    standin = None
    del llm, eng, runner
    import gc
    gc.collect()
    torch.cuda.empty_cache()
    if not args.no_standin:
        try:
            standin = library_standin(cfg, (args.batch,) if args.no_points else (1, args.batch, 64), P, min(K, 64), W,
                                      windows)
        except Exception as e:                             # a stand-in must never take the measurement down with it
            standin = {"unavailable": f"{type(e).__name__}: {e}"[:200]}
        gc.collect()
        torch.cuda.empty_cache()
    if not args.no_workloads and args.layers is None:
        workloads["llama3b_continuous_batching"] = workload_3b(pk, windows)
        workloads["llama8b_shared_prefix"] = workload_8b(pk, windows)
    clocks.stop()

    nbytes = decode_bytes(cfg, layers, args.batch, ctx_mid)
    achieved = nbytes / (ms_step / 1e3) / 1e9
    out = {
        "metric": f"decode tok/s at batch {args.batch}, 2,048-token prompts + 256 tokens (Llama-3.2-1B shape, bf16)",
        "value": round(value, 1),
        "unit": "tok/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": round(ms_step, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic (random weights N(0,0.02) seed 0, uniform random token ids)", "impl": "ours",
        "config": {"model": "Llama-3.2-1B shape", "layers": layers, "layers_of_model": LLAMA_1B["num_hidden_layers"],
                   "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
                   "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
                   "global_batch": args.batch, "seq_len": P + SETTLE_STEPS + W + K, "prompt_len": P, "context_cap": CONTEXT_LEN,
                   "block_size": BLOCK_SIZE, "prefill_tokens": PREFILL_TOKENS, "parallelism": "single GPU",
                   "cuda_graphs": True, "l2": "inputs larger than L2 (2.5 GB of weights per step)",
                   "peaks": pk["source"], "settle_steps": SETTLE_STEPS},
        "load_s": round(load_s, 1), "value_runs_ms": " ".join(f"{r[1]:.4f}" for r in runs),
        "e2e": {k: (round(v, 3) if isinstance(v, float) else v) for k, v in e2e.items()},
        "gpu_launches": int(per_step * K),
        "prefill": prefill, "prefill_idle_s": PREFILL_IDLE_S,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
        "workloads": workloads,
        "library_standin": standin,
        "clocks": clocks.summary(windows),
        "launches_per_decode_step": int(per_step), "launches_per_prefill": int(prefill_launches),
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
