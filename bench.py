#!/usr/bin/env python3
"""Benchmark of the engine on one GPU: decode tokens/s of a Qwen3-8B-shaped model with random
weights (batch 8, context 4096 by default), prefill tokens/s of one 2048-token prompt, and the
fraction of the memory / tensor-core roofline each reaches.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch B] [--context C] [--layers L]
    python bench.py --shape 32b             # the same at the Qwen3-32B (or 0.6b) layer sizes
    python bench.py --serving               # 32 requests through LLM.generate at the Qwen3-0.6B shape
    python bench.py --shape 0.6b --closed-loop 8,128,128    # the reference's "c8 p128 o128" at engine level
    python bench.py --impl reference        # the reference engine, where it can be installed

Prints ONE JSON line.  A "step" is one decode step of the whole batch.  ``value`` times K steps on
the device (CUDA events); ``e2e`` is the same K steps through the Python entry point ``LLM.step()``,
each step copying its plan (token ids, positions, page tables) host->device from pinned memory and
reading sampled tokens device->host; the engine keeps one step in flight (it launches a step, then
reads the tokens of the step before), so K calls cover K steps' launches, copies and read-backs.
The cache is filled by really prefilling the prompts through the engine.
"""
from __future__ import annotations

import argparse
import json
import os
import random
import subprocess
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# Qwen3-8B shape: the benchmark configuration
QWEN3_8B = dict(architectures=["Qwen3ForCausalLM"], model_type="qwen3", vocab_size=151936, hidden_size=4096,
                intermediate_size=12288, num_hidden_layers=36, num_attention_heads=32, num_key_value_heads=8,
                head_dim=128, rms_norm_eps=1e-6, rope_theta=1000000.0, max_position_embeddings=40960,
                tie_word_embeddings=False, attention_bias=False, hidden_act="silu")
# the other two shapes the reference's architecture is quoted at (python bench.py --shape ...)
QWEN3_32B = dict(QWEN3_8B, hidden_size=5120, intermediate_size=25600, num_hidden_layers=64, num_attention_heads=64)
QWEN3_06B = dict(QWEN3_8B, hidden_size=1024, intermediate_size=3072, num_hidden_layers=28, num_attention_heads=16,
                 tie_word_embeddings=True)
SHAPES = {"8b": ("Qwen3-8B shape", QWEN3_8B), "32b": ("Qwen3-32B shape", QWEN3_32B), "0.6b": ("Qwen3-0.6B shape", QWEN3_06B)}
FULL_LAYERS = 36
PREFILL_TOKENS = 2048


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(p):
        d = json.load(open(p))
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]),
                "bf16_tflops_sustained": float(d.get("bf16_tflops_sustained", d["bf16_tflops"])), "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}


class ClockSampler:
    """nvidia-smi sampling of SM clocks and throttle reasons while the timed region runs."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.proc = None
        self.lines = []

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            out, _ = self.proc.communicate(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
            out = ""
        sm, mx, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in out.splitlines():
            f = [x.strip() for x in line.split(",")]
            if len(f) < 6:
                continue
            try:
                sm.append(float(f[0]))
                mx = float(f[1])
            except ValueError:
                continue
            for n, v in zip(names, f[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx, "reasons": sorted(reasons),
                "samples": len(sm)}


def model_numbers(cfg, layers):
    h, I, H, Hkv, D, V = (cfg["hidden_size"], cfg["intermediate_size"], cfg["num_attention_heads"],
                          cfg["num_key_value_heads"], cfg["head_dim"], cfg["vocab_size"])
    per_layer = (H + 2 * Hkv) * D * h + h * H * D + 3 * I * h            # linear parameters
    norms = 2 * h + 2 * D
    weight_bytes = 2 * (layers * (per_layer + norms) + V * h + h)         # read once per decode step (bf16)
    kv_bytes_per_token = layers * 2 * Hkv * D * 2
    return dict(per_layer=per_layer, weight_bytes=weight_bytes, kv_bytes_per_token=kv_bytes_per_token)


def prefill_flops(cfg, layers, T):
    n = model_numbers(cfg, layers)
    H, D, V, h = cfg["num_attention_heads"], cfg["head_dim"], cfg["vocab_size"], cfg["hidden_size"]
    return 2.0 * T * n["per_layer"] * layers + layers * 2.0 * T * T * H * D + 2.0 * V * h


def make_llm(cfg, layers, max_seqs, context, seed=42, **engine):
    from dinfer_b200 import LLM
    from dinfer_b200.weights.random_init import RandomSource
    c = dict(cfg, num_hidden_layers=layers)
    blocks = max_seqs * ((context + 64 + 15) // 16) + (PREFILL_TOKENS + 64) // 16 + 64
    return LLM(config=c, weights=RandomSource(c, seed, std=0.02, norm_jitter=0.0), dtype="bfloat16",
               max_model_len=max(context, PREFILL_TOKENS) + 64, max_num_seqs=max(max_seqs, 1), max_num_batched_tokens=2048,
               num_blocks=blocks, block_size=16, enable_cuda_graph=True, **{"split_norms": "auto", **engine})


def count_launches(fn):
    """Kernel launches of ``fn()``: every call into this package's kernel libraries and every library
    matrix product counts one (a replayed CUDA graph counts the launches it captured)."""
    from dinfer_b200.kernels import lib
    n0 = lib.launch_count()
    fn()
    return lib.launch_count() - n0


def decode_run(llm, cfg, batch, context, steps, warmup, rng, measure_e2e, want_launches=False):
    """Prefill ``batch`` prompts so that the timed steps end at ``context`` tokens, then time decode."""
    import torch
    from dinfer_b200 import SamplingParams
    V = cfg["vocab_size"]
    total_steps = warmup + (steps if measure_e2e else 1)
    # requests that finish their prompt early decode while the others still prefill (two portions each),
    # so leave room for that drift; the bytes of the roofline use the contexts actually reached
    prompt_len = context - total_steps - 2 * batch - 1
    sp = SamplingParams(temperature=0.0, max_tokens=1 << 20, ignore_eos=True)
    for _ in range(batch):
        llm.add_request([rng.randrange(V) for _ in range(prompt_len)], sp)
    while any(r.num_computed < len(r.prompt_ids) for r in llm._requests.values()) or llm.scheduler.waiting:
        llm.step()
    for _ in range(warmup):
        llm.step()
    res = {}
    torch.cuda.synchronize()
    sampler = ClockSampler()
    sampler.start()
    if measure_e2e:
        # end to end: K steps through the Python entry point; every step copies its plan (token ids,
        # positions, page tables) host->device from pinned memory and reads the sampled tokens back
        host0 = (llm.stats.host_schedule_s, llm.stats.host_launch_s, llm.stats.host_collect_s)
        t0 = time.perf_counter()
        for _ in range(steps):
            llm.step()
        torch.cuda.synchronize()
        res["e2e_ms_per_step"] = (time.perf_counter() - t0) * 1e3 / steps
        st = llm.stats
        res["host_us"] = [round((x - y) * 1e6 / steps, 1) for x, y in zip(
            (st.host_schedule_s, st.host_launch_s, st.host_collect_s), host0)]
        res["h2d_bytes_per_step"] = llm.runner.plan.h2d_bytes
        res["d2h_bytes_per_step"] = 4 * batch
    else:
        llm.step()
    # device time of one decode step: the step's captured graph (forward of the whole batch) replayed K
    # times back to back at the context just reached, timed with CUDA events, no host in between
    res["mean_context"] = sum(r.num_tokens + r.num_placeholders for r in llm._requests.values()) / batch - 1
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    from dinfer_b200.kernels import lib as _lib
    l0 = _lib.launch_count()
    e0.record()
    from dinfer_b200.sampling.sampler import argmax
    tokens = torch.empty(llm.runner.engine.max_num_seqs, dtype=torch.int32, device=llm.runner.device)
    llm.runner.replay_last_decode(steps, after=lambda logits: argmax(logits[:batch], out=tokens[:batch]))
    e1.record()
    torch.cuda.synchronize()
    res["ms_per_step"] = e0.elapsed_time(e1) / steps
    res["launches_per_step"] = (_lib.launch_count() - l0) // steps
    res["clocks"] = sampler.stop()
    for rid in list(llm._requests):
        llm.abort(rid)
    return res


def prefill_run(llm, cfg, tokens, rng, reps=3):
    import torch
    from dinfer_b200.engine.batch import StepEntry
    V = cfg["vocab_size"]
    best = None
    for i in range(reps + 1):
        ids = [rng.randrange(V) for _ in range(tokens)]
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        llm.runner.step([StepEntry(("prefill", i), ids, [tokens - 1])])
        e1.record()
        torch.cuda.synchronize()
        llm.runner.finish(("prefill", i))
        ms = e0.elapsed_time(e1)
        if i > 0:
            best = ms if best is None else min(best, ms)
    return best


def profile_region(a) -> int:
    """For a profiler: set up a small case, then bracket ONE decode step (or one prefill step) with
    cudaProfilerStart/Stop, so that ``ncu --profile-from-start off`` sees only that step's kernels.
    Prints no benchmark line: a run under a profiler is never a measurement."""
    import torch
    from dinfer_b200 import SamplingParams
    from dinfer_b200.engine.batch import StepEntry
    cfg = QWEN3_8B
    rng = random.Random(42)
    # the bracketed prefill step launches its kernels one by one (a profiler then lists them once, in order)
    llm = make_llm(cfg, a.layers, max(a.batch, 1), a.context, mixed_cuda_graph=False)
    V = cfg["vocab_size"]
    if a.profile == "prefill":
        ids = [rng.randrange(V) for _ in range(PREFILL_TOKENS)]
        llm.runner.step([StepEntry("w", ids, [PREFILL_TOKENS - 1])])
        llm.runner.finish("w")
        torch.cuda.synchronize()
        torch.cuda.profiler.start()
        llm.runner.step([StepEntry("p", ids, [PREFILL_TOKENS - 1])])
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
        return 0
    sp = SamplingParams(temperature=0.0, max_tokens=1 << 20, ignore_eos=True)
    for _ in range(a.batch):
        llm.add_request([rng.randrange(V) for _ in range(a.context - 16)], sp)
    while any(r.num_computed < len(r.prompt_ids) for r in llm._requests.values()) or llm.scheduler.waiting:
        llm.step()
    for _ in range(3):
        llm.step()
    torch.cuda.synchronize()
    torch.cuda.profiler.start()
    llm.step()
    torch.cuda.synchronize()
    torch.cuda.profiler.stop()
    return 0


def serving_run() -> int:
    """32 requests with prompts of 16..1024 tokens (seed 3) through ``LLM.generate`` at the Qwen3-0.6B shape:
    prompts cut into portions of 512 tokens beside decoding requests, 256 tokens each at temperature 0.7."""
    import torch
    from dinfer_b200 import LLM, SamplingParams
    from dinfer_b200.weights.random_init import RandomSource
    cfg = QWEN3_06B
    llm = LLM(config=cfg, weights=RandomSource(cfg, 3, std=0.02, norm_jitter=0.0), dtype="bfloat16", max_model_len=2048,
              max_num_seqs=32, max_num_batched_tokens=512, num_blocks=32 * 129, block_size=16)
    rng = random.Random(3)
    prompts = [[rng.randrange(cfg["vocab_size"]) for _ in range(rng.randint(16, 1024))] for _ in range(32)]
    sp = [SamplingParams(temperature=0.7, max_tokens=256, ignore_eos=True, seed=100 + i) for i in range(32)]
    best = None
    for _ in range(3):                                  # the first pass also captures the decode graphs
        steps0 = llm.stats.steps
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        outs = llm.generate(prompts, sp)
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        gen = sum(len(o.output_ids) for o in outs)
        mid = len(outs) // 2
        rec = {"seconds": round(dt, 4), "steps": llm.stats.steps - steps0, "generated": gen,
               # as the reference's bench reports them: time to the first token and time per token after it, medians
               "ttft_ms_p50": round(sorted(o.ttft_s for o in outs)[mid] * 1e3, 2),
               "tpot_ms_p50": round(sorted(o.tpot_s for o in outs)[mid] * 1e3, 3)}
        if best is None or dt < best["seconds"]:
            best = rec
    print(json.dumps({"metric": "serving: generated tok/s (Qwen3-0.6B shape, bf16, 32 requests, prompts 16..1024, "
                                "portions of 512, 256 tokens each at temperature 0.7)",
                      "value": round(best["generated"] / best["seconds"], 1), "unit": "tokens/s",
                      "prompt_tokens": sum(map(len, prompts)), "ms_per_step": round(best["seconds"] * 1e3 / best["steps"], 3),
                      **best, "impl": "ours", "data": "synthetic"}))
    return 0


def closed_loop_run(shape: str, clients: int, prompt_len: int, output_len: int, requests_per_client: int = 6) -> int:
    """The reference's serving measurement without the HTTP in between (its ``bench`` tool,
    scripts/verify/bench_compare.sh: "cN pP oO" = N clients, each sending its next request when the last has ended,
    prompts of P tokens, O generated tokens, temperature 0, ignore_eos, the first 2 requests of each client left
    out): output tokens a second over the measured requests, time to the first token and time per token after it."""
    import torch
    from dinfer_b200 import LLM, SamplingParams
    from dinfer_b200.weights.random_init import RandomSource
    name, cfg = SHAPES[shape]
    llm = LLM(config=cfg, weights=RandomSource(cfg, 3, std=0.02, norm_jitter=0.0), dtype="bfloat16",
              max_model_len=max(2048, prompt_len + output_len + 64), max_num_seqs=max(16, clients),
              max_num_batched_tokens=2048, block_size=16, split_norms="auto")
    rng = random.Random(11)
    sp = SamplingParams(temperature=0.0, max_tokens=output_len, ignore_eos=True)

    def prompt():
        return [rng.randrange(cfg["vocab_size"]) for _ in range(prompt_len)]
    sent = {c: 0 for c in range(clients)}
    owner, outs = {}, []
    for c in range(clients):
        owner[llm.add_request(prompt(), sp)] = c
        sent[c] += 1
    t_start = None
    while llm.has_unfinished():
        for o in llm.step():
            c = owner.pop(o.req_id)
            if sent[c] > 2:                                   # measured (the first two of a client warm up)
                outs.append(o)
            if sent[c] == 2 and t_start is None and all(n >= 2 for n in sent.values()):
                torch.cuda.synchronize()
                t_start = time.perf_counter()
            if sent[c] < requests_per_client:
                owner[llm.add_request(prompt(), sp)] = c
                sent[c] += 1
    torch.cuda.synchronize()
    dt = time.perf_counter() - (t_start or 0.0)
    gen = sum(len(o.output_ids) for o in outs)
    mid = len(outs) // 2
    print(json.dumps({"metric": f"closed loop c{clients} p{prompt_len} o{output_len}: output tok/s ({name}, bf16, random "
                                "weights, engine level, no HTTP)",
                      "value": round(gen / dt, 1), "unit": "tokens/s", "requests": len(outs),
                      "ttft_ms_p50": round(sorted(o.ttft_s for o in outs)[mid] * 1e3, 2),
                      "tpot_ms_p50": round(sorted(o.tpot_s for o in outs)[mid] * 1e3, 3),
                      "e2e_ms_p50": round(sorted(o.e2e_s for o in outs)[mid] * 1e3, 1),
                      "seconds": round(dt, 3), "impl": "ours", "data": "synthetic"}))
    return 0


# ---------------------------------------------------------------- Dobedra beside Qwen3 at equal layer sizes
def _dobedra_cfg(width, heads, dim, rot, vdim, kv_rank, q_rank, dense_ff, experts, top, ff, shared, vocab=32768):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "rot": {"base": 10000.0, "dims": rot}, "scale": (dim + rot) ** -0.5}
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    layers = [{"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": dense_ff}},
              {"type": "latent_attention", "mixer": m, "mlp": moe},
              {"type": "latent_attention", "mixer": m, "mlp": moe},
              {"type": "latent_attention", "mixer": dict(m, kv_from=2), "mlp": moe}]
    return {"architecture": "Dobedra", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": layers}


def _qwen3_cfg(width, heads, kv_heads, head_dim, inter, vocab=32768):
    return dict(QWEN3_8B, vocab_size=vocab, hidden_size=width, intermediate_size=inter, num_hidden_layers=4,
                num_attention_heads=heads, num_key_value_heads=kv_heads, head_dim=head_dim)


# layer sizes that resemble real models of the design's kind (a latent of 512 + 64 under 16 or 32 heads of 128 + 64,
# 64 experts of which a token uses 6, a shared expert), and a smaller one; beside each the dense Qwen3 layer of the same
# width and head count whose feed-forward has about the weights a Dobedra token uses
DESIGN_SIZES = {
    "small": (_dobedra_cfg(1024, 8, 64, 32, 64, 256, 512, 4096, 16, 2, 512, 1024), _qwen3_cfg(1024, 8, 2, 128, 2048)),
    "medium": (_dobedra_cfg(2048, 16, 128, 64, 128, 512, 1536, 10944, 64, 6, 1408, 2816), _qwen3_cfg(2048, 16, 4, 128, 7680)),
    "large": (_dobedra_cfg(4096, 32, 128, 64, 128, 512, 1536, 12288, 64, 6, 2048, 4096), _qwen3_cfg(4096, 32, 8, 128, 12288)),
}


# ---------------------------------------------------------------- Zasipel beside Qwen3 at equal layer sizes
def _zasipel_cfg(width, heads, kv_heads, dim, window, delta_heads, delta_kv, experts, top, ff, shared, vocab=32768):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window},
            "rot": {"base": 10000.0, "dims": dim // 2}}
    right = {"heads": delta_heads, "kv_heads": delta_kv, "dim": dim, "vdim": dim, "conv": 4}
    channel = dict(right, kv_heads=delta_heads, decay_rank=dim // 2, gate_rank=dim // 2)
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    par = {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": moe}
    return {"architecture": "Zasipel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "layers": [par, par, {"type": "channel_delta", "mixer": channel, "mlp": moe}, par]}


# four layers (three with attention over a window beside a delta rule, one with the per-channel delta rule alone), heads
# of 64 or 128, a window of 1024, 16 or 64 experts of which a token uses 2 or 6, a shared expert; beside each the dense
# Qwen3 layers of the same width and head count whose feed-forward has about the weights a Zasipel token uses
ZASIPEL_SIZES = {
    "small": (_zasipel_cfg(1024, 16, 4, 64, 1024, 16, 8, 16, 2, 512, 1024), _qwen3_cfg(1024, 16, 4, 64, 2048)),
    "medium": (_zasipel_cfg(2048, 16, 4, 128, 1024, 16, 8, 64, 6, 1408, 2816), _qwen3_cfg(2048, 16, 4, 128, 7680)),
    "large": (_zasipel_cfg(4096, 32, 8, 128, 1024, 32, 16, 64, 6, 2048, 4096), _qwen3_cfg(4096, 32, 8, 128, 12288)),
}


# ---------------------------------------------------------------- Sobivik beside Qwen3 at equal layer sizes
def _sobivik_cfg(width, heads, kv_heads, dim, kv_rank, q_rank, window, ff, vocab=32768):
    decay = [1.0 - 2.0 ** (-5.0 - 6.0 * i / max(1, heads - 1)) for i in range(heads)]
    ret = {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": dim, "decay": decay}}
    lat = {"type": "latent_attention",
           "mixer": {"heads": heads, "dim": dim, "rot_dim": dim // 2, "vdim": dim, "kv_rank": kv_rank, "q_rank": q_rank,
                     "scale": (1.5 * dim) ** -0.5, "mask": {"size": window},
                     "rot": {"base": 1e6, "dims": dim // 2, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    dif = {"type": "attention",
           "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim // 2, "vdim": dim, "scale": (dim // 2) ** -0.5,
                     "diff": 0.5, "mask": {"size": window, "keep_first": 4}}}
    mlp = {"kind": "dense", "ff": ff}
    return {"architecture": "Sobivik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "logit_scale": 1.0, "canon": {"taps": 4}, "layers": [dict(l, mlp=mlp) for l in (ret, lat, dif, ret)]}


# four layers (retention, latent attention over a window, differential attention over a window with kept first tokens,
# retention), heads of 64 or 128 (each differential map half a head), a window of 1024, a convolution of four taps on
# every mixer's input, the dense feed-forward of the Qwen3 layers beside them
SOBIVIK_SIZES = {
    "small": (_sobivik_cfg(1024, 16, 4, 64, 256, 512, 1024, 2048), _qwen3_cfg(1024, 16, 4, 64, 2048)),
    "medium": (_sobivik_cfg(2048, 16, 4, 128, 512, 1536, 1024, 7680), _qwen3_cfg(2048, 16, 4, 128, 7680)),
    "large": (_sobivik_cfg(4096, 32, 8, 128, 512, 1536, 1024, 12288), _qwen3_cfg(4096, 32, 8, 128, 12288)),
}


# ---------------------------------------------------------------- Porovik beside Zasipel at equal layer sizes
def _porovik_cfg(width, heads, kv_heads, dim, experts, top, ff_expert, ff_dense, vocab=32768):
    gw = {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": dim}}
    gd = {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "decay_rank": dim // 2}}
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
                                          "q_temp": {"coef": 0.4, "every": 128}, "v_mix": True}}
    dense = {"kind": "dense", "ff": ff_dense}
    moe = {"kind": "moe", "expert": {"ff": ff_expert}, "router": {"experts": experts, "top": top}}
    return {"architecture": "Porovik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "max_positions": 8192,
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 131, "mul_cur": 37}},
            "layers": [dict(gw, mlp=dense), dict(att, mlp=moe), dict(gd, mlp=dense), dict(att, mlp=moe)]}


# four layers (gate-write linear attention, attention with a distance bias, the general delta rule, attention again:
# the second one mixes the first one's values into its own), heads of 64 or 128, a dense feed-forward behind the
# recurrent mixers and 16 or 64 experts of which a token uses 2 or 6 behind the attention layers; beside each the
# Zasipel layers of the same width, heads and experts (the closest design: a delta rule with a decay per channel,
# attention, routed experts)
POROVIK_SIZES = {
    "small": (_porovik_cfg(1024, 16, 4, 64, 16, 2, 512, 2048), ZASIPEL_SIZES["small"][0]),
    "medium": (_porovik_cfg(2048, 16, 4, 128, 64, 6, 1408, 7680), ZASIPEL_SIZES["medium"][0]),
    "large": (_porovik_cfg(4096, 32, 8, 128, 64, 6, 2048, 12288), ZASIPEL_SIZES["large"][0]),
}


# ---------------------------------------------------------------- Datozen beside Qwen3 at equal layer sizes
def _datozen_cfg(width, heads, kv_heads, dim, experts, identity, groups, keep, top, ff_expert, shared, ff_dense, side, vocab=32768):
    def att(chunk):
        return {"type": "attention",
                "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": chunk},
                          "rot": {"base": 1e6, "dims": dim // 2,
                                  "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    dense = {"kind": "dense", "ff": ff_dense}
    moe = {"kind": "moe", "expert": {"ff": ff_expert}, "shared": {"ff": shared},
           "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}}}
    return {"architecture": "Datozen", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "max_positions": 8192,
            "token_side": {"dim": side},
            "layers": [dict(att(1024), mlp=dense), dict(att(8192), mlp=moe), dict(att(1024), mlp=dense), dict(att(8192), mlp=moe)]}


# four layers (chunks of 1024 and 8192 positions in turn; a dense feed-forward behind the first and third, 16 or 64 experts
# and a quarter as many identity experts, of which a token uses 2 or 6, with a shared expert behind the others), heads of 64
# or 128, a token input of 64 to 256; no loop, so that four layers run; beside each the dense Qwen3 layers of the same width
# and heads, whose feed-forward has as many weights as the dense one here
DATOZEN_SIZES = {
    "small": (_datozen_cfg(1024, 16, 4, 64, 16, 4, 4, 2, 2, 512, 1024, 3072, 64), _qwen3_cfg(1024, 16, 4, 64, 2048)),
    "medium": (_datozen_cfg(2048, 16, 4, 128, 64, 16, 8, 4, 6, 1408, 2816, 11520, 128), _qwen3_cfg(2048, 16, 4, 128, 7680)),
    "large": (_datozen_cfg(4096, 32, 8, 128, 64, 16, 8, 4, 6, 2048, 4096, 18432, 256), _qwen3_cfg(4096, 32, 8, 128, 12288)),
}


# ---------------------------------------------------------------- Rorutar beside Zasipel at equal layer sizes
def _rorutar_cfg(width, heads, kv_heads, dim, window, state_heads, vdim, state, groups, experts, expert_groups, keep, top, ff,
                 vocab=32768):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "softcap": 30.0,
            "mask": {"size": window, "keep_first": 4}, "rot": {"base": 10000.0, "dims": dim, "scaling": {"factor": 4.0}}}
    right = {"heads": state_heads, "vdim": vdim, "state": state, "groups": groups, "conv": 4, "norm_groups": groups}
    moe = {"kind": "moe", "expert": {"ff": ff, "limit": 7.0},
           "router": {"experts": experts, "top": top, "groups": {"count": expert_groups, "keep": keep}}}
    layer = {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.5, "right_scale": 0.7}, "mlp": moe}
    return {"architecture": "Rorutar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "layers": [layer] * 4}


# four layers (attention over a window of 1024 and four kept tokens, heads of 64 or 128, beside a state-space mixer whose
# state is as large as the delta rule's of the Zasipel layers at that size, 16 or 64 experts of which a token uses 4 or 8: the
# weights of Zasipel's chosen experts and its shared one); no loop, so that four layers run; beside each the Zasipel
# layers of the same width, heads and experts (the closest design: two mixers side by side, attention over a window with a
# sink and a recurrence with a short convolution, routed gated experts)
RORUTAR_SIZES = {
    "small": (_rorutar_cfg(1024, 16, 4, 64, 1024, 16, 64, 64, 2, 16, 4, 2, 4, 512), ZASIPEL_SIZES["small"][0]),
    "medium": (_rorutar_cfg(2048, 16, 4, 128, 1024, 32, 64, 128, 4, 64, 8, 4, 8, 1408), ZASIPEL_SIZES["medium"][0]),
    "large": (_rorutar_cfg(4096, 32, 8, 128, 1024, 64, 64, 128, 8, 64, 8, 4, 8, 2048), ZASIPEL_SIZES["large"][0]),
}
DESIGNS = {"rorutar": RORUTAR_SIZES, "datozen": DATOZEN_SIZES, "dobedra": DESIGN_SIZES, "zasipel": ZASIPEL_SIZES, "sobivik": SOBIVIK_SIZES, "porovik": POROVIK_SIZES}
# the model a design stands beside (the closest one this package has)
BESIDE = {"porovik": "zasipel", "rorutar": "zasipel"}


def _time_model(cfg, batch, context, prefill_tokens, steps, seed=5, profile=None):
    """(prefill ms of one prompt, decode ms per step of ``batch`` requests at ``context``, launches per decode step) of
    four layers of ``cfg`` with random weights: the prompt through the step function (best of three), the decode
    step as its captured graph replayed ``steps`` times between CUDA events."""
    import torch
    from dinfer_b200.config.engine_config import EngineConfig
    from dinfer_b200.engine.batch import StepEntry
    from dinfer_b200.engine.runner import ModelRunner
    from dinfer_b200.kernels import lib
    from dinfer_b200.weights.random_init import RandomSource
    vocab = cfg.get("vocab_size", cfg.get("vocab"))
    longest = max(context, prefill_tokens) + 64
    eng = EngineConfig(max_model_len=longest, max_num_seqs=batch, max_num_batched_tokens=max(2048, prefill_tokens),
                       num_blocks=(batch + 1) * ((longest + 15) // 16) + 8, block_size=16, dtype="bfloat16",
                       mixed_cuda_graph=False)
    runner = ModelRunner(cfg, RandomSource(cfg, seed, std=0.02, norm_jitter=0.0), eng)
    rng = random.Random(seed)
    pre = None
    for i in range(4):
        ids = [rng.randrange(vocab) for _ in range(prefill_tokens)]
        torch.cuda.synchronize()
        if profile == "prefill" and i == 3:
            torch.cuda.profiler.start()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        runner.step([StepEntry(("p", i), ids, [prefill_tokens - 1])])
        e1.record()
        torch.cuda.synchronize()
        if profile == "prefill" and i == 3:
            torch.cuda.profiler.stop()
        runner.finish(("p", i))
        if i > 0:
            pre = e0.elapsed_time(e1) if pre is None else min(pre, e0.elapsed_time(e1))
    for b in range(batch):                                     # fill the cache up to the context, one request a step
        runner.step([StepEntry(b, [rng.randrange(vocab) for _ in range(context - 4)], [])])
    for _ in range(3):
        runner.step([StepEntry(b, [rng.randrange(vocab)], [0]) for b in range(batch)])
    torch.cuda.synchronize()
    if profile == "decode":
        runner._graph_ok = False
        torch.cuda.profiler.start()
        runner.step([StepEntry(b, [rng.randrange(vocab)], [0]) for b in range(batch)])
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
        return pre, 0.0, 0
    l0 = lib.launch_count()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    runner.replay_last_decode(steps)
    e1.record()
    torch.cuda.synchronize()
    dec = e0.elapsed_time(e1) / steps
    launches = (lib.launch_count() - l0) // steps
    del runner
    torch.cuda.empty_cache()
    return pre, dec, launches


def design_run(a) -> int:
    """``--design dobedra|zasipel|sobivik|porovik|datozen|rorutar``: prefill and decode throughput of four layers of the design beside four
    layers of the model it is compared with (Qwen3, or ``BESIDE``) at the same width and head count, at the sizes of
    ``DESIGNS``; one JSON line."""
    rows = {}
    table = DESIGNS[a.design]
    beside = BESIDE.get(a.design, "qwen3")
    sizes = [a.design_size] if a.design_size else list(table)
    for name in sizes:
        ours, theirs = table[name]
        row = {}
        for label, cfg in ((a.design, ours), (beside, theirs)):
            if a.profile and label != (a.design_model or a.design):
                continue
            pre, dec, launches = _time_model(cfg, a.batch, a.context, PREFILL_TOKENS, a.steps, profile=a.profile)
            row[label] = {"prefill_ms": round(pre, 3), "prefill_tok_s": round(PREFILL_TOKENS * 1e3 / pre, 1),
                          "decode_ms_per_step": round(dec, 4), "decode_tok_s": round(a.batch * 1e3 / dec, 1) if dec else None,
                          "launches_per_decode_step": launches}
        rows[name] = row
    if a.profile:
        return 0
    print(json.dumps({"metric": f"{a.design.capitalize()} beside {beside.capitalize()}, four layers at equal width and heads (bf16, random weights): "
                                f"prefill of {PREFILL_TOKENS} tokens, decode at batch {a.batch} context {a.context}",
                      "sizes": rows, "steps": a.steps, "impl": "ours", "data": "synthetic"}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--profile", choices=["decode", "prefill"], default=None,
                    help="run one bracketed step for a profiler instead of the benchmark")
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=FULL_LAYERS)
    ap.add_argument("--no-points", action="store_true", help="skip the batch-1 and batch-64 points")
    ap.add_argument("--shape", choices=sorted(SHAPES), default="8b", help="layer sizes of the model (default: the benchmark's)")
    ap.add_argument("--serving", action="store_true",
                    help="the mixed serving workload instead: 32 requests, prompts of 16..1024 tokens, portions of "
                         "512, 256 tokens each at temperature 0.7, at the Qwen3-0.6B shape")
    ap.add_argument("--closed-loop", default=None, metavar="C,P,O",
                    help="the reference's serving measurement at engine level instead: C clients, each sending its "
                         "next request when the last has ended, prompts of P tokens, O generated tokens (--shape applies)")
    ap.add_argument("--design", choices=["dobedra", "zasipel", "sobivik", "porovik", "datozen", "rorutar"], default=None,
                    help="instead of the benchmark: four layers of this design beside four Qwen3 layers of equal width, "
                         "prefill and decode, at a few layer sizes")
    ap.add_argument("--design-size", choices=["small", "medium", "large"], default=None, help="only this size")
    ap.add_argument("--design-model", choices=["dobedra", "zasipel", "sobivik", "porovik", "datozen", "rorutar", "qwen3"], default=None, help="with --profile: which of the two")
    a = ap.parse_args()
    if a.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "rayze-ai/dinfer is a Rust workspace: no cargo/rustc in this image and pip finds no "
                          "Python project in it (no setup.py / pyproject.toml), so it cannot be installed offline"}))
        return 0
    if a.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {a.gpus} is not supported")
        return 2
    a.warmup = max(a.warmup, 3)
    import torch
    if a.design:
        if a.context == 4096:
            a.context = 2048
        return design_run(a)
    if a.profile:
        return profile_region(a)
    if a.serving:
        return serving_run()
    if a.closed_loop:
        c, p_len, o_len = (int(x) for x in a.closed_loop.split(","))
        return closed_loop_run(a.shape, c, p_len, o_len)
    shape_name, cfg = SHAPES[a.shape]
    full_layers = cfg["num_hidden_layers"]
    if a.shape != "8b" and a.layers == FULL_LAYERS:
        a.layers = full_layers
    pk = peaks()
    rng = random.Random(42)
    nums = model_numbers(cfg, a.layers)
    llm = make_llm(cfg, a.layers, max(a.batch, 1 if a.no_points else 64), a.context)

    main_run = decode_run(llm, cfg, a.batch, a.context, a.steps, a.warmup, rng, measure_e2e=True, want_launches=True)
    ms = main_run["ms_per_step"]
    value = a.batch * 1e3 / ms
    # context of the device-timed step (the graph is replayed at the context the requests had reached)
    ctx_mid = main_run["mean_context"]
    step_bytes = nums["weight_bytes"] + a.batch * ctx_mid * nums["kv_bytes_per_token"]
    achieved = step_bytes / (ms * 1e-3) / 1e9

    pre_ms = prefill_run(llm, cfg, PREFILL_TOKENS, rng)
    pf = prefill_flops(cfg, a.layers, PREFILL_TOKENS)
    points = {}
    if not a.no_points:
        for b in (1, 64):
            r = decode_run(llm, cfg, b, a.context, max(8, a.steps // 2), a.warmup, rng, measure_e2e=False)
            points[f"decode_b{b}"] = round(b * 1e3 / r["ms_per_step"], 1)

    out = {
        "metric": f"decode tok/s ({shape_name}, bf16, random weights)", "value": round(value, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": a.steps, "warmup": a.warmup, "ms_per_step": round(ms, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "impl": "ours",
        "config": {"model": shape_name, "layers": a.layers, "layers_full": full_layers, "hidden": cfg["hidden_size"],
                   "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
                   "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"],
                   "vocab": cfg["vocab_size"], "global_batch": a.batch, "seq_len": a.context, "mean_context_timed": round(ctx_mid, 1),
                   "block_size": 16, "parallelism": "single GPU", "prefill_tokens": PREFILL_TOKENS,
                   "l2": "inputs larger than L2 (weights + cache read per step)", "peaks": pk["source"],
                   # the engine option this run sets: each decode graph in the faster of its two forms, measured at start
                   "split_norms": "auto: norms taken apart at batch sizes " + (",".join(map(str, llm.runner.split_norms_buckets())) or "none")},
        "e2e": {"value": round(a.batch * 1e3 / main_run["e2e_ms_per_step"], 1), "unit": "tokens/s",
                "h2d_bytes_per_step": main_run["h2d_bytes_per_step"],
                "d2h_bytes_per_step": main_run["d2h_bytes_per_step"],
                # the host's share of a step in us: deciding it, plan + launch, waiting for and applying the tokens
                # of the step before (one step is in flight, so the wait is where the device's time shows)
                "host_us_schedule_launch_collect": main_run.get("host_us")},
        "gpu_launches": main_run["launches_per_step"] * a.steps,
        "prefill": {"value": round(PREFILL_TOKENS * 1e3 / pre_ms, 1), "tokens": PREFILL_TOKENS,
                    "ms": round(pre_ms, 3), "frac": round(pf / (pre_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
        "clocks": main_run["clocks"],
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
