#!/usr/bin/env python3
"""Benchmark of the engine on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--impl ours|reference]
    python bench.py --workload mix14b | 32b
    python bench.py --workload zidivik | tidavik | toredra | korirax | tuganex | fasanex [--size a|b]

Default run (the headline): decode tokens a second at batch 8, at batch 1 and 64, prefill of
2,048 tokens, and the same decode through the Python entry point with host tokens in and out.
Model: the sizes of Qwen3-8B (36 layers, width 4096, 32/8 heads of 128, feed-forward 12288,
vocabulary 151936), bfloat16, random weights; prompts are uniform random token ids.  A step is
one decode step of the whole batch at a context that ends at 4,096 tokens; the ids a step picks
are the next step's input (on the device), and the cache pages are handed out in a scattered
order, as after long serving.  `--layers` runs fewer layers of the same sizes (the record names
both numbers); layer sizes never shrink.

`--workload mix14b`: 32 requests with prompts of 128 to 2,048 tokens (seed-fixed) and 256 greedy
tokens each at the sizes of Qwen3-14B, through `LLM.add_request` / `LLM.step`, prompt portions
mixed with decode tokens under a budget of 512 tokens a step (two token tiles of the products).  `--workload 32b`: 16 requests of 1,024 + 128 tokens at
the sizes of Qwen3-32B (64 query heads of 128 on a width of 5,120).  Each prints one JSON line
with total, prompt and generated tokens a second, the time of all steps on the device, the
wall-clock time over it, and the steps' fraction of their roofline.

`--workload zidivik`: the Zidivik decoder (window attention with kept first tokens and shared keys,
gated delta rule, routed experts) at layer sizes of a real model, random weights, beside the Qwen3
dense decoder of equal width, heads, depth and active feed-forward size: a prompt of 2,048 tokens in
one step and decode steps of 8 requests at a context of 2,048, device-timed through `Engine.step`,
plus the device time of every kind of operation in one step of each (CUDA events around each call,
which switch the overlap of neighbours off: compare shares).

`--workload tidavik`: the Tidavik decoder (window attention with sigmoid weights and a distance term,
window attention with a softmax that has one more term, attention over cached latents; dense gated
feed-forward) the same way, beside the Qwen3 dense decoder of equal width, heads, depth, feed-forward
and window.

`--workload toredra`: the Toredra decoder (rotary attention whose softmax has a learned term per head beside a
forget-gate recurrence, a generalised delta rule, gated and twice-normed sublayers, an ungated feed-forward with
the square of relu) the same way, beside the Qwen3 dense decoder of equal width, heads, depth, vocabulary and
feed-forward weights.

`--workload korirax`: the Korirax decoder (attention with a table of distance terms, a query temperature and a gate per
element; attention over cached latents with a rotated key part that all heads share; a gated diagonal recurrence; dense
gated feed-forward and routed experts with a sigmoid router, groups and a shared expert; a token input per layer) the same
way, beside the Qwen3 dense decoder of equal width, heads, depth, vocabulary and active feed-forward weights.

`--workload tuganex`: the Tuganex decoder (differential attention, also on another layer's keys; retention; a dense feed-forward
with xIELU and routed experts with a softmax router, groups, identity experts and a gated shared expert; norms on the
sublayers' results only) the same way.

`--workload fasanex`: the Fasanex decoder (a state-space mixer with a scalar decay per head; window attention whose values are its keys
beside time mixing; a delta rule with one decay per head; a bounded gated feed-forward; twice-normed sublayers) the same way, beside the
Qwen3 dense decoder of equal width, heads, depth, feed-forward, vocabulary and window.

Timing: CUDA events on the launching stream around exactly K steps after W warm-up steps, with
a synchronize on both sides.  Every step streams all weights (15 GB) and the live requests'
cache from HBM, far more than the 126 MB of L2, so nothing a step reads is still cached from
the step before.  SM clocks and throttle reasons are sampled with nvidia-smi during the timed
regions.  One JSON line is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_8B = dict(architectures=["Qwen3ForCausalLM"], model_type="qwen3", num_hidden_layers=36, hidden_size=4096,
                num_attention_heads=32, num_key_value_heads=8, head_dim=128, intermediate_size=12288,
                vocab_size=151936, rope_theta=1000000.0, rms_norm_eps=1e-6, tie_word_embeddings=False,
                attention_bias=False, max_position_embeddings=40960, hidden_act="silu")
QWEN3_14B = dict(QWEN3_8B, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408)
QWEN3_32B = dict(QWEN3_8B, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, intermediate_size=25600)
# The reference cannot run this benchmark.  It is a CMake C11 project ("Neither 'setup.py' nor
# 'pyproject.toml' found" is pip's answer), its engine reads only its own quantized VQF files,
# and its one bfloat16-free route to the same numbers, the float32 CPU forward that
# tests/golden compiles, takes 35 ms a token and layer at these layer sizes on this machine's
# 8 cores (measured: 24 tokens through one layer, less 4 tokens through it, over 20) - 1.4 s a
# token for 36 layers and the output head - and prefills token by token
# (src/model/vllm_safetensors.c:17964-17971): the 8 x 2,048 prompt tokens of this benchmark
# alone would take more than six hours, and the float32 weights 33 GB of host memory.
REFERENCE_UNAVAILABLE = ("the reference is a CPU-only C11 engine (CMake, no Python package: pip install finds no setup.py or "
                         "pyproject.toml) that loads only its own quantized VQF files; its float32 forward, the one path "
                         "that takes these weights, was compiled and measured here at 35 ms per token and layer of this "
                         "size on 8 cores = 1.4 s a token, prefill token by token: batch 8 x context 4,096 would take hours")
CONTEXT = 4096
PREFILL_TOKENS = 2048
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                p = json.load(f)
            out = dict(FALLBACK_PEAKS)
            for k in out:
                if isinstance(p.get(k), (int, float)) and p[k] > 0:
                    out[k] = float(p[k])
            out["source"] = "measured"
            return out
        except Exception:
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """nvidia-smi clocks and throttle reasons, sampled every 200 ms while `active`."""
    Q = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
         "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
         "clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.rows = []
        self.active = False
        self._stop = False
        self._proc = None
        try:
            self._proc = subprocess.Popen(["nvidia-smi", f"--id={index}", f"--query-gpu={self.Q}",
                                           "--format=csv,noheader,nounits", "-lms", "200"],
                                          stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self._t = threading.Thread(target=self._read, daemon=True)
            self._t.start()
        except OSError:
            self._proc = None

    def _read(self):
        for line in self._proc.stdout:
            if self._stop:
                break
            if self.active:
                self.rows.append([c.strip() for c in line.split(",")])

    def close(self):
        self._stop = True
        if self._proc:
            self._proc.terminate()

    def summary(self):
        sm, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for r in self.rows:
            try:
                sm.append(int(float(r[0])))
                mx = max(mx, int(float(r[1])))
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, r[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(sm)}


def run_workload(args) -> int:
    """A whole workload through the scheduler: requests are added to `LLM`, `LLM.step` is called
    until all are done; every step leaves CUDA events, from which the time on the device and the
    host's share follow."""
    import numpy as np
    import torch
    from kestrel_llm_b200 import LLM, SamplingParams
    from kestrel_llm_b200.config import EngineOptions, Qwen3Config
    from kestrel_llm_b200.config.registry import resolve_architecture
    from kestrel_llm_b200.weights import fill_random_

    if args.workload == "mix14b":
        raw, label = dict(QWEN3_14B), "Qwen3-14B shape"
        n_req, gen = args.requests or 32, args.generate or 256
        rng = np.random.default_rng(14)
        lengths = rng.integers(128, 2049, size=n_req).tolist()
        chunk = 512
        what = f"{n_req} requests, prompts of 128 to 2,048 tokens (seed 14), {gen} greedy tokens each, prompt portions of {chunk} mixed with decode tokens"
    else:
        raw, label = dict(QWEN3_32B), "Qwen3-32B shape"
        n_req, gen = args.requests or 16, args.generate or 128
        rng = np.random.default_rng(32)
        lengths = [1024] * n_req
        chunk = 512
        what = f"{n_req} requests of 1,024 prompt tokens, {gen} greedy tokens each, prompt portions of {chunk} mixed with decode tokens"
    full_layers = raw["num_hidden_layers"]
    if args.layers:
        raw["num_hidden_layers"] = min(args.layers, full_layers)
    cfg = Qwen3Config.from_dict(raw)
    L = cfg.num_hidden_layers
    dev = "cuda:0"
    torch.cuda.set_device(0)
    model = resolve_architecture(cfg.architecture).build(cfg, torch.bfloat16, dev)
    fill_random_(model, 0)
    longest = max(lengths) + gen + 64
    opts = EngineOptions(dtype="bfloat16", page_size=args.page_size, batch_max=n_req, max_model_len=longest,
                         max_tokens=sum(l + gen + 64 for l in lengths), max_step_tokens=max(args.step_tokens, chunk), prefill_batch=chunk)
    llm = LLM(model, dtype="bfloat16", options=opts)
    llm.engine.cache.shuffle_free(0)
    prompts = [rng.integers(0, cfg.vocab_size, size=n).tolist() for n in lengths]
    sp = SamplingParams(temperature=0.0, max_tokens=gen, ignore_eos=True)
    pk = peaks()
    # warm-up: a short run of the same kind, so that modules are loaded, graphs of the first buckets are captured and
    # the workspace has its size
    llm.generate([p[:300] for p in prompts[:min(4, n_req)]], SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True))
    llm.warm_up()
    clocks = ClockSampler(0)
    llm.record_steps = True
    llm.step_records.clear()
    for p in prompts:
        llm.add_request(p, sp)
    contexts = []           # per step: (tokens, sum over entries of count * (start + (count + 1) / 2), live context tokens)
    sched_plan = llm.scheduler.schedule
    seen = []

    def watching():
        plan = sched_plan()
        seen.append(plan)
        return plan
    llm.scheduler.schedule = watching
    torch.cuda.synchronize()
    clocks.active = True
    t0 = time.perf_counter()
    done = llm.run_until_done()
    wall = time.perf_counter() - t0
    clocks.active = False
    clocks.close()
    llm.scheduler.schedule = sched_plan
    recs = llm.step_records
    dev_ms = [r.start.elapsed_time(r.end) for r in recs]
    device_s = sum(dev_ms) / 1000.0
    n_prompt, n_gen = sum(lengths), sum(len(o.token_ids) for o in done.values())
    # the steps' bound: every weight once, the live requests' cache, and the arithmetic, whichever is larger
    per_layer = (cfg.q_size + 2 * cfg.kv_size) * cfg.hidden_size + cfg.hidden_size * cfg.q_size + 3 * cfg.intermediate_size * cfg.hidden_size
    weight_bytes = 2 * (L * per_layer + cfg.vocab_size * cfg.hidden_size)
    kv_bytes_per_token = L * 2 * cfg.kv_size * 2
    plans = [p for p in seen if p]
    ideal_s, prefill_dev, decode_dev, mixed = 0.0, 0.0, 0.0, 0
    for plan, ms in zip(plans, dev_ms):
        T = sum(s.count for s in plan)
        ctx = sum(s.start + s.count for s in plan)
        pairs = sum(s.count * (s.start + (s.count + 1) / 2.0) for s in plan)
        flops = 2.0 * T * L * per_layer + 2.0 * sum(1 for s in plan if s.wants_token) * cfg.vocab_size * cfg.hidden_size \
            + L * 4.0 * cfg.num_attention_heads * cfg.head_dim * pairs
        byts = weight_bytes + ctx * kv_bytes_per_token
        ideal_s += max(byts / (pk["hbm_gbs"] * 1e9), flops / (pk["bf16_tflops_sustained"] * 1e12))
        if all(s.count == 1 for s in plan):
            decode_dev += ms
        else:
            prefill_dev += ms
            mixed += 1 if any(s.count == 1 for s in plan) else 0
    m = [o.metrics for o in done.values()]
    rec = {
        "metric": f"tokens/s (prompt + generated) of the workload, {label} bf16", "value": round((n_prompt + n_gen) / wall, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": len(recs), "warmup": 1, "ms_per_step": round(1000 * wall / max(1, len(recs)), 3),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights, uniform random token ids; " + what, "impl": "ours", "workload": args.workload,
        "config": {"model": label, "layers": L, "layers_of_model": full_layers, "hidden": cfg.hidden_size,
                   "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size, "requests": n_req, "generate": gen,
                   "prompt_tokens": n_prompt, "prefill_batch": chunk, "max_step_tokens": opts.max_step_tokens,
                   "page_size": args.page_size, "pages": "scattered", "parallelism": "single GPU", "peaks": pk["source"]},
        "wall_s": round(wall, 4), "device_s": round(device_s, 4), "wall_over_device": round(wall / device_s, 4),
        "prompt_tok_s": round(n_prompt / wall, 1), "generated_tok_s": round(n_gen / wall, 1),
        "steps_with_prompt_portions": {"steps": sum(1 for p in plans if any(s.count > 1 for s in p)), "of_them_mixed": mixed,
                                       "device_ms": round(prefill_dev, 2)},
        "decode_only_steps": {"steps": sum(1 for p in plans if all(s.count == 1 for s in p)), "device_ms": round(decode_dev, 2)},
        "roofline": {"bound": "per step max(bytes / HBM, flops / sustained bf16)", "ideal_s": round(ideal_s, 4),
                     "frac_of_device_time": round(ideal_s / device_s, 4), "frac_of_wall": round(ideal_s / wall, 4)},
        "requests": {"ttft_ms_mean": round(sum(x.ttft_ms for x in m) / len(m), 1), "ttft_ms_max": round(max(x.ttft_ms for x in m), 1),
                     "tpot_ms_mean": round(sum(x.tpot_ms for x in m) / len(m), 2), "preemptions": int(llm.scheduler.num_preemptions)},
        "gpu_launches": int(llm.engine.native_launches + llm.engine.graph_launches), "clocks": clocks.summary(),
    }
    print(json.dumps(rec))
    return 0


ZIDIVIK_SIZES = {
    # width, heads, kv heads, head sizes, window, experts x ff (top 4), delta heads, ranks, side dim, vocab
    "a": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, window=1024, keep=4, experts=32, top=4, ff=768,
              d_heads=16, d_kv=4, rank=64, side=128, vocab=32000),
    "b": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, window=2048, keep=4, experts=64, top=4, ff=1024,
              d_heads=32, d_kv=8, rank=128, side=256, vocab=64000),
}


def zidivik_raw(z):
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "scale": z["dim"] ** -0.5,
           "mask": {"size": z["window"], "keep_first": z["keep"]}}
    dlt = {"heads": z["d_heads"], "kv_heads": z["d_kv"], "dim": z["dim"], "vdim": z["vdim"], "conv": 4, "decay_rank": z["rank"], "gate_rank": z["rank"]}
    mlp = {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["ff"], "limit": 7.0}}
    layers = [{"type": "attention", "mixer": att, "mlp": mlp}, {"type": "attention", "mixer": dict(att, kv_from=0), "mlp": mlp},
              {"type": "channel_delta", "mixer": dlt, "mlp": mlp}, {"type": "attention", "mixer": att, "mlp": mlp}]
    return {"architecture": "Zidivik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "token_side": {"dim": z["side"]},
            "max_positions": 8192, "layers": layers}


TIDAVIK_SIZES = {
    # width, heads, kv heads, head sizes, window, ranks of the latent layer, feed-forward, vocab
    "a": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, window=1024, q_rank=768, kv_rank=256, ff=6144, vocab=32000),
    "b": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, window=2048, q_rank=1536, kv_rank=256, ff=12288, vocab=64000),
}


def tidavik_raw(z):
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "scale": z["dim"] ** -0.5, "softcap": 50.0,
           "mask": {"size": z["window"]}}
    lat = {"heads": z["heads"], "dim": z["dim"], "vdim": z["vdim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"], "scale": z["dim"] ** -0.5,
           "mask": {"size": z["window"]}}
    mlp = {"kind": "dense", "ff": z["ff"]}
    layers = [{"type": "attention", "mixer": att, "mlp": mlp}, {"type": "attention_2", "mixer": att, "mlp": mlp},
              {"type": "latent_attention", "mixer": lat, "mlp": mlp}, {"type": "attention_2", "mixer": att, "mlp": mlp}]
    return {"architecture": "Tidavik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "max_positions": 8192, "layers": layers}


TOREDRA_SIZES = {
    # width, attention heads / kv heads x head sizes, rotated dimensions, recurrence heads x key / value size, delta heads x size, rank of
    # the decay's projection, feed-forward (two matrices: as many weights as a gated one of two thirds the size), vocab
    "a": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, rot=64, r_heads=16, r_dim=64, r_vdim=128, d_heads=16, d_dim=128, rank=64,
              ff=9216, vocab=32000),
    "b": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, rot=64, r_heads=32, r_dim=64, r_vdim=128, d_heads=32, d_dim=128, rank=128,
              ff=18432, vocab=64000),
}


def toredra_raw(z):
    par = {"left": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "scale": z["dim"] ** -0.5,
                    "rot": {"dims": z["rot"], "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}},
           "right": {"heads": z["r_heads"], "dim": z["r_dim"], "vdim": z["r_vdim"]}}
    dlt = {"heads": z["d_heads"], "dim": z["d_dim"], "decay_rank": z["rank"]}
    mlp = {"kind": "dense", "ff": z["ff"]}
    layers = [{"type": "parallel", "mixer": par, "mlp": mlp}, {"type": "general_delta", "mixer": dlt, "mlp": mlp},
              {"type": "general_delta", "mixer": dlt, "mlp": mlp}, {"type": "parallel", "mixer": par, "mlp": mlp}]
    return {"architecture": "Toredra", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "max_positions": 8192,
            "logit_scale": 0.5, "logit_softcap": 30.0, "layers": layers}


KORIRAX_SIZES = {
    # width, attention heads / kv heads x head sizes, rows of the distance table, latent heads x (unrotated + rotated) / value size and ranks,
    # recurrence channels and blocks, dense feed-forward, experts x ff (top 4 of groups) and the shared expert, token input, vocab
    "a": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, rows=32, l_heads=16, l_dim=128, l_rot=64, l_vdim=128, q_rank=768, kv_rank=192,
              channels=2048, blocks=16, ff=6144, experts=32, top=4, e_ff=768, groups=4, keep=2, shared=768, side=128, vocab=32000),
    "b": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, rows=32, l_heads=32, l_dim=128, l_rot=64, l_vdim=128, q_rank=1536, kv_rank=192,
              channels=4096, blocks=16, ff=12288, experts=64, top=4, e_ff=1024, groups=8, keep=4, shared=1024, side=256, vocab=64000),
}


def korirax_raw(z):
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "scale": z["dim"] ** -0.5, "bias_max": 512,
           "bias_rows": z["rows"], "q_temp": {"coef": 0.1, "every": 1024}}
    lat = {"heads": z["l_heads"], "dim": z["l_dim"], "rot_dim": z["l_rot"], "vdim": z["l_vdim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"],
           "scale": (z["l_dim"] + z["l_rot"]) ** -0.5,
           "rot": {"dims": z["l_rot"], "base": 10000.0, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    rec = {"width": z["channels"], "blocks": z["blocks"], "conv": 4}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["e_ff"]}, "router": {"experts": z["experts"], "top": z["top"], "scale": 2.5,
                                                                  "groups": {"count": z["groups"], "keep": z["keep"]}}, "shared": {"ff": z["shared"]}}
    layers = [{"type": "attention", "mixer": att, "mlp": dense}, {"type": "latent_attention", "mixer": lat, "mlp": moe},
              {"type": "rglru", "mixer": rec, "mlp": dense}, {"type": "latent_attention", "mixer": lat, "mlp": moe}]
    return {"architecture": "Korirax", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "token_side": {"dim": z["side"]}, "max_positions": 8192, "layers": layers}


TUGANEX_SIZES = {
    # width, attention heads / kv heads x (map, value) sizes, rotated dimensions of a map, recurrence heads x key / value size, dense feed-forward
    # (two matrices), experts x ff (top of experts + identity outputs in groups) and the shared expert, vocab
    "a": dict(width=2048, heads=16, kv_heads=4, dim=64, vdim=128, rot=64, r_heads=16, r_dim=128, r_vdim=128, ff=9216, experts=32, identity=8, top=4,
              e_ff=768, groups=4, keep=2, shared=768, vocab=32000),
    "b": dict(width=4096, heads=32, kv_heads=8, dim=64, vdim=128, rot=64, r_heads=32, r_dim=128, r_vdim=128, ff=18432, experts=64, identity=16, top=4,
              e_ff=1024, groups=8, keep=4, shared=1024, vocab=64000),
}


def tuganex_raw(z):
    rot = {"dims": z["rot"], "base": 500000.0}
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "scale": z["dim"] ** -0.5, "diff": 0.5, "rot": rot}
    # decays from a memory of 32 tokens to one of 4,096, as far apart as the heads are many
    ret = {"heads": z["r_heads"], "dim": z["r_dim"], "vdim": z["r_vdim"], "decay": [1.0 - 2.0 ** (-5 - 7.0 * h / (z["r_heads"] - 1)) for h in range(z["r_heads"])],
           "rot": {"dims": z["r_dim"], "base": 10000.0}}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["e_ff"]}, "router": {"experts": z["experts"], "identity": z["identity"], "top": z["top"],
                                                                  "groups": {"count": z["groups"], "keep": z["keep"]}}, "shared": {"ff": z["shared"]}}
    layers = [{"type": "attention", "mixer": att, "mlp": dense}, {"type": "attention", "mixer": att, "mlp": moe},
              {"type": "retention", "mixer": ret, "mlp": dense}, {"type": "attention", "mixer": dict(att, kv_from=1), "mlp": moe}]
    return {"architecture": "Tuganex", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "max_positions": 8192, "layers": layers}


FASANEX_SIZES = {
    # width, attention heads / kv heads x size and window, time-mixing heads x size and decay rank, state-space heads x value size, state, groups,
    # delta heads / key heads x key / value size, feed-forward, vocab
    "a": dict(width=2048, heads=16, kv_heads=4, dim=128, window=1024, t_heads=32, t_dim=64, rank=64, s_heads=64, s_vdim=64, s_state=128, s_groups=8,
              d_heads=16, d_kv=8, d_dim=128, d_vdim=128, ff=6144, vocab=32000),
    "b": dict(width=4096, heads=32, kv_heads=8, dim=128, window=2048, t_heads=64, t_dim=64, rank=128, s_heads=128, s_vdim=64, s_state=128, s_groups=8,
              d_heads=32, d_kv=16, d_dim=128, d_vdim=128, ff=12288, vocab=64000),
}


def fasanex_raw(z):
    left = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "conv": 4, "scale": z["dim"] ** -0.5, "softcap": 30.0,
            "mask": {"size": z["window"]}, "rot": {"dims": z["dim"], "base": 500000.0, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    par = {"left": left, "right": {"heads": z["t_heads"], "dim": z["t_dim"], "decay_rank": z["rank"]}, "left_scale": 0.8, "right_scale": 1.1}
    ssm = {"heads": z["s_heads"], "vdim": z["s_vdim"], "state": z["s_state"], "groups": z["s_groups"], "norm_groups": z["s_groups"], "conv": 4}
    dlt = {"heads": z["d_heads"], "kv_heads": z["d_kv"], "dim": z["d_dim"], "vdim": z["d_vdim"], "conv": 4}
    mlp = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    layers = [{"type": "mamba2", "mixer": ssm, "mlp": mlp}, {"type": "parallel", "mixer": par, "mlp": mlp}, {"type": "delta", "mixer": dlt, "mlp": mlp},
              {"type": "parallel", "mixer": par, "mlp": mlp}]
    return {"architecture": "Fasanex", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 12.0}, "max_positions": 8192,
            "layers": layers}


def run_zidivik(args) -> int:
    """Prefill and decode of the Zidivik, the Tidavik, the Toredra, the Korirax, the Tuganex or the Fasanex decoder at real layer sizes, beside the Qwen3 dense decoder of equal size."""
    import numpy as np
    import torch
    from kestrel_llm_b200.config import EngineOptions, Qwen3Config, TidavikConfig, ToredraConfig, ZidivikConfig
    from kestrel_llm_b200.config.korirax_config import KoriraxConfig
    from kestrel_llm_b200.config.tuganex_config import TuganexConfig
    from kestrel_llm_b200.config.fasanex_config import FasanexConfig
    from kestrel_llm_b200.config.registry import resolve_architecture
    from kestrel_llm_b200.csrc import ops
    from kestrel_llm_b200.engine import Engine, Entry
    from kestrel_llm_b200.weights import fill_random_

    dev = "cuda:0"
    torch.cuda.set_device(0)
    tidavik, toredra, korirax = args.workload == "tidavik", args.workload == "toredra", args.workload == "korirax"
    tuganex = args.workload == "tuganex"
    fasanex = args.workload == "fasanex"
    z = (FASANEX_SIZES if fasanex else TUGANEX_SIZES if tuganex else KORIRAX_SIZES if korirax else TOREDRA_SIZES if toredra else TIDAVIK_SIZES if tidavik else ZIDIVIK_SIZES)[args.size]
    T, B, CTX = args.prefill_tokens, args.batch, 2048
    W, K = max(3, args.warmup), max(1, min(args.steps, 32))
    pk = peaks()
    clocks = ClockSampler(0)
    rng = np.random.default_rng(0)
    timed_names = ["linear", "add_rmsnorm", "attn_prepare", "attn_prepare_ex", "attention", "attention_plain_ex", "attention_window", "qkv_prepare_fused",
                   "gate_up_swiglu", "moe_route", "moe_experts", "short_conv", "delta_gates", "delta_scan", "delta_out", "partial_columns",
                   "add_two", "gelu_table_mul", "add_normed", "embed", "add_sinusoid", "linear_add_into", "latent_prepare", "head_gemm", "attention_tc",
                   "forget_gates", "removal_gates", "recurrence_scan", "head_norm_gate", "combine_normed", "add_gated_normed", "partial_columns_act",
                   "embed_add", "logit_scale_cap", "linear_act", "rglru_branches", "rglru_scan", "moe_route_sigmoid", "moe_experts_ungated",
                   "gate_columns_mul", "latent_rotate_queries", "add_row", "differential_combine", "retention_prepare", "retention_step", "retention_chunks",
                   "moe_route_scored", "attention_tc_maps", "attention_window_maps", "attention_decode_maps", "post_norm_add", "embed_copy",
                   "attn_prepare_conv", "token_shift", "linear_groups", "time_mix_gates", "recurrence_scan_bonus", "ssm_expand", "ssm_out", "ssm_step", "ssm_chunks", "part_norm", "delta_head_step",
                   "delta_chunks", "time_mix_step", "time_mix_chunks", "post_norm_add_norm", "attention_decode_capped"]

    def measure(cfg, label):
        model = resolve_architecture(cfg.architecture).build(cfg, torch.bfloat16, dev)
        fill_random_(model, 0)
        for b in model.blocks:                  # decays and gates of a trained model's size, not of N(0, 0.02)
            m = b.mixer
            if hasattr(m, "dt_bias"):
                m.dt_bias.normal_(-1.0, 1.0)
                m.A_log.normal_(-0.5, 0.5)
            for r in (m, getattr(m, "right", None)):        # forget gates and decays that keep a state for hundreds of tokens
                if hasattr(r, "f_bias"):
                    r.f_bias.normal_(2.0, 1.0)
                if hasattr(r, "w0"):
                    r.w0.normal_(-1.0, 1.0)
            if hasattr(m, "lam"):               # decays that keep a state for hundreds of tokens
                m.lam.normal_(-4.0, 1.0)
        opts = EngineOptions(dtype="bfloat16", page_size=args.page_size, batch_max=B + 1, max_model_len=CTX + T + 64,
                             max_tokens=B * (CTX + 128) + T + 64, max_step_tokens=max(T, B), prefill_batch=T)
        engine = Engine(model, opts)
        engine.cache.shuffle_free(0)
        for t in engine.cache.k + engine.cache.v:
            if t is not None:
                t.normal_(0.0, 0.5)

        def timed(fn, n):
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            for _ in range(n):
                fn()
            b.record()
            torch.cuda.synchronize()
            return a.elapsed_time(b) / 1000.0

        clocks.active = True                     # the timed regions are milliseconds long: sample over the whole measurement
        counter = {"i": 0}

        def prefill():
            counter["i"] += 1
            toks = rng.integers(0, cfg.vocab_size, size=T).tolist()
            engine.step([Entry(5000 + counter["i"], toks, (T - 1,))])
            engine.release(5000 + counter["i"])
        for _ in range(3):
            prefill()
        pre = min(timed(prefill, 5) / 5 for _ in range(4))      # the host prepares 2,048 ids a step: the best of four rounds of five
        rids = list(range(100, 100 + B))
        ctx0 = CTX - (W + K)
        for r in rids:                           # a context whose pages hold random values and whose state slots are as a prompt left them
            engine.admit(r)
            engine.cache.reserve(r, ctx0)
            engine.cache.commit(r, ctx0)
        engine.cache.clear_admitted()
        nxt = torch.from_numpy(rng.integers(0, cfg.vocab_size, size=B).astype(np.int32)).to(dev)

        def decode():
            if engine.graphs is not None:
                logits = engine.step([Entry(r, (0,), (0,)) for r in rids], token_ids_dev=nxt)
            else:
                logits = engine.step([Entry(r, (int(t),), (0,)) for r, t in zip(rids, nxt.tolist())])
            ops.argmax(logits, nxt)
        for _ in range(W):
            decode()
        before = ops.launches + engine.graph_launches + engine.native_launches
        dec = timed(decode, K) / K
        launches = (ops.launches + engine.graph_launches + engine.native_launches - before) // K
        if not clocks.rows:                      # the timed regions were shorter than the sampler's period: the same steps
            until = time.time() + 0.7            # once more, untimed, so that the record has clocks under this load; decode
            extra = 0                            # steps while the requests' page head-room lasts, prompt steps after that
            while time.time() < until:
                if extra < 64:
                    decode()
                else:
                    prefill()
                extra += 1
            torch.cuda.synchronize()

        # device time per kind of operation, one step of each
        split = {}
        if True:
            saved, acc = {}, {}

            def wrap(name, fn):
                def inner(*a, **kw):
                    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                    e0.record()
                    out = fn(*a, **kw)
                    e1.record()
                    acc.setdefault(name, []).append((e0, e1))
                    return out
                return inner
            for name in timed_names:
                if hasattr(ops, name):
                    saved[name] = getattr(ops, name)
                    setattr(ops, name, wrap(name, saved[name]))
            graphs, engine.graphs = engine.graphs, None
            runner, engine.runner = engine.runner, None        # the parts' forward methods from Python: the same kernels
            for what, fn in (("prefill", prefill), ("decode", decode)):
                fn()                                 # once untimed: what this walk does for the first time (tensor maps, attributes)
                torch.cuda.synchronize()
                acc.clear()
                fn()
                torch.cuda.synchronize()
                split[what] = {n: round(sum(a.elapsed_time(b) for a, b in ev) * 1000.0, 1) for n, ev in acc.items()}
            engine.graphs, engine.runner = graphs, runner
            for name, fn in saved.items():
                setattr(ops, name, fn)
        clocks.active = False
        for r in rids:
            engine.release(r)
        del engine, model
        torch.cuda.empty_cache()
        return {"model": label, "prefill_tokens": T, "prefill_ms": round(1000 * pre, 3), "prefill_tok_s": round(T / pre, 1),
                "decode_batch": B, "decode_context": CTX, "decode_ms": round(1000 * dec, 4), "decode_tok_s": round(B / dec, 1),
                "launches_per_decode_step": int(launches), "device_us_per_operation": split}

    raw = fasanex_raw(z) if fasanex else tuganex_raw(z) if tuganex else korirax_raw(z) if korirax else toredra_raw(z) if toredra else tidavik_raw(z) if tidavik else zidivik_raw(z)
    zc = (FasanexConfig if fasanex else TuganexConfig if tuganex else KoriraxConfig if korirax else ToredraConfig if toredra else TidavikConfig if tidavik else ZidivikConfig).from_dict(raw)
    L = len(raw["layers"])
    dense_raw = dict(QWEN3_8B, num_hidden_layers=L, hidden_size=z["width"], num_attention_heads=z["heads"],
                     num_key_value_heads=z["kv_heads"], head_dim=z["vdim"] if tuganex else z["dim"],
                     intermediate_size=(z["ff"] * 2 // 3 + z["top"] * z["e_ff"] + z["shared"]) // 2 // 256 * 256 if tuganex else
                     (z["ff"] + (z["top"] * z["e_ff"] + z["shared"]) * 2 // 3) // 2 // 256 * 256 if korirax else
                     z["ff"] * 2 // 3 if toredra else z["ff"] if tidavik or fasanex else z["top"] * z["ff"],
                     vocab_size=z["vocab"], max_position_embeddings=8192)
    if tidavik or fasanex:                   # the dense model's layers look through the same window
        dense_raw.update(sliding_window=z["window"], use_sliding_window=True, layer_types=["sliding_attention"] * L)
    qc = Qwen3Config.from_dict(dense_raw)
    ours = measure(zc, "Fasanex" if fasanex else "Tuganex" if tuganex else "Korirax" if korirax else "Toredra" if toredra else "Tidavik" if tidavik else "Zidivik")
    dense = measure(qc, "Qwen3 dense, equal size" + (" and window" if tidavik or fasanex else ""))
    clocks.close()
    if fasanex:
        D, H, G, d, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["ff"]
        inner, gn, tn, dq, dvv = z["s_heads"] * z["s_vdim"], z["s_groups"] * z["s_state"], z["t_heads"] * z["t_dim"], z["d_kv"] * z["d_dim"], z["d_heads"] * z["d_vdim"]
        ssm_w = D * (2 * inner + 2 * gn + z["s_heads"]) + inner * D
        par_w = D * (2 * H * d + G * d) + 4 * D * tn + z["rank"] * (D + tn) + (H * d + tn) * D
        dlt_w = D * (2 * dq + 2 * dvv + 2 * z["d_heads"]) + dvv * D
        active = ssm_w + 2 * par_w + dlt_w + L * 3 * ff * D
        win = min(z["window"], T)
        pairs = win * (win + 1) / 2 + (T - win) * win           # (query, key) pairs inside the window
        state = z["s_heads"] * z["s_state"] * z["s_vdim"] + 2 * tn * z["t_dim"] + z["d_heads"] * z["d_dim"] * z["d_vdim"]
        # products, attention, and the recurrences' three passes over their states a token
        flops_prefill = 2.0 * T * active + 2 * 4.0 * H * d * pairs + 6.0 * T * state
        cache_bytes = 2.0 * B * min(CTX, z["window"]) * 2 * G * 2 * d
        rec = {"metric": f"Fasanex prefill tokens/s at size {args.size}, bf16, beside Qwen3 dense of equal size", "value": ours["prefill_tok_s"],
               "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": ours["prefill_ms"], "higher_is_better": True,
               "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "impl": "ours", "workload": "fasanex",
               "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
               "config": dict(z, layers=[l["type"] + "+" + l["mlp"]["kind"] for l in raw["layers"]], page_size=args.page_size, peaks=pk["source"],
                              parallelism="single GPU"),
               "fasanex": ours, "dense": dense,
               "ratio_to_dense": {"prefill": round(ours["prefill_tok_s"] / dense["prefill_tok_s"], 3), "decode": round(ours["decode_tok_s"] / dense["decode_tok_s"], 3)},
               "prefill_flops_frac_of_peak": round(flops_prefill / (ours["prefill_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
               "decode_bytes_frac_of_hbm": round((2.0 * (active + z["vocab"] * D) + 8.0 * B * state + cache_bytes) / (ours["decode_ms"] / 1000.0) / (pk["hbm_gbs"] * 1e9), 4),
               "gpu_launches": ours["launches_per_decode_step"] * K, "clocks": clocks.summary()}
        print(json.dumps(rec))
        return 0
    if tuganex:
        D, H, G, d, dv, ff, n = z["width"], z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["ff"], z["experts"] + z["identity"]
        q_w, kv_w, o_w = D * H * 2 * d, D * G * (2 * d + dv), H * dv * D
        rq, rv = z["r_heads"] * z["r_dim"], z["r_heads"] * z["r_vdim"]
        mixers = 3 * (q_w + o_w) + 2 * kv_w + D * (2 * rq + 2 * rv) + rv * D
        share = z["experts"] / n                 # of a token's choices, those that are experts with matrices (random router)
        moe_fixed = 3 * z["shared"] * D + (n + 1) * D
        active = mixers + 2 * 2 * ff * D + 2 * (3 * z["e_ff"] * D * z["top"] * share + moe_fixed)
        touched = mixers + 2 * 2 * ff * D + 2 * (3 * z["e_ff"] * D * min(z["experts"], B * z["top"] * share) + moe_fixed) + z["vocab"] * D
        # products, two causal maps a head over one value each (half of the T x T scores), three passes over a head's state a token
        flops_prefill = 2.0 * T * active + 3 * 2.0 * H * (2 * d + 2 * dv) * T * T / 2 + T * 6.0 * rq * z["r_vdim"]
        state_bytes, cache_bytes = 4.0 * B * rq * z["r_vdim"] * 2, 2.0 * B * CTX * 3 * G * (2 * d + dv)
        rec = {"metric": f"Tuganex prefill tokens/s at size {args.size}, bf16, beside Qwen3 dense of equal size", "value": ours["prefill_tok_s"],
               "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": ours["prefill_ms"], "higher_is_better": True,
               "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "impl": "ours", "workload": "tuganex",
               "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
               "config": dict(z, layers=[l["type"] + ("/shared keys" if "kv_from" in l["mixer"] else "") + "+" + l["mlp"]["kind"] for l in raw["layers"]],
                              page_size=args.page_size, peaks=pk["source"], parallelism="single GPU"),
               "tuganex": ours, "dense": dense,
               "ratio_to_dense": {"prefill": round(ours["prefill_tok_s"] / dense["prefill_tok_s"], 3), "decode": round(ours["decode_tok_s"] / dense["decode_tok_s"], 3)},
               "prefill_flops_frac_of_peak": round(flops_prefill / (ours["prefill_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
               "decode_bytes_frac_of_hbm": round((2.0 * touched + state_bytes + cache_bytes) / (ours["decode_ms"] / 1000.0) / (pk["hbm_gbs"] * 1e9), 4),
               "gpu_launches": ours["launches_per_decode_step"] * K, "clocks": clocks.summary()}
        print(json.dumps(rec))
        return 0
    if korirax:
        D, H, G, d, dv, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["ff"]
        LH, ld, lr, lv, qr, kr, C = z["l_heads"], z["l_dim"], z["l_rot"], z["l_vdim"], z["q_rank"], z["kv_rank"], z["channels"]
        att_w = D * (H * d + G * (d + dv) + H * dv) + H * dv * D
        lat_w = D * (qr + kr + lr + LH * lv) + qr * LH * (ld + lr) + LH * ld * kr + LH * lv * kr + LH * lv * D
        rec_w = D * 2 * C + 2 * C * (C // z["blocks"]) + C * D
        moe_active = 2 * z["e_ff"] * D * z["top"] + 2 * z["shared"] * D + z["experts"] * D
        moe_touched = 2 * z["e_ff"] * D * min(z["experts"], B * z["top"]) + 2 * z["shared"] * D + z["experts"] * D      # a decode step of B tokens
        side_w = L * 2 * z["side"] * D
        mixers = att_w + 2 * lat_w + rec_w
        active = mixers + 2 * 3 * ff * D + 2 * moe_active + side_w
        touched = mixers + 2 * 3 * ff * D + 2 * moe_touched + side_w + z["vocab"] * D
        row = kr + lr
        # products, causal attention (half of the T x T scores; the latent layers over rows of kv_rank + rot_dim for keys and values alike)
        flops_prefill = 2.0 * T * active + 2.0 * H * (d + dv) * T * T / 2 + 2 * 2.0 * LH * 2 * row * T * T / 2
        cache_bytes = 2.0 * B * CTX * (G * (d + dv) + 2 * row)
        rec = {"metric": f"Korirax prefill tokens/s at size {args.size}, bf16, beside Qwen3 dense of equal size", "value": ours["prefill_tok_s"],
               "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": ours["prefill_ms"], "higher_is_better": True,
               "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "impl": "ours", "workload": "korirax",
               "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
               "config": dict(z, layers=[l["type"] + "+" + l["mlp"]["kind"] for l in raw["layers"]], page_size=args.page_size, peaks=pk["source"],
                              parallelism="single GPU"),
               "korirax": ours, "dense": dense,
               "ratio_to_dense": {"prefill": round(ours["prefill_tok_s"] / dense["prefill_tok_s"], 3), "decode": round(ours["decode_tok_s"] / dense["decode_tok_s"], 3)},
               "prefill_flops_frac_of_peak": round(flops_prefill / (ours["prefill_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
               "decode_bytes_frac_of_hbm": round((2.0 * touched + cache_bytes) / (ours["decode_ms"] / 1000.0) / (pk["hbm_gbs"] * 1e9), 4),
               "gpu_launches": ours["launches_per_decode_step"] * K, "clocks": clocks.summary()}
        print(json.dumps(rec))
        return 0
    if toredra:
        D, H, G, d, dv, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["ff"]
        rn, rv, dn = z["r_heads"] * z["r_dim"], z["r_heads"] * z["r_vdim"], z["d_heads"] * z["d_dim"]
        par_w = D * (H * d + G * (d + dv)) + H * dv * D + D * (2 * rn + rv) + rv * D
        dlt_w = D * (5 * dn + z["rank"]) + z["rank"] * dn + dn * D
        n_par = sum(1 for l in raw["layers"] if l["type"] == "parallel")
        weights = n_par * par_w + (L - n_par) * dlt_w + L * (2 * ff * D + 2 * D * D) + z["vocab"] * D
        # products, causal attention (half of the T x T scores), and the scans' three (delta rule: five) passes over each head's state a token
        flops_prefill = 2.0 * T * (weights - z["vocab"] * D) + n_par * 2.0 * H * (d + dv) * T * T / 2 + \
            T * (n_par * 6.0 * rn * z["r_vdim"] + (L - n_par) * 10.0 * dn * z["d_dim"])
        state_bytes = 4.0 * B * (n_par * rn * z["r_vdim"] + (L - n_par) * dn * z["d_dim"]) * 2        # read and written every decode step
        cache_bytes = 2.0 * B * CTX * n_par * G * (d + dv)
        rec = {"metric": f"Toredra prefill tokens/s at size {args.size}, bf16, beside Qwen3 dense of equal size", "value": ours["prefill_tok_s"],
               "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": ours["prefill_ms"], "higher_is_better": True,
               "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "impl": "ours", "workload": "toredra",
               "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
               "config": dict(z, layers=[l["type"] for l in raw["layers"]], page_size=args.page_size, peaks=pk["source"], parallelism="single GPU"),
               "toredra": ours, "dense": dense,
               "ratio_to_dense": {"prefill": round(ours["prefill_tok_s"] / dense["prefill_tok_s"], 3), "decode": round(ours["decode_tok_s"] / dense["decode_tok_s"], 3)},
               "prefill_flops_frac_of_peak": round(flops_prefill / (ours["prefill_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
               "decode_bytes_frac_of_hbm": round((2.0 * weights + state_bytes + cache_bytes) / (ours["decode_ms"] / 1000.0) / (pk["hbm_gbs"] * 1e9), 4),
               "gpu_launches": ours["launches_per_decode_step"] * K, "clocks": clocks.summary()}
        print(json.dumps(rec))
        return 0
    if tidavik:
        D, H, G, d, dv, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["vdim"], z["ff"]
        grouped_w = D * (H * d + G * (d + dv)) + H * dv * D
        latent_w = D * (z["q_rank"] + z["kv_rank"] + H) + z["q_rank"] * H * d + H * d * z["kv_rank"] + H * dv * z["kv_rank"] + H * dv * D
        weights = 3 * grouped_w + latent_w + L * 3 * ff * D + z["vocab"] * D
        seen = min(T, z["window"])
        attn = 3 * 2.0 * H * (d + dv) * T * seen + 2.0 * H * 2 * z["kv_rank"] * T * seen       # all keys of the window for every query: an upper bound
        flops_prefill = 2.0 * T * (weights - z["vocab"] * D) + attn
        rec = {"metric": f"Tidavik prefill tokens/s at size {args.size}, bf16, beside Qwen3 dense of equal size", "value": ours["prefill_tok_s"],
               "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": ours["prefill_ms"], "higher_is_better": True,
               "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "impl": "ours", "workload": "tidavik",
               "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
               "config": dict(z, layers=[l["type"] for l in raw["layers"]], page_size=args.page_size, peaks=pk["source"], parallelism="single GPU"),
               "tidavik": ours, "dense": dense,
               "ratio_to_dense": {"prefill": round(ours["prefill_tok_s"] / dense["prefill_tok_s"], 3), "decode": round(ours["decode_tok_s"] / dense["decode_tok_s"], 3)},
               "prefill_flops_frac_of_peak": round(flops_prefill / (ours["prefill_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
               "decode_weight_bytes_frac_of_hbm": round(2.0 * weights / (ours["decode_ms"] / 1000.0) / (pk["hbm_gbs"] * 1e9), 4),
               "gpu_launches": ours["launches_per_decode_step"] * K, "clocks": clocks.summary()}
        print(json.dumps(rec))
        return 0
    # what a Zidivik step has to do: the weights it touches once, and its arithmetic
    D, ff, top, E = z["width"], z["ff"], z["top"], z["experts"]
    att_w = D * (z["heads"] * z["dim"] + z["kv_heads"] * (z["dim"] + z["vdim"]) + z["heads"]) + z["heads"] * z["vdim"] * D
    moe_active = 3 * ff * D * top
    flops_prefill = 2.0 * T * (L * (att_w + moe_active + E * D)) + L * 4.0 * z["heads"] * z["dim"] * T * min(T, z["window"])
    rec = {"metric": f"Zidivik prefill tokens/s at size {args.size}, bf16, beside Qwen3 dense of equal size", "value": ours["prefill_tok_s"],
           "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": ours["prefill_ms"], "higher_is_better": True,
           "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "impl": "ours", "workload": "zidivik",
           "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
           "config": dict(z, layers=[l["type"] + ("/shared keys" if "kv_from" in l["mixer"] else "") for l in raw["layers"]],
                          page_size=args.page_size, peaks=pk["source"], parallelism="single GPU"),
           "zidivik": ours, "dense": dense,
           "ratio_to_dense": {"prefill": round(ours["prefill_tok_s"] / dense["prefill_tok_s"], 3), "decode": round(ours["decode_tok_s"] / dense["decode_tok_s"], 3)},
           "prefill_flops_frac_of_peak": round(flops_prefill / (ours["prefill_ms"] / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
           "gpu_launches": ours["launches_per_decode_step"] * K, "clocks": clocks.summary()}
    print(json.dumps(rec))
    return 0


def main() -> int:
    global CONTEXT, PREFILL_TOKENS
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--layers", type=int, default=0, help="run this many layers of the model's 36 (0 = all)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--skip-points", action="store_true", help="leave out batch 1 and 64")
    ap.add_argument("--page-size", type=int, default=16, help="tokens per cache page (default 16)")
    ap.add_argument("--context", type=int, default=CONTEXT, help="context length at which the decode steps end (default 4096)")
    ap.add_argument("--prefill-tokens", type=int, default=PREFILL_TOKENS, help="tokens of the prefill step (default 2048)")
    ap.add_argument("--workload", default="decode8b", choices=["decode8b", "mix14b", "32b", "zidivik", "tidavik", "toredra", "korirax", "tuganex", "fasanex"],
                    help="decode8b: the headline run; mix14b / 32b: whole workloads through the scheduler; zidivik / tidavik / toredra / korirax / tuganex / fasanex: that decoder "
                         "at real layer sizes beside Qwen3 dense of equal size")
    ap.add_argument("--size", default="a", choices=sorted(ZIDIVIK_SIZES), help="layer sizes of --workload zidivik / tidavik / toredra / korirax / tuganex / fasanex")
    ap.add_argument("--requests", type=int, default=0, help="requests of a workload (0: 32 for mix14b, 16 for 32b)")
    ap.add_argument("--generate", type=int, default=0, help="tokens to generate per request of a workload (0: 256 / 128)")
    ap.add_argument("--step-tokens", type=int, default=2048,
                    help="token budget of a workload's step (the engine's default 2,048: up to four portions of 512 beside the decode tokens)")
    args = ap.parse_args()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": REFERENCE_UNAVAILABLE}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on ONE GPU; --gpus {args.gpus} is not supported (no multi-GPU path exists)")
        return 2
    if args.workload in ("zidivik", "tidavik", "toredra", "korirax", "tuganex", "fasanex"):
        return run_zidivik(args)
    if args.workload != "decode8b":
        return run_workload(args)
    W, K = max(3, args.warmup), max(1, args.steps)
    CONTEXT, PREFILL_TOKENS = max(256, args.context), max(16, args.prefill_tokens)      # the defaults unless asked otherwise

    import numpy as np
    import torch
    from kestrel_llm_b200 import LLM, SamplingParams
    from kestrel_llm_b200.config import EngineOptions, Qwen3Config
    from kestrel_llm_b200.config.registry import resolve_architecture
    from kestrel_llm_b200.csrc import ops
    from kestrel_llm_b200.engine import Entry
    from kestrel_llm_b200.weights import fill_random_

    raw = dict(QWEN3_8B)
    full_layers = raw["num_hidden_layers"]
    if args.layers:
        raw["num_hidden_layers"] = min(args.layers, full_layers)
    cfg = Qwen3Config.from_dict(raw)
    L = cfg.num_hidden_layers
    dev = "cuda:0"
    torch.cuda.set_device(0)
    model = resolve_architecture(cfg.architecture).build(cfg, torch.bfloat16, dev)
    fill_random_(model, 0)
    max_batch = 64 if not args.skip_points else max(args.batch, 1)
    longest = max(CONTEXT, PREFILL_TOKENS) + 64
    opts = EngineOptions(dtype="bfloat16", page_size=args.page_size, batch_max=max_batch, max_model_len=longest,
                         max_tokens=max(max_batch * (CONTEXT + 64), longest), max_step_tokens=max(PREFILL_TOKENS, max_batch),
                         prefill_batch=PREFILL_TOKENS)
    llm = LLM(model, dtype="bfloat16", options=opts)
    engine = llm.engine
    engine.cache.shuffle_free(0)                     # pages in a scattered order, as after long serving
    for t in engine.cache.k + engine.cache.v:        # cache contents for the synthetic contexts
        if t is not None:
            t.normal_(0.0, 0.5)
    rng = np.random.default_rng(0)
    pk = peaks()
    clocks = ClockSampler(0)

    # bytes a decode step has to read: every weight it uses once, and the live requests' cache
    esz = 2
    per_layer = (cfg.q_size + 2 * cfg.kv_size) * cfg.hidden_size + cfg.hidden_size * cfg.q_size \
        + 3 * cfg.intermediate_size * cfg.hidden_size
    weight_bytes = esz * (L * per_layer + cfg.vocab_size * cfg.hidden_size)
    kv_bytes_per_token = L * 2 * cfg.kv_size * esz

    def timed(fn, n):
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        clocks.active = True
        a.record()
        for _ in range(n):
            fn()
        b.record()
        torch.cuda.synchronize()
        clocks.active = False
        return a.elapsed_time(b) / 1000.0

    def decode_point(B):
        """K timed decode steps of B requests whose context ends at CONTEXT; device-timed, the
        step function called directly, tokens picked on the device."""
        ctx0 = CONTEXT - (W + K)
        rids = list(range(1000, 1000 + B))
        for r in rids:
            engine.admit(r)
            engine.cache.reserve(r, ctx0)       # a context of ctx0 tokens whose cache holds random values
            engine.cache.commit(r, ctx0)
        nxt = torch.from_numpy(rng.integers(0, cfg.vocab_size, size=B).astype(np.int32)).to(dev)
        entries = [Entry(r, (0,), (0,)) for r in rids]       # the ids are on the device: those the step before picked

        def one():
            logits = engine.step(entries, token_ids_dev=nxt)
            ops.argmax(logits, nxt)

        for _ in range(W):
            one()
        before = ops.launches + engine.graph_launches + engine.native_launches
        secs = timed(one, K)
        launched = ops.launches + engine.graph_launches + engine.native_launches - before
        for r in rids:
            engine.release(r)
        mean_ctx = ctx0 + W + (K - 1) / 2.0 + 1
        bytes_step = weight_bytes + B * mean_ctx * kv_bytes_per_token
        return {"tok_s": B * K / secs, "ms": 1000.0 * secs / K, "bytes_step": bytes_step, "launches": launched}

    # prefill of one 2,048-token prompt in one step (logits of the last token); measured first: it
    # is bound by the tensor cores, whose clock sinks under the power cap once the GPU has been busy
    # for seconds, and its fraction is taken against the burst figure of the peak
    def prefill_once(rid):
        toks = rng.integers(0, cfg.vocab_size, size=PREFILL_TOKENS).tolist()
        engine.step([Entry(rid, toks, (PREFILL_TOKENS - 1,))])
        engine.release(rid)
    for i in range(2):
        prefill_once(2000 + i)
    pre_runs = 3
    counter = {"i": 0}

    def pf():
        counter["i"] += 1
        prefill_once(2100 + counter["i"])
    pre_secs = timed(pf, pre_runs) / pre_runs
    T = PREFILL_TOKENS
    gemm_flops = 2.0 * T * L * per_layer + 2.0 * cfg.vocab_size * cfg.hidden_size     # head: one row
    attn_flops = L * 4.0 * cfg.num_attention_heads * cfg.head_dim * (T * (T + 1) / 2.0)
    pre_flops = gemm_flops + attn_flops
    prefill = {"value": round(T / pre_secs, 1), "tokens": T, "ms": round(1000 * pre_secs, 3),
               "frac": round(pre_flops / pre_secs / (pk["bf16_tflops"] * 1e12), 4)}

    out_points = {}
    main_pt = decode_point(args.batch)
    if not args.skip_points:
        out_points["decode_b1"] = round(decode_point(1)["tok_s"], 2)
        out_points["decode_b64"] = round(decode_point(64)["tok_s"], 2)

    # end to end: the same decode through the Python entry point (scheduler, one H2D copy of the
    # step's description from pinned memory, sampling on the device, token ids read back)
    B = args.batch
    # while the prompts are still being prefilled (2,048 tokens a step) the first requests
    # already decode; every request must still be live when the timed steps end
    prefill_steps = -(-B * CONTEXT // opts.max_step_tokens)
    spare = prefill_steps + W + K + 8
    ctx0 = max(256, CONTEXT - spare)
    prompts = [rng.integers(0, cfg.vocab_size, size=ctx0).tolist() for _ in range(B)]
    sp = SamplingParams(temperature=0.0, max_tokens=spare + 32, ignore_eos=True)
    rids = [llm.add_request(p, sp) for p in prompts]
    while any(len(llm._live[r].out.token_ids) == 0 for r in rids):      # prompts, untimed
        llm.step()
    for _ in range(W):
        llm.step()
    h0, d0 = llm.stats.h2d_bytes, llm.stats.d2h_bytes
    torch.cuda.synchronize()
    clocks.active = True
    t0 = time.perf_counter()
    for _ in range(K):
        llm.step()                               # launches a step and reads back the ids of the one before
    torch.cuda.synchronize()
    e2e_secs = time.perf_counter() - t0
    clocks.active = False
    e2e = {"value": round(B * K / e2e_secs, 2), "unit": "tokens/s", "ms_per_step": round(1000 * e2e_secs / K, 3),
           "h2d_bytes_per_step": (llm.stats.h2d_bytes - h0) // K, "d2h_bytes_per_step": (llm.stats.d2h_bytes - d0) // K}
    for r in rids:
        llm.abort_request(r)
    clocks.close()

    achieved = main_pt["bytes_step"] / (main_pt["ms"] / 1000.0) / 1e9
    rec = {
        "metric": f"decode tokens/s, Qwen3-8B bf16, batch {args.batch}, context {CONTEXT}", "value": round(main_pt["tok_s"], 2),
        "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": round(main_pt["ms"], 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights, uniform random token ids, cache of the context filled with random values",
        "impl": "ours",
        "config": {"model": "Qwen3-8B shape", "layers": L, "layers_of_model": full_layers, "hidden": cfg.hidden_size,
                   "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size, "global_batch": args.batch,
                   "seq_len": CONTEXT, "page_size": args.page_size, "parallelism": "single GPU",
                   "cache_flush": "inputs larger than L2: each step streams all weights and cache from HBM",
                   "pages": "scattered", "token_feedback": "device",
                   "peaks": pk["source"]},
        "e2e": e2e, "gpu_launches": int(main_pt["launches"]), "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": out_points, "clocks": clocks.summary(),
    }
    print(json.dumps(rec))
    return 0


if __name__ == "__main__":
    sys.exit(main())
