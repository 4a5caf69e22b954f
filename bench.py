"""Benchmark of zinfer_b200: decode tokens per second of an LFM2-1.2B-shaped model with random
weights on one B200, with the prefill rate, the decode roofline and batch-1/64 points beside it.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]

A "step" is one decode step: one new token for each of the batch's sequences.  After W warm-up
steps exactly K steps are timed with CUDA events on the launching stream.  The step reads 2.3 GB
of weights and the live requests' cache, far more than the 126 MB L2, so no flush is needed
between iterations.  The line printed is one JSON object; `value` is device-timed, `e2e` is the
same metric through `Engine.generate` with token ids going in from and coming back to the host
every step.  The reference engine (a Zig program for CPUs) cannot be installed as a Python
package, so `--impl reference` prints an `unavailable` line.  This library runs on one GPU: for
--gpus > 1 the program says so and exits with 2.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent

# LFM2-1.2B: the sizes of the published checkpoint's config.json
LFM2_1_2B = dict(
    architectures=["Lfm2ForCausalLM"], model_type="lfm2", vocab_size=65536, hidden_size=2048, num_hidden_layers=16,
    num_attention_heads=32, num_key_value_heads=8, max_position_embeddings=128000,
    layer_types=["conv", "conv", "full_attention", "conv", "conv", "full_attention", "conv", "conv", "full_attention",
                 "conv", "full_attention", "conv", "full_attention", "conv", "full_attention", "conv"],
    block_ff_dim=12288, block_auto_adjust_ff_dim=True, block_ffn_dim_multiplier=1.0, block_multiple_of=256,
    conv_L_cache=3, conv_bias=False, rope_theta=1000000.0, norm_eps=1e-5, tie_word_embeddings=True, eos_token_id=7)


def _lfm2(hidden, layers, attn_at, heads, ffn):
    """An LFM2 configuration of the given sizes with the effective SwiGLU width `ffn`."""
    d = dict(LFM2_1_2B, hidden_size=hidden, num_hidden_layers=layers, num_attention_heads=heads,
             layer_types=["full_attention" if i in attn_at else "conv" for i in range(layers)],
             block_ff_dim=ffn, block_auto_adjust_ff_dim=False)
    return d


# The secondary workloads: (configuration, batch, prompt lengths, decode steps, longest sequence)
SECONDARY = {
    "2.6b": (_lfm2(2048, 30, {2, 6, 10, 14, 18, 21, 24, 27}, 32, 10752), 16, (64, 4096), 256, 4096 + 512),
    "350m": (_lfm2(1024, 16, {2, 5, 8, 10, 12, 14}, 16, 4608), 64, (1024, 32768), 128, 32768 + 256),
}
CONTEXT = 4096
PROMPT_RANGE = (512, 2048)
PREFILL_TOKENS = 2048
POINT_STEPS = 64            # the batch-1 and batch-64 points are timed over at least this many steps
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def peaks() -> dict:
    p = ROOT / "MEASURED_PEAKS.json"
    if p.is_file():
        try:
            d = json.loads(p.read_text())
            return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]),
                    "bf16_tflops_sustained": float(d.get("bf16_tflops_sustained", d["bf16_tflops"])), "source": "measured"}
        except (KeyError, ValueError, json.JSONDecodeError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.proc = None
        self.lines: list[str] = []

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def __exit__(self, *exc):
        if self.proc is not None:
            time.sleep(0.15)
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self) -> dict:
        sm, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for l in self.lines:
            f = [x.strip() for x in l.split(",")]
            if len(f) < 6 or not f[0].isdigit():
                continue
            sm.append(int(f[0]))
            mx = max(mx, int(f[1]) if f[1].isdigit() else 0)
            for n, v in zip(names, f[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": int(statistics.median(sm)) if sm else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(sm)}


def model_numbers(cfg, n_layers_run: int) -> dict:
    """Weight bytes a decode step reads and FLOPs a prefill needs, from the configuration."""
    D, F, Q, KV, V = cfg.hidden_size, cfg.ffn_dim, cfg.q_dim, cfg.kv_dim, cfg.vocab_size
    kinds = cfg.layer_types[:n_layers_run]
    conv = 3 * D * D + D * D
    attn = (Q + 2 * KV) * D + D * Q
    ffn = 3 * D * F
    layer_params = sum((conv if k == "conv" else attn) + ffn for k in kinds)
    n_attn = sum(k != "conv" for k in kinds)
    return {"layer_params": layer_params, "head_params": V * D, "n_attn": n_attn, "n_conv": len(kinds) - n_attn,
            "kv_bytes_per_token": n_attn * 2 * KV * 2, "conv_state_bytes": (len(kinds) - n_attn) * (cfg.conv_L_cache - 1) * D * 4}


def time_decode(engine, torch, rng, batch: int, steps: int, warmup: int, vocab: int, prompt_range=None):
    """Prefills `batch` prompts of lengths uniform in `prompt_range` (default PROMPT_RANGE), then times
    `steps` decode steps.  Every CUDA graph the timed steps replay is recorded before the timing
    starts; `captures` counts the steps that had to record one all the same (expected: 0).
    Returns (ms per step, total cached tokens at the middle of the timed region, launches per step,
    captures)."""
    from zinfer_b200 import kernels
    lo, hi = prompt_range or PROMPT_RANGE
    lens = rng.integers(lo, hi + 1, size=batch).tolist()
    prompts = [rng.integers(0, vocab, size=n).tolist() for n in lens]
    slots = engine.start(batch)
    try:
        engine.step(slots, prompts, want=[[] for _ in prompts])
        toks = rng.integers(0, vocab, size=(warmup + steps, batch))
        launches = None
        for i in range(warmup):
            before = kernels.launch_count
            engine.decode(slots, toks[i].tolist())
            if launches is None:
                launches = kernels.launch_count - before
        longest = max(lens) + warmup
        engine.prepare_decode(batch, longest, longest + steps + 1)
        torch.cuda.synchronize()
        captures = engine.graph_captures
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        for i in range(warmup, warmup + steps):
            engine.decode(slots, toks[i].tolist())
        stop.record()
        torch.cuda.synchronize()
        engine.check_status()
        ms = start.elapsed_time(stop) / steps
        cached = sum(lens) + batch * (warmup + steps // 2)
        captures = engine.graph_captures - captures
    finally:
        engine.finish(slots)
    return ms, cached, launches, captures


def time_prefill(engine, torch, rng, cfg, warmup: int, num: dict, pk: dict, tokens: int = PREFILL_TOKENS) -> dict:
    """One sequence of `tokens` tokens in one step; median of 5 after the warm-up."""
    toks = rng.integers(0, cfg.vocab_size, size=tokens).tolist()
    times = []
    for i in range(warmup + 5):
        slot = engine.start(1)
        torch.cuda.synchronize()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        engine.step(slot, [toks], check=False)
        stop.record()
        torch.cuda.synchronize()
        engine.finish(slot)
        if i >= warmup:
            times.append(start.elapsed_time(stop))
    pre_ms = statistics.median(times)
    T = tokens
    flops = 2 * T * num["layer_params"] + 2 * num["head_params"] + num["n_attn"] * 2 * T * T * cfg.q_dim
    return {"value": round(T / (pre_ms * 1e-3), 1), "tokens": T, "ms": round(pre_ms, 3),
            "frac": round(flops / (pre_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}


def secondary_arm(args) -> dict:
    """One of the secondary workloads: unequal long prompts, then `steps` timed decode steps."""
    import numpy as np
    import torch
    import zinfer_b200 as z
    from zinfer_b200 import kernels

    kernels.require_cuda()
    pk = peaks()
    cfg_dict, batch, prompt_range, steps, longest = SECONDARY[args.model]
    cfg = z.config_from_dict(cfg_dict)
    model = z.random(cfg, seed=0, dtype="bf16", fill_on_device=True)
    rng = np.random.default_rng(0)
    lens = np.random.default_rng(0).integers(prompt_range[0], prompt_range[1] + 1, size=batch)   # as time_decode draws them
    page = 64
    room = int(sum(-(-(int(n) + args.warmup + steps + 1) // page) * page for n in lens))
    engine = z.Engine(model, max_batch=batch, max_seq_len=longest, max_tokens=room, page_size=page)
    num = model_numbers(cfg, cfg.num_hidden_layers)
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    with ClockSampler() as clocks:
        ms, cached, launches, captures = time_decode(engine, torch, rng, batch, steps, args.warmup, cfg.vocab_size,
                                                     prompt_range=prompt_range)
    wall = time.perf_counter() - t0
    weight_bytes = 2 * (num["layer_params"] + num["head_params"])
    step_bytes = weight_bytes + cached * num["kv_bytes_per_token"] + batch * num["conv_state_bytes"] * 2
    achieved = step_bytes / (ms * 1e-3) / 1e9
    return {"metric": f"decode tokens/s at batch {batch} (LFM2-{args.model.upper()} shape, random weights)",
            "value": round(batch / (ms * 1e-3), 1), "unit": "tokens/s", "ms_per_step": round(ms, 4), "steps": steps,
            "warmup": args.warmup, "dtype": "bf16", "impl": "zinfer_b200",
            "config": {"model": f"LFM2-{args.model.upper()}", "global_batch": batch, "layers": cfg.num_hidden_layers,
                       "hidden": cfg.hidden_size, "ffn": cfg.ffn_dim, "prompt_lens": f"uniform[{prompt_range[0]},{prompt_range[1]}]",
                       "cached_tokens": int(cached), "peaks": pk["source"]},
            "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                         "frac": round(achieved / pk["hbm_gbs"], 4), "weight_gb": round(weight_bytes / 1e9, 3),
                         "cache_gb": round(cached * num["kv_bytes_per_token"] / 1e9, 3)},
            "clocks": clocks.summary(), "gpu_launches": int(launches or 0) * steps,
            "graph_captures_in_timed_steps": captures, "wall_s_with_prompts": round(wall, 1)}


# Ponusun beside the closest existing architecture at equal size: width, layers, heads, window and vocabulary
# are the same, and LFM2's SwiGLU is as wide as the experts one Ponusun token runs (top * ff + shared).
PONUSUN_SIZES = {
    "w1024": dict(width=1024, layers=8, heads=16, kv=4, dim=64, window=512, experts=16, top=2, ff=1024, shared=1024,
                  dense_ff=4096, vocab=32768, taps=3),
    "w2048": dict(width=2048, layers=8, heads=32, kv=8, dim=64, window=1024, experts=16, top=2, ff=2048, shared=2048,
                  dense_ff=8192, vocab=65536, taps=3),
}


def ponusun_config(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                 "mask": {"size": sz["window"]}}
        if i >= 2 and i % 2 == 0:
            mixer["kv_from"] = i - 1                   # every second layer reads the keys and values of the one before
        mlp = ({"kind": "dense", "ff": sz["dense_ff"]} if i == 0 else
               {"kind": "moe", "expert": {"ff": sz["ff"]}, "router": {"experts": sz["experts"], "top": sz["top"]},
                "shared": {"ff": sz["shared"]}})
        layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Ponusun", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "canon": {"taps": sz["taps"]}, "logit_softcap": 20.0, "layers": layers}


def lfm2_like(sz: dict) -> dict:
    return dict(LFM2_1_2B, vocab_size=sz["vocab"], hidden_size=sz["width"], num_hidden_layers=sz["layers"],
                num_attention_heads=sz["heads"], num_key_value_heads=sz["kv"], head_dim=sz["dim"],
                max_position_embeddings=CONTEXT, layer_types=["sliding_attention"] * sz["layers"],
                sliding_window=sz["window"], block_ff_dim=sz["top"] * sz["ff"] + sz["shared"], block_auto_adjust_ff_dim=False)


# Zosurax beside the closest existing architecture at equal size: width, layers, vocabulary and the attention
# layers' heads are the same; LFM2 has a short convolution where Zosurax has its HGRN2 recurrence, plain
# grouped-query attention where Zosurax has either of its attention kinds, and a SwiGLU of two thirds the
# hidden units (three matrices) where Zosurax has its squared-relu feed-forward of two: the same parameters.
ZOSURAX_SIZES = {
    "w1024": dict(width=1024, layers=8, heads=16, kv=4, dim=64, rec_heads=8, rec_dim=128, ff=4096, vocab=32768),
    "w2048": dict(width=2048, layers=8, heads=32, kv=8, dim=64, rec_heads=16, rec_dim=128, ff=8192, vocab=65536),
}
ZOSURAX_KINDS = ["hgrn2", "attention", "attention_2", "hgrn2", "attention", "attention_2", "hgrn2", "attention"]


def zosurax_config(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        kind = ZOSURAX_KINDS[i % len(ZOSURAX_KINDS)]
        if kind == "hgrn2":
            mixer = {"heads": sz["rec_heads"], "dim": sz["rec_dim"], "vdim": sz["width"] // sz["rec_heads"]}
        else:
            mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["dim"] if kind == "attention" else sz["dim"] // 2}}
        layers.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": sz["ff"]}})
    return {"architecture": "Zosurax", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "layers": layers}


def lfm2_like_zosurax(sz: dict) -> dict:
    kinds = ["conv" if ZOSURAX_KINDS[i % len(ZOSURAX_KINDS)] == "hgrn2" else "full_attention" for i in range(sz["layers"])]
    return dict(LFM2_1_2B, vocab_size=sz["vocab"], hidden_size=sz["width"], num_hidden_layers=sz["layers"],
                num_attention_heads=sz["heads"], num_key_value_heads=sz["kv"], head_dim=sz["dim"],
                max_position_embeddings=CONTEXT, layer_types=kinds, block_ff_dim=-(-(sz["ff"] * 2 // 3) // 256) * 256,
                block_auto_adjust_ff_dim=False)


# Kerotar beside the closest existing architecture at equal size, Ponusun without its convolutions, shared experts,
# borrowed keys and logit cap: width, layers, vocabulary, the heads and window of the windowed layers, the dense
# feed-forwards' hidden units and the experts are the same.  Kerotar's even layers attend through a latent (Ponusun:
# windowed attention there too), its windowed layers keep a sequence's first tokens and have a sink, its router is
# learned (Ponusun: a table by token id), and one norm feeds both sublayers of a layer.
KEROTAR_SIZES = {
    "w1024": dict(width=1024, layers=8, heads=16, kv=4, dim=64, window=512, keep=4, lat_dim=64, lat_rot=32, lat_vdim=64,
                  kv_rank=256, q_rank=512, experts=16, top=2, ff=1024, dense_ff=4096, vocab=32768),
    "w2048": dict(width=2048, layers=8, heads=32, kv=8, dim=64, window=1024, keep=4, lat_dim=64, lat_rot=32, lat_vdim=64,
                  kv_rank=512, q_rank=768, experts=16, top=2, ff=2048, dense_ff=8192, vocab=65536),
}


def kerotar_config(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        if i % 2 == 0:
            kind = "latent_attention"
            mixer = {"heads": sz["heads"], "dim": sz["lat_dim"], "rot_dim": sz["lat_rot"], "vdim": sz["lat_vdim"],
                     "kv_rank": sz["kv_rank"], "q_rank": sz["q_rank"], "scale": (sz["lat_dim"] + sz["lat_rot"]) ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["lat_rot"]}}
            mlp = {"kind": "dense", "ff": sz["dense_ff"], "limit": 7.0}
        else:
            kind = "attention"
            mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["dim"] // 2}, "mask": {"size": sz["window"], "keep_first": sz["keep"]}}
            mlp = {"kind": "moe", "expert": {"ff": sz["ff"]}, "router": {"experts": sz["experts"], "top": sz["top"]}}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Kerotar", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "layers": layers}


def ponusun_like_kerotar(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                 "mask": {"size": sz["window"]}}
        mlp = ({"kind": "dense", "ff": sz["dense_ff"]} if i % 2 == 0 else
               {"kind": "moe", "expert": {"ff": sz["ff"]}, "router": {"experts": sz["experts"], "top": sz["top"]}})
        layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Ponusun", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "layers": layers}


# Pirisun beside the closest existing architecture at equal size, Kerotar (parallel layers, attention through a latent,
# routed experts): width, layers, vocabulary, heads, the latent's sizes and the experts are the same.  Where Kerotar has
# grouped-query attention with a sink (here without a window, so that both attend to every earlier token), Pirisun has
# its pair of mixers: attention with capped scores and a query temperature beside retention; its latent attention has
# no query latent but a sink and a gate per value; its router has a correction and two identity experts, and every
# layer also runs a shared expert.
PIRISUN_SIZES = {
    "w1024": dict(width=1024, layers=8, heads=16, kv=4, dim=64, ret_heads=8, ret_dim=128, lat_dim=64, lat_rot=32, lat_vdim=64,
                  kv_rank=256, q_rank=512, experts=16, top=2, identity=2, ff=1024, shared=1024, vocab=32768),
    "w2048": dict(width=2048, layers=8, heads=32, kv=8, dim=64, ret_heads=16, ret_dim=128, lat_dim=64, lat_rot=32, lat_vdim=64,
                  kv_rank=512, q_rank=768, experts=16, top=2, identity=2, ff=2048, shared=2048, vocab=65536),
}


def pirisun_config(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        if i % 2 == 0:
            kind = "parallel"
            mixer = {"left": {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                              "softcap": 50.0, "q_temp": {"coef": 0.1, "every": 256}},
                     "right": {"heads": sz["ret_heads"], "dim": sz["ret_dim"], "vdim": sz["width"] // sz["ret_heads"],
                               "decay": [1.0 - 1.0 / (24.0 * (h + 1)) for h in range(sz["ret_heads"])],
                               "rot": {"base": 10000.0, "dims": sz["ret_dim"]}}}
        else:
            kind = "latent_attention"
            mixer = {"heads": sz["heads"], "dim": sz["lat_dim"], "rot_dim": sz["lat_rot"], "vdim": sz["lat_vdim"],
                     "kv_rank": sz["kv_rank"], "scale": (sz["lat_dim"] + sz["lat_rot"]) ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["lat_rot"]}}
        mlp = {"kind": "moe", "expert": {"ff": sz["ff"]}, "shared": {"ff": sz["shared"]},
               "router": {"experts": sz["experts"], "top": sz["top"], "identity": sz["identity"]}}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Pirisun", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": layers}


def kerotar_like_pirisun(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        if i % 2 == 0:
            kind = "attention"
            mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["dim"] // 2}}
        else:
            kind = "latent_attention"
            mixer = {"heads": sz["heads"], "dim": sz["lat_dim"], "rot_dim": sz["lat_rot"], "vdim": sz["lat_vdim"],
                     "kv_rank": sz["kv_rank"], "q_rank": sz["q_rank"], "scale": (sz["lat_dim"] + sz["lat_rot"]) ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["lat_rot"]}}
        mlp = {"kind": "moe", "expert": {"ff": sz["ff"]}, "router": {"experts": sz["experts"], "top": sz["top"]}}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Kerotar", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "layers": layers}


# Varolorn beside the closest existing architecture at equal size, Zosurax (pre-norm, a recurrence in some layers and
# softmax attention in the others, a dense feed-forward, the head tied to the embedding): width, layers, vocabulary and the
# attention layers' heads are the same; Varolorn has the Mamba-2 recurrence (inner width twice the model's) where Zosurax has
# HGRN2, attention within stretches of positions with a distance table and a gate where Zosurax has its first, rotated kind
# (every earlier token), and a gated feed-forward of two thirds the hidden units (three matrices) where Zosurax has its
# squared-relu one of two.
VAROLORN_SIZES = {
    "w1024": dict(width=1024, layers=8, heads=16, kv=4, dim=64, chunk=1024, ssm_heads=32, ssm_vdim=64, ssm_state=128, ssm_groups=4,
                  conv=4, streams=4, ff=4096, vocab=32768, rec_heads=8, rec_dim=128),
    "w2048": dict(width=2048, layers=8, heads=32, kv=8, dim=64, chunk=1024, ssm_heads=64, ssm_vdim=64, ssm_state=128, ssm_groups=8,
                  conv=4, streams=4, ff=8192, vocab=65536, rec_heads=16, rec_dim=128),
}


def varolorn_config(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        if ZOSURAX_KINDS[i % len(ZOSURAX_KINDS)] == "hgrn2":
            kind = "mamba2"
            mixer = {"heads": sz["ssm_heads"], "vdim": sz["ssm_vdim"], "state": sz["ssm_state"], "groups": sz["ssm_groups"],
                     "conv": sz["conv"], "norm_groups": sz["ssm_groups"]}
        else:
            kind = "attention"
            mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                     "bias_max": 600, "mask": {"size": sz["chunk"]}, "v_mix": True}
        layers.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": -(-(sz["ff"] * 2 // 3) // 256) * 256}})
    return {"architecture": "Varolorn", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT, "streams": sz["streams"],
            "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0, "bigram": {"buckets": 2 * sz["vocab"] - 1, "mul_prev": 7919, "mul_cur": 271}},
            "layers": layers}


def zosurax_like_varolorn(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        if ZOSURAX_KINDS[i % len(ZOSURAX_KINDS)] == "hgrn2":
            kind, mixer = "hgrn2", {"heads": sz["rec_heads"], "dim": sz["rec_dim"], "vdim": sz["width"] // sz["rec_heads"]}
        else:
            kind = "attention"
            mixer = {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                     "rot": {"base": 10000.0, "dims": sz["dim"]}}
        layers.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": sz["ff"]}})
    return {"architecture": "Zosurax", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "layers": layers}


# Nipizen beside the closest existing architecture at equal size, Pirisun (attention beside a recurrence, routed experts): width,
# layers, vocabulary, the attention heads, the recurrence's heads and sizes and the number of experts are the same, and the
# experts have the same parameters (two matrices of one and a half times the hidden units here, three there).  Every Pirisun layer is
# its pair of mixers, without identity and shared experts and with no temperature or cap; every fourth Nipizen layer is an mLSTM in
# place of the pair.
NIPIZEN_SIZES = {
    "w1024": dict(width=1024, layers=8, heads=16, kv=4, dim=64, rec_heads=8, rec_dim=128, conv=4, mem_heads=4, mem_dim=128, mem_vdim=256,
                  experts=16, top=2, ff=1024, vocab=32768),
    "w2048": dict(width=2048, layers=8, heads=32, kv=8, dim=64, rec_heads=16, rec_dim=128, conv=4, mem_heads=8, mem_dim=128, mem_vdim=256,
                  experts=16, top=2, ff=2048, vocab=65536),
}


def nipizen_config(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        if i % 4 == 3:
            kind, mixer = "mlstm", {"heads": sz["mem_heads"], "dim": sz["mem_dim"], "vdim": sz["mem_vdim"], "gate_cap": 15.0}
        else:
            kind = "parallel"
            mixer = {"left": {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5,
                              "rot": {"base": 10000.0, "dims": sz["dim"],
                                      "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}},
                     "right": {"heads": sz["rec_heads"], "kv_heads": sz["rec_heads"], "dim": sz["rec_dim"],
                               "vdim": sz["width"] // sz["rec_heads"], "conv": sz["conv"]},
                     "left_scale": 0.5, "right_scale": 0.5}
        mlp = {"kind": "moe", "expert": {"ff": sz["ff"] * 3 // 2}, "router": {"experts": sz["experts"], "top": sz["top"]}}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Nipizen", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "layers": layers}


def pirisun_like_nipizen(sz: dict) -> dict:
    layers = []
    for i in range(sz["layers"]):
        mixer = {"left": {"heads": sz["heads"], "kv_heads": sz["kv"], "dim": sz["dim"], "vdim": sz["dim"], "scale": sz["dim"] ** -0.5},
                 "right": {"heads": sz["rec_heads"], "dim": sz["rec_dim"], "vdim": sz["width"] // sz["rec_heads"],
                           "decay": [1.0 - 1.0 / (24.0 * (h + 1)) for h in range(sz["rec_heads"])],
                           "rot": {"base": 10000.0, "dims": sz["rec_dim"]}}}
        mlp = {"kind": "moe", "expert": {"ff": sz["ff"]}, "router": {"experts": sz["experts"], "top": sz["top"]}}
        layers.append({"type": "parallel", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Pirisun", "vocab": sz["vocab"], "width": sz["width"], "max_positions": CONTEXT,
            "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": layers}


# new architecture -> (sizes, its configuration, the configuration of the architecture beside it, that one's name)
COMPARISONS = {"ponusun": (PONUSUN_SIZES, ponusun_config, lfm2_like, "lfm2"),
               "zosurax": (ZOSURAX_SIZES, zosurax_config, lfm2_like_zosurax, "lfm2"),
               "kerotar": (KEROTAR_SIZES, kerotar_config, ponusun_like_kerotar, "ponusun"),
               "pirisun": (PIRISUN_SIZES, pirisun_config, kerotar_like_pirisun, "kerotar"),
               "varolorn": (VAROLORN_SIZES, varolorn_config, zosurax_like_varolorn, "zosurax"),
               "nipizen": (NIPIZEN_SIZES, nipizen_config, pirisun_like_nipizen, "pirisun")}


def ponusun_arm(args) -> dict:
    """Prompt and single-token throughput of Ponusun (or Zosurax, Kerotar, Pirisun, Varolorn, Nipizen: `--model`) and of the closest earlier
    architecture (LFM2; for Kerotar, Ponusun; for Pirisun, Kerotar; for Varolorn, Zosurax; for Nipizen, Pirisun) at equal size, random
    weights, bfloat16: one prompt of --prefill-tokens tokens in one step (median of 5), then --steps single-token
    steps of --batch sequences replayed from CUDA graphs (prompts of 512..2,048 tokens)."""
    import numpy as np
    import torch
    import zinfer_b200 as z
    from zinfer_b200 import kernels

    kernels.require_cuda()
    new = args.model
    sizes, new_config, like_config, like = COMPARISONS[new]
    like_title = {"lfm2": "LFM2"}.get(like, like.capitalize())
    out = {"metric": f"prompt and single-token tokens/s, {new.capitalize()} beside {like_title} at equal size (random weights)", "unit": "tokens/s",
           "dtype": "bf16", "data": "synthetic", "steps": args.steps, "warmup": args.warmup, "batch": args.batch,
           "prefill_tokens": args.prefill_tokens, "sizes": {}}
    wanted = [args.size] if args.size else list(sizes)
    with ClockSampler() as clocks:
        for name in wanted:
            sz = sizes[name]
            row = {}
            for arch, cfg_dict in ((new, new_config(sz)), (like, like_config(sz))):
                if args.arch and arch != args.arch:
                    continue
                cfg = z.config_from_dict(cfg_dict)
                model = z.random(cfg, seed=0, dtype="bf16", fill_on_device=True, std=sz["width"] ** -0.5)
                engine = z.Engine(model, max_batch=args.batch, max_seq_len=CONTEXT, use_graphs=not args.no_graphs)
                rng = np.random.default_rng(0)
                res = {}
                if args.only in ("all", "prefill"):
                    toks = rng.integers(0, cfg.vocab_size, size=args.prefill_tokens).tolist()
                    times = []
                    for i in range(args.warmup + 5):
                        slot = engine.start(1)
                        torch.cuda.synchronize()
                        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                        start.record()
                        engine.step(slot, [toks], check=False)
                        stop.record()
                        torch.cuda.synchronize()
                        engine.finish(slot)
                        if i >= args.warmup:
                            times.append(start.elapsed_time(stop))
                    engine.check_status()
                    ms = statistics.median(times)
                    res["prefill"] = {"tokens_per_s": round(args.prefill_tokens / (ms * 1e-3), 1), "ms": round(ms, 3)}
                if args.only in ("all", "decode"):
                    ms, cached, launches, captures = time_decode(engine, torch, rng, args.batch, args.steps, args.warmup,
                                                                 cfg.vocab_size)
                    res["decode"] = {"tokens_per_s": round(args.batch / (ms * 1e-3), 1), "ms_per_step": round(ms, 4),
                                     "launches_per_step": launches, "graph_captures_in_timed_steps": captures}
                row[arch] = res
                del engine, model
                torch.cuda.empty_cache()
            if new in row and like in row:
                row[f"{new}_over_{like}"] = {k: round(row[new][k]["tokens_per_s"] / row[like][k]["tokens_per_s"], 3)
                                           for k in row[new]}
            out["sizes"][name] = dict(row, config={k: sz[k] for k in sz})
    out["clocks"] = clocks.summary()
    return out


def own_arm(args) -> dict:
    import numpy as np
    import torch

    sys.path.insert(0, str(ROOT))
    import zinfer_b200 as z
    from zinfer_b200 import kernels

    kernels.require_cuda()
    pk = peaks()
    cfg_dict = dict(LFM2_1_2B)
    layers_cfg = cfg_dict["num_hidden_layers"]
    if args.layers and args.layers < layers_cfg:
        cfg_dict["num_hidden_layers"] = args.layers
        cfg_dict["layer_types"] = cfg_dict["layer_types"][:args.layers]
    cfg = z.config_from_dict(cfg_dict)
    model = z.random(cfg, seed=0, dtype="bf16", fill_on_device=True)
    B = args.batch
    engine = z.Engine(model, max_batch=64, max_seq_len=max(CONTEXT, args.prefill_tokens), page_size=64,
                      max_tokens=max(64 * CONTEXT, args.prefill_tokens), max_step_tokens=max(8192, args.prefill_tokens),
                      use_graphs=not args.no_graphs)
    if args.only == "prefill":
        return {"prefill": time_prefill(engine, torch, np.random.default_rng(0), cfg, args.warmup,
                                        model_numbers(cfg, cfg.num_hidden_layers), pk, args.prefill_tokens)}
    rng = np.random.default_rng(0)
    num = model_numbers(cfg, cfg.num_hidden_layers)
    weight_bytes = 2 * (num["layer_params"] + num["head_params"])

    # decode at the headline batch, device-timed, with the clocks sampled meanwhile
    with ClockSampler() as clocks:
        ms, cached, launches, captures = time_decode(engine, torch, rng, B, args.steps, args.warmup, cfg.vocab_size)
    value = B / (ms * 1e-3)
    step_bytes = weight_bytes + cached * num["kv_bytes_per_token"] + B * num["conv_state_bytes"] * 2
    achieved = step_bytes / (ms * 1e-3) / 1e9

    if args.only == "decode":
        return {"value": round(value, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                "roofline_frac": round(achieved / pk["hbm_gbs"], 4)}

    # other batch sizes, each over at least POINT_STEPS steps whatever --steps says
    points = {}
    for b in (1, 64):
        pms, pcached, _, pcap = time_decode(engine, torch, rng, b, max(POINT_STEPS, args.steps), args.warmup,
                                            cfg.vocab_size)
        captures += pcap
        pbytes = weight_bytes + pcached * num["kv_bytes_per_token"] + b * num["conv_state_bytes"] * 2
        points[f"decode_b{b}"] = round(b / (pms * 1e-3), 1)
        points[f"decode_b{b}_hbm_frac"] = round(pbytes / (pms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)

    prefill = time_prefill(engine, torch, rng, cfg, args.warmup, num, pk)
    T = PREFILL_TOKENS

    # the same metric end to end through the public entry point: host token ids in and out every step
    prompts = [rng.integers(0, cfg.vocab_size, size=int(n)).tolist()
               for n in rng.integers(PROMPT_RANGE[0], PROMPT_RANGE[1] + 1, size=B)]
    n_new = max(POINT_STEPS, args.steps) + 1       # at least 64 steps, as the other points
    # warm-up: the same generation once, so that every graph the timed one replays is captured
    engine.generate(prompts, max_new_tokens=n_new, temp=0.0, stop_ids=[])
    engine.generate(prompts, max_new_tokens=n_new, temp=0.0, stop_ids=[])
    st = engine.stats
    e2e_value = B * st.n_decode_steps / st.t_gen_s
    from zinfer_b200.engine.context import batch_layout
    e2e = {"value": round(e2e_value, 1), "unit": "tokens/s", "h2d_bytes_per_step": 4 * batch_layout(B, B)["_total"][0],
           "d2h_bytes_per_step": 4 * (B + 1)}

    return {
        "metric": "decode tokens/s at batch 8 (LFM2-1.2B shape, random weights, context 4096)" if B == 8
        else f"decode tokens/s at batch {B} (LFM2-1.2B shape, random weights, context 4096)",
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic token ids, random-init weights N(0, 0.02)", "impl": "zinfer_b200",
        "config": {"model": "LFM2-1.2B", "global_batch": B, "seq_len": CONTEXT, "parallelism": "none",
                   "vocab": cfg.vocab_size, "hidden": cfg.hidden_size, "layers": cfg.num_hidden_layers,
                   "layers_of_config": layers_cfg, "attn_layers": num["n_attn"], "heads": cfg.num_attention_heads,
                   "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim, "ffn": cfg.ffn_dim,
                   "conv_window": cfg.conv_L_cache, "prompt_lens": "uniform[512,2048]", "prefill_tokens": T,
                   "l2": "inputs larger than L2 (2.3 GB of weights per step)", "peaks": pk["source"]},
        "clocks": clocks.summary(),
        "e2e": e2e,
        "gpu_launches": int(launches or 0) * args.steps,
        "graph_captures_in_timed_steps": captures,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
    }


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="own", choices=["own", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=0, help="run only the first L layers (named in `config`)")
    ap.add_argument("--only", default="all", choices=["all", "decode", "prefill"],
                    help="measure one part only (for profiling); the JSON line then lacks the other parts")
    ap.add_argument("--no-graphs", action="store_true", help="launch decode steps kernel by kernel")
    ap.add_argument("--prefill-tokens", type=int, default=PREFILL_TOKENS,
                    help="with --only prefill: the prompt's length (the headline line always uses 2,048)")
    ap.add_argument("--model", default="1.2b", choices=["1.2b"] + list(COMPARISONS) + sorted(SECONDARY),
                    help="1.2b: the headline benchmark; 2.6b, 350m: the secondary workloads (decode only); ponusun, zosurax, "
                         "kerotar, pirisun, varolorn, nipizen: that architecture beside the closest earlier one at equal size, prompt and single-token steps")
    ap.add_argument("--size", default="", choices=[""] + sorted(PONUSUN_SIZES), help="with --model ponusun, zosurax, kerotar, pirisun, varolorn or nipizen: one size only")
    ap.add_argument("--arch", default="", choices=["", "lfm2"] + list(COMPARISONS),
                    help="with --model ponusun, zosurax, kerotar, pirisun, varolorn or nipizen: one architecture of the two only")
    args = ap.parse_args()
    args.warmup = max(3, args.warmup)
    if args.impl == "reference":
        print(json.dumps({"impl": "reference",
                          "unavailable": "pylypenko99/zinfer is a Zig program for CPUs: pip cannot install it "
                                         "(no setup.py or pyproject.toml) and no Zig compiler is on this image"}))
        return 0
    if args.gpus != 1 or int(os.environ.get("WORLD_SIZE", "1")) != 1:
        print(f"bench.py: zinfer_b200 runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.model in COMPARISONS:
        print(json.dumps(ponusun_arm(args)))
        return 0
    print(json.dumps(own_arm(args) if args.model == "1.2b" else secondary_arm(args)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
