#!/usr/bin/env python3
"""Benchmark of the engine's decode step on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--impl reference]

Default: the layer sizes of the Qwen3-8B shape, random bfloat16 weights, batch 8,
each request holding a 2,048-token prompt, engine context limit 4,096; token ids
are seeded uniform-random (no dataset).  A step is one decode step (one new token
for every request).  Prints ONE JSON line:

  value     decoded tokens per second at batch 8, timed on the device with CUDA events
  e2e       the same through the Python entry point (Engine.step), host tokens in
            and out, with the step's host->device and device->host bytes; "points"
            inside it: the same at batch 1 and 64; "sampled": the same at batch 8 with
            the reference's default sampling options instead of greedy
  prefill   one step of 2,048 prompt tokens: tokens/s, ms, fraction of the bf16 peak;
            "chunks_512" inside it: the same prompt as four steps of 512 tokens
  roofline  bytes the decode step must read (every weight once + the live
            requests' cache) / time, against the measured copy bandwidth
  points    decode tokens/s at batch 1 and 64

With ``--design luvavik`` it runs another measurement instead and prints a JSON line of its own: prefill
(2,048 tokens) and decode (batch 8, 2,048 cached tokens each) throughput of the Luvavik design at layer
sizes of real models (widths 2048 and 4096; ``--design-sizes``), beside Qwen3 dense at the same width,
layer count and multiply-adds per token; ``--design rogosun`` does the same for the Rogosun design, beside
Luvavik (the nearest design the engine has) and Qwen3, and ``--design vumezen`` for the Vumezen design, beside
Rogosun (whose attention with a sink and routed experts beside a shared one are the nearest the engine has) and Qwen3, and
``--design sepitar`` for the Sepitar design, beside Vumezen, Luvavik and Qwen3, and ``--design kesitar`` for the Kesitar
design, beside Rogosun (the nearest recurrence; its feed-forwards all dense here), Vumezen (the nearest attention) and Qwen3
with the same feed-forward, and ``--design sumozen`` for the Sumozen design, beside Rogosun (the nearest mixers and experts; experts
in every layer here) and Qwen3; ``--profile PATH`` adds both models' per-kernel-class times and
roofline fractions.  The default workload and its output line are untouched.

Peaks come from MEASURED_PEAKS.json when the driver wrote it, else the fallback
figures (6.65 TB/s, 1.59 PFLOP/s).  Weights (15 GB) exceed L2 (126 MB), so every
step streams its inputs from HBM without a flush.  For --gpus > 1 it says that
the engine is single-GPU and exits with 2.
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

REPO = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, REPO)

QWEN3_8B = dict(
    architectures=["Qwen3ForCausalLM"], model_type="qwen3", vocab_size=151936, hidden_size=4096,
    intermediate_size=12288, num_hidden_layers=36, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
    max_position_embeddings=40960, rms_norm_eps=1e-6, rope_theta=1000000.0, tie_word_embeddings=False,
    torch_dtype="bfloat16")
PROMPT_LEN = 2048
CONTEXT_LEN = 4096
PREFILL_TOKENS = 2048


def peaks() -> tuple[float, float, str]:
    """(HBM GB/s, bf16 TFLOP/s, source)."""
    path = os.path.join(REPO, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            with open(path) as f:
                d = json.load(f)
            return float(d["hbm_gbs"]), float(d["bf16_tflops"]), "measured"
        except (OSError, ValueError, KeyError):
            pass
    return 6650.0, 1590.0, "fallback"


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.index = index
        self.rows: list[list[str]] = []
        self.proc = None

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", str(self.index), f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "50"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 6:
                self.rows.append(parts)

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()   # the exact process started above
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self) -> dict:
        if not self.rows:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["no samples"]}
        sm = [int(r[0]) for r in self.rows if r[0].isdigit()]
        mx = [int(r[1]) for r in self.rows if r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(r[2 + i].lower().startswith("active") for r in self.rows)]
        return {"sm_mhz": int(statistics.median(sm)) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(self.rows)}


def matmul_params(cfg, n_layers: int) -> int:
    """Weight elements every token multiplies with (layers + output head)."""
    H, I = cfg.hidden_size, cfg.intermediate_size
    q, kv = cfg.num_attention_heads * cfg.head_dim, cfg.num_key_value_heads * cfg.head_dim
    per_layer = H * (q + 2 * kv) + q * H + 3 * H * I
    return n_layers * per_layer


# ------------------------------------------------------------ another design beside Qwen3
def luvavik_shape(width: int, heads: int, experts: int, top: int, expert_ff: int, dense_ff: int) -> dict:
    """A Luvavik configuration with layers the size of a real model's: latent attention with heads of
    128 + 64 rotated dimensions over a latent of 512, recurrent blocks as wide as the model in blocks of
    128 channels with four taps, a dense feed-forward in the first layer and experts elsewhere; layers
    1..2 run twice.  Seven layer runs in all."""
    attn = {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
                      "rot": {"base": 10000.0, "dims": 64}}}
    rec = {"type": "rglru", "mixer": {"width": width, "blocks": width // 128, "conv": 4}}
    moe = {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top, "identity": 2}}
    dense = {"kind": "dense", "ff": dense_ff}
    layers = [dict(attn, mlp=dense), dict(rec, mlp=moe), dict(attn, mlp=moe), dict(attn, mlp=moe), dict(rec, mlp=moe)]
    return {"architecture": "Luvavik", "vocab": 32768, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "residual_mult": 0.5, "logit_scale": 1.0, "loop": {"start": 1, "stop": 3, "times": 2},
            "max_position_embeddings": 8192}


def rogosun_shape(width: int, heads: int, experts: int, top: int, expert_ff: int, dense_ff: int) -> dict:
    """A Rogosun configuration with layers the size of a real model's: gated linear attention with key heads of 128
    and value heads of 256 channels (keys half as wide as the model, values as wide), parallel layers of attention
    (heads of 128 of which 64 dimensions rotate, four query heads per kv head, a sink, the raw keys as values) beside
    a gated delta rule (heads of 128 x 256 behind convolutions of four taps), dense feed-forwards and routed experts
    in groups of four with a shared expert.  Seven layers."""
    g = max(1, width // 256)
    gla = {"type": "gla", "mixer": {"heads": g, "dim": 128, "vdim": 256, "tau": 16.0}}
    par = {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "rot": {"base": 1000000.0, "dims": 64, "scaling": {"factor": 4.0}}},
        "right": {"heads": g, "kv_heads": max(1, g // 2), "dim": 128, "vdim": 256, "conv": 4},
        "left_scale": 0.8, "right_scale": 0.5}}
    moe = {"kind": "moe", "expert": {"ff": expert_ff}, "shared": {"ff": expert_ff},
           "router": {"experts": experts, "top": top, "scale": 2.0, "groups": {"count": 4, "keep": 2}}}
    dense = {"kind": "dense", "ff": dense_ff}
    layers = [dict(gla, mlp=dense), dict(par, mlp=moe), dict(gla, mlp=moe), dict(gla, mlp=moe), dict(par, mlp=dense),
              dict(gla, mlp=moe), dict(par, mlp=moe)]
    return {"architecture": "Rogosun", "vocab": 32768, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "max_position_embeddings": 8192}


def vumezen_shape(width: int, heads: int, experts: int, top: int, expert_ff: int, dense_ff: int) -> dict:
    """A Vumezen configuration with layers the size of a real model's: blocks whose two sublayers read the same
    stream; attention heads of 128 of which 64 dimensions rotate, four query heads per kv head, values of 128, a
    sink, a window of 1,024 tokens that keeps a request's first four; every second layer reads the keys and values
    of the layer before it; relu-squared experts chosen by sigmoid scores beside a shared expert in every layer; a
    table of token pairs beside the embedding.  Seven layers."""
    def mixer(src=None):
        m = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
             "rot": {"base": 1000000.0, "dims": 64}, "mask": {"size": 1024, "keep_first": 4}}
        if src is not None:
            m["kv_from"] = src
        return m
    moe = {"kind": "moe", "expert": {"ff": expert_ff}, "shared": {"ff": expert_ff},
           "router": {"experts": experts, "top": top, "scale": 2.0}}
    layers = [{"type": "attention", "mixer": mixer(i - 1 if i % 2 else None), "mlp": moe} for i in range(7)]
    return {"architecture": "Vumezen", "vocab": 32768, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0, "bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 17}},
            "max_position_embeddings": 8192}


def sepitar_shape(width: int, heads: int, experts: int, top: int, expert_ff: int, dense_ff: int) -> dict:
    """A Sepitar configuration with layers the size of a real model's: blocks with one norm whose two sublayers read it;
    latent attention with heads of 128 + 64 rotated dimensions over a latent of 512, queries through a latent of 1,536,
    a window of 1,024 tokens and a learned sink; attention with biases, a distance table and a gate per channel (heads
    of 128, four query heads per kv head, a window of 1,024); attention with a norm over the whole of q and k, 64
    rotated dimensions, a capped score, a sink and a gate per head, over all earlier keys; clamped gated experts chosen
    by their logits beside a shared expert in every layer.  Five layers of which 1..2 run twice: seven layer runs."""
    lat = {"type": "latent_attention",
           "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": 1536, "scale": 192 ** -0.5,
                     "mask": {"size": 1024},
                     "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}}}}
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128,
                                          "scale": 128 ** -0.5, "bias_max": 2048, "mask": {"size": 1024}}}
    att2 = {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128,
                                             "scale": 128 ** -0.5, "softcap": 50.0,
                                             "rot": {"base": 1000000.0, "dims": 64,
                                                     "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}}}
    moe = {"kind": "moe", "expert": {"ff": expert_ff, "limit": 7.0}, "shared": {"ff": expert_ff, "limit": 7.0},
           "router": {"experts": experts, "top": top}}
    layers = [dict(lat, mlp=moe), dict(att, mlp=moe), dict(att2, mlp=moe), dict(lat, mlp=moe), dict(lat, mlp=moe)]
    return {"architecture": "Sepitar", "vocab": 32768, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "loop": {"start": 1, "stop": 3, "times": 2}, "max_position_embeddings": 8192}


def kesitar_shape(width: int, heads: int, dense_ff: int) -> dict:
    """A Kesitar configuration with layers the size of a real model's: HGRN2 with heads of 128 key and 128 value channels,
    as wide as the model; attention with biases, head norms, heads of 128 of which 64 dimensions rotate, four query heads
    per kv head, mixed values, a window of 512 tokens and pooled blocks of 16 tokens before it; dense gated
    feed-forwards; layer norms before and after every sublayer.  Seven layers."""
    ff = {"kind": "dense", "ff": dense_ff}
    rec = {"type": "hgrn2", "mixer": {"heads": width // 128, "dim": 128, "vdim": 128}, "mlp": ff}
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                          "rot": {"base": 1000000.0, "dims": 64}, "mask": {"size": 512, "pool": 16}, "v_mix": True},
           "mlp": ff}
    return {"architecture": "Kesitar", "vocab": 32768, "width": width, "layers": [rec, att, rec, rec, att, rec, att],
            "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0}, "logit_scale": 1.0, "max_position_embeddings": 8192}


def sumozen_shape(width: int, heads: int, experts: int, top: int, expert_ff: int) -> dict:
    """A Sumozen configuration with layers the size of a real model's: Mamba-2 as wide as the model (heads of 64 channels, a
    state of 128, two groups, four norm groups, four taps); parallel layers of attention with biases, convolutions of
    three taps and a capped score (heads of 128, four query heads per kv head, rescaled rotation of the whole head) beside a
    gated delta rule (heads of 128 x 256 behind convolutions of four taps); experts whose inputs are weighted beside a gated
    shared expert in every layer.  Seven layers."""
    g = max(1, width // 256)
    mam = {"type": "mamba2", "mixer": {"heads": width // 64, "vdim": 64, "state": 128, "groups": 2, "norm_groups": 4, "conv": 4}}
    par = {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "conv": 3, "softcap": 50.0,
                 "rot": {"base": 1000000.0, "dims": 128, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}},
        "right": {"heads": g, "kv_heads": max(1, g // 2), "dim": 128, "vdim": 256, "conv": 4}, "left_scale": 0.8, "right_scale": 0.5}}
    moe = {"kind": "moe", "expert": {"ff": expert_ff}, "shared": {"ff": expert_ff}, "router": {"experts": experts, "top": top}}
    layers = [dict(lay, mlp=moe) for lay in (mam, par, mam, mam, par, mam, par)]
    return {"architecture": "Sumozen", "vocab": 32768, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "max_position_embeddings": 8192}


DESIGN_SIZES = {
    # name: (width, heads, experts, chosen, expert ff, dense ff); Qwen3 beside it: the same width, layer runs and
    # heads of 128, a feed-forward as wide as the chosen experts together (equal products per token)
    "2048": (2048, 16, 16, 4, 1024, 5632),
    "4096": (4096, 32, 32, 4, 2048, 11264),
}


def compare_designs(args) -> int:
    """Prefill and decode throughput of the Luvavik design at layer sizes of real models, beside Qwen3
    dense at equal width, layer count and products per token; with --profile the per-kernel-class times
    and roofline fractions of both.  Prints one JSON line of its own (the default benchmark is untouched)."""
    import torch
    from zinfer_b200 import ops
    from zinfer_b200.config import LuvavikConfig, Qwen3Config
    from zinfer_b200.engine import StepEntry
    from zinfer_b200.engine.api import Engine

    hbm_gbs, bf16_tflops, peak_src = peaks()
    gen = torch.Generator().manual_seed(99)
    steps, warmup, batch = args.steps, max(3, args.warmup), args.batch
    tokens, context = 2048, 2048
    results, profiles = {}, {}

    def event_ms(fn, n):
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        for _ in range(n):
            fn()
        end.record()
        torch.cuda.synchronize()
        return start.elapsed_time(end) / n

    def measure(name, cfg, vocab):
        engine = Engine(config=cfg, random_weights_seed=7, dtype="bfloat16", device="cuda:0", page_size=16,
                        kv_cache_tokens=batch * (context + steps + warmup + 64) + tokens + 64,
                        max_batched_tokens=tokens, max_requests=batch + 1, max_model_len=8192)
        runner = engine.runner
        rand = lambda n: torch.randint(0, vocab, (n,), generator=gen).tolist()
        prompt = rand(tokens)

        def prefill_once():
            runner.step([StepEntry("prefill", prompt, [tokens - 1])])
            runner.end_request("prefill")

        for _ in range(2):
            prefill_once()
        pf_ms = event_ms(prefill_once, 3)
        ids = [f"d{i}" for i in range(batch)]
        for rid in ids:
            runner.step([StepEntry(rid, rand(context), [])])
        cur = rand(batch)
        one = lambda: runner.step_argmax([StepEntry(rid, [t], [0]) for rid, t in zip(ids, cur)])
        for _ in range(warmup):
            one()
        dec_ms = event_ms(one, steps)
        out = {"prefill_tokens_per_s": round(tokens / (pf_ms * 1e-3), 1), "prefill_ms": round(pf_ms, 3),
               "decode_tokens_per_s": round(batch / (dec_ms * 1e-3), 1), "decode_ms_per_step": round(dec_ms, 4),
               "weight_gb": round(runner.model.weight_bytes() / 1e9, 3)}
        if args.profile:
            with engine.profile(hbm_gbs, bf16_tflops) as prof:
                for _ in range(3):
                    one()
                dec = prof.summary()
            with engine.profile(hbm_gbs, bf16_tflops) as prof:
                prefill_once()
                pf = prof.summary()
            profiles[name] = {"decode": dec, "prefill": pf}
        for rid in ids:
            runner.end_request(rid)
        ops.require_kernel_status_ok(name)
        del engine, runner
        torch.cuda.empty_cache()
        return out

    for size in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
        width, heads, experts, top, eff, dff = DESIGN_SIZES[size]
        raw = luvavik_shape(width, heads, experts, top, eff, dff)
        if args.design == "rogosun":
            # beside Luvavik, the nearest design the engine has (recurrent layers, attention, routed experts), and Qwen3
            from zinfer_b200.config import RogosunConfig
            own = rogosun_shape(width, heads, experts, top, eff, dff)
            results[f"rogosun_{size}"] = measure(f"rogosun_{size}", RogosunConfig.from_dict(own), own["vocab"])
        if args.design == "vumezen":
            # beside Rogosun, whose attention (a sink, the same tensor-core kernels) and experts (sigmoid scores, a shared
            # expert) are the nearest the engine has, and Qwen3
            from zinfer_b200.config import RogosunConfig, VumezenConfig
            own = vumezen_shape(width, heads, experts, top, eff, dff)
            results[f"vumezen_{size}"] = measure(f"vumezen_{size}", VumezenConfig.from_dict(own), own["vocab"])
            other = rogosun_shape(width, heads, experts, top, eff, dff)
            results[f"rogosun_{size}"] = measure(f"rogosun_{size}", RogosunConfig.from_dict(other), other["vocab"])
        elif args.design == "sumozen":
            # beside Rogosun (attention beside a delta rule on the same input, linear recurrences with a matrix state, experts
            # beside a shared one) with routed experts in every layer, and Qwen3
            from zinfer_b200.config import RogosunConfig, SumozenConfig
            own = sumozen_shape(width, heads, experts, top, eff)
            results[f"sumozen_{size}"] = measure(f"sumozen_{size}", SumozenConfig.from_dict(own), own["vocab"])
            other = rogosun_shape(width, heads, experts, top, eff, dff)
            routed = next(lay["mlp"] for lay in other["layers"] if lay["mlp"]["kind"] == "moe")
            for lay in other["layers"]:
                lay["mlp"] = routed
            results[f"rogosun_{size}"] = measure(f"rogosun_{size}", RogosunConfig.from_dict(other), other["vocab"])
        elif args.design == "sepitar":
            # beside Vumezen (blocks whose sublayers read one stream, attention with a window and a sink on the same
            # tensor-core kernels, experts beside a shared one), Luvavik (latent attention) and Qwen3
            from zinfer_b200.config import SepitarConfig, VumezenConfig
            own = sepitar_shape(width, heads, experts, top, eff, dff)
            results[f"sepitar_{size}"] = measure(f"sepitar_{size}", SepitarConfig.from_dict(own), own["vocab"])
            other = vumezen_shape(width, heads, experts, top, eff, dff)
            results[f"vumezen_{size}"] = measure(f"vumezen_{size}", VumezenConfig.from_dict(other), other["vocab"])
            results[f"luvavik_{size}"] = measure(f"luvavik_{size}", LuvavikConfig.from_dict(raw), raw["vocab"])
        elif args.design == "kesitar":
            # beside Rogosun (a linear recurrence with a decay per key channel, norms of the sublayers' outputs) with dense
            # feed-forwards of equal products, Vumezen (windowed attention with a sink on the same tensor-core kernels)
            # and Qwen3 with the same dense feed-forward
            from zinfer_b200.config import KesitarConfig, RogosunConfig, VumezenConfig
            own = kesitar_shape(width, heads, dff)
            results[f"kesitar_{size}"] = measure(f"kesitar_{size}", KesitarConfig.from_dict(own), own["vocab"])
            other = rogosun_shape(width, heads, experts, top, eff, dff)
            for lay in other["layers"]:
                lay["mlp"] = {"kind": "dense", "ff": dff * 3 // 2}
            results[f"rogosun_dense_{size}"] = measure(f"rogosun_dense_{size}", RogosunConfig.from_dict(other), other["vocab"])
            other = vumezen_shape(width, heads, experts, top, eff, dff)
            results[f"vumezen_{size}"] = measure(f"vumezen_{size}", VumezenConfig.from_dict(other), other["vocab"])
        else:
            results[f"luvavik_{size}"] = measure(f"luvavik_{size}", LuvavikConfig.from_dict(raw), raw["vocab"])
        # two products of an expert against three of the gated feed-forward: equal multiply-adds per token
        qwen_ff = dff if args.design == "kesitar" else (2 * top * eff) // 3 // 64 * 64
        qwen = dict(QWEN3_8B, vocab_size=raw["vocab"], hidden_size=width, intermediate_size=qwen_ff,
                    num_hidden_layers=7, num_attention_heads=heads, num_key_value_heads=max(1, heads // 4), head_dim=128,
                    max_position_embeddings=8192)
        results[f"qwen3_{size}"] = measure(f"qwen3_{size}", Qwen3Config.from_dict(qwen), raw["vocab"])
    if args.profile:
        with open(args.profile, "w") as f:
            json.dump(profiles, f, indent=1)
    names = {"rogosun": "Rogosun beside Luvavik and Qwen3 dense", "vumezen": "Vumezen beside Rogosun and Qwen3 dense",
             "sumozen": "Sumozen beside Rogosun (routed experts in every layer) and Qwen3 dense",
             "sepitar": "Sepitar beside Vumezen, Luvavik and Qwen3 dense",
             "kesitar": "Kesitar beside Rogosun (dense feed-forwards), Vumezen and Qwen3 dense"}.get(
        args.design, "Luvavik beside Qwen3 dense")
    print(json.dumps({"metric": f"prefill and decode tokens/s, {names} at equal width and layer runs",
                      "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16",
                      "data": "synthetic", "config": {"prefill_tokens": tokens, "decode_batch": batch, "context": context,
                                                      "layer_runs": 7, "peaks": peak_src}, "results": results}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the model has (reported in config)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--impl", default="zinfer_b200", choices=["zinfer_b200", "reference"])
    ap.add_argument("--skip-points", action="store_true", help="only the headline batch (for profiling runs)")
    ap.add_argument("--profile", default=None, metavar="PATH",
                    help="also run one prefill and a few decode steps under the per-kernel-class profiler "
                         "(uncaptured, outside every timed region) and write its summary there as JSON")
    ap.add_argument("--timeline", default=None, metavar="PATH",
                    help="with ZINFER_B200_TRACE=1 in the environment: write the timeline of one decode step at the "
                         "headline batch (every kernel's start, the completion of what it depends on, and what it adds "
                         "to the chain) there as JSON, and do nothing else")
    ap.add_argument("--design", default=None, choices=["luvavik", "rogosun", "vumezen", "sepitar", "kesitar", "sumozen"],
                    help="instead of the default benchmark: prefill and decode throughput of this design at layer sizes "
                         "of real models beside Qwen3 dense at equal size (a JSON line of its own)")
    ap.add_argument("--design-sizes", default=None, help="with --design: widths to run, e.g. 2048 or 2048,4096")
    args = ap.parse_args()

    if args.design and args.impl != "reference" and args.gpus == 1:
        return compare_designs(args)
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "NeoZedAtlas/Zinfer is a Zig program (needs zig >= 0.15.2); no Zig toolchain exists here and "
                          "pip cannot install it: it has neither setup.py nor pyproject.toml"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch
    from zinfer_b200 import ops
    from zinfer_b200.config import Qwen3Config
    from zinfer_b200.engine import StepEntry
    from zinfer_b200.engine.api import Engine
    from zinfer_b200.sampling import SamplingParams

    full_layers = QWEN3_8B["num_hidden_layers"]
    n_layers = args.layers or full_layers
    cfg = Qwen3Config.from_dict({**QWEN3_8B, "num_hidden_layers": n_layers})
    hbm_gbs, bf16_tflops, peak_src = peaks()
    dev = torch.device("cuda:0")
    gen = torch.Generator().manual_seed(1234)
    max_batch = args.batch if args.skip_points else max(64, args.batch)
    steps, warmup = args.steps, args.warmup

    engine = Engine(config=cfg, random_weights_seed=20240, dtype="bfloat16", device="cuda:0", page_size=16,
                    kv_cache_tokens=max_batch * (PROMPT_LEN + steps + warmup + 64) + PREFILL_TOKENS + 64,
                    max_batched_tokens=max(PREFILL_TOKENS, 2048), max_requests=max_batch)
    runner = engine.runner
    weight_bytes = runner.model.weight_bytes() - cfg.vocab_size * cfg.hidden_size * 2   # the embedding table is only gathered
    kv_bytes_per_token = 2 * n_layers * cfg.num_key_value_heads * cfg.head_dim * 2

    def rand_tokens(n):
        return torch.randint(0, cfg.vocab_size, (n,), generator=gen).tolist()

    def event_ms(fn, n):
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        for _ in range(n):
            fn()
        end.record()
        torch.cuda.synchronize()
        return start.elapsed_time(end)

    if args.timeline:
        from zinfer_b200 import profiling

        ids = [f"t{i}" for i in range(args.batch)]
        for rid in ids:
            runner.step([StepEntry(rid, rand_tokens(PROMPT_LEN), [])])
        cur = torch.randint(0, cfg.vocab_size, (args.batch,), generator=gen).tolist()

        def one_step():
            runner.step_argmax([StepEntry(rid, [t], [0]) for rid, t in zip(ids, cur)])

        kernels = profiling.chain_timeline(one_step, warm=4)
        # the chain of a decode step of this architecture, when its kernel count says that it is the one meant
        per_layer = ["input norm", "qkv product", "attention (fused)", "attention combine", "o product", "post-attention norm",
                     "gate_up product", "swiglu", "down product"]
        names = ["embedding"] + per_layer * n_layers + ["final norm", "output head", "argmax (candidates)"]
        for i, k in enumerate(kernels):
            k["kernel"] = names[i] if len(names) == len(kernels) else f"kernel {i}"
        with open(args.timeline, "w") as f:
            json.dump({"batch": args.batch, "context": PROMPT_LEN, "layers": n_layers, "kernels": kernels}, f, indent=1)
        per = {}
        for k in kernels:
            if k["own_us"] is not None:
                per.setdefault(k["kernel"], []).append(k["own_us"])
        for name, v in per.items():
            print(f"{name:24s} {statistics.median(v):8.2f} us (median of {len(v)})")
        return 0

    # ---------------------------------------------------------------- prefill
    def prefill_once():
        runner.step([StepEntry("prefill", prompt, [PREFILL_TOKENS - 1])])
        runner.end_request("prefill")

    prompt = rand_tokens(PREFILL_TOKENS)
    for _ in range(2):
        prefill_once()
    pf_ms = event_ms(prefill_once, 3) / 3
    attn_flops = n_layers * 4 * cfg.num_attention_heads * cfg.head_dim * (PREFILL_TOKENS * (PREFILL_TOKENS + 1) // 2)
    pf_flops = 2 * PREFILL_TOKENS * matmul_params(cfg, n_layers) + attn_flops + 2 * cfg.vocab_size * cfg.hidden_size
    prefill = {"value": round(PREFILL_TOKENS / (pf_ms * 1e-3), 1), "tokens": PREFILL_TOKENS, "ms": round(pf_ms, 3),
               "frac": round(pf_flops / (pf_ms * 1e-3) / (bf16_tflops * 1e12), 4)}

    def prefill_chunked():
        for c in range(0, PREFILL_TOKENS, 512):
            last = c + 512 >= PREFILL_TOKENS
            runner.step([StepEntry("prefill", prompt[c:c + 512], [511] if last else [])])
        runner.end_request("prefill")

    prefill_chunked()
    ck_ms = event_ms(prefill_chunked, 3) / 3
    prefill["chunks_512"] = {"value": round(PREFILL_TOKENS / (ck_ms * 1e-3), 1), "ms": round(ck_ms, 3),
                             "frac": round(pf_flops / (ck_ms * 1e-3) / (bf16_tflops * 1e12), 4)}

    # ----------------------------------------------------------------- decode
    def decode_point(batch: int, n_steps: int, sample_clocks: bool = False):
        """Device-timed decode at `batch`: every request holds PROMPT_LEN cached tokens
        (their cache is filled by real prefill steps), then n_steps steps of one token each."""
        ids = [f"d{batch}_{i}" for i in range(batch)]
        for rid in ids:
            runner.step([StepEntry(rid, rand_tokens(PROMPT_LEN), [])])
        cur = torch.randint(0, cfg.vocab_size, (batch,), generator=gen).tolist()

        def one():
            nonlocal cur
            return runner.step_argmax([StepEntry(rid, [t], [0]) for rid, t in zip(ids, cur)])[1]

        for _ in range(warmup):
            one()
        launches0 = ops.LAUNCHES + runner.graph_launches if hasattr(runner, "graph_launches") else ops.LAUNCHES
        sampler = ClockSampler() if sample_clocks else None
        if sampler:
            sampler.__enter__()
        ms = event_ms(one, n_steps)
        if sampler:
            sampler.__exit__()
        launches = (ops.LAUNCHES + runner.graph_launches if hasattr(runner, "graph_launches") else ops.LAUNCHES) - launches0
        mean_ctx = PROMPT_LEN + warmup + n_steps / 2
        for rid in ids:
            runner.end_request(rid)
        return ms / n_steps, launches, mean_ctx, (sampler.summary() if sampler else None)

    ms_step, launches, mean_ctx, clocks = decode_point(args.batch, steps, sample_clocks=True)
    value = args.batch / (ms_step * 1e-3)
    step_bytes = weight_bytes + args.batch * mean_ctx * kv_bytes_per_token
    achieved = step_bytes / (ms_step * 1e-3) / 1e9
    points = {}
    if not args.skip_points:
        for b in (1, 64):
            m, _, _, _ = decode_point(b, min(steps, 32))
            points[f"decode_b{b}"] = round(b / (m * 1e-3), 1)

    # ------------------------------------------------- end to end through the API
    def e2e_point(batch: int, n_steps: int, **sampling) -> tuple[float, int]:
        """Decoded tokens a second through Engine.step (host tokens in and out), and the bytes of
        the step's one host->device copy.  Greedy unless sampling options are given.  Prompts are
        admitted one a step, so the first request has decoded `batch` tokens before the last one is
        in: every request may generate enough to stay live through the timed steps, and the tokens
        counted are the ones the requests really gained."""
        params = SamplingParams(**{"temperature": 0.0, **sampling}, max_new_tokens=batch + n_steps + warmup + 8, ignore_eos=True)
        rids = [engine.add_request(rand_tokens(PROMPT_LEN), params) for _ in range(batch)]
        reqs = [engine._live[rid] for rid in rids]
        while any(r.num_computed < len(r.prompt) for r in engine.scheduler.running) or engine.scheduler.waiting:
            engine.step()
        for _ in range(warmup):
            engine.step()
        torch.cuda.synchronize()
        before = sum(len(r.output) for r in reqs)
        t0 = time.perf_counter()
        for _ in range(n_steps):
            engine.step()
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        gained = sum(len(r.output) for r in reqs) - before
        if gained != batch * n_steps or len(engine.scheduler.running) != batch:
            raise RuntimeError(f"e2e at batch {batch}: {gained} tokens in {n_steps} steps, {len(engine.scheduler.running)} requests live")
        h2d_bytes = runner.last_h2d_bytes
        while engine.has_unfinished():
            engine.step()
        return gained / dt, int(h2d_bytes)

    e2e_value, h2d = e2e_point(args.batch, steps)
    e2e = {"value": round(e2e_value, 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * args.batch}
    if not args.skip_points:
        e2e["points"] = {f"decode_b{b}": round(e2e_point(b, min(steps, 32))[0], 1) for b in (1, 64)}
        # the same with the reference's default sampling options instead of greedy (src/app/cli/args.zig:364-370)
        e2e["sampled"] = {"value": round(e2e_point(args.batch, min(steps, 32), temperature=0.7, top_k=20, top_p=0.8,
                                                   repetition_penalty=1.1, seed=7)[0], 1),
                          "options": "temperature 0.7, top-k 20, top-p 0.8, repetition penalty 1.1"}

    # -------------------------------- where the time goes (uncaptured, never a timed number)
    if args.profile:
        ids = [f"p{i}" for i in range(args.batch)]
        for rid in ids:
            runner.step([StepEntry(rid, rand_tokens(PROMPT_LEN), [])])
        cur = torch.randint(0, cfg.vocab_size, (args.batch,), generator=gen).tolist()
        with engine.profile(hbm_gbs, bf16_tflops) as prof:
            for _ in range(4):
                runner.step_argmax([StepEntry(rid, [t], [0]) for rid, t in zip(ids, cur)])
            decode_profile = prof.summary()
        for rid in ids:
            runner.end_request(rid)
        with engine.profile(hbm_gbs, bf16_tflops) as prof:
            prefill_once()
            prefill_profile = prof.summary()
        with open(args.profile, "w") as f:
            json.dump({"decode": {"batch": args.batch, "context": PROMPT_LEN, **decode_profile},
                       "prefill": {"tokens": PREFILL_TOKENS, **prefill_profile}}, f, indent=1)

    out = {
        "metric": "decode tok/s at batch 8 (Qwen3-8B shape, bf16)", "value": round(value, 1), "unit": "tokens/s",
        "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": round(ms_step, 4), "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "impl": "zinfer_b200",
        "config": {
            "model": "Qwen3-8B shape, random weights", "global_batch": args.batch, "seq_len": CONTEXT_LEN,
            "prompt_len": PROMPT_LEN, "parallelism": "single GPU", "layers": n_layers, "layers_full_model": full_layers,
            "hidden_size": cfg.hidden_size, "intermediate_size": cfg.intermediate_size,
            "num_attention_heads": cfg.num_attention_heads, "num_key_value_heads": cfg.num_key_value_heads,
            "head_dim": cfg.head_dim, "vocab_size": cfg.vocab_size, "page_size": 16, "kv_dtype": "bf16",
            "l2": "inputs larger than L2 (weights streamed every step)", "peaks": peak_src,
        },
        "e2e": e2e, "gpu_launches": int(launches), "clocks": clocks,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": hbm_gbs, "unit": "GB/s",
                     "frac": round(achieved / hbm_gbs, 4)},
        "points": points,
    }
    ops.require_kernel_status_ok("bench")   # a kernel whose bounded wait ran out would make every number above void
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
