#!/usr/bin/env python3
"""Benchmark of the engine's decode step (and a 2,048-token prefill) at Qwen3-8B layer sizes.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--layers L] [--impl ours|reference]

Prints ONE JSON line.  ``value`` is decoded tokens per second at the given batch (default 8), each
sequence holding ``context_len`` tokens of context, timed on the device with CUDA events around
exactly K decode steps after W warm-up steps; a step includes the greedy pick of every sequence's
next token on the device.  ``e2e`` is the same measured through the Python entry point (the
scheduler, the step function and the sampler): every step copies its inputs from pinned host memory
to the device and reads the sampled tokens back to the host.  ``prefill`` is one 2,048-token prompt
in one step; ``roofline`` compares the bytes a decode step has to read (every weight once, and the
cache of the live requests) with the measured copy bandwidth; ``points`` holds decode at batch 1 and
64 and the main batch without the pick; ``check`` (outside every timed region) says whether a short greedy
continuation by the timed engine is what a float32 engine of the same weights picks, ties apart.
``--profile`` prints a per-kernel table instead.
Weights are random (seeded), token ids are uniform-random (seeded): no dataset is involved.
The weights alone (over 15 GB) exceed the L2 cache many times over, so no flush is needed between
steps.  Runs on one GPU only.
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

SIZES_8B = dict(num_hidden_layers=36, hidden_size=4096, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
                intermediate_size=12288, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6,
                tie_word_embeddings=False, max_position_embeddings=40960)
SIZES_14B = dict(SIZES_8B, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408)
SIZES_32B = dict(SIZES_8B, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, intermediate_size=25600)
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            with open(path) as fh:
                p = json.load(fh)
            return {"hbm_gbs": float(p["hbm_gbs"]), "bf16_tflops": float(p["bf16_tflops"]),
                    "bf16_tflops_sustained": float(p.get("bf16_tflops_sustained", p["bf16_tflops"])), "source": "measured"}
        except (OSError, ValueError, KeyError):
            pass
    return dict(FALLBACK_PEAKS, bf16_tflops_sustained=1400.0, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.time(), line.strip()))

    def mark(self):
        return time.time()

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()

    def summary(self, t0, t1):
        mhz, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for t, line in self.samples:
            if not (t0 - 0.05 <= t <= t1 + 0.15):
                continue
            f = [x.strip() for x in line.split(",")]
            try:
                mhz.append(int(f[0])); mx = max(mx, int(f[1]))
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, f[2:]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": int(statistics.median(mhz)) if mhz else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(mhz)}


def decode_bytes(cfg, layers, batch, ctx, el=2):
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    q, kv = cfg["num_attention_heads"] * cfg["head_dim"], cfg["num_key_value_heads"] * cfg["head_dim"]
    per_layer = (q + 2 * kv) * H + H * q + 3 * H * I + 2 * H + 2 * cfg["head_dim"]
    weights = layers * per_layer + V * H + H + batch * H            # head, final norm, the embedding rows that are read
    cache = layers * 2 * kv * ctx * batch
    return (weights + cache) * el


def prefill_flops(cfg, layers, T):
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nh, d = cfg["num_attention_heads"], cfg["head_dim"]
    q, kv = nh * d, cfg["num_key_value_heads"] * d
    linear = 2 * T * ((q + 2 * kv) * H + H * q + 3 * H * I)
    attn = 4 * d * nh * T * (T + 1) // 2
    return layers * (linear + attn) + 2 * V * H


def serve_workload(args, BenchHarness) -> int:
    """The two serving workloads of the larger model sizes, through the engine's public entry point."""
    import numpy as np
    if args.workload == "mixed-14b":
        sizes, name, n_req, new_tokens, budget = SIZES_14B, "Qwen3-14B sizes", 32, 128, 2048
        lens = np.random.default_rng(1).integers(128, 3073, size=n_req).tolist()
    else:
        sizes, name, n_req, new_tokens, budget = SIZES_32B, "Qwen3-32B sizes", 16, 256, 4096
        lens = [1024] * n_req
    layers = args.layers if args.layers != SIZES_8B["num_hidden_layers"] else sizes["num_hidden_layers"]
    h = BenchHarness(dict(sizes, num_hidden_layers=layers), max_batch=n_req, context=max(lens), new_tokens=new_tokens,
                     graphs=not args.no_graphs, step_tokens=budget)
    h.serve(lens, new_tokens)                      # once untimed: kernels, graphs and allocations are warm afterwards
    clocks = ClockSampler()
    clocks.start()
    time.sleep(0.3)
    t0 = clocks.mark()
    r = h.serve(lens, new_tokens)
    t1 = clocks.mark()
    clocks.stop()
    print(json.dumps({
        "metric": f"tokens/s (prompt + generated) of the {args.workload} workload ({name}, bf16)", "value": round(r["tokens_per_s"], 1),
        "unit": "tokens/s", "n_gpus": 1, "generated_tokens_per_s": round(r["generated_per_s"], 1), "seconds": round(r["seconds"], 3),
        "steps": r["steps"], "ms_per_step": round(r["seconds"] / r["steps"] * 1e3, 3), "prompt_tokens": r["prompt_tokens"],
        "generated_tokens": r["generated_tokens"], "higher_is_better": True, "dtype": "bf16", "impl": "ours",
        "data": "synthetic: seeded random weights, seeded uniform-random token ids",
        "config": {"model": name, "layers": layers, "layers_of_model": sizes["num_hidden_layers"], "hidden_size": sizes["hidden_size"],
                   "heads": sizes["num_attention_heads"], "kv_heads": sizes["num_key_value_heads"], "head_dim": sizes["head_dim"],
                   "intermediate_size": sizes["intermediate_size"], "vocab_size": sizes["vocab_size"], "requests": n_req,
                   "prompt_tokens_min": int(min(lens)), "prompt_tokens_max": int(max(lens)), "new_tokens": new_tokens,
                   "step_token_budget": budget, "page_size": h.page_size, "cuda_graphs": h.graphs},
        "clocks": clocks.summary(t0, t1), "gpu_launches": r["launches"]}))
    return 0


# Layer sizes for the comparison of the two designs: width, query heads, key/value heads, feed-forward width
COMPARE_SIZES = {"1b": (2048, 16, 4, 6144), "4b": (2560, 20, 4, 9728), "8b": (4096, 32, 8, 12288)}


def munizen_config(width, heads, kv_heads, ff, layers, vocab):
    """A Munizen model whose layers alternate between the recurrent mixer and differential attention, every
    layer with a feed-forward: per layer the same projection and feed-forward sizes as the Qwen3 model beside it
    (a query head's two maps of 64 take the place of one head of 128; state heads of 64)."""
    from carbon_engine_b200.config.munizen import MunizenConfig
    attn = {"type": "attention", "mlp": {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": 64, "vdim": 128, "diff": 0.3, "scale": 0.125,
                      "rot": {"dims": 32, "base": 1e6}, "mask": {"size": 1024}}}
    delta = {"type": "general_delta", "mlp": {"kind": "dense", "ff": ff},
             "mixer": {"heads": width // 64, "dim": 64, "rank": 64}}
    return MunizenConfig.from_dict({"architecture": "Munizen", "vocab": vocab, "width": width,
                                    "layers": [delta if i % 2 == 0 else attn for i in range(layers)],
                                    "norm": {"eps": 1e-6, "groups": 2}, "streams": 2, "max_position_embeddings": 8192})


def lunerax_config(width, heads, kv_heads, ff, layers, vocab):
    """A Lunerax model of the usual proportions at the Qwen3 model's layer sizes: layers go attention (heads of 128, capped
    scores, a window of 1,024 that keeps 4 first tokens, blended values), delta rule, delta rule (state heads of 128 x 128,
    4 taps), latent attention (a cached row of 256 + 32 per token, a window of 1,024); every layer with the feed-forward
    and a per-layer token input of 128."""
    from carbon_engine_b200.config.lunerax import LuneraxConfig
    ffn = {"kind": "dense", "ff": ff}
    attn = {"type": "attention", "mlp": ffn,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                      "mask": {"size": 1024, "keep_first": 4}, "v_mix": True}}
    delta = {"type": "channel_delta", "mlp": ffn,
             "mixer": {"heads": width // 128, "kv_heads": width // 128, "dim": 128, "vdim": 128, "conv": 4, "a_rank": 64, "g_rank": 64}}
    latent = {"type": "latent_attention", "mlp": ffn,
              "mixer": {"heads": heads, "dim": 128, "rot_dim": 32, "vdim": 128, "q_rank": width // 4, "kv_rank": 256,
                        "scale": 160 ** -0.5, "rot": {"dims": 32, "base": 1e6}, "mask": {"size": 1024}}}
    kinds = (attn, delta, delta, latent)
    return LuneraxConfig.from_dict({"architecture": "Lunerax", "vocab": vocab, "width": width,
                                    "layers": [kinds[i % 4] for i in range(layers)], "norm": {"eps": 1e-6},
                                    "embedding": {"scale": float(width) ** 0.5}, "logit_softcap": 30.0,
                                    "token_side": {"dim": 128}, "max_position_embeddings": 8192})


def vamadra_config(width, heads, kv_heads, ff, layers, vocab):
    """A Vamadra model at the Qwen3 model's layer sizes: every layer latent attention with the Lunerax latent layer's sizes
    (heads of 128 + 32, values of 128, a cached row of 256 + 32 per token; no window), a sink and a gate per head, stretched
    rotary frequencies; of every two layers the second reads the rows the first cached.  The feed-forward alternates between
    the dense one and a mixture of 32 experts in 4 groups (2 kept), 4 per token, each an eighth of the dense width, beside a
    shared expert of half the dense width: a token's products are as wide as the dense layer's."""
    from carbon_engine_b200.config.vamadra import VamadraConfig
    rotation = {"dims": 32, "base": 1e6, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    out = []
    for i in range(layers):
        m = {"heads": heads, "dim": 128, "rot_dim": 32, "vdim": 128, "kv_rank": 256, "scale": 160 ** -0.5, "rot": rotation}
        if i % 2:
            m["kv_from"] = i - 1
        mlp = {"kind": "dense", "ff": ff} if i % 2 == 0 else {
            "kind": "moe", "expert": {"ff": ff // 8}, "shared": {"ff": ff // 2},
            "router": {"experts": 32, "top": 4, "groups": {"count": 4, "keep": 2}, "scale": 2.5}}
        out.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return VamadraConfig.from_dict({"architecture": "Vamadra", "vocab": vocab, "width": width, "layers": out,
                                    "norm": {"eps": 1e-6}, "max_position_embeddings": 8192})


def pugozen_config(width, heads, kv_heads, ff, layers, vocab):
    """A Pugozen model of the usual proportions at the Qwen3 model's layer sizes: layers go delta rule with a decay per head
    (state heads of 128 x 128, half as many key heads, 4 taps), the pair (attention with heads of 128 whose values are the
    projected keys, a quarter of a head rotated, a temperature and a sink per head, beside the delta rule with a decay per
    key channel: state heads of 128 x 128, 3 taps), the pair again, retention (state heads of 128 x 128, whole heads rotated);
    every layer with the dense squared-ReLU feed-forward; no layer shares weights."""
    from carbon_engine_b200.config.pugozen import PugozenConfig
    ffn = {"kind": "dense", "ff": ff}
    n = width // 128
    delta = {"type": "delta", "mlp": ffn, "mixer": {"heads": n, "kv_heads": max(1, n // 2), "dim": 128, "vdim": 128, "conv": 4}}
    pair = {"type": "parallel", "mlp": ffn,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                               "rot": {"dims": 32, "base": 1e6}},
                      "right": {"heads": n, "kv_heads": n, "dim": 128, "vdim": 128, "conv": 3, "a_rank": 64, "g_rank": 64},
                      "left_scale": 0.7, "right_scale": 0.6}}
    retention = {"type": "retention", "mlp": ffn,
                 "mixer": {"heads": n, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - (6 * j) // n) for j in range(n)],
                           "rot": {"dims": 128, "base": 1e6}}}
    kinds = (delta, pair, pair, retention)
    return PugozenConfig.from_dict({"architecture": "Pugozen", "vocab": vocab, "width": width,
                                    "layers": [kinds[i % 4] for i in range(layers)], "norm": {"eps": 1e-6},
                                    "embedding": {"scale": float(width) ** 0.5}, "max_position_embeddings": 8192})


def rapovik_config(width, heads, kv_heads, ff, layers, vocab):
    """A Rapovik model of the usual proportions at the Qwen3 model's layer sizes: layers go state space (state heads of 128 x 128
    filling the width, 1 group, 4 taps), matrix memory (state heads of 128 x 128), latent attention (heads of 128 + 32, values of
    128, a cached row of 256 + 32 per token, a window of 1,024), state space again.  The feed-forward alternates between the dense
    gated one and a mixture of 32 gated experts in 4 groups (2 kept), 4 per token, each an eighth of the dense width, beside a shared expert of
    half the dense width: a token's products are as wide as the dense layer's.  No layer is looped."""
    from carbon_engine_b200.config.rapovik import RapovikConfig
    n = width // 128
    ssm = {"type": "mamba2", "mixer": {"heads": n, "vdim": 128, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1}}
    memory = {"type": "mlstm", "mixer": {"heads": n, "dim": 128, "vdim": 128, "gate_cap": 15.0}}
    latent = {"type": "latent_attention",
              "mixer": {"heads": heads, "dim": 128, "rot_dim": 32, "vdim": 128, "kv_rank": 256, "scale": 160 ** -0.5,
                        "rot": {"dims": 32, "base": 1e6}, "mask": {"size": 1024}}}
    dense = {"kind": "dense", "ff": ff, "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": ff // 8, "limit": 7.0}, "shared": {"ff": ff // 2, "limit": 7.0},
           "router": {"experts": 32, "top": 4, "groups": {"count": 4, "keep": 2}}}
    kinds = (ssm, memory, latent, ssm)
    return RapovikConfig.from_dict({"architecture": "Rapovik", "vocab": vocab, "width": width,
                                    "layers": [dict(kinds[i % 4], mlp=dense if i % 2 == 0 else moe) for i in range(layers)],
                                    "norm": {"eps": 1e-6}, "max_position_embeddings": 8192})


def lanirax_config(width, heads, kv_heads, ff, layers, vocab):
    """A Lanirax model of the usual proportions at the Qwen3 model's layer sizes: layers go the pair (attention with heads of 128
    whose values are the projected keys, a window of 1,024, half of a head rotated, a sink per head, beside the delta rule with a
    decay per head: state heads of 128 x 128 filling the width, half as many key heads, 4 taps) and attention (heads of 128 over
    all keys, a penalty on distance) and again, each with a mixture of 32 gated experts, 4 per token, each an eighth of the dense
    width: a token's products are half as wide as the dense layer's.  No layer shares weights."""
    from carbon_engine_b200.config.lanirax import LaniraxConfig
    n = width // 128
    moe = {"kind": "moe", "expert": {"ff": ff // 8}, "router": {"experts": 32, "top": 4}}
    pair = {"type": "parallel", "mlp": moe,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024},
                               "rot": {"dims": 64, "base": 1e6, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}},
                      "right": {"heads": n, "kv_heads": max(1, n // 2), "dim": 128, "vdim": 128, "conv": 4}}}
    attention = {"type": "attention", "mlp": moe,
                 "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                           "q_temp": {"coef": 0.1, "every": 1024}}}
    kinds = (pair, attention)
    return LaniraxConfig.from_dict({"architecture": "Lanirax", "vocab": vocab, "width": width,
                                    "layers": [kinds[i % 2] for i in range(layers)], "norm": {"eps": 1e-6}, "postln_alpha": 1.5,
                                    "max_position_embeddings": 8192})


def compare_designs(args, BenchHarness, pk) -> int:
    """Prefill and decode throughput of the engine's other designs (--designs: munizen, lunerax, vamadra, pugozen, rapovik, lanirax) beside the
    Qwen3 dense design at equal layer sizes (random weights, a few layers), with the kernels of each and their distance from the roofline."""
    import torch
    makers = {"munizen": munizen_config, "lunerax": lunerax_config, "vamadra": vamadra_config, "pugozen": pugozen_config,
              "rapovik": rapovik_config, "lanirax": lanirax_config}
    designs = [x for x in args.designs.split(",") if x != "qwen3"]
    for x in designs:
        if x not in makers:
            raise SystemExit(f"--designs {x}: munizen, lunerax, vamadra, pugozen, rapovik, lanirax and qwen3 are built")
    layers = args.layers if args.layers != SIZES_8B["num_hidden_layers"] else 4
    vocab, out = 32768, {}
    for name in args.sizes.split(","):
        width, heads, kv_heads, ff = COMPARE_SIZES[name]
        qwen = dict(SIZES_8B, num_hidden_layers=layers, hidden_size=width, num_attention_heads=heads,
                    num_key_value_heads=kv_heads, head_dim=128, intermediate_size=ff, vocab_size=vocab, max_position_embeddings=8192)
        row = {}
        for design, cfg in [(x, makers[x](width, heads, kv_heads, ff, layers, vocab)) for x in designs] + [("qwen3", qwen)]:
            h = BenchHarness(cfg, max_batch=max(args.batch, 2), context=args.context, new_tokens=256, graphs=not args.no_graphs,
                             step_tokens=max(4096, args.prefill_tokens))
            pf = h.prefill(args.prefill_tokens, 3, 2)
            dec = h.decode(args.batch, args.steps, args.warmup)
            r = {"prefill_tokens_per_s": round(args.prefill_tokens / (pf["ms"] / 1e3), 1), "prefill_ms": round(pf["ms"], 3),
                 "decode_tokens_per_s": round(dec["tokens_per_s"], 1), "decode_ms_per_step": round(dec["ms_per_step"], 4)}
            if args.profile:
                prof = h.profile(args.batch, args.prefill_tokens, pk["hbm_gbs"], pk["bf16_tflops"])
                r["kernels"] = {part: [dict(k) for k in prof[part]["kernels"]] for part in ("decode", "prefill")}
                for part in ("decode", "prefill"):
                    print(f"\n{design} {name}, {part}: {prof[part]['us']:.0f} us with kernels one after another", file=sys.stderr)
                    for k in prof[part]["kernels"]:
                        frac = "" if k["frac_of_peak"] is None else f"{k['frac_of_peak']:.3f}"
                        print(f"{k['kernel'][:58]:58s} {k['launches']:6d} {k['us']:10.1f} {k['share']:6.3f} {k['gb_s']:8.0f} "
                              f"{k['tflop_s']:8.1f} {frac:>8s}", file=sys.stderr)
            row[design] = r
            del h
            torch.cuda.empty_cache()
        out[name] = row
    print(json.dumps({"workload": "compare-designs", "layers": layers, "batch": args.batch, "context": args.context,
                      "prefill_tokens": args.prefill_tokens, "dtype": "bf16", "peaks": pk["source"],
                      "data": "synthetic: seeded random weights, seeded uniform-random token ids", "sizes": out}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=2048, help="tokens of context each sequence holds when decoding starts")
    ap.add_argument("--layers", type=int, default=SIZES_8B["num_hidden_layers"])
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 / 64 points and the prefill")
    ap.add_argument("--no-graphs", action="store_true")
    ap.add_argument("--prefill-only", action="store_true",
                    help="run only the prefill of one prompt (for profiling, and for other prompt lengths) and print its time")
    ap.add_argument("--prefill-tokens", type=int, default=2048, help="with --prefill-only: tokens of the prompt (one step)")
    ap.add_argument("--profile", action="store_true",
                    help="instead of the default JSON line: time every kernel of a decode step and of a 2,048-token prefill "
                         "with CUDA events (eager, kernels one after another) and print a table per kernel: launches, "
                         "microseconds, share, GB/s, TFLOP/s and the fraction of the measured peak")
    ap.add_argument("--between-steps", action="store_true",
                    help="instead of the default JSON line: the device activities between two decode steps through the entry "
                         "point (pick, read-back copies, upload, token copy) and the steps' period")
    ap.add_argument("--no-check", action="store_true", help="skip the comparison of a short greedy continuation with float32")
    ap.add_argument("--sizes", default="1b,8b", help="with --workload compare-designs: which of the layer sizes "
                    "1b, 4b, 8b (width / heads / feed-forward of models of about that size), with commas between them")
    ap.add_argument("--designs", default="munizen,qwen3", help="with --workload compare-designs: the designs set beside one another "
                    "(munizen, lunerax, vamadra, pugozen, rapovik, lanirax; qwen3 is always the last)")
    ap.add_argument("--workload", default="decode", choices=["decode", "mixed-14b", "batch16-32b", "compare-designs"],
                    help="decode: the headline line (default).  mixed-14b: 32 requests with prompts of 128 to 3,072 tokens at "
                         "Qwen3-14B sizes, prompts cut under a 2,048-token step budget beside the decoding requests, 128 new "
                         "tokens each.  batch16-32b: 16 prompts of 1,024 tokens at Qwen3-32B sizes, 256 new tokens each.  Both "
                         "run through the scheduler and print a line of their own.  compare-designs: prefill and decode throughput of "
                         "the Munizen design beside the Qwen3 dense design at equal layer sizes (--sizes, --layers, default 4; "
                         "with --profile also every kernel of both against the roofline)")
    args = ap.parse_args()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": "the reference is a Rust crate on the candle library: no "
                          "Python package to install offline, and neither cargo/rustc nor its crates are on this machine"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU only; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch
    from carbon_engine_b200.bench_support import BenchHarness
    pk = peaks()
    if args.workload == "compare-designs":
        return compare_designs(args, BenchHarness, pk)
    if args.workload != "decode":
        return serve_workload(args, BenchHarness)
    cfg = dict(SIZES_8B, num_hidden_layers=args.layers)
    if args.prefill_only:
        T = args.prefill_tokens
        h = BenchHarness(cfg, max_batch=2, context=max(args.context, T), new_tokens=256, graphs=not args.no_graphs,
                         step_tokens=max(4096, T))
        pf = h.prefill(T, 3, 2)
        flops = prefill_flops(cfg, args.layers, T)
        print(json.dumps({"prefill_ms": round(pf["ms"], 3), "tokens": T, "layers": args.layers,
                          "tokens_per_s": round(T / (pf["ms"] / 1e3), 1), "tflops": round(flops / (pf["ms"] / 1e3) / 1e12, 1),
                          "frac": round(flops / (pf["ms"] / 1e3) / (pk["bf16_tflops"] * 1e12), 4), "peaks": pk["source"]}))
        return 0
    h = BenchHarness(cfg, max_batch=max(64 if not args.no_points else args.batch, args.batch),
                     context=args.context,
                     new_tokens=max(256, args.steps + max(args.warmup, 32) + 8 + args.batch * ((args.context + 4095) // 4096 + 1)),
                     graphs=not args.no_graphs)
    if args.between_steps:
        print(json.dumps({"between_steps": h.between_steps(args.batch), "batch": args.batch, "context": args.context,
                          "layers": args.layers}, indent=1))
        return 0
    if args.profile:
        prof = h.profile(args.batch, 2048, pk["hbm_gbs"], pk["bf16_tflops"])
        for part in ("decode", "prefill"):
            p = prof[part]
            what = f"decode step, batch {p['batch']}, {args.context}-token contexts" if part == "decode" else f"prefill of {p['tokens']} tokens"
            print(f"\n{what}, {args.layers} layers: {p['us']:.0f} us with kernels one after another (peaks {pk['source']}: "
                  f"{pk['hbm_gbs']:.0f} GB/s, {pk['bf16_tflops']:.0f} TFLOP/s)", file=sys.stderr)
            print(f"{'kernel':58s} {'launches':>8s} {'us':>10s} {'share':>6s} {'GB/s':>8s} {'TFLOP/s':>8s} {'of peak':>8s}", file=sys.stderr)
            for r in p["kernels"]:
                frac = "" if r["frac_of_peak"] is None else f"{r['frac_of_peak']:.2f}"
                print(f"{r['kernel'][:58]:58s} {r['launches']:8d} {r['us']:10.1f} {r['share']:6.3f} {r['gb_s']:8.0f} {r['tflop_s']:8.0f} {frac:>8s}",
                      file=sys.stderr)
        print(json.dumps({"profile": prof, "layers": args.layers, "peaks": pk["source"]}))
        return 0
    clocks = ClockSampler()
    clocks.start()
    time.sleep(0.3)

    t0 = clocks.mark()
    main_run = h.decode(args.batch, args.steps, args.warmup)
    t1 = clocks.mark()
    e2e = h.decode_e2e(args.batch, args.steps, args.warmup)
    t2 = clocks.mark()
    points, prefill = {}, None
    if not args.no_points:
        pf = h.prefill(2048, 3, 3)
        flops = prefill_flops(cfg, args.layers, 2048)
        prefill = {"value": round(2048 / (pf["ms"] / 1e3), 1), "tokens": 2048, "ms": round(pf["ms"], 3),
                   "frac": round(flops / (pf["ms"] / 1e3) / (pk["bf16_tflops"] * 1e12), 4)}
        for b in (1, 64):
            r = h.decode(b, min(args.steps, 32), 3)
            points[f"decode_b{b}"] = round(r["tokens_per_s"], 1)
        # the same step without the greedy pick at its end (the logits are the step's result)
        points[f"decode_b{args.batch}_without_pick"] = round(h.decode(args.batch, min(args.steps, 32), 3, pick=False)["tokens_per_s"], 1)
    clocks.stop()
    check = None if args.no_check else h.check_against_float32()

    ms = main_run["ms_per_step"]
    need = decode_bytes(cfg, args.layers, args.batch, args.context + args.warmup + args.steps // 2)
    achieved = need / (ms / 1e3) / 1e9
    out = {
        "metric": f"decode tok/s at batch {args.batch} (Qwen3-8B sizes, bf16, {args.context}-token contexts)", "value": round(main_run["tokens_per_s"], 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(ms, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: seeded random weights, seeded uniform-random token ids", "impl": "ours",
        "config": {"model": "Qwen3-8B sizes", "layers": args.layers, "layers_of_model": SIZES_8B["num_hidden_layers"],
                   "hidden_size": cfg["hidden_size"], "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
                   "head_dim": cfg["head_dim"], "intermediate_size": cfg["intermediate_size"], "vocab_size": cfg["vocab_size"],
                   "global_batch": args.batch, "seq_len": args.context, "max_seq_len": h.max_seq_len, "new_tokens": args.steps,
                   "page_size": h.page_size, "parallelism": "single GPU", "cuda_graphs": h.graphs,
                   "l2": "inputs larger than L2 (weights over 15 GB per step)", "peaks": pk["source"]},
        "clocks": clocks.summary(t0, t1),
        "e2e": {"value": round(e2e["tokens_per_s"], 1), "unit": "tokens/s", "ms_per_step": round(e2e["ms_per_step"], 4),
                "h2d_bytes_per_step": e2e["h2d_bytes"], "d2h_bytes_per_step": e2e["d2h_bytes"],
                # timed steps that were launched before the step before them had been read back
                "steps_launched_ahead": e2e["launched_ahead"],
                # over the whole e2e run: its prompts' prefill (which may meet the power cap), warm-up and timed steps
                "clocks": clocks.summary(t1, t2)},
        "gpu_launches": main_run["launches"],
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
    }
    if prefill is not None:
        out["prefill"] = prefill
        out["points"] = points
    if check is not None:
        out["check"] = check
    print(json.dumps(out))
    return 0 if check is None or check["ok"] else 1


if __name__ == "__main__":
    sys.exit(main())
