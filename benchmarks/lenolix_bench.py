"""Prefill and decode throughput of the Lenolix family beside the closest dense model (Llama layers, bf16) at equal
width, heads, feed-forward, vocabulary and depth, with random weights:

  python bench.py --design lenolix [--sizes 1b,3b,8b] [--layers 8] [--window 512] [--keep-first 64]

One JSON line per size: device time and tokens/s of one prefill step and one decode step (CUDA graphs, CUDA events,
median of several replays; the weights of the layers are larger than L2), and every kernel class with its algorithmic
bytes and operations, its time and its distance from the measured roofline (time / roofline time). ``like``: for each
kernel of the new family the distance divided by the distance of the same job's kernel in the dense model. A third
variant repeats a middle third of the layers twice (the family's loop).
"""
from __future__ import annotations

import json
import os

HERE = os.path.dirname(os.path.abspath(__file__))
# width, query heads, key/value heads, head size, feed-forward
SIZES = {"1b": (2048, 32, 8, 64, 8192), "3b": (3072, 32, 8, 96, 8192), "8b": (4096, 32, 8, 128, 14336)}
VOCAB = 32768


def peaks():
    try:
        with open(os.path.join(HERE, "..", "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]) * 1e9, float(p["bf16_tflops"]) * 1e12, "of measured"
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15, "of fallback"


def lenolix_model(size, layers, window, keep, loop):
    W, H, G, D, ff = SIZES[size]
    entry = {"type": "attention", "mlp": {"kind": "dense", "ff": ff, "limit": 7.0},
             "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": window, "keep_first": keep},
                       "rot": {"base": 500000.0, "dims": D // 2, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    c = {"architecture": "Lenolix", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": [entry] * layers,
         "embedding": {"scale": 1.0, "bigram": {"buckets": 20011, "mul_prev": 31, "mul_cur": 17}}}
    if loop:
        c["loop"] = {"start": layers // 3, "stop": layers - layers // 3, "times": 2}
    return c


def visible_pairs(n, window, keep):
    """(query, key) pairs of a prompt of n tokens under the mask."""
    if window <= 0:
        return n * (n + 1) // 2
    total = 0
    for i in range(n):
        lo = max(0, i - window + 1)
        total += i + 1 - lo + min(keep, lo)
    return total


def cost(ctx):
    """Cost function (entry point, arguments) -> (job, bytes, operations) for a step whose sequences hold ``ctx`` tokens."""
    def f(name, a):
        n = name.replace("ksana_", "")
        if n == "gemm_smallm":
            M, N, K, res, f32 = a[14], a[15], a[16], a[12], a[9]
        elif n == "gemm_bf16":
            M, N, K, res, f32 = a[10], a[11], a[12], a[8], a[5]
        elif n == "gemm_bf16_tall":
            M, N, K, res, f32 = a[9], a[10], a[11], a[7], a[5]
        else:
            M = None
        if M is not None:
            return f"gemm {N}x{K}", 2 * (M * K + N * K) + M * N * ((4 if f32 else 2) + (2 if res else 0)), 2 * M * N * K
        if n == "norm":
            return "norm", a[8] * a[9] * (4 + (4 if a[1] else 0)), 0
        if n == "residual_norm":
            b = 4 + (6 if a[4] else 0) + (2 if a[12] else 0)
            return ("norm", "norm alone")[0 if a[4] else 1], a[14] * a[15] * b, 0
        if n == "act_mul":
            return "gated unit", a[5] * a[6] * 6, 0
        if n == "glu_clamp":
            return "gated unit", a[2] * a[3] * 6, 0
        if n == "rope_kv_append":
            return "rotation", a[8] * a[11] * 2 * (2 * a[9] + 4 * a[10]), 0
        if n == "qkv_rope_append":
            T, Hq, Hkv, D, Dv, rot = a[10:16]
            return "rotation", T * 2 * (2 * Hq * rot + 2 * Hkv * (D + Dv)), 0
        if n in ("paged_prefill_tc", "paged_prefill"):
            i = 15 if n.endswith("tc") else 14
            B, _, Hq, Hkv, D, Dv, win, keep = a[i:i + 8]
            return "attention", B * ctx * (Hq + Hkv) * (D + Dv) * 2, 2 * Hq * (D + Dv) * B * visible_pairs(ctx, win, keep)
        if n == "paged_decode":
            B, Hq, Hkv, D, Dv, win, keep = a[13:20]
            vis = min(ctx, win + min(keep, max(0, ctx - win))) if win > 0 else ctx
            return "attention", B * (vis * Hkv + Hq) * (D + Dv) * 2, 2 * Hq * (D + Dv) * B * vis
        if n == "embedding":
            return "embedding", a[5] * a[6] * 4, 0
        if n == "embed_pair":
            return "embedding", a[7] * a[8] * (2 + (2 if a[3] else 0) + 4 + (2 if a[5] else 0)), 0
        return n, 0, 0
    return f


def main(args):
    import torch

    from benchmarks.step_breakdown import run_breakdown
    from ksanallm_b200.config import ModelConfig, model_config_from_hf
    from ksanallm_b200.models.weights import RandomSource, build_model
    from ksanallm_b200.utils.clocks import ClockSampler
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    hbm, flops, note = peaks()
    phases = (("prefill", args.prefill_batch, args.prefill_len), ("decode", args.decode_batch, args.decode_ctx))
    for size in args.sizes.split(","):
        W, H, G, D, ff = SIZES[size]
        out = {"metric": "tokens/s of one step", "design": "lenolix", "size": size, "layers": args.layers, "dtype": "bf16",
               "data": "synthetic", "n_gpus": 1, "config": {
                   "width": W, "heads": H, "kv_heads": G, "head_dim": D, "ff": ff, "vocab": VOCAB, "window": args.window,
                   "keep_first": args.keep_first, "l2": "weights larger than L2; no explicit flush"}, "roofline": note, "results": {}}
        sampler = ClockSampler(0)
        sampler.start()
        tables = {}
        for variant in ("llama", "lenolix", "lenolix_loop"):
            if variant == "llama":
                mc = ModelConfig(model_type="llama", hidden_size=W, num_layers=args.layers, num_heads=H, num_kv_heads=G, head_dim=D,
                                 intermediate_size=ff, vocab_size=VOCAB, rms_norm_eps=1e-5, rope_theta=500000.0,
                                 max_position_embeddings=8192, max_token_len=8192, tie_word_embeddings=True)
            else:
                mc = model_config_from_hf(lenolix_model(size, args.layers, args.window, args.keep_first, variant.endswith("loop")))
            model = build_model(mc, RandomSource(seed=1, on_device=True), device=dev, dtype=torch.bfloat16, max_positions=8192)
            for phase, batch, ctx in phases:
                r = run_breakdown(model, phase, batch, ctx, ctx, args.reps, cost=cost(ctx), classes=variant != "lenolix_loop")
                toks = batch * (ctx if phase == "prefill" else 1)
                res = {"us_per_step": r["full_graph_us"], "tokens_per_s": round(toks / r["full_graph_us"] * 1e6), "batch": batch, "ctx": ctx,
                       "launches": r["native_launches"]}
                rows = []
                for c in r["classes"]:
                    roof = max(c["bytes"] / hbm, c["flops"] / flops) * 1e6
                    rows.append({"job": c["job"], "class": c["class"], "n": c["launches"], "us": c["us_each"],
                                 "roofline_us": round(roof, 2), "distance": round(c["us_each"] / roof, 2) if roof > 0 else None})
                if rows:
                    res["kernels"] = rows
                    tables[(variant, phase)] = rows
                out["results"].setdefault(phase, {})[variant] = res
                model.kv_cache = None
            del model
            torch.cuda.empty_cache()
        out["clocks"] = sampler.stop()
        total = lambda c: c["us"] * c["n"]  # noqa: E731
        for phase, _, _ in phases:
            like = {}
            for job in dict.fromkeys(c["job"] for c in tables[("lenolix", phase)]):
                mine = [c for c in tables[("lenolix", phase)] if c["job"] == job and c["distance"]]
                base = [c for c in tables[("llama", phase)] if c["job"] == job and c["distance"]]
                if mine and base:
                    # of several classes of a job the one that takes the most time
                    like[job] = round(max(mine, key=total)["distance"] / max(base, key=total)["distance"], 2)
            out["results"][phase]["like"] = like
        print(json.dumps(out), flush=True)
    return 0
