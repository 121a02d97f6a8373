"""Throughput of a design whose layers are configured one by one beside the framework's closest existing model at equal
sizes, kernel by kernel: the loop that the benchmarks/<design>_bench.py files share.

Per size, one JSON line: device time and tokens/s of one prefill step and one decode step of every variant (CUDA graphs,
CUDA events, median of several replays; the weights of the layers are larger than L2), and every kernel class with its
algorithmic bytes and operations, its time and its distance from the measured roofline (time / roofline time). ``like``:
for each job of the design the distance divided by the distance of the same job's kernel in the closest model.
"""
from __future__ import annotations

import json
import os

HERE = os.path.dirname(os.path.abspath(__file__))
VOCAB = 32768


def peaks():
    try:
        with open(os.path.join(HERE, "..", "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]) * 1e9, float(p["bf16_tflops"]) * 1e12, "of measured"
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15, "of fallback"


def visible_pairs(n, window, keep=0):
    """(query, key) pairs of a prompt of n tokens under the mask."""
    if window <= 0:
        return n * (n + 1) // 2
    total = 0
    for i in range(n):
        lo = max(0, i - window + 1)
        total += i + 1 - lo + min(keep, lo)
    return total


def common_cost(n, a):
    """(job, bytes, operations) of the entry points that every family calls, None for others."""
    if n == "gemm_smallm":
        M, N, K, res, f32 = a[14], a[15], a[16], a[12], a[9]
    elif n == "gemm_bf16":
        M, N, K, res, f32 = a[10], a[11], a[12], a[8], a[5]
    elif n == "gemm_bf16_tall":
        M, N, K, res, f32 = a[9], a[10], a[11], a[7], a[5]
    elif n == "gemm_pair":
        M, N, K, res, f32 = a[13], a[14], a[15], a[11], None
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
        return "unit", a[5] * a[6] * 6, 0
    if n == "embedding":
        return "embedding", a[5] * a[6] * 4, 0
    if n == "embed_pair":
        return "embedding", a[7] * a[8] * (2 + (2 if a[3] else 0) + 4 + (2 if a[5] else 0)), 0
    return None


def run(args, design, sizes, describe, variants, cost, base, mine, timed_only=(), match=None):
    """``variants(size)``: name -> function giving the variant's ModelConfig; ``base`` and ``mine``: the variants whose kernels
    are compared (``base`` may be several names: a job is compared with the first that has it); ``timed_only``: variants
    without a kernel table; ``match``: job of the design -> job of the base model where the names differ. A GEMM without a
    counterpart of its own shape is compared with the base models' GEMMs together."""
    import torch

    from benchmarks.step_breakdown import run_breakdown
    from ksanallm_b200.models.weights import RandomSource, build_model
    from ksanallm_b200.utils.clocks import ClockSampler
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    hbm, flops, note = peaks()
    phases = (("prefill", args.prefill_batch, args.prefill_len), ("decode", args.decode_batch, args.decode_ctx))
    for size in args.sizes.split(","):
        if size not in sizes:
            raise SystemExit(f"unknown size {size!r}: {', '.join(sizes)}")
        out = {"metric": "tokens/s of one step", "design": design, "size": size, "layers": args.layers, "dtype": "bf16",
               "data": "synthetic", "n_gpus": 1, "config": {**describe(size), "vocab": VOCAB, "l2": "weights larger than L2; no explicit flush"},
               "roofline": note, "results": {}}
        sampler = ClockSampler(0)
        sampler.start()
        tables = {}
        for variant, make in variants(size).items():
            model = build_model(make(), RandomSource(seed=1, on_device=True), device=dev, dtype=torch.bfloat16, max_positions=8192)
            for phase, batch, ctx in phases:
                r = run_breakdown(model, phase, batch, ctx, ctx, args.reps, cost=cost(phase, ctx), classes=variant not in timed_only)
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
                model.kv_cache = model.state = None
            del model
            torch.cuda.empty_cache()
        out["clocks"] = sampler.stop()
        total = lambda c: c["us"] * c["n"]  # noqa: E731

        def distance(rows, job):
            # of several classes of a job the one that takes the most time
            rows = [c for c in rows if c["job"] == job and c["distance"]]
            return max(rows, key=total)["distance"] if rows else None

        def gemms(rows):
            rows = [c for c in rows if c["job"].startswith("gemm ") and c["distance"]]
            return sum(map(total, rows)) / sum(total(c) / c["distance"] for c in rows)

        for phase, _, _ in phases:
            bases = [tables[(name, phase)] for name in ([base] if isinstance(base, str) else base)]
            a, like = tables[(mine, phase)], {}
            for job in dict.fromkeys(c["job"] for c in a):
                x = distance(a, job)
                y = next((d for b in bases if (d := distance(b, (match or {}).get(job, job)))), None)
                y = y or (gemms([c for b in bases for c in b]) if job.startswith("gemm ") else None)
                if x and y:
                    like[job] = round(x / y, 2)
            out["results"][phase]["like"] = like
        print(json.dumps(out), flush=True)
    return 0
