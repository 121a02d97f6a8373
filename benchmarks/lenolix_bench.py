"""Prefill and decode throughput of the Lenolix family beside the closest dense model (Llama layers, bf16) at equal
width, heads, feed-forward, vocabulary and depth, with random weights:

  python bench.py --design lenolix [--sizes 1b,3b,8b] [--layers 8] [--window 512] [--keep-first 64]

One JSON line per size (see benchmarks/design_bench.py). A third variant repeats a middle third of the layers twice (the
family's loop).
"""
from __future__ import annotations

from benchmarks.design_bench import VOCAB, common_cost, run, visible_pairs

# width, query heads, key/value heads, head size, feed-forward
SIZES = {"1b": (2048, 32, 8, 64, 8192), "3b": (3072, 32, 8, 96, 8192), "8b": (4096, 32, 8, 128, 14336)}


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


def cost(phase, ctx):
    """Cost function (entry point, arguments) -> (job, bytes, operations) for a step whose sequences hold ``ctx`` tokens."""
    def f(name, a):
        n = name.replace("ksana_", "")
        known = common_cost(n, a)
        if known:
            return known
        if n == "glu_clamp":
            return "unit", a[2] * a[3] * 6, 0
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
        return n, 0, 0
    return f


def main(args):
    from ksanallm_b200.config import ModelConfig, model_config_from_hf

    def variants(size):
        W, H, G, D, ff = SIZES[size]
        make = lambda loop: lambda: model_config_from_hf(lenolix_model(size, args.layers, args.window, args.keep_first, loop))  # noqa: E731
        return {"llama": lambda: ModelConfig(
            model_type="llama", hidden_size=W, num_layers=args.layers, num_heads=H, num_kv_heads=G, head_dim=D, intermediate_size=ff,
            vocab_size=VOCAB, rms_norm_eps=1e-5, rope_theta=500000.0, max_position_embeddings=8192, max_token_len=8192,
            tie_word_embeddings=True), "lenolix": make(False), "lenolix_loop": make(True)}

    def describe(size):
        W, H, G, D, ff = SIZES[size]
        return {"width": W, "heads": H, "kv_heads": G, "head_dim": D, "ff": ff, "window": args.window, "keep_first": args.keep_first}

    return run(args, "lenolix", SIZES, describe, variants, cost, "llama", "lenolix", timed_only=("lenolix_loop",))
