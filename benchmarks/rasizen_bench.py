"""Prefill and decode throughput of the Rasizen family beside the closest existing model (DeepSeek-style latent attention
with dense feed-forwards, bf16) at equal width, heads, latent sizes, feed-forward, vocabulary and depth, with random
weights:

  python bench.py --design rasizen [--sizes 1b,3b,8b] [--layers 8] [--window 512]

One JSON line per size (see benchmarks/design_bench.py). Of four layers two are recurrences (as wide as the model), one is
latent attention and one reads that layer's latents again; every layer has a feed-forward. The recurrence has no
counterpart in the other model: it streams its operands once like the gated unit, which it is compared with.
"""
from __future__ import annotations

from benchmarks.design_bench import VOCAB, common_cost, run, visible_pairs

# width, heads, feed-forward
SIZES = {"1b": (2048, 16, 8192), "3b": (3072, 24, 8192), "8b": (4096, 32, 14336)}
DIM, ROT, VDIM, RANK, BASE = 128, 64, 128, 512, 500000.0


def rasizen_model(size, layers, window):
    W, H, ff = SIZES[size]

    def latent(kv_from):
        m = {"heads": H, "dim": DIM, "rot_dim": ROT, "vdim": VDIM, "kv_rank": RANK, "scale": (DIM + ROT) ** -0.5,
             "rot": {"base": BASE, "dims": ROT}, "mask": {"size": window} if window else None}
        return {"type": "latent_attention", "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}

    out = []
    for i in range(layers):
        e = {"type": "mingru", "mixer": {"width": W}} if i % 4 < 2 else latent(i - 1 if i % 4 == 3 else None)
        out.append({**e, "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Rasizen", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-5, "groups": 4}, "residual_mult": 0.5, "layers": out}


def cost(phase, ctx):
    """Cost function (entry point, arguments) -> (job, bytes, operations) for a step whose sequences hold ``ctx`` tokens."""
    def f(name, a):
        n = name.replace("ksana_", "")
        known = common_cost(n, a)
        if known:
            return known
        if n == "xielu":
            return "unit", a[4] * a[5] * 4, 0
        if n == "gated_recurrence":
            B, W, bt = a[15], a[16], a[8]
            rows, states = (B * ctx, B * (ctx // bt)) if phase == "prefill" else (B, 2 * B)
            return "recurrence", rows * W * 8 + states * W * 4, 0
        if n == "mla_rope_append":
            T, G, rank, rot = a[14:18]
            return "rotation" if a[3] else "rotation of queries", T * (G * rot * 4 + ((rank + rot) * 4 if a[3] else 0)), 0
        if n == "gemm_bf16_batched":
            B, M, N, K = a[9:13]
            return "absorb" if N > K else "expand", 2 * B * (M * K + N * K + M * N * (2 if a[13] else 1)), 2 * B * M * N * K
        if n == "mla_attention":
            T, B, G, dk, dv, win = a[1], a[11], a[13], a[14], a[15], a[16]
            vis = min(ctx, win) if win > 0 else ctx
            keys, pairs = (ctx, visible_pairs(ctx, win)) if phase == "prefill" else (vis, vis)
            return "attention", B * keys * dk * 2 + T * G * (dk + dv) * 2, 2 * G * (dk + dv) * B * pairs
        return n, 0, 0
    return f


def main(args):
    from ksanallm_b200.config import ModelConfig, model_config_from_hf

    def variants(size):
        W, H, ff = SIZES[size]
        return {"deepseek": lambda: ModelConfig(
            model_type="deepseek_v3", hidden_size=W, num_layers=args.layers, num_heads=H, num_kv_heads=H, head_dim=DIM + ROT,
            intermediate_size=ff, vocab_size=VOCAB, rms_norm_eps=1e-5, rope_theta=BASE, rope_neox=False, max_position_embeddings=8192,
            max_token_len=8192, tie_word_embeddings=True, kv_lora_rank=RANK, qk_nope_head_dim=DIM, qk_rope_head_dim=ROT, v_head_dim=VDIM),
            "rasizen": lambda: model_config_from_hf(rasizen_model(size, args.layers, args.window))}

    def describe(size):
        W, H, ff = SIZES[size]
        return {"width": W, "heads": H, "dim": DIM, "rot_dim": ROT, "vdim": VDIM, "kv_rank": RANK, "ff": ff, "channels": W, "window": args.window}

    return run(args, "rasizen", SIZES, describe, variants, cost, "deepseek", "rasizen",
               match={"recurrence": "unit", "rotation of queries": "rotation"})
