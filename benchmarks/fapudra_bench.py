"""Prefill and decode throughput of the Fapudra family beside the closest existing models at equal sizes, with random weights:

  python bench.py --design fapudra [--sizes 1b,3b,8b] [--layers 8] [--window 512] [--keep-first 64]

One JSON line per size (see benchmarks/design_bench.py). Of four layers three are state spaces and one is windowed sigmoid
attention beside a delta rule; every layer has a mixture of experts. Experts, projections and norms are compared with a
Qwen2-MoE model (same width, heads, experts), windowed attention with a Lenolix model (same heads, window, kept tokens), the
recurrences with the Rasizen family's, and passes over rows that have no counterpart with the pass that streams its operands like
them (named in ``match``).
"""
from __future__ import annotations

from benchmarks.design_bench import VOCAB, common_cost, run, visible_pairs

# width, query heads, key/value heads, heads of the state space, heads of the delta rule, expert feed-forward
SIZES = {"1b": (2048, 16, 4, 64, 16, 768), "3b": (3072, 24, 8, 96, 24, 1024), "8b": (4096, 32, 8, 128, 32, 1536)}
DIM, VDIM, STATE, SPACE_GROUPS, TAPS = 128, 64, 128, 8, 4
EXPERTS, TOP, GROUPS, KEEP = 64, 8, 8, 4


def fapudra_model(size, layers, window, keep):
    W, H, G, S, R, ff = SIZES[size]
    moe = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP, "groups": {"count": GROUPS, "keep": KEEP}}, "expert": {"ff": ff, "limit": 7.0}}
    space = {"type": "mamba2", "mixer": {"heads": S, "vdim": VDIM, "state": STATE, "groups": SPACE_GROUPS, "conv": TAPS, "norm_groups": SPACE_GROUPS}}
    both = {"type": "parallel", "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": DIM, "vdim": DIM, "scale": DIM ** -0.5, "bias_max": 128,
                 "mask": {"size": window, "keep_first": keep} if window else None},
        "right": {"heads": R, "kv_heads": R, "dim": DIM, "vdim": DIM, "conv": TAPS}, "left_scale": 1.0, "right_scale": 1.0}}
    return {"architecture": "Fapudra", "width": W, "vocab": VOCAB, "max_positions": 8192, "norm": {"eps": 1e-5}, "embedding": {"scale": W ** 0.5},
            "logit_softcap": 30.0, "layers": [{**(both if i % 4 == 1 else space), "mlp": moe} for i in range(layers)]}


def cost(batch):
    """Cost function factory: (phase, context) -> ((entry point, arguments) -> (job, bytes, operations)); ``batch``: sequences of
    a phase."""
    def of(phase, ctx):
        rows = batch[phase] * (ctx if phase == "prefill" else 1)               # tokens of the step
        used = min(EXPERTS, rows * TOP)

        def f(name, a):
            n = name.replace("ksana_", "")
            if n in ("act_mul", "glu_clamp"):
                M, I = (a[5], a[6]) if n == "act_mul" else (a[2], a[3])
                return ("expert unit", rows * TOP * I * 6, 0) if M != rows else ("unit", M * I * 6, 0)
            if n == "residual_norm" and a[24]:
                return "norm with expert sum", rows * a[15] * (8 + 2 * TOP + (2 if a[29] else 0) + (2 if a[12] else 0)), 0
            known = common_cost(n, a)
            if known and known[0].startswith("gemm ") and int(known[0][5:].split("x")[0]) <= EXPERTS + 8:
                return ("router", *known[1:])
            if known:
                return known
            if n == "gemm_grouped":
                N, K = a[11], a[12]
                return "expert down" if K < N else "expert gate, up", 2 * (rows * TOP * (N + K) + used * N * K), 2 * rows * TOP * N * K
            if n == "moe_route":
                return "choice", rows * (a[1] * 4 + TOP * 8), 0
            if n == "moe_align":
                return "expert rows", rows * TOP * 8, 0
            if n == "moe_permute":
                return "gather", rows * (1 + TOP) * a[5] * 2, 0
            if n == "moe_combine":
                return "combine", rows * (1 + TOP) * a[6] * 2, 0
            if n in ("rope_kv_append", "qkv_rope_append"):
                Hq, Hkv, D = (a[9], a[10], a[11]) if n == "rope_kv_append" else (a[11], a[12], a[13])
                return "rotation", rows * D * 2 * (2 * Hq + 4 * Hkv), 0
            if n in ("paged_prefill_tc", "paged_prefill"):
                i = 15 if n.endswith("tc") else 14
                B, _, Hq, Hkv, D, Dv, win, keep = a[i:i + 8]
                kv = D if a[5 if n.endswith("tc") else 4] == a[6 if n.endswith("tc") else 5] else D + Dv
                return ("window attention" if win else "attention", B * ctx * (Hq * (D + Dv) + Hkv * kv) * 2,
                        2 * Hq * (D + Dv) * B * visible_pairs(ctx, win, keep))
            if n == "paged_decode":
                B, Hq, Hkv, D, Dv, win, keep = a[13:20]
                vis = min(ctx, win + min(keep, max(0, ctx - win))) if win > 0 else ctx
                kv = D if a[4] == a[5] else D + Dv
                return "window attention" if win else "attention", B * (vis * Hkv * kv + Hq * (D + Dv)) * 2, 2 * Hq * (D + Dv) * B * vis
            if n == "gated_recurrence":
                B, W, bt = a[15], a[16], a[8]
                states = B * (ctx // bt) if phase == "prefill" else 2 * B
                return "recurrence", rows * W * 8 + states * W * 4, 0
            if n == "xielu":
                return "unit", a[4] * a[5] * 4, 0
            if n == "embed_normed":
                return "embedding", a[6] * a[7] * 8, 0
            if n == "token_shift":
                return "token shift", rows * a[13] * 4, 0
            if n == "causal_conv":
                return "convolution", rows * a[7] * 4, 0
            if n == "state_space":
                B, H, G, P, N = a[22:27]
                # x in, y out, B and C in, the state in (decode) and out; decay, write and read-out of a state element per token
                return ("state space", rows * (H * P * 4 + 2 * G * N * 2 + H * 2) + B * H * P * N * (8 if phase == "decode" else 4),
                        rows * H * P * N * 4)
            if n == "delta_rule":
                B, H, G, K, V = a[22:27]
                return ("delta rule", rows * (2 * G * K * 2 + H * V * 4 + H * K * 2 + H * 2) + B * H * K * V * (8 if phase == "decode" else 4),
                        rows * H * K * V * 6)
            if n == "gated_norm":
                return "gated norm", a[9] * a[10] * 6, 0
            if n == "panel_append":
                return "append", a[9] * a[7] * a[8] * 4, 0
            if n == "softcap":
                return "soft cap", a[2] * a[3] * 8, 0
            return n, 0, 0
        return f
    return of


def main(args):
    from benchmarks import lenolix_bench, rasizen_bench
    from ksanallm_b200.config import ModelConfig, model_config_from_hf

    def lenolix(size):
        W, H, G, _, _, ff = SIZES[size]
        c = lenolix_bench.lenolix_model("1b", 2, args.window, args.keep_first, False)
        c["width"] = W
        for e in c["layers"]:
            e["mixer"].update(heads=H, kv_heads=G, dim=DIM, vdim=DIM, scale=DIM ** -0.5)
            e["mixer"]["rot"].update(dims=DIM // 2)
        return model_config_from_hf(c)

    def rasizen(size):
        c = rasizen_bench.rasizen_model(size, 4, args.window)
        return model_config_from_hf(c)

    def variants(size):
        W, H, G, _, _, ff = SIZES[size]
        return {"qwen2_moe": lambda: ModelConfig(
            model_type="qwen2_moe", hidden_size=W, num_layers=args.layers, num_heads=H, num_kv_heads=G, head_dim=DIM, vocab_size=VOCAB,
            rms_norm_eps=1e-5, max_position_embeddings=8192, max_token_len=8192, num_experts=EXPERTS, num_experts_per_tok=TOP, norm_topk_prob=True,
            moe_intermediate_size=ff, intermediate_size=ff),
            "lenolix": lambda: lenolix(size), "rasizen": lambda: rasizen(size),
            "fapudra": lambda: model_config_from_hf(fapudra_model(size, args.layers, args.window, args.keep_first))}

    def describe(size):
        W, H, G, S, R, ff = SIZES[size]
        return {"width": W, "heads": H, "kv_heads": G, "dim": DIM, "space_heads": S, "vdim": VDIM, "state": STATE, "delta_heads": R, "experts": EXPERTS,
                "top": TOP, "expert_ff": ff, "window": args.window, "keep_first": args.keep_first}

    batch = {"prefill": args.prefill_batch, "decode": args.decode_batch}
    return run(args, "fapudra", SIZES, describe, variants, cost(batch), ("qwen2_moe", "lenolix", "rasizen"), "fapudra",
               match={"state space": "recurrence", "delta rule": "recurrence", "norm with expert sum": "combine", "norm alone": "norm",
                      "token shift": "norm", "gated norm": "norm", "convolution": "unit", "append": "rotation", "soft cap": "unit"})
