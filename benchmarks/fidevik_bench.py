"""Prefill and decode throughput of the Fidevik family beside the closest existing models at equal sizes, with random
weights:

  python bench.py --design fidevik [--sizes 1b,3b,8b] [--layers 8]

One JSON line per size (see benchmarks/design_bench.py). Every other layer is latent attention, the rest grouped-query
attention; the first layer's feed-forward is dense, the others are mixtures of experts with a shared expert. Latent attention
and the experts are compared with a DeepSeek model (same latent sizes, router and experts, latent attention in every layer),
grouped-query attention with a Qwen2-MoE model (same heads, experts and shared expert's gate). A further variant repeats the
middle layers (half of eight) twice (the family's loop).
"""
from __future__ import annotations

from benchmarks.design_bench import VOCAB, common_cost, run, visible_pairs

# width, heads, key/value heads, query latent, dense feed-forward, expert feed-forward, shared expert's
SIZES = {"1b": (2048, 16, 4, 768, 8192, 768, 1536), "3b": (3072, 24, 8, 1024, 8192, 1024, 2048),
         "8b": (4096, 32, 8, 1536, 14336, 1536, 3072)}
DIM, RANK, BASE, EXPERTS, TOP, GROUPS, KEEP = 128, 512, 500000.0, 64, 8, 8, 4


def fidevik_model(size, layers, loop):
    W, H, G, QR, ff, xff, sff = SIZES[size]
    latent = {"type": "latent_attention", "mixer": {"heads": H, "dim": DIM, "vdim": DIM, "q_rank": QR, "kv_rank": RANK, "scale": DIM ** -0.5}}
    attn = {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": DIM, "vdim": DIM, "scale": DIM ** -0.5,
                                           "rot": {"dims": DIM, "base": BASE}}}
    moe = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP, "groups": {"count": GROUPS, "keep": KEEP}}, "expert": {"ff": xff},
           "shared": {"ff": sff}}
    out = [{**(attn if i % 2 else latent), "mlp": moe if i else {"kind": "dense", "ff": ff}} for i in range(layers)]
    c = {"architecture": "Fidevik", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-5}, "logit_scale": 0.5, "layers": out}
    if loop:
        c["loop"] = {"start": layers // 3, "stop": layers - layers // 3, "times": 2}
    return c


def cost(batch):
    """Cost function factory: (phase, context) -> ((entry point, arguments) -> (job, bytes, operations)); ``batch``: sequences of
    a phase."""
    def of(phase, ctx):
        rows = batch[phase] * (ctx if phase == "prefill" else 1)               # tokens of the step
        used = min(EXPERTS, rows * TOP)

        def f(name, a):
            n = name.replace("ksana_", "")
            if n == "act_mul" and a[5] != rows:                                # a buffer with the experts' padding rows
                return "expert unit", rows * TOP * a[6] * 6, 0
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
            if n == "mla_rope_append":
                T, G, rank, rot = a[14:18]
                return "latent norms", T * (G * rot * 4 + (rank + rot) * 4), 0
            if n == "latent_norms":
                return "latent norms", a[14] * (a[7] + a[8]) * 4, 0
            if n == "rope_kv_append":
                return "rotation", a[8] * a[11] * 2 * (2 * a[9] + 4 * a[10]), 0
            if n == "qkv_norm_rope_append":
                T, Hq, Hkv, D, Dv = a[16:21]
                return "norms, rotation", T * 2 * (2 * Hq * D + 2 * Hkv * (D + Dv)), 0
            if n == "gemm_bf16_batched":
                B, M, N, K = a[9:13]
                return "absorb" if N > K else "expand", 2 * B * (M * K + N * K + M * N), 2 * B * M * N * K
            if n == "mla_attention":
                T, B, G, dk, dv = a[1], a[11], *a[13:16]
                pairs = visible_pairs(ctx, 0) if phase == "prefill" else ctx
                return "latent attention", B * ctx * dk * 2 + T * G * (dk + dv) * 2, 2 * G * (dk + dv) * B * pairs
            if n in ("paged_prefill_tc", "paged_prefill"):
                i = 15 if n.endswith("tc") else 14
                B, _, Hq, Hkv, D, Dv = a[i:i + 6]
                return "attention", B * ctx * (Hq + Hkv) * (D + Dv) * 2, 2 * Hq * (D + Dv) * B * visible_pairs(ctx, 0)
            if n == "paged_decode":
                B, Hq, Hkv, D, Dv = a[13:18]
                return "attention", B * (ctx * Hkv + Hq) * (D + Dv) * 2, 2 * Hq * (D + Dv) * B * ctx
            return n, 0, 0
        return f
    return of


def main(args):
    from ksanallm_b200.config import ModelConfig, model_config_from_hf

    def variants(size):
        W, H, G, QR, ff, xff, sff = SIZES[size]
        common = dict(hidden_size=W, num_layers=args.layers, num_heads=H, vocab_size=VOCAB, rms_norm_eps=1e-5, rope_theta=BASE,
                      max_position_embeddings=8192, max_token_len=8192, num_experts=EXPERTS, num_experts_per_tok=TOP, norm_topk_prob=False,
                      moe_intermediate_size=xff, shared_expert_intermediate_size=sff, intermediate_size=ff)
        make = lambda loop: lambda: model_config_from_hf(fidevik_model(size, args.layers, loop))  # noqa: E731
        return {"deepseek": lambda: ModelConfig(
            model_type="deepseek_v3", num_kv_heads=H, head_dim=DIM + 64, rope_neox=False, q_lora_rank=QR, kv_lora_rank=RANK,
            qk_nope_head_dim=DIM, qk_rope_head_dim=64, v_head_dim=DIM, moe_scoring="sigmoid", n_group=GROUPS, topk_group=KEEP,
            first_k_dense_replace=1, **common),
            "qwen2_moe": lambda: ModelConfig(model_type="qwen2_moe", num_kv_heads=G, head_dim=DIM, shared_expert_gate=True, **common),
            "fidevik": make(False), "fidevik_loop": make(True)}

    def describe(size):
        W, H, G, QR, ff, xff, sff = SIZES[size]
        return {"width": W, "heads": H, "kv_heads": G, "dim": DIM, "q_rank": QR, "kv_rank": RANK, "ff": ff, "experts": EXPERTS, "top": TOP,
                "expert_ff": xff, "shared_ff": sff}

    def match():
        """GEMMs of latent attention whose counterparts have other row counts: no rotated part, several projections in one."""
        out = {}
        for W, H, _, QR, _, _, _ in SIZES.values():
            out.update({f"gemm {H * DIM}x{QR}": f"gemm {H * (DIM + 64)}x{QR}", f"gemm {QR + RANK + (H + 7) // 8 * 8}x{W}": f"gemm {QR}x{W}"})
        return out

    batch = {"prefill": args.prefill_batch, "decode": args.decode_batch}
    return run(args, "fidevik", SIZES, describe, variants, cost(batch), ("deepseek", "qwen2_moe"), "fidevik", timed_only=("fidevik_loop",),
               match={**match(), "norms, rotation": "rotation", "norm with expert sum": "combine", "norm alone": "norm"})
