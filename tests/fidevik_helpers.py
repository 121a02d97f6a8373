"""Small Fidevik models for the tests: configurations and seeded weights that make attention sharp, sinks matter and the
experts' choice depend on the token, the groups and the corrections."""
import torch

from decoder_helpers import build, engine, error, run_portions, save_checkpoint, tokens  # noqa: F401


def attn(heads, kv, dim, vdim, rot, base=500.0, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                         "rot": {"dims": rot, "base": base} if rot else None}


def latent(heads, dim, vdim, q_rank, kv_rank, scale=None):
    return "latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale or dim ** -0.5}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, count, keep, ff, shared):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}, "expert": {"ff": ff},
            "shared": {"ff": shared}}


def config(width, vocab, layers, loop, logit_scale, eps=1e-5):
    return {"architecture": "Fidevik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "layers": [{"type": t, "mixer": m, "mlp": ff} for (t, m), ff in layers]}


CONFIGS = {
    # layers before and behind the repeated ones, three passes, every kind of feed-forward behind each kind of mixer
    "unequal": config(72, 203, [(latent(3, 16, 24, 24, 40), dense(40)), (attn(6, 2, 24, 16, 8), moe(12, 4, 4, 2, 24, 40)),
                                (latent(5, 8, 16, 56, 16), None), (attn(4, 4, 16, 32, 16), dense(56)), (latent(2, 32, 8, 16, 48), moe(10, 3, 1, 1, 16, 8))],
                      (1, 4, 3), 0.7),
    # nothing is a multiple of 8, the first layer opens the loop
    "odd": config(70, 101, [(attn(3, 1, 10, 6, 6, 70.0), moe(9, 2, 3, 2, 13, 11)), (latent(3, 10, 12, 13, 22, 0.4), dense(33)),
                            (attn(4, 2, 14, 20, 14, 30.0, 0.2), None)], (0, 1, 2), 1.3, 1e-4),
    # no loop, no rotation, no experts, one key/value head
    "plain": config(64, 96, [(attn(8, 1, 16, 24, 0), dense(48)), (attn(2, 2, 40, 8, 4, 1e5), None), (latent(4, 24, 24, 32, 64), None)], None, 1.0),
    # every layer repeats; more experts than a warp has lanes, groups of one expert and of many
    "long": config(128, 320, [(latent(8, 32, 32, 64, 128), moe(64, 6, 8, 3, 40, 96)), (attn(8, 2, 64, 48, 32, 5000.0), moe(40, 8, 40, 12, 24, 16)),
                              (attn(6, 3, 128, 64, 64, 1000.0), dense(200))], (0, 3, 2), 0.5),
    # degenerate values: one head, one pair, one expert, one pass, ranks of one column, factor 1
    "ones": config(64, 90, [(latent(1, 1, 1, 1, 3, 1.0), moe(1, 1, 1, 1, 1, 1)), (attn(1, 1, 2, 1, 2), moe(2, 1, 2, 1, 8, 8))], (1, 2, 1), 1.0),
    # heads beyond the tensor-core prefill kernel, latent rows of two output halves and beyond the tensor-core kernel
    "wide": config(96, 150, [(latent(2, 40, 16, 24, 520), dense(64)), (attn(2, 1, 136, 200, 96), dense(64)), (latent(24, 16, 8, 40, 264), None)],
                   (0, 2, 2), 0.8),
}

# layouts that split evenly over ranks, with sizes that do not
SPLIT = {
    "split2": config(70, 151, [(latent(2, 20, 12, 13, 22), moe(6, 2, 3, 1, 13, 21)), (attn(4, 2, 10, 12, 6), dense(51)), (attn(6, 1, 12, 8, 4), None)],
                     (0, 2, 2), 0.7),
    "split4": config(72, 90, [(attn(8, 2, 16, 8, 8), moe(8, 3, 2, 2, 30, 25)), (latent(4, 24, 16, 40, 16), dense(50))], (1, 2, 2), 1.1),
}


def shapes(c):
    W = c["width"]
    out = {"embed": (c["vocab"], W), "head": (c["vocab"], W), "final.norm": (W,), "final.norm.b": (W,)}
    if c["loop"]:
        out["loop.step"] = (c["loop"]["times"], W)
    for i, e in enumerate(c["layers"]):
        m, f, p = e["mixer"], e["mlp"], f"l{i}."
        x, y = p + "mix.", p + "mlp."
        H, d, v = m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "norm1.b": (W,), x + "o": (W, H * v)})
        if e["type"] == "attention":
            G = m["kv_heads"]
            out.update({x + "q": (H * d, W), x + "k": (G * d, W), x + "v": (G * v, W), x + "q.norm": (H * d,), x + "k.norm": (G * d,)})
        else:
            q, k = m["q_rank"], m["kv_rank"]
            out.update({x + "dq": (q, W), x + "dq.norm": (q,), x + "uq": (H * d, q), x + "dkv": (k, W), x + "dkv.norm": (k,),
                        x + "uk": (H * d, k), x + "uv": (H * v, k), x + "sink": (H,), x + "g": (H, W)})
        if not f:
            continue
        out.update({p + "norm2": (W,), p + "norm2.b": (W,)})
        parts = [(y, f["ff"])] if f["kind"] == "dense" else \
            [(f"{y}e{j}.", f["expert"]["ff"]) for j in range(f["router"]["experts"])] + [(y + "shared.", f["shared"]["ff"])]
        for name, n in parts:
            out.update({name + "gate": (n, W), name + "up": (n, W), name + "down": (W, n)})
        if f["kind"] == "moe":
            out.update({y + "router": (f["router"]["experts"], W), y + "correction": (f["router"]["experts"],), y + "shared.sg": (1, W)})
    return out


def weights(c, seed=0):
    """bf16-representable fp32 weights. Normed queries and keys are large, so a softmax row rests on a few keys and a wrong or
    missing one shows; sinks are of the size of the largest scores; norm weights are far from one. Corrections are large and
    mostly negative. One expert's share is kept small: a choice between two nearly equal scores may fall either way in bf16 and
    must not decide such a test, while in 32 bits a wrong expert is far beyond the limit."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, s in shapes(c).items():
        t = torch.randn(s, generator=g)
        last = name.split(".")[-1]
        if last == "sink":
            t = t * 1.5 + 2
        elif last == "correction":
            t = t * 0.4 - 0.6
        elif last == "b":
            t = t * 0.3
        elif name == "loop.step":
            t = t * 0.7
        elif last in ("uq", "uk", "router"):
            t = t * 1.6 / s[-1] ** 0.5
        elif name.endswith(("q.norm", "k.norm")) and "d" not in name.split(".")[-2]:
            t = 1.5 + 0.4 * t
        elif last == "down" and ".e" in name:
            t = t * 0.05 / s[-1] ** 0.5
        elif len(s) == 2 and last != "embed":
            t = t * 1.2 / s[-1] ** 0.5
        elif len(s) == 1:                          # norm weights
            t = 0.9 + 0.3 * t
        w[name] = t.bfloat16().float()
    return w
