"""Small Fapudra models for the tests: configurations and seeded weights whose recurrences remember for hundreds of tokens, whose
attention rests on a few keys and whose distance biases differ from bucket to bucket."""
import math

import torch

from decoder_helpers import build, engine, error, run_portions, save_checkpoint, tokens  # noqa: F401


def space(heads, vdim, state, groups, conv, norm_groups):
    return "mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def both(left, mask, right, scales=(1.25, 0.8), bias_max=40, scale=None):
    """left: heads, kv_heads, dim; right: heads, kv_heads, dim, vdim, conv."""
    H, G, d = left
    names = ("heads", "kv_heads", "dim", "vdim", "conv")
    return "parallel", {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": scale or d ** -0.5, "bias_max": bias_max,
                                 "mask": {"size": mask[0], "keep_first": mask[1]} if mask else None},
                        "right": dict(zip(names, right)), "left_scale": scales[0], "right_scale": scales[1]}


def moe(experts, top, groups, ff, limit=1.3):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": dict(zip(("count", "keep"), groups)) if groups else None},
            "expert": {"ff": ff, "limit": limit}}


def config(width, vocab, layers, cap=24.0, scale=3.0, eps=1e-5, max_positions=512):
    return {"architecture": "Fapudra", "width": width, "vocab": vocab, "max_positions": max_positions, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "logit_softcap": cap,
            "layers": [{"type": t, "mixer": m, "mlp": ff} for (t, m), ff in layers]}


CONFIGS = {
    # both mixers with and without experts, groups of heads, a norm of several parts, unequal key and value sizes
    "unequal": config(72, 203, [(space(6, 16, 24, 2, 3, 3), moe(15, 4, (5, 3), 24)), (both((6, 2, 24), (20, 5), (4, 2, 16, 24, 4)), None),
                                (space(4, 24, 16, 4, 4, 1), None), (both((4, 4, 16), (33, 0), (2, 2, 24, 8, 2), (0.7, 1.4), 25), moe(10, 2, None, 16, 0.8))]),
    # nothing is a multiple of 8, norm parts that cross heads
    "odd": config(70, 101, [(both((3, 1, 10), (17, 3), (3, 3, 10, 6, 3), (0.5, 2.0), 23, 0.4), moe(9, 2, (3, 1), 13, 1.1)),
                            (space(3, 10, 13, 3, 2, 5), moe(5, 5, None, 11, 2.0)), (space(6, 5, 9, 1, 5, 2), None)], 7.0, 5.5, 1e-4),
    # no window, no kept tokens, no experts, one key/value head
    "plain": config(64, 96, [(both((8, 1, 16), None, (4, 1, 8, 32, 4), (1.0, 1.0), 60), None), (space(2, 32, 32, 1, 4, 2), None)], 50.0),
    # sizes of the fast paths, more experts than a warp has lanes
    "long": config(128, 320, [(space(8, 64, 128, 2, 4, 8), moe(64, 6, (8, 3), 40)), (both((8, 2, 64), (64, 20), (4, 2, 64, 64, 4), bias_max=100), moe(40, 8, (40, 12), 24)),
                              (both((6, 3, 128), (100, 7), (2, 1, 128, 128, 3)), None)]),
    # degenerate values: one head, one column, one tap, one expert, one bucket per distance (a large eps: norms of single columns
    # would be signs)
    "ones": config(64, 90, [(space(1, 1, 1, 1, 1, 1), moe(1, 1, (1, 1), 1)), (both((1, 1, 1), (1, 1), (1, 1, 2, 1, 1), (1.0, 1.0), 9, 1.0), moe(2, 1, (2, 1), 8))],
                   eps=0.1),
    # heads beyond the tensor-core prefill kernel, many heads per key/value head, long keys, many taps
    "wide": config(96, 150, [(both((2, 1, 136), (40, 9), (2, 1, 136, 40, 6)), None), (space(2, 72, 136, 2, 6, 4), None),
                             (both((40, 2, 8), (21, 4), (2, 2, 40, 136, 1), bias_max=700), None)]),
}
BUCKETS = {"unequal": 16, "odd": 10, "plain": 32, "long": 32, "ones": 4, "wide": 24}
RANKS = {"unequal": (12, 20), "odd": (7, 5), "plain": (8, 16), "long": (64, 24), "ones": (1, 3), "wide": (30, 9)}


def shapes(c, buckets=16, ranks=(12, 20)):
    W = c["width"]
    out = {"embed": (c["vocab"], W), "pos": (c["max_positions"], W), "embed.norm": (), "head": (c["vocab"], W), "final.norm": ()}
    for i, e in enumerate(c["layers"]):
        m, f, p = e["mixer"], e["mlp"], f"l{i}."
        x, y = p + "mix.", p + "mlp."
        out.update({p + "norm1": (), p + "shift": (W,)})
        if e["type"] == "mamba2":
            H, inner, ch = m["heads"], m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            out.update({x + "in": (inner + ch + H, W), x + "conv": (ch, m["conv"]), x + "conv.b": (ch,), x + "dt_bias": (H,), x + "A_log": (H,),
                        x + "D": (H,), x + "norm": (inner,), x + "o": (W, inner)})
        else:
            a, d, le, ri = m["left"], m["right"], x + "left.", x + "right."
            q, k = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            out.update({le + "q": (q, W), le + "q.b": (q,), le + "k": (k, W), le + "k.b": (k,), le + "rel": (buckets, a["heads"]),
                        le + "pb": (a["heads"],), le + "g": (q, W), le + "o": (W, q)})
            k, v = d["kv_heads"] * d["dim"], d["heads"] * d["vdim"]
            for name, n in (("q", k), ("k", k), ("v", v)):
                out.update({ri + name: (n, W), f"{ri}{name}.conv": (n, d["conv"])})
            keys = d["heads"] * d["dim"]
            out.update({ri + "b": (d["heads"], W), ri + "A_log": (d["heads"],), ri + "norm": (d["vdim"],), ri + "a1": (ranks[0], W),
                        ri + "a2": (keys, ranks[0]), ri + "dt_bias": (keys,), ri + "g1": (ranks[1], W), ri + "g2": (v, ranks[1]), ri + "o": (W, v)})
        if f:
            out[y + "router"] = (f["router"]["experts"], W)
            for j in range(f["router"]["experts"]):
                n = f["expert"]["ff"]
                out.update({f"{y}e{j}.gate": (n, W), f"{y}e{j}.up": (n, W), f"{y}e{j}.down": (W, n)})
    return out


def weights(c, seed=0, buckets=16, ranks=(12, 20)):
    """bf16-representable fp32 weights. Step sizes and decays are small enough that a state keeps what it saw for hundreds of tokens.
    Queries and keys are large and the heads' offsets strongly negative: few keys get a weight that counts, a wrong or missing
    one shows. One expert's share is kept small: a choice between two nearly equal scores may fall either way in bf16 and must
    not decide such a test, while in 32 bits a wrong expert is far beyond the limit."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, s in shapes(c, buckets, ranks).items():
        t = torch.randn(s, generator=g)
        last = name.split(".")[-1]
        if last == "A_log":
            t = -1.0 + 0.8 * t
        elif last == "dt_bias":
            t = -4.5 + 0.8 * t
        elif last in ("q", "k") and ".left." in name:
            t = t * 1.7 / s[-1] ** 0.5
        elif last == "pb":
            t = -4.0 + 0.5 * t
        elif last == "rel":
            t = t * 1.2
        elif last == "shift":
            t = 0.4 + 0.3 * t
        elif last == "conv":
            t = t * 0.6 + (torch.arange(s[-1]) == s[-1] - 1)
        elif last == "D":
            t = 0.5 + 0.3 * t
        elif last == "router":
            t = t * 1.6 / s[-1] ** 0.5
        elif last == "down":
            t = t * 0.06 / s[-1] ** 0.5
        elif last in ("norm1", "norm") or name.endswith("norm"):
            t = 1.0 + 0.2 * t
        elif last == "b":
            t = t * (0.3 if len(s) == 1 else 1.2 / math.sqrt(s[-1]))
        elif name == "pos":
            t = t * 1.0
        elif len(s) == 2 and last != "embed":
            t = t * 1.2 / s[-1] ** 0.5
        w[name] = t.bfloat16().float()
    return w


def of(name):
    """Weights of a configuration of ``CONFIGS``."""
    return weights(CONFIGS[name], sorted(CONFIGS).index(name), BUCKETS[name], RANKS[name])
