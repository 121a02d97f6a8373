"""Small Lenolix models for the tests: configurations and seeded weights that make attention sharp."""
import torch

from decoder_helpers import PLACES, build, engine, error, run_portions, save_checkpoint, tokens  # noqa: F401
ROTATION = {"base": 5000.0, "dims": 8, "scaling": {"factor": 3.0, "low": 1.5, "high": 6.0, "original": 120}}


def mixer(heads, kv_heads, dim, vdim, mask=None, rot=None, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "mask": mask, "rot": rot}


def entry(mix, ff=None, limit=1.5):
    return {"type": "attention", "mixer": mix, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(width, vocab, layers, loop=None, bigram=None, scale=3.0, eps=1e-5):
    c = {"architecture": "Lenolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
         "layers": layers}
    if bigram:
        c["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def _rot(dims, base=900.0, scaling=None):
    return {"base": base, "dims": dims, "scaling": scaling}


CONFIGS = {
    # unequal layers, key and value sizes differ, a layer without a feed-forward, the loop starts at the first layer
    "unequal": config(72, 203, [entry(mixer(6, 2, 24, 16, {"size": 13, "keep_first": 3}, ROTATION), 88),
                                entry(mixer(4, 4, 32, 40, None, _rot(32))),
                                entry(mixer(4, 1, 48, 24, {"size": 40, "keep_first": 18}, _rot(14)), 40, 0.7)], (0, 2, 2), (61, 7, 3)),
    # nothing is a multiple of 8; no loop, no pair embedding, no kept tokens
    "odd": config(70, 101, [entry(mixer(3, 1, 20, 12, {"size": 20, "keep_first": 0}, _rot(10)), 50),
                            entry(mixer(5, 5, 12, 20, {"size": 7, "keep_first": 2}, _rot(12, 70.0)), 33, 3.0)]),
    # grouped heads, the loop is the last layer, a window longer than a cache page, large pair multipliers
    "grouped": config(128, 320, [entry(mixer(8, 1, 64, 64, {"size": 70, "keep_first": 5}, ROTATION), 96),
                                 entry(mixer(8, 2, 64, 64, {"size": 33, "keep_first": 16}, _rot(64)), 160)], (1, 2, 3), (97, 99991, 65537)),
    # degenerate values: a window of one token, more kept tokens than the window, one pass, one head, no rotation
    "ones": config(64, 96, [entry(mixer(1, 1, 16, 16, {"size": 1, "keep_first": 1}, None, 1.0), 24),
                            entry(mixer(2, 2, 16, 8, {"size": 4, "keep_first": 30}, _rot(2)), 16)], (0, 2, 1), (1, 1, 1), 1.0),
    # head sizes above 128 and a head group that does not divide a tile
    "wide": config(96, 150, [entry(mixer(3, 1, 136, 72, {"size": 25, "keep_first": 4}, _rot(16)), 64),
                             entry(mixer(2, 2, 200, 256, {"size": 90, "keep_first": 0}, _rot(64)), 64)], None, (31, 5, 2)),
}


# layouts that split evenly over ranks, with sizes that do not
SPLIT = {
    "wide2": config(70, 151, [entry(mixer(4, 2, 20, 12, {"size": 9, "keep_first": 2}, _rot(10)), 51)], None, (31, 5, 2)),
    "unequal4": config(72, 90, [entry(mixer(4, 2, 24, 16, {"size": 13, "keep_first": 3}, ROTATION), 50),
                                entry(mixer(8, 4, 8, 8, None, _rot(8)))], (0, 1, 2)),
}


def shapes(c):
    W, out = c["width"], {}
    out["embed"] = (c["vocab"], W)
    b = c["embedding"].get("bigram")
    if b:
        out["bigram"] = (b["buckets"] + 1, W)
    if c.get("loop"):
        out["loop.in"], out["loop.step"] = (W, 2 * W), (c["loop"]["times"], W)

    def norm(n):
        out[n], out[n + ".b"] = (W,), (W,)

    for i, e in enumerate(c["layers"]):
        m, p = e["mixer"], f"l{i}."
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * dv, W), p + "mix.sink": (H,),
                    p + "mix.o": (W, H * dv), p + "ls1": (W,)})
        norm(p + "norm1"), norm(p + "norm1b")
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff), p + "ls2": (W,)})
            norm(p + "norm2"), norm(p + "norm2b")
    norm("final.norm")
    return out


def weights(c, seed=0):
    """bf16-representable fp32 weights. Queries and keys are large, so a softmax row rests on a few keys and a wrong or
    missing one shows; sinks, layer scales, norm weights and biases are all far from neutral."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, s in shapes(c).items():
        t = torch.randn(s, generator=g)
        last = name.split(".")[-1]
        if last in ("q", "k"):
            t = t * 2.2 / s[-1] ** 0.5
        elif last in ("v", "o", "gate", "up", "down", "in"):
            t = t * 1.2 / s[-1] ** 0.5
        elif last in ("embed", "bigram"):
            t = t * 0.4
        elif last == "sink":
            t = t * 2
        elif last == "step" or last == "b":
            t = t * 0.3
        else:                                      # norm weights and layer scales
            t = 0.8 + 0.3 * t
        w[name] = t.bfloat16().float()
    return w
