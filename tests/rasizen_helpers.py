"""Small Rasizen models for the tests: configurations and seeded weights that make attention sharp and the recurrences'
memories of unequal length."""
import torch

from decoder_helpers import build, engine, error, run_portions, save_checkpoint, tokens  # noqa: F401


def latent(heads, dim, rot, vdim, rank, window, base=900.0, kv_from=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot) ** -0.5,
         "rot": {"base": base, "dims": rot}, "mask": None if window is None else {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def mingru(width):
    return "mingru", {"width": width}


def config(width, vocab, layers, groups, mult, eps=1e-5):
    return {"architecture": "Rasizen", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "residual_mult": mult,
            "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}


CONFIGS = {
    # the recurrence first, a feed-forward on one layer of each kind, latents read again with other heads and another window
    "unequal": config(72, 203, [(mingru(56), 40), (latent(3, 16, 8, 24, 40, 13), 88), (latent(5, 24, 8, 8, 40, 20, kv_from=1), None),
                                (mingru(96), None)], 3, 0.6),
    # nothing is a multiple of 8, norm groups that cut through vectors
    "odd": config(70, 101, [(latent(3, 10, 6, 12, 22, 7, 70.0), 33), (mingru(45), 50), (latent(2, 20, 6, 20, 22, 33, 70.0, kv_from=0), None)],
                  5, 1.3, 1e-4),
    # windows longer than a page and than a tile, two layers with latents of their own, one group
    "long": config(128, 320, [(latent(8, 32, 16, 32, 64, 70), None), (mingru(128), 96), (latent(4, 24, 32, 16, 136, 24, 5000.0), 64),
                              (latent(2, 48, 32, 40, 136, 101, 5000.0, kv_from=2), 80), (mingru(64), None)], 1, 0.35),
    # degenerate values: a window of one token, one head, one pair, factor 1, the smallest sizes
    "ones": config(64, 96, [(latent(1, 8, 2, 8, 8, 1, scale=1.0), 8), (mingru(8), None), (latent(2, 1, 2, 1, 3, 2, scale=0.2), 1)], 8, 1.0),
    # recurrences only
    "recurrent": config(48, 90, [(mingru(40), 24), (mingru(136), None), (mingru(48), 48)], 2, 0.8),
    # no recurrence, no mask, latent rows of more than one output half and beyond the tensor-core kernel
    "wide": config(96, 150, [(latent(2, 16, 64, 24, 520, 90), 64), (latent(3, 40, 64, 48, 300, None), 64),
                             (latent(6, 16, 64, 8, 300, 35, kv_from=1), None)], 2, 0.5),
}

# layouts that split evenly over ranks, with sizes that do not
SPLIT = {
    "split2": config(70, 151, [(latent(2, 20, 6, 12, 22, 9), 51), (mingru(45), None), (latent(4, 12, 6, 20, 22, 30, kv_from=0), None)], 5, 0.7),
    "split4": config(72, 90, [(mingru(100), 50), (latent(4, 24, 8, 16, 40, 13), None), (latent(8, 8, 8, 8, 40, 5, kv_from=1), 33)], 3, 1.1),
}


def shapes(c):
    W = c["width"]
    out = {"embed": (c["vocab"], W), "final.norm": (W,)}
    for i, e in enumerate(c["layers"]):
        m, p = e["mixer"], f"l{i}."
        x = p + "mix."
        out[p + "norm1"] = (W,)
        if e["type"] == "mingru":
            n = m["width"]
            out.update({x + "z": (n, W), x + "z.b": (n,), x + "x": (n, W), x + "x.b": (n,), x + "g": (n, W), x + "o": (W, n)})
        else:
            H, d, r, v, k = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            out.update({x + "q": (H * (d + r), W), x + "uk": (H * d, k), x + "uv": (H * v, k), x + "g": (H * v, W), x + "o": (W, H * v)})
            if m.get("kv_from") is None:
                out.update({x + "dkv": (k + r, W), x + "dkv.norm": (k,)})
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff), p + "mlp.act": (2,)})
    return out


def weights(c, seed=0):
    """bf16-representable fp32 weights. Queries, rotary keys and key products are large, so a softmax row rests on a few
    keys and a wrong or missing one shows; the recurrence's gates are mostly small, some very small (a state that is lost
    or mixed up stays visible for hundreds of tokens); norm weights are far from one."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, s in shapes(c).items():
        t = torch.randn(s, generator=g)
        last = name.split(".")[-1]
        if name.endswith("z.b"):
            t = t * 1.5 - 3
        elif name.endswith("x.b") or last == "act":
            t = t * 0.7
        elif last in ("q", "uk", "dkv"):
            t = t * 2.0 / s[-1] ** 0.5
        elif last == "embed":
            t = t * 0.7
        elif len(s) == 2:
            t = t * 1.5 / s[-1] ** 0.5
        else:                                      # norm weights
            t = 0.9 + 0.3 * t
        w[name] = t.bfloat16().float()
    return w
