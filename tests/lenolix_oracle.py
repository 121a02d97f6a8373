"""Plain, slow statement of the Lenolix decoder: whole sequences, no cache, one function per mechanism. Shares no code
with the package; every function works in the dtype of its inputs (float32 or float64)."""
import functools
import math

import torch


def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """Row of the pair table for every token of a sequence; a sequence's first token has a row of its own."""
    rows = []
    for i, t in enumerate(tokens):
        rows.append(buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets)
    return rows


def embed(tokens, cfg, w):
    e = cfg["embedding"]
    x = w["embed"][torch.tensor(tokens)] * e["scale"]
    b = e.get("bigram")
    if b:
        x = x + w["bigram"][torch.tensor(bigram_rows(tokens, b["mul_prev"], b["mul_cur"], b["buckets"]))]
    return x


def layer_norm(x, w, b, eps):
    mean = x.sum(-1, keepdim=True) / x.shape[-1]
    d = x - mean
    var = (d * d).sum(-1, keepdim=True) / x.shape[-1]
    return d / torch.sqrt(var + eps) * w + b


def rope_frequencies(dims, base, scaling):
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wavelength = 2 * math.pi / f
            if wavelength > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif wavelength >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wavelength - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate(x, position, freqs):
    """x [..., dim] of one position: dimension i turns with dimension i + n (n = number of frequencies)."""
    n = len(freqs)
    c = torch.tensor([math.cos(position * f) for f in freqs], dtype=x.dtype)
    s = torch.tensor([math.sin(position * f) for f in freqs], dtype=x.dtype)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def visible(i, j, mask):
    if j > i:
        return False
    return mask is None or i - j < mask["size"] or j < mask["keep_first"]


@functools.lru_cache(maxsize=None)
def _visibility(T, size, keep_first):
    mask = None if size is None else {"size": size, "keep_first": keep_first}
    return torch.tensor([[visible(i, j, mask) for j in range(T)] for i in range(T)])


def attend(q, k, v, sink, scale, mask):
    """One head: q [T, dim], k [T, dim], v [T, vdim]; ``sink``: extra logit in the denominator (or None)."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    see = _visibility(T, None if mask is None else mask["size"], None if mask is None else mask["keep_first"])
    s = (q @ k.t()) * scale
    for i in range(T):
        si = s[i][see[i]]
        top = si.max()
        if sink is not None:
            top = torch.maximum(top, sink)
        p = torch.exp(si - top)
        den = p.sum() + (torch.exp(sink - top) if sink is not None else 0)
        out[i] = (p / den) @ v[see[i]]
    return out


def attention(h, m, w, pre):
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].t()).view(T, H, dim)
    k = (h @ w[pre + "k"].t()).view(T, G, dim)
    v = (h @ w[pre + "v"].t()).view(T, G, vdim)
    rot = m.get("rot")
    if rot:
        fr = rope_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q = torch.stack([rotate(q[p], p, fr) for p in range(T)])
        k = torch.stack([rotate(k[p], p, fr) for p in range(T)])
    sink = w.get(pre + "sink")
    heads = [attend(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], None if sink is None else sink[a], m["scale"],
                    m.get("mask")) for a in range(H)]
    return torch.cat(heads, dim=1) @ w[pre + "o"].t()


def feed_forward(h, mlp, w, pre):
    lim = mlp["limit"]
    g = torch.clamp(h @ w[pre + "gate"].t(), max=lim)
    u = torch.clamp(h @ w[pre + "up"].t(), min=-lim, max=lim)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w[pre + "down"].t()


def layer(x, i, cfg, w):
    e, p = cfg["layers"][i], f"l{i}."
    eps = cfg["norm"]["eps"]

    def norm(name, t):
        return layer_norm(t, w[p + name], w[p + name + ".b"], eps)

    x = x + norm("norm1b", attention(norm("norm1", x), e["mixer"], w, p + "mix.")) * w[p + "ls1"]
    if e.get("mlp"):
        x = x + norm("norm2b", feed_forward(norm("norm2", x), e["mlp"], w, p + "mlp.")) * w[p + "ls2"]
    return x


def layer_runs(cfg):
    """(layer, pass or None, first layer of a pass) in running order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    runs = [(i, None, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None, False) for i in range(loop["stop"], n)]


def forward(tokens, cfg, w, streams=None):
    """Logits [T, vocab] of one sequence. ``streams`` (a list) receives the residual stream after every layer run."""
    x0 = x = embed(tokens, cfg, w)
    for i, t, first in layer_runs(cfg):
        if first:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].t() + w["loop.step"][t]
        x = layer(x, i, cfg, w)
        if streams is not None:
            streams.append(x.clone())
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"])
    return x @ w["embed"].t()
