"""Plain, slow statement of the Fidevik decoder: whole sequences, no cache, one function per mechanism. Shares no code
with the package; every function works in the dtype of its inputs (float32 or float64)."""
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps) * w


def layer_norm(x, w, b, eps):
    d = x - x.sum(-1, keepdim=True) / x.shape[-1]
    return d / torch.sqrt((d * d).sum(-1, keepdim=True) / x.shape[-1] + eps) * w + b


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * sigmoid(z)


# ------------------------------------------------------------------------------------------------ attention
def rotate(x, position, dims, base):
    """x [..., n]: of the first ``dims`` dimensions the neighbours 2i and 2i + 1 turn by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = position * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - v * math.sin(a)
        out[..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def attend(q, k, v, scale, sink=None):
    """One head: q, k [T, d], v [T, dv]; a row sees itself and all earlier ones. ``sink``: a logit that takes its share of
    the weights and gives nothing."""
    s = (q @ k.t()) * scale
    s = s.masked_fill(torch.ones(s.shape, dtype=torch.bool).triu(1), float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    p = torch.exp(s - top)
    total = p.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return (p / total) @ v


def attention(h, m, w, pre, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[pre + "q"].t(), w[pre + "q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ w[pre + "k"].t(), w[pre + "k.norm"], eps).view(T, G, d)
    v = (h @ w[pre + "v"].t()).view(T, G, dv)
    if m.get("rot"):
        dims, base = m["rot"]["dims"], m["rot"]["base"]
        q = torch.stack([rotate(q[p], p, dims, base) for p in range(T)])
        k = torch.stack([rotate(k[p], p, dims, base) for p in range(T)])
    heads = [attend(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"]) for a in range(H)]
    return torch.cat(heads, 1) @ w[pre + "o"].t()


def latent_attention(h, m, w, pre, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[pre + "dq"].t(), w[pre + "dq.norm"], eps) @ w[pre + "uq"].t()
    c = rms_norm(h @ w[pre + "dkv"].t(), w[pre + "dkv.norm"], eps)
    k, v = c @ w[pre + "uk"].t(), c @ w[pre + "uv"].t()
    gate = sigmoid(h @ w[pre + "g"].t())
    heads = []
    for a in range(H):
        qa, ka, va = q[:, a * d:(a + 1) * d], k[:, a * d:(a + 1) * d], v[:, a * dv:(a + 1) * dv]
        heads.append(attend(qa, ka, va, m["scale"], w[pre + "sink"][a]) * gate[:, a:a + 1])
    return torch.cat(heads, 1) @ w[pre + "o"].t()


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_unit(h, w, pre, act):
    return (act(h @ w[pre + "gate"].t()) * (h @ w[pre + "up"].t())) @ w[pre + "down"].t()


def choose(z, correction, top, count, keep):
    """Router logits [experts] of one token -> {expert: weight}."""
    s = sigmoid(z)
    choice = (s + correction).tolist()
    size = len(choice) // count
    score = [sum(sorted(choice[g * size:(g + 1) * size])[-2:]) for g in range(count)]
    kept = sorted(range(count), key=lambda g: -score[g])[:keep]
    allowed = [e for e in range(len(choice)) if e // size in kept]
    best = sorted(allowed, key=lambda e: -choice[e])[:top]
    return {e: s[e] for e in best}


def experts(h, m, w, pre):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[pre + "router"].t()
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for e, weight in choose(z[t], w[pre + "correction"], r["top"], groups["count"], groups["keep"]).items():
            y = y + weight * gated_unit(h[t], w, f"{pre}e{e}.", silu)
        rows.append(y)
    y = torch.stack(rows)
    if m.get("shared"):
        y = y + gated_unit(h, w, pre + "shared.", silu) * sigmoid(h @ w[pre + "shared.sg"].t())
    return y


def feed_forward(h, m, w, pre):
    return gated_unit(h, w, pre, gelu) if m["kind"] == "dense" else experts(h, m, w, pre)


# ------------------------------------------------------------------------------------------------ model
def order(cfg):
    """(layer, number of the pass that it opens or None) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    inner = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + inner + [(i, None) for i in range(b, n)]


def forward(tokens, cfg, w, streams=None):
    """Logits [T, vocab] of one sequence. ``streams`` (a list) receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    first = w["embed"][torch.tensor(tokens)]
    x = first
    for i, opens in order(cfg):
        if opens is not None:
            if opens > 0:
                x = x + first
            x = x + w["loop.step"][opens]
        e, p = cfg["layers"][i], f"l{i}."
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        mixer = {"attention": attention, "latent_attention": latent_attention}[e["type"]]
        x = x + mixer(h, e["mixer"], w, p + "mix.", eps)
        if e.get("mlp"):
            x = x + feed_forward(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), e["mlp"], w, p + "mlp.")
        if streams is not None:
            streams.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].t() * cfg["logit_scale"]
