"""Plain, slow statement of the Rasizen decoder: whole sequences, no cache, one function per mechanism. Shares no code
with the package; every function works in the dtype of its inputs (float32 or float64)."""
import math

import torch


def group_norm(x, w, groups, eps):
    """RMS norm part by part (``groups`` parts of equal size), then the weight over the whole row."""
    size = x.shape[-1] // groups
    parts = []
    for g in range(groups):
        p = x[..., g * size:(g + 1) * size]
        ms = (p * p).sum(-1, keepdim=True) / size
        parts.append(p / torch.sqrt(ms + eps))
    return torch.cat(parts, dim=-1) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


# ------------------------------------------------------------------------------------------------ gated recurrence
def recurrence(z, u, state):
    """z, u [T, width] (gate and candidate pre-activations), state [width]: the states after every token."""
    out = []
    for t in range(z.shape[0]):
        gate = sigmoid(z[t])
        cand = torch.where(u[t] >= 0, u[t] + 0.5, sigmoid(u[t]))
        state = (1 - gate) * state + gate * cand
        out.append(state)
    return torch.stack(out)


def mingru(h, m, w, pre):
    z = h @ w[pre + "z"].t() + w[pre + "z.b"]
    u = h @ w[pre + "x"].t() + w[pre + "x.b"]
    g = h @ w[pre + "g"].t()
    s = recurrence(z, u, torch.zeros(m["width"], dtype=h.dtype))
    return (s * g * sigmoid(g)) @ w[pre + "o"].t()


# ------------------------------------------------------------------------------------------------ latent attention
def rotate(x, position, base):
    """x [..., n]: neighbouring dimensions 2i and 2i + 1 turn by position * base^(-2i / n)."""
    n = x.shape[-1]
    out = x.clone()
    for i in range(n // 2):
        a = position * base ** (-2.0 * i / n)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - v * math.sin(a)
        out[..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def latents(h, m, w, pre, eps):
    """(latent [T, rank], rotated shared key [T, rot]) of a sequence."""
    y = h @ w[pre + "dkv"].t()
    c = group_norm(y[:, :m["kv_rank"]], w[pre + "dkv.norm"], 1, eps)
    r = torch.stack([rotate(y[p, m["kv_rank"]:], p, m["rot"]["base"]) for p in range(h.shape[0])])
    return c, r


def attend(q, k, v, scale, window):
    """One head: q, k [T, d], v [T, dv]; ``window`` None: every earlier token is visible."""
    out = []
    for i in range(q.shape[0]):
        lo = 0 if window is None else max(0, i - window + 1)
        s = (k[lo:i + 1] @ q[i]) * scale
        p = torch.exp(s - s.max())
        out.append((p / p.sum()) @ v[lo:i + 1])
    return torch.stack(out)


def latent_attention(h, m, w, pre, c, r):
    T, H, dim, rot, vdim, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[pre + "q"].t()).view(T, H, dim + rot)
    uk, uv = w[pre + "uk"].view(H, dim, rank), w[pre + "uv"].view(H, vdim, rank)
    window = m["mask"]["size"] if m.get("mask") else None
    heads = []
    for a in range(H):
        qr = torch.stack([rotate(q[p, a, dim:], p, m["rot"]["base"]) for p in range(T)])
        heads.append(attend(torch.cat([q[:, a, :dim], qr], 1), torch.cat([c @ uk[a].t(), r], 1), c @ uv[a].t(), m["scale"], window))
    return (torch.cat(heads, dim=1) * sigmoid(h @ w[pre + "g"].t())) @ w[pre + "o"].t()


# ------------------------------------------------------------------------------------------------ feed-forward
def softplus(x):
    return max(x, 0.0) + math.log1p(math.exp(-abs(x)))


def xielu(z, p, q):
    z0 = torch.clamp(z, max=0)
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(z0) - z0)) + z / 2


def feed_forward(h, w, pre):
    p, q = (float(t) for t in w[pre + "act"])
    return xielu(h @ w[pre + "up"].t(), p, q) @ w[pre + "down"].t()


# ------------------------------------------------------------------------------------------------ model
def forward(tokens, cfg, w, streams=None):
    """Logits [T, vocab] of one sequence. ``streams`` (a list) receives the residual stream after every layer."""
    eps, groups, mult = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(tokens)]
    cached = {}
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        h = group_norm(x, w[p + "norm1"], groups, eps)
        if e["type"] == "mingru":
            y = mingru(h, m, w, p + "mix.")
        else:
            if m.get("kv_from") is None:
                cached[i] = latents(h, m, w, p + "mix.", eps)
            y = latent_attention(h, m, w, p + "mix.", *cached[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + mult * y
        if e.get("mlp"):
            x = x + mult * feed_forward(group_norm(x, w[p + "norm2"], groups, eps), w, p + "mlp.")
        if streams is not None:
            streams.append(x.clone())
    return group_norm(x, w["final.norm"], groups, eps) @ w["embed"].t()
