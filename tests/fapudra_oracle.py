"""Plain, slow statement of the Fapudra decoder: whole sequences, no cache, one function per mechanism. Shares no code
with the package; every function works in the dtype of its inputs (float32 or float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------------------------ token mixing
def token_shift(h, mu):
    """Row t moves towards row t - 1 (zeros before the first) by ``mu``, column by column."""
    before = torch.zeros_like(h)
    before[1:] = h[:-1]
    return h + (before - h) * mu


def causal_conv(x, taps, bias=None):
    """x [T, C], taps [C, n]: the last tap multiplies the row itself, the ones before it earlier rows."""
    out = torch.zeros_like(x) if bias is None else bias.expand_as(x).clone()
    n = taps.shape[1]
    for j in range(n):
        back = n - 1 - j
        for t in range(back, x.shape[0]):
            out[t] = out[t] + x[t - back] * taps[:, j]
    return out


def state_space(x, B, C, dt, A_log, D):
    """One head: x [T, P], B and C [T, N], dt [T] (positive). S is [N, P]."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=x.dtype)
    rows = []
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(A_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        rows.append(S.t() @ C[t] + D * x[t])
    return torch.stack(rows)


def mamba2(h, m, w, pre, eps):
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, x, B, C, dt = (h @ w[pre + "in"].t()).split([inner, inner, G * N, G * N, H], dim=1)
    c = silu(causal_conv(torch.cat([x, B, C], 1), w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = c.split([inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[pre + "dt_bias"])
    y = []
    for a in range(H):
        g = a // (H // G)
        y.append(state_space(x[:, a * P:(a + 1) * P], B[:, g * N:(g + 1) * N], C[:, g * N:(g + 1) * N], dt[:, a], w[pre + "A_log"][a],
                             w[pre + "D"][a]))
    y = torch.cat(y, 1) * silu(z)
    y = rms(y.unflatten(1, (m["norm_groups"], -1)), eps).flatten(1) * w[pre + "norm"]
    return y @ w[pre + "o"].t()


def delta_rule(q, k, v, beta, g):
    """One head: q, k, g [T, K], v [T, V], beta [T]. The read-out sees the row's own write."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    rows = []
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        rows.append(S.t() @ q[t])
    return torch.stack(rows)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def gated_delta(h, m, w, pre, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[pre + n].t(), w[pre + n + ".conv"])) for n in "qkv")
    q, k, v = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d)), v.view(T, H, dv)
    beta = sigmoid(h @ w[pre + "b"].t())
    step = softplus((h @ w[pre + "a1"].t()) @ w[pre + "a2"].t() + w[pre + "dt_bias"]).view(T, H, d)
    decay = torch.exp(-torch.exp(w[pre + "A_log"])[None, :, None] * step)
    o = torch.stack([delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], decay[:, a]) for a in range(H)], 1)
    gate = sigmoid((h @ w[pre + "g1"].t()) @ w[pre + "g2"].t()).view(T, H, dv)
    return (rms(o, eps) * w[pre + "norm"] * gate).flatten(1) @ w[pre + "o"].t()


# ------------------------------------------------------------------------------------------------ attention
def bucket(n, count, far):
    half = count // 2
    if n < half:
        return n
    return min(count - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (count - half)))


def attend(q, k, v, scale, bias, window, keep):
    """One head with independent sigmoid weights: q, k [T, d], v [T, dv]; ``bias(n)``: what distance n adds to a score."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    table = torch.stack([bias(n) for n in range(T)])
    for i in range(T):
        j = torch.arange(i + 1)
        j = j[(i - j < window) | (j < keep)]
        out[i] = sigmoid((k[j] @ q[i]) * scale + table[i - j]) @ v[j]
    return out


def sigmoid_attention(h, m, w, pre):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[pre + "q"].t() + w[pre + "q.b"]).view(T, H, d)
    k = (h @ w[pre + "k"].t() + w[pre + "k.b"]).view(T, G, d)
    rel = w[pre + "rel"]
    mask = m.get("mask") or {"size": T + 1}
    heads = []
    for a in range(H):
        def bias(n):
            return rel[bucket(n, rel.shape[0], m["bias_max"]), a] + w[pre + "pb"][a]
        kv = k[:, a // (H // G)]
        heads.append(attend(q[:, a], kv, kv, m["scale"], bias, mask["size"], mask.get("keep_first", 0)))
    return (torch.cat(heads, 1) * sigmoid(h @ w[pre + "g"].t())) @ w[pre + "o"].t()


def parallel(h, m, w, pre, eps):
    return (m["left_scale"] * sigmoid_attention(h, m["left"], w, pre + "left.") +
            m["right_scale"] * gated_delta(h, m["right"], w, pre + "right.", eps))


# ------------------------------------------------------------------------------------------------ feed-forward
def expert(h, w, pre, limit):
    g = torch.clamp(h @ w[pre + "gate"].t(), max=limit)
    u = torch.clamp(h @ w[pre + "up"].t(), -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[pre + "down"].t()


def choose(z, top, count, keep):
    """Router logits [experts] of one token -> {expert: weight}."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    p, size = s.tolist(), len(s) // count
    kept = sorted(range(count), key=lambda g: -max(p[g * size:(g + 1) * size]))[:keep]
    best = sorted([e for e in range(len(p)) if e // size in kept], key=lambda e: -p[e])[:top]
    total = sum(s[e] for e in best) + 1e-20
    return {e: s[e] / total for e in best}


def experts(h, m, w, pre):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[pre + "router"].t()
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for e, weight in choose(z[t], r["top"], groups["count"], groups["keep"]).items():
            y = y + weight * expert(h[t], w, f"{pre}e{e}.", m["expert"]["limit"])
        rows.append(y)
    return torch.stack(rows)


# ------------------------------------------------------------------------------------------------ model
def forward(tokens, cfg, w, streams=None, splice=None):
    """Logits [T, vocab] of one sequence. ``streams`` (a list) receives the residual stream after every layer; ``splice`` {row:
    vector} replaces rows of the first stream."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"] + w["pos"][:len(tokens)]
    x = rms(x, eps) * w["embed.norm"]
    for row, vector in (splice or {}).items():
        x[row] = vector
    for i, e in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        mixer = {"mamba2": mamba2, "parallel": parallel}[e["type"]]
        y = mixer(token_shift(h, w[p + "shift"]), e["mixer"], w, p + "mix.", eps)
        if e.get("mlp"):
            y = y + experts(h, e["mlp"], w, p + "mlp.")
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    z = (rms(x, eps) * w["final.norm"]) @ w["head"].t()
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(z / cap)
