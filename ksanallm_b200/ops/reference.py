"""Plain PyTorch statements of every op (fp32 math). They are the oracles the CUDA kernels are
tested against and the execution path for CPU tensors (unit tests, the CPU end-to-end slice).
Signatures mirror :mod:`ksanallm_b200.ops.native`.
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn.functional as F

E4M3_MAX = 448.0


def gemm(x, w, bias=None, residual=None, out_dtype=None):
    y = x.float() @ w.float().t()
    if bias is not None:
        y = y + bias.float()
    if residual is not None:
        y = y + residual.float()
    return y.to(out_dtype or x.dtype)


def pow2_scale(amax):
    """Smallest power of two >= amax / 448 (UE8M0 scale), computed on the fp32 bit pattern like the kernels do."""
    s = amax.float().clamp_min(1e-10) * (1.0 / E4M3_MAX)
    bits = s.contiguous().view(torch.int32)
    e = (bits >> 23) + ((bits & 0x7FFFFF) != 0).to(torch.int32)
    return (e << 23).view(torch.float32)


def is_pow2(scale) -> bool:
    """True when every (positive, normal) fp32 scale is an exact power of two."""
    bits = scale.float().contiguous().view(torch.int32)
    return bool(((bits & 0x7FFFFF) == 0).all() and (bits > 0).all())


def quant_fp8(x):
    """Per (row, 128 columns) e4m3 quantisation with power-of-two scales; scales returned as [K/128, M]
    (k-group major)."""
    M, K = x.shape
    g = x.float().reshape(M, K // 128, 128)
    scale = pow2_scale(g.abs().amax(dim=-1))
    q = (g / scale.unsqueeze(-1)).clamp(-E4M3_MAX, E4M3_MAX).to(torch.float8_e4m3fn).reshape(M, K)
    return q, scale.t().contiguous()


WEIGHT_SCALE_POW2 = True   # default scale rule of quant_weight_fp8_block (engine option quantization.fp8_scale_mode)


def quant_weight_fp8_block(w, block=128, pow2=None):
    """[N,K] weight -> e4m3 + one fp32 scale per (128 x 128) block, scales [ceil(N/128), ceil(K/128)].
    pow2: power-of-two scales (what the tensor cores can apply themselves); False: amax / 448 exactly;
    None: the module default ``WEIGHT_SCALE_POW2``."""
    if pow2 is None:
        pow2 = WEIGHT_SCALE_POW2
    N, K = w.shape
    nb, kb = (N + block - 1) // block, (K + block - 1) // block
    wp = torch.zeros(nb * block, kb * block, dtype=torch.float32, device=w.device)
    wp[:N, :K] = w.float()
    blocks = wp.reshape(nb, block, kb, block)
    amax = blocks.abs().amax(dim=(1, 3)).clamp_min(1e-10)
    scale = pow2_scale(amax) if pow2 else amax / E4M3_MAX
    q = (blocks / scale[:, None, :, None]).clamp(-E4M3_MAX, E4M3_MAX).reshape(nb * block, kb * block)[:N, :K]
    return q.to(torch.float8_e4m3fn).contiguous(), scale.contiguous()


def dequant_weight_fp8_block(wq, ws, block=128):
    N, K = wq.shape
    s = ws.repeat_interleave(block, 0)[:N].repeat_interleave(block, 1)[:, :K]
    return wq.float() * s


def gemm_fp8(xq, xs, wq, ws, bias=None, residual=None, out_dtype=torch.bfloat16):
    M, K = xq.shape
    x = xq.float().reshape(M, K // 128, 128) * xs[:, :M].t().unsqueeze(-1)
    y = x.reshape(M, K) @ dequant_weight_fp8_block(wq, ws).t()
    if bias is not None:
        y = y + bias.float()
    if residual is not None:
        y = y + residual.float()
    return y.to(out_dtype)


def norm(x, w, eps, residual=None, beta=None, layernorm=False):
    """Returns (y, new_residual). With a residual the sum is rounded to the activation dtype first."""
    h = x.float()
    if residual is not None:
        h = (h + residual.float()).to(x.dtype).float()
    if layernorm:
        mu = h.mean(-1, keepdim=True)
        var = (h - mu).pow(2).mean(-1, keepdim=True)
        y = (h - mu) * torch.rsqrt(var + eps) * w.float()
    else:
        y = h * torch.rsqrt(h.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    if beta is not None:
        y = y + beta.float()
    return y.to(x.dtype), h.to(x.dtype)


def act(x, kind="silu"):
    if kind in ("silu", "swiglu"):
        return F.silu(x)
    if kind in ("gelu", "gelu_new", "gelu_pytorch_tanh"):
        return F.gelu(x, approximate="tanh")
    if kind == "relu":
        return F.relu(x)
    raise ValueError(kind)


def act_mul(x, kind="silu", gated=True):
    xf = x.float()
    if gated:
        inter = x.shape[-1] // 2
        return (act(xf[..., :inter], kind) * xf[..., inter:]).to(x.dtype)
    return act(xf, kind).to(x.dtype)


def embedding(ids, table, vocab_lo=0, vocab_hi=None, positions=None, pos_table=None, scale=1.0):
    hi = vocab_lo + table.shape[0] if vocab_hi is None else vocab_hi
    mine = (ids >= vocab_lo) & (ids < hi)
    local = torch.where(mine, ids - vocab_lo, torch.zeros_like(ids)).long()
    out = table[local].float() * scale
    if pos_table is not None:
        out = out + pos_table[positions.long()].float()
    out = out * mine.unsqueeze(-1)
    return out.to(table.dtype)


def build_cos_sin_cache(rot_dim, max_pos, base=10000.0, scaling=None, device="cpu"):
    """[max_pos, rot_dim] = cos | sin. ``scaling`` follows HF ``rope_scaling`` dicts
    (linear, dynamic, llama3, yarn) as handled by the reference
    (3rdparty/LLM_kernels/csrc/kernels/nvidia/rotary_embedding/rotary_embedding.cu:202-340)."""
    half = rot_dim // 2
    inv_freq = 1.0 / (base ** (torch.arange(0, half, dtype=torch.float64) * 2 / rot_dim))
    t = torch.arange(max_pos, dtype=torch.float64)
    mscale = 1.0
    if scaling:
        kind = scaling.get("rope_type", scaling.get("type", "default"))
        factor = float(scaling.get("factor", 1.0))
        if kind == "linear":
            t = t / factor
        elif kind == "dynamic":
            orig = scaling.get("original_max_position_embeddings", max_pos)
            alpha = scaling.get("alpha")
            if alpha is not None:   # NTK-alpha variant
                nb = base * float(alpha) ** (rot_dim / (rot_dim - 2))
            else:
                nb = base * ((factor * max_pos / orig) - (factor - 1)) ** (rot_dim / (rot_dim - 2)) if max_pos > orig else base
            inv_freq = 1.0 / (nb ** (torch.arange(0, half, dtype=torch.float64) * 2 / rot_dim))
        elif kind == "llama3":
            low, high = float(scaling.get("low_freq_factor", 1.0)), float(scaling.get("high_freq_factor", 4.0))
            orig = float(scaling.get("original_max_position_embeddings", 8192))
            wavelen = 2 * math.pi / inv_freq
            smooth = ((orig / wavelen) - low) / (high - low)
            scaled = torch.where(wavelen > orig / low, inv_freq / factor, inv_freq)
            mid = (wavelen <= orig / low) & (wavelen >= orig / high)
            inv_freq = torch.where(mid, (1 - smooth) * inv_freq / factor + smooth * inv_freq, scaled)
        elif kind == "yarn":
            orig = float(scaling.get("original_max_position_embeddings", 4096))
            beta_fast, beta_slow = float(scaling.get("beta_fast", 32)), float(scaling.get("beta_slow", 1))

            def corr_dim(rot):
                return rot_dim * math.log(orig / (rot * 2 * math.pi)) / (2 * math.log(base))

            lo = max(math.floor(corr_dim(beta_fast)), 0)
            hi = min(math.ceil(corr_dim(beta_slow)), rot_dim - 1)
            ramp = ((torch.arange(half, dtype=torch.float64) - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
            mask = 1 - ramp
            inv_freq = inv_freq / factor * (1 - mask) + inv_freq * mask
            ms = float(scaling.get("mscale", 1.0))
            ms_all = float(scaling.get("mscale_all_dim", 0.0))

            def get_mscale(s, m):
                return 1.0 if s <= 1 else 0.1 * m * math.log(s) + 1.0

            mscale = get_mscale(factor, ms) / get_mscale(factor, ms_all) if ms_all else get_mscale(factor, 1.0)
    freqs = torch.outer(t, inv_freq)
    return torch.cat([freqs.cos() * mscale, freqs.sin() * mscale], dim=-1).float().to(device)


def apply_rope(x, positions, cos_sin, rot_dim, neox=True, mrope_sections=None):
    """x [T, H, D]; positions [T] or [3, T] with mrope_sections."""
    T, H, D = x.shape
    half = rot_dim // 2
    if mrope_sections is not None:
        s0, s1 = mrope_sections[0], mrope_sections[0] + mrope_sections[1]
        j = torch.arange(half, device=x.device)
        sec = torch.where(j < s0, 0, torch.where(j < s1, 1, 2))
        pos = positions.long()[sec, :].t()                     # [T, half]
        cs_cos = cos_sin[:, :half][pos, j]                     # [T, half]
        cs_sin = cos_sin[:, half:][pos, j]
    else:
        cs = cos_sin[positions.long()]
        cs_cos, cs_sin = cs[:, :half], cs[:, half:]
    cos, sin = cs_cos.unsqueeze(1).float(), cs_sin.unsqueeze(1).float()
    xf = x.float()
    rot = xf[..., :rot_dim]
    if neox:
        x0, x1 = rot[..., :half], rot[..., half:]
        r = torch.cat([x0 * cos - x1 * sin, x1 * cos + x0 * sin], dim=-1)
    else:
        x0, x1 = rot[..., 0::2], rot[..., 1::2]
        r = torch.stack([x0 * cos - x1 * sin, x1 * cos + x0 * sin], dim=-1).flatten(-2)
    return torch.cat([r, xf[..., rot_dim:]], dim=-1).to(x.dtype)


def rope_kv_append(qkv, positions, slots, cos_sin, cache_layer, block_tokens, Hq, Hkv, D, rot_dim, neox=True,
                   mrope_sections=None, k_scale=1.0, v_scale=1.0, apply=True):
    """In place on qkv [T,(Hq+2Hkv)*D]; cache_layer viewed as [blocks, 2, Hkv, block_tokens, D]."""
    T = qkv.shape[0]
    q = qkv[:, : Hq * D].reshape(T, Hq, D)
    k = qkv[:, Hq * D: (Hq + Hkv) * D].reshape(T, Hkv, D)
    v = qkv[:, (Hq + Hkv) * D:].reshape(T, Hkv, D)
    if apply:
        q.copy_(apply_rope(q, positions, cos_sin, rot_dim, neox, mrope_sections))
        k.copy_(apply_rope(k, positions, cos_sin, rot_dim, neox, mrope_sections))
    if cache_layer is None:
        return
    ok = slots >= 0
    sl = slots[ok].long()
    blk, off = sl // block_tokens, sl % block_tokens
    if cache_layer.dtype == torch.float8_e4m3fn:
        cache_layer[blk, 0, :, off] = (k[ok].float() / k_scale).clamp(-E4M3_MAX, E4M3_MAX).to(torch.float8_e4m3fn)
        cache_layer[blk, 1, :, off] = (v[ok].float() / v_scale).clamp(-E4M3_MAX, E4M3_MAX).to(torch.float8_e4m3fn)
    else:
        cache_layer[blk, 0, :, off] = k[ok].to(cache_layer.dtype)
        cache_layer[blk, 1, :, off] = v[ok].to(cache_layer.dtype)


def paged_attention(q, cache_layer, block_table, cu_q, kv_lens, Hq, Hkv, D, scale, alibi=None, k_scale=1.0,
                    v_scale=1.0):
    """q [T, Hq*D] (new tokens only); returns [T, Hq*D]. Query i of sequence s sits at absolute position
    kv_len - q_len + i and sees cache positions <= its own."""
    T = q.shape[0]
    out = torch.zeros(T, Hq * D, dtype=q.dtype, device=q.device)
    B = kv_lens.numel()
    G = Hq // Hkv
    bt = cache_layer.shape[3]
    for s in range(B):
        q0, q1 = int(cu_q[s]), int(cu_q[s + 1])
        ql, kl = q1 - q0, int(kv_lens[s])
        if ql == 0:
            continue
        nblk = (kl + bt - 1) // bt
        blocks = block_table[s, :nblk].long()
        kv = cache_layer[blocks].float()                                  # [nblk, 2, Hkv, bt, D]
        k = kv[:, 0].permute(1, 0, 2, 3).reshape(Hkv, nblk * bt, D)[:, :kl] * k_scale
        v = kv[:, 1].permute(1, 0, 2, 3).reshape(Hkv, nblk * bt, D)[:, :kl] * v_scale
        qs = q[q0:q1].float().reshape(ql, Hkv, G, D).permute(1, 2, 0, 3)  # [Hkv, G, ql, D]
        att = torch.einsum("hgqd,hkd->hgqk", qs, k) * scale
        qpos = torch.arange(kl - ql, kl, device=q.device).unsqueeze(1)
        kpos = torch.arange(kl, device=q.device).unsqueeze(0)
        if alibi is not None:
            att = att + alibi.float().reshape(Hkv, G, 1, 1) * (kpos - qpos).float()
        att = att.masked_fill(kpos > qpos, float("-inf"))
        p = torch.softmax(att, dim=-1)
        o = torch.einsum("hgqk,hkd->hgqd", p, v).permute(2, 0, 1, 3).reshape(ql, Hq * D)
        out[q0:q1] = o.to(q.dtype)
    return out


# ------------------------------------------------------------------------------- 32-bit residual stream
def embed_pair(ids, prev, table, pair, scale, buckets=0, mul_prev=0, mul_cur=0):
    x = table[ids.long()].float() * scale
    if pair is not None:
        a = prev.long()
        row = torch.where(a < 0, torch.full_like(a, buckets), (a * mul_prev + ids.long() * mul_cur) % buckets)
        x = x + pair[row].float()
    return x


def stream_norm(x, norm):
    """fp32 norm over the first ``norm.size`` columns (of each of ``norm.groups`` equal parts of them); pad columns come
    out as zeros."""
    h = x[:, :norm.size].float()
    if norm.rms:
        p = h.unflatten(-1, (norm.groups, -1))
        y = (p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + norm.eps)).flatten(-2)
    else:
        d = h - h.mean(-1, keepdim=True)
        y = d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + norm.eps)
    y = y * norm.w[:norm.size].float()
    if norm.b is not None:
        y = y + norm.b[:norm.size].float()
    return F.pad(y, (0, x.shape[1] - norm.size))


def glu_clamp(x, limit, alpha, offset):
    g, u = x.float().chunk(2, dim=-1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(alpha * g) * (u + offset)).to(x.dtype)


def xielu(x, pos, neg, lin):
    z = x.float()
    low = z.clamp(max=0)
    return (torch.where(z > 0, pos * z * z, neg * (torch.expm1(low) - low)) + lin * z).to(x.dtype)


def gated_recurrence(z, u, g, state, block_tokens, block_table, cu_q, kv_lens, offset):
    """See dispatch.gated_recurrence; ``state`` [blocks, W] is updated in place."""
    out = torch.zeros(z.shape, dtype=z.dtype, device=z.device)
    for s in range(kv_lens.numel()):
        q0, q1 = int(cu_q[s]), int(cu_q[s + 1])
        pos = int(kv_lens[s]) - (q1 - q0)
        if q1 == q0 or pos < 0:
            continue
        S = state[int(block_table[s, (pos - 1) // block_tokens])].clone() if pos > 0 else torch.zeros_like(state[0])
        gate = torch.sigmoid(z[q0:q1].float())
        uf = u[q0:q1].float()
        inc = gate * torch.where(uf >= 0, uf + offset, torch.sigmoid(uf))
        for i in range(q1 - q0):
            S = (1 - gate[i]) * S + inc[i]
            out[q0 + i] = (S * F.silu(g[q0 + i].float())).to(out.dtype)
            if i == q1 - q0 - 1 or (pos + i + 1) % block_tokens == 0:
                state[int(block_table[s, (pos + i) // block_tokens])] = S
    return out


def _new_rows(cu_q, kv_lens, slots):
    """(state slot, rows, position of the first new token) of every sequence with new rows."""
    for s in range(kv_lens.numel()):
        q0, q1 = int(cu_q[s]), int(cu_q[s + 1])
        if q1 > q0 and int(slots[s]) >= 0:
            yield int(slots[s]), slice(q0, q1), int(kv_lens[s]) - (q1 - q0)


def _with_history(x, ring, slot, past):
    """x with the ring's rows that come before it in front (zeros before the sequence); the ring takes x's last rows."""
    n = ring.shape[1]
    back = [ring[slot, (past - b) % n] if past - b >= 0 else torch.zeros_like(x[0]) for b in range(n - 1, 0, -1)]
    out = torch.cat([torch.stack(back), x]) if back else x
    for t in range(max(0, x.shape[0] - n), x.shape[0]):
        ring[slot, (past + t) % n] = x[t]
    return out


def token_shift(h, mu, ring, cu_q, kv_lens, slots):
    out = torch.empty_like(h)
    for slot, r, past in _new_rows(cu_q, kv_lens, slots):
        f = _with_history(h[r], ring, slot, past).float()
        out[r] = (f[1:] + (f[:-1] - f[1:]) * mu.float()).to(h.dtype)
    return out


def gated_norm(y, w, pad, real, parts, eps, z=None, g=None, factor=1.0):
    v = y.float() if z is None else y.float() * torch.nn.functional.silu(z.float())
    v = v.unflatten(1, (-1, pad))
    parts_ = v[..., :real].flatten(1).unflatten(1, (parts, -1))
    rstd = torch.rsqrt(parts_.pow(2).mean(-1, keepdim=True) + eps)
    n = torch.zeros_like(v)
    n[..., :real] = (parts_ * rstd).flatten(1).unflatten(1, (-1, real))
    n = n.flatten(1) * w.float() * factor
    return (n if g is None else n * torch.sigmoid(g.float())).to(y.dtype)


def _convolved(x, conv, slot, past):
    f, taps = _with_history(x, conv.ring, slot, past).float(), conv.w.shape[0]
    y = sum(f[j:j + x.shape[0]] * conv.w[j].float() for j in range(taps))
    return torch.nn.functional.silu(y if conv.bias is None else y + conv.bias.float())


def state_space(x, conv, dt, dt_bias, A, D, state, groups, step):
    n, H, P, N = state.shape
    out = torch.zeros(x.shape[0], H * P)
    for slot, r, past in _new_rows(step.cu_q, step.kv_lens, step.state_slots):
        c = _convolved(x[r], conv, slot, past).to(x.dtype).float()
        xs = c[:, :H * P].unflatten(1, (H, P))
        B, C = (t.unflatten(1, (groups, N)).repeat_interleave(H // groups, 1) for t in c[:, H * P:].chunk(2, 1))
        d = torch.nn.functional.softplus(dt[r][:, :H].float() + dt_bias)
        S = state[slot] if past > 0 else torch.zeros_like(state[slot])
        for t in range(xs.shape[0]):
            S = S * torch.exp(-A * d[t])[:, None, None] + (d[t][:, None] * xs[t])[:, :, None] * B[t][:, None, :]
            out[r.start + t] = ((S * C[t][:, None, :]).sum(-1) + D[:, None] * xs[t]).flatten()
        state[slot] = S
    return out


def delta_rule(x, conv, beta, decay, decay_bias, A, state, groups, q_scale, step):
    n, H, V, K = state.shape
    out = torch.zeros(x.shape[0], H * V)
    for slot, r, past in _new_rows(step.cu_q, step.kv_lens, step.state_slots):
        c = _convolved(x[r], conv, slot, past).to(x.dtype).float()
        q, k = (t.unflatten(1, (groups, K)) for t in c[:, :2 * groups * K].chunk(2, 1))
        q, k = ((t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)).repeat_interleave(H // groups, 1) for t in (q, k))
        q, v = q * q_scale, c[:, 2 * groups * K:].unflatten(1, (H, V))
        b = torch.sigmoid(beta[r][:, :H].float())
        g = torch.exp(-A[:, None] * torch.nn.functional.softplus(decay[r].float() + decay_bias).unflatten(1, (H, K)))
        S = state[slot] if past > 0 else torch.zeros_like(state[slot])
        for t in range(v.shape[0]):
            S = S * g[t][:, None, :]
            u = b[t][:, None] * (v[t] - (S * k[t][:, None, :]).sum(-1))
            S = S + u[:, :, None] * k[t][:, None, :]
            out[r.start + t] = (S * q[t][:, None, :]).sum(-1).flatten()
        state[slot] = S
    return out


def latent_append(q, nope, kv, norm_w, eps, rank, positions, slots, cos_sin, qfull, cache, block_tokens):
    """q [T, G, nope + rotary] -> rotary columns of qfull [T, G, DK]; normed latents | rotated key of kv [T, DK] into the
    panel [blocks, block tokens, DK]."""
    R, rot = q.shape[2] - nope, cos_sin.shape[1]
    rank_p = qfull.shape[2] - R
    qfull[..., rank_p:] = apply_rope(q[..., nope:], positions, cos_sin, rot, neox=False).to(qfull.dtype)
    if kv is None:
        return
    c = kv[:, :rank_p].float()
    c = c * torch.rsqrt(c.pow(2).sum(-1, keepdim=True) / rank + eps) * norm_w.float()
    r = apply_rope(kv[:, None, rank_p:], positions, cos_sin, rot, neox=False)[:, 0]
    ok = slots >= 0
    sl = slots[ok].long()
    cache[sl // block_tokens, sl % block_tokens] = torch.cat([c.to(cache.dtype), r.to(cache.dtype)], -1)[ok]


def qkv_rope_append(qkv, positions, slots, cos_sin, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim):
    """In place on q of qkv [T, Hq*D + Hkv*D + Hkv*Dv]; rotated k and v into panels [blocks, Hkv, block_tokens, size]."""
    T, D, Dv = qkv.shape[0], k_cache.shape[-1], v_cache.shape[-1]
    q, k = qkv[:, :Hq * D].reshape(T, Hq, D), qkv[:, Hq * D:(Hq + Hkv) * D].reshape(T, Hkv, D)
    v = qkv[:, (Hq + Hkv) * D:].reshape(T, Hkv, Dv)
    if rot_dim:
        qkv[:, :Hq * D] = apply_rope(q, positions, cos_sin, rot_dim).reshape(T, Hq * D)
        k = apply_rope(k, positions, cos_sin, rot_dim)
    ok = slots >= 0
    blk, off = slots[ok].long() // block_tokens, slots[ok].long() % block_tokens
    k_cache[blk, :, off] = k[ok].to(k_cache.dtype)
    v_cache[blk, :, off] = v[ok].to(v_cache.dtype)


def qkv_norm_rope_append(qkv, positions, slots, cos_sin, qw, kw, eps, nq, nk, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim,
                         sums=None):
    """In place on q of qkv [T, Hq*D + Hkv*D + Hkv*Dv], k and v into panels; see native.qkv_norm_rope_append."""
    T, D, Dv = qkv.shape[0], k_cache.shape[-1], v_cache.shape[-1]
    q, k = qkv[:, :Hq * D].float(), qkv[:, Hq * D:(Hq + Hkv) * D].float()
    sq, sk = (q.pow(2).sum(-1), k.pow(2).sum(-1)) if sums is None else sums.unbind(1)
    q = (q * torch.rsqrt(sq / nq + eps).unsqueeze(1) * qw.float()).view(T, Hq, D)
    k = (k * torch.rsqrt(sk / nk + eps).unsqueeze(1) * kw.float()).view(T, Hkv, D)
    if rot_dim:
        q = apply_rope(q, positions, cos_sin, rot_dim, neox=False)
        k = apply_rope(k, positions, cos_sin, rot_dim, neox=False)
    qkv[:, :Hq * D] = q.reshape(T, Hq * D).to(qkv.dtype)
    ok = slots >= 0
    blk, off = slots[ok].long() // block_tokens, slots[ok].long() % block_tokens
    k_cache[blk, :, off] = k[ok].to(k_cache.dtype)
    v_cache[blk, :, off] = qkv[:, (Hq + Hkv) * D:].reshape(T, Hkv, Dv)[ok].to(v_cache.dtype)


def latent_norms(q, kv, q_w, kv_w, eps, q_rank, kv_rank, slots, cache, block_tokens):
    def normed(x, w, n):
        f = x.float()
        return f * torch.rsqrt(f.pow(2).sum(-1, keepdim=True) / n + eps) * w.float()
    ok = slots >= 0
    sl = slots[ok].long()
    cache[sl // block_tokens, sl % block_tokens] = normed(kv, kv_w, kv_rank)[ok].to(cache.dtype)
    return normed(q, q_w, q_rank).to(q.dtype)


def moe_route(logits, K, scoring="softmax", renorm=True, scale=1.0, bias=None, n_group=1, topk_group=1, E=None, gate_col=-1, group_top=2):
    """(ids [T, K] int64, weights fp32 [T, K (+ 1)]); see native.moe_route."""
    z = logits[:, :logits.shape[1] if E is None else E].float()
    score = torch.sigmoid(z) if scoring == "sigmoid" else torch.softmax(z, dim=-1)
    sel = score + (bias.float() if bias is not None else 0.0)
    if n_group > 1 and topk_group < n_group:
        grp = sel.unflatten(-1, (n_group, -1))
        gscore = grp.topk(min(group_top, grp.shape[-1]), dim=-1).values.sum(-1)
        keep = torch.zeros_like(gscore, dtype=torch.bool).scatter_(1, gscore.topk(topk_group, dim=-1).indices, True)
        sel = grp.masked_fill(~keep.unsqueeze(-1), float("-inf")).flatten(-2)
    ids = sel.topk(K, dim=-1).indices
    w = score.gather(1, ids)
    if renorm:
        w = w / w.sum(-1, keepdim=True).clamp_min(1e-20)
    w = w * scale
    if gate_col >= 0:
        w = torch.cat([w, torch.sigmoid(logits[:, gate_col:gate_col + 1].float())], 1)
    return ids, w


def expert_sum(y, dst_row, w, shared=None):
    """fp32 rows: sum over k of w[t, k] * y[dst_row[t, k]] (negative: left out), plus w[t, K] * shared[t] (without such a
    weight: plus shared[t])."""
    rows = y.float()[dst_row.clamp_min(0).long()].masked_fill((dst_row < 0).unsqueeze(-1), 0.0)
    out = (rows * w[:, :dst_row.shape[1], None]).sum(1)
    if shared is None:
        return out
    return out + (shared.float() * w[:, dst_row.shape[1], None] if w.shape[1] > dst_row.shape[1] else shared.float())


def panel_attention(q, k_cache, v_cache, block_table, cu_q, kv_lens, Hq, Hkv, scale, window=0, keep=0, sinks=None, weights=None):
    """q [T, Hq*D] (new tokens only) -> [T, Hq*Dv]; see the sliding window, the sink and the unnormalised weights in
    dispatch.panel_attention."""
    T, G, D, Dv, bt = q.shape[0], Hq // Hkv, k_cache.shape[-1], v_cache.shape[-1], k_cache.shape[2]
    out = torch.zeros(T, Hq * Dv, dtype=q.dtype, device=q.device)
    for s in range(kv_lens.numel()):
        q0, q1 = int(cu_q[s]), int(cu_q[s + 1])
        ql, kl = q1 - q0, int(kv_lens[s])
        if ql == 0:
            continue
        blocks = block_table[s, :(kl + bt - 1) // bt].long()
        k = k_cache[blocks].float().permute(1, 0, 2, 3).reshape(Hkv, -1, D)[:, :kl]
        v = v_cache[blocks].float().permute(1, 0, 2, 3).reshape(Hkv, -1, Dv)[:, :kl]
        qs = q[q0:q1].float().reshape(ql, Hkv, G, D).permute(1, 2, 0, 3)
        att = torch.einsum("hgqd,hkd->hgqk", qs, k) * scale
        qpos = torch.arange(kl - ql, kl, device=q.device).unsqueeze(1)
        kpos = torch.arange(kl, device=q.device).unsqueeze(0)
        hide = kpos > qpos
        if window > 0:
            hide = hide | ((qpos - kpos >= window) & (kpos >= keep))
        if weights is not None:
            far = (qpos - kpos).clamp(0, weights.bias.shape[1] - 1)
            att = torch.sigmoid(att + weights.bias[:, far].unflatten(0, (Hkv, G)))
            o = torch.einsum("hgqk,hkd->hgqd", att.masked_fill(hide, 0.0), v).permute(2, 0, 1, 3).reshape(ql, Hq * Dv)
            if weights.gate is not None:
                o = o * torch.sigmoid(weights.gate[q0:q1].float()) * weights.factor
            out[q0:q1] = o.to(q.dtype)
            continue
        att = att.masked_fill(hide, float("-inf"))
        if sinks is not None:
            att = torch.cat([att, sinks.float().reshape(Hkv, G, 1, 1).expand(-1, -1, ql, 1)], dim=-1)
        p = torch.softmax(att, dim=-1)[..., :kl]
        out[q0:q1] = torch.einsum("hgqk,hkd->hgqd", p, v).permute(2, 0, 1, 3).reshape(ql, Hq * Dv).to(q.dtype)
    return out


def sample(logits, temperature, top_k, top_p, uniforms, num_logprobs=0):
    """Row-wise reference of the fused sampler; ``uniforms`` [B] in [0,1) replaces the device RNG."""
    B, V = logits.shape
    tokens = torch.zeros(B, dtype=torch.int64)
    lp_ids = torch.full((B, num_logprobs), -1, dtype=torch.int64)
    lp_vals = torch.full((B, num_logprobs), float("-inf"))
    for b in range(B):
        row = logits[b].float()
        t = float(temperature[b]) if float(temperature[b]) > 0 else 1.0
        k = max(1, min(int(top_k[b]), 1024, V))
        vals, idx = torch.sort(row, descending=True, stable=True)
        if num_logprobs:
            n = min(num_logprobs, V)
            lp = torch.log_softmax(vals[:n] / t, dim=-1)
            lp_ids[b, :n], lp_vals[b, :n] = idx[:n], lp
        if k == 1:
            tokens[b] = idx[0]
            continue
        w = torch.exp(vals[:k] / t - vals[0] / t)
        p = float(top_p[b]) if 0 < float(top_p[b]) < 1 else 1.0
        cum = torch.cumsum(w, 0)
        keep = k if p >= 1 else int((cum >= p * cum[-1]).nonzero()[0]) + 1
        mass = cum[keep - 1] if p < 1 else cum[-1]
        u = float(uniforms[b]) * float(mass)
        pick = int((cum[:keep] > u).nonzero()[0]) if bool((cum[:keep] > u).any()) else keep - 1
        tokens[b] = idx[pick]
    return tokens, lp_ids, lp_vals


# ------------------------------------------------------------------------------------- NVFP4
# e2m1 values in blocks of 16 along K, one e4m3 scale per block and one fp32 scale per tensor:
#   x ~= e2m1 * e4m3_block_scale * tensor_scale.  Two values per byte, the even element in the low nibble.
_E2M1_VALUES = (0.0, 0.5, 1.0, 1.5, 2.0, 3.0, 4.0, 6.0)


def quant_nvfp4(x, tensor_scale=None):
    """[M, K] -> (packed uint8 [M, K/2], block scales float8_e4m3fn [M, K/16], tensor scale fp32 scalar tensor).
    K must be a multiple of 16. ``tensor_scale`` None: amax / (448 * 6), so that block scales use the e4m3 range."""
    M, K = x.shape
    xf = x.float()
    if tensor_scale is None:
        tensor_scale = (xf.abs().amax().clamp_min(1e-12) / (448.0 * 6.0)).reshape(())
    tensor_scale = torch.as_tensor(tensor_scale, dtype=torch.float32, device=x.device).reshape(())
    g = xf.reshape(M, K // 16, 16) / tensor_scale
    bs = (g.abs().amax(dim=-1) / 6.0).clamp(max=448.0).to(torch.float8_e4m3fn)       # e4m3 rounding of amax / 6
    bsf = bs.float().clamp_min(2.0 ** -9)
    v = (g / bsf.unsqueeze(-1)).clamp(-6.0, 6.0)
    grid = torch.tensor(_E2M1_VALUES, device=x.device)
    # round to nearest e2m1 magnitude, ties to the even code (codes 0..7)
    mag = v.abs()
    mids = (grid[1:] + grid[:-1]) / 2
    code = torch.bucketize(mag, mids, right=False)            # mag == midpoint -> lower code
    tie = mag == mids[(code).clamp(max=6)]
    up = tie & (code % 2 == 1) & (code < 7)
    code = torch.where(up, code + 1, code)
    code = (code | ((v < 0).to(code.dtype) << 3)).to(torch.uint8).reshape(M, K)
    packed = code[:, 0::2] | (code[:, 1::2] << 4)
    return packed.contiguous(), bs.contiguous(), tensor_scale


def dequant_nvfp4(packed, block_scale, tensor_scale):
    M, K2 = packed.shape
    grid = torch.tensor(_E2M1_VALUES, device=packed.device)
    lo, hi = packed & 0xF, packed >> 4
    codes = torch.stack([lo, hi], dim=-1).reshape(M, K2 * 2).long()
    val = grid[codes & 7] * torch.where((codes & 8) != 0, -1.0, 1.0)
    return (val.reshape(M, -1, 16) * block_scale.float().unsqueeze(-1)).reshape(M, K2 * 2) * tensor_scale


def gemm_nvfp4(aq, a_bs, a_ts, wq, w_bs, w_ts, bias=None, residual=None, out_dtype=torch.bfloat16):
    y = dequant_nvfp4(aq, a_bs, a_ts) @ dequant_nvfp4(wq, w_bs, w_ts).t()
    if bias is not None:
        y = y + bias.float()
    if residual is not None:
        y = y + residual.float()
    return y.to(out_dtype)


def mla_attention(qfull, cache_layer, block_table, cu_q, kv_lens, scale, lora=512, window=0, sinks=None, gate=None):
    """Absorbed multi-head latent attention, plain fp32 statement. qfull [T, G, lora+rope] (q_lat | q_pe),
    cache_layer [blocks, block_tokens, lora+rope] (c_kv | k_pe). Returns [T, G, lora] fp32. ``sinks`` [G]: logits in the
    denominator only, ``gate`` [T, G]: outputs are multiplied by its sigmoid."""
    T, G, _ = qfull.shape
    bt = cache_layer.shape[1]
    out = torch.zeros(T, G, lora, dtype=torch.float32, device=qfull.device)
    cu, kvl = cu_q.tolist(), kv_lens.tolist()
    for s in range(len(kvl)):
        q0, q1, kl = cu[s], cu[s + 1], kvl[s]
        if q1 == q0:
            continue
        nblk = (kl + bt - 1) // bt
        rows = cache_layer[block_table[s, :nblk].long()].reshape(nblk * bt, -1)[:kl].float()
        sc = torch.einsum("qhd,kd->hqk", qfull[q0:q1].float(), rows) * scale
        qpos = torch.arange(kl - (q1 - q0), kl, device=qfull.device).unsqueeze(1)
        kpos = torch.arange(kl, device=qfull.device).unsqueeze(0)
        hide = (kpos > qpos) | (qpos - kpos >= window) if window > 0 else kpos > qpos
        sc = sc.masked_fill(hide, float("-inf"))
        if sinks is not None:
            sc = torch.cat([sc, sinks.float().view(G, 1, 1).expand(-1, q1 - q0, 1)], dim=-1)
        out[q0:q1] = torch.einsum("hqk,kl->qhl", torch.softmax(sc, -1)[..., :kl], rows[:, :lora])
    return out if gate is None else out * torch.sigmoid(gate.float()).unsqueeze(-1)


# ----------------------------------------------------------------------------- 4-bit weight-only groups (W4A16)
def quant_w4(w, group=128):
    """Asymmetric 4-bit group quantisation along K of w [N, K]: returns (packed uint8 [N, K/2] with the even k in
    the low nibble, scale fp16 [N, K/g], zs = zero_point * scale fp16 [N, K/g]); w ~= q * scale - zs.
    Per group the step is (max - min) / n for the n in 15..12 with the smallest error, so a group whose values
    already sit on a 16-level lattice (a dequantised GPTQ / AWQ group, which need not use all 16 levels) is
    reproduced up to the fp16 rounding of zs."""
    N, K = w.shape
    g = min(group, K)
    wf = w.float().reshape(N, K // g, g)
    lo, hi = wf.amin(-1, keepdim=True), wf.amax(-1, keepdim=True)
    best = None
    for n in (15.0, 14.0, 13.0, 12.0):
        scale = ((hi - lo) / n).clamp_min(1e-8).to(torch.float16).float()
        zp = torch.round(-lo / scale)
        q = torch.round(wf / scale + zp).clamp(0, 15)
        zs = (zp * scale).to(torch.float16).float()
        err = (q * scale - zs - wf).abs().amax(-1, keepdim=True)
        if best is None:
            best = [err, q, scale, zs]
        else:
            take = err < best[0] * 0.5          # a coarser step must be clearly better (an exact lattice hit)
            best = [torch.where(take, err, best[0]), torch.where(take, q, best[1]), torch.where(take, scale, best[2]),
                    torch.where(take, zs, best[3])]
    _, q, scale, zs = best
    q = q.to(torch.uint8).reshape(N, K)
    packed = (q[:, 0::2] | (q[:, 1::2] << 4)).contiguous()
    return packed, scale.to(torch.float16).reshape(N, K // g).contiguous(), zs.to(torch.float16).reshape(N, K // g).contiguous()


def pack_w4(q, scale, zero):
    """From integer levels q [N, K] (0..15), scales and integer zero points [N, K/g] to the packed form."""
    q = q.to(torch.uint8)
    packed = (q[:, 0::2] | (q[:, 1::2] << 4)).contiguous()
    sb = scale.to(torch.float16)
    return packed, sb.contiguous(), (zero.float() * sb.float()).to(torch.float16).contiguous()


def dequant_w4(packed, scale, zs):
    N, K2 = packed.shape
    K = K2 * 2
    q = torch.empty(N, K, dtype=torch.float32, device=packed.device)
    q[:, 0::2] = (packed & 15).float()
    q[:, 1::2] = (packed >> 4).float()
    g = K // scale.shape[1]
    s = scale.float().repeat_interleave(g, dim=1)
    z = zs.float().repeat_interleave(g, dim=1)
    return q * s - z
