"""Device dispatch for the operator layer: CUDA tensors go to the hand-written sm_100a kernels
(:mod:`.native`), CPU tensors to the PyTorch statements (:mod:`.reference`). Model code calls
only this module, so the same model definition runs the CPU test slice and the B200 path.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import native, reference as ref
from .native import SigmoidWeights  # noqa: F401


@dataclass
class QTensor:
    """FP8 GEMM operand: e4m3 values [M,K] and fp32 scales [K/128, ld] (one per row and 128 columns)."""
    q: torch.Tensor
    s: torch.Tensor

    @property
    def shape(self):
        return self.q.shape


class LinearWeight:
    """[N,K] weight of y = x W^T (+bias): dense bf16/fp32, or e4m3 with one fp32 scale per 128x128 block."""

    def __init__(self, w: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None,
                 wq: Optional[torch.Tensor] = None, ws: Optional[torch.Tensor] = None):
        self.w, self.bias, self.wq, self.ws = w, bias, wq, ws
        # NVFP4 form: packed e2m1 [N, K/2], e4m3 scales per 16 elements [N, K/16], fp32 tensor scale
        self.w4 = self.w4_bs = self.w4_ts = None
        # weight-only 4-bit groups (GPTQ / AWQ family): packed levels [N, K/2], fp16 scale and zero*scale [N, K/g]
        self.q4 = self.q4_scale = self.q4_zs = None
        # power-of-two block scales: the tensor cores can apply them (hardware block-scaled MMA)
        self.ue8m0 = ws is not None and ref.is_pow2(ws)

    @property
    def fp8(self) -> bool:
        return self.wq is not None

    @property
    def nvfp4(self) -> bool:
        return self.w4 is not None

    @property
    def w4a16(self) -> bool:
        return self.q4 is not None

    def _any(self) -> torch.Tensor:
        if self.w4a16:
            return self.q4
        return self.w4 if self.nvfp4 else (self.wq if self.fp8 else self.w)

    @property
    def out_features(self) -> int:
        return self._any().shape[0]

    @property
    def in_features(self) -> int:
        return self._any().shape[1] * 2 if (self.nvfp4 or self.w4a16) else self._any().shape[1]

    @property
    def device(self):
        return self._any().device

    def without_bias(self) -> "LinearWeight":
        """Shallow copy that shares the weight tensors and has no bias (row-parallel ranks other than the first)."""
        if self.bias is None:
            return self
        if getattr(self, "_nb", None) is None:
            import copy
            self._nb = copy.copy(self)
            self._nb.bias = None
        return self._nb

    def quantize_nvfp4(self) -> "LinearWeight":
        """e2m1 weights with e4m3 scales per 16 input features (in_features must be a multiple of 256)."""
        if not self.nvfp4 and not self.fp8:
            self.w4, self.w4_bs, self.w4_ts = ref.quant_nvfp4(self.w)
            self.w = None
        return self

    def quantize_w4(self, group: int = 128) -> "LinearWeight":
        """4-bit weight-only groups along the input features (in_features must be a multiple of 32)."""
        if not (self.w4a16 or self.nvfp4 or self.fp8):
            self.q4, self.q4_scale, self.q4_zs = ref.quant_w4(self.w, group)
            self.w = None
        return self

    def quantize_fp8_block(self) -> "LinearWeight":
        if not self.fp8:
            self.wq, self.ws = ref.quant_weight_fp8_block(self.w)
            self.w = None
            self.ue8m0 = True
        return self

    def dense(self) -> torch.Tensor:
        if self.w4a16:
            return ref.dequant_w4(self.q4, self.q4_scale, self.q4_zs)
        if self.nvfp4:
            return ref.dequant_nvfp4(self.w4, self.w4_bs, self.w4_ts)
        return ref.dequant_weight_fp8_block(self.wq, self.ws) if self.fp8 else self.w

    def nbytes(self) -> int:
        t = [x for x in (self.w, self.wq, self.ws, self.bias, self.w4, self.w4_bs, self.q4, self.q4_scale, self.q4_zs)
             if x is not None]
        return sum(x.numel() * x.element_size() for x in t)


def _is_cuda(x) -> bool:
    return (x.q if isinstance(x, QTensor) else x).is_cuda


def quantize(x: torch.Tensor) -> QTensor:
    if x.is_cuda:
        return QTensor(*native.quant_fp8(x))
    return QTensor(*ref.quant_fp8(x))


def linear(x, W: LinearWeight, residual=None, out=None, out_f32: bool = False):
    """y = x W^T (+bias) (+residual). ``x`` may be a QTensor when W is FP8. ``out`` may alias ``residual``."""
    if W.w4a16:
        if isinstance(x, QTensor):
            raise TypeError("4-bit weight-only layers take bf16 activations")
        if x.is_cuda:
            if out_f32:
                return native.linear_w4(x, W.q4, W.q4_scale, W.q4_zs, bias=W.bias, residual=residual).float()
            return native.linear_w4(x, W.q4, W.q4_scale, W.q4_zs, out=out, bias=W.bias, residual=residual)
        y = ref.gemm(x, W.dense().to(x.dtype), W.bias, residual, torch.float32 if out_f32 else None)
        if out is not None:
            out.copy_(y)
            return out
        return y
    if W.nvfp4:
        # activations are quantised to NVFP4 too (per-tensor scale from the tensor's own maximum, no host sync)
        if x.is_cuda and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 and x.stride(1) == 1 and x.stride(0) % 8 == 0:
            a_ts = native.absmax_scale(x, 448.0 * 6.0)          # one pass over x, scale stays on the device
        else:
            a_ts = (x.float().abs().amax() / (448.0 * 6.0)).clamp_min(1e-12).reshape(())
        if x.is_cuda:
            aq, a_bs, _ = native.quant_nvfp4(x, a_ts)
            if out_f32:
                o = torch.empty(x.shape[0], W.out_features, dtype=torch.float32, device=x.device)
                return native.gemm_nvfp4(aq, a_bs, a_ts, W.w4, W.w4_bs, W.w4_ts, bias=W.bias, residual=residual, out_f32=o)
            return native.gemm_nvfp4(aq, a_bs, a_ts, W.w4, W.w4_bs, W.w4_ts, out=out, bias=W.bias, residual=residual)
        aq, a_bs, _ = ref.quant_nvfp4(x, a_ts)
        y = ref.gemm_nvfp4(aq, a_bs, a_ts, W.w4, W.w4_bs, W.w4_ts, W.bias, residual, torch.float32 if out_f32 else x.dtype)
        if out is not None:
            out.copy_(y)
            return out
        return y
    if _is_cuda(x):
        if W.fp8:
            if not isinstance(x, QTensor):
                x = quantize(x)
            if out_f32:
                o = torch.empty(x.q.shape[0], W.out_features, dtype=torch.float32, device=x.q.device)
                return native.gemm_fp8(x.q, x.s, W.wq, W.ws, bias=W.bias, residual=residual, out_f32=o, hw_scale=W.ue8m0)
            return native.gemm_fp8(x.q, x.s, W.wq, W.ws, out=out, bias=W.bias, residual=residual, hw_scale=W.ue8m0)
        if W.w.dtype == torch.float32:
            return native.gemm_f32(x, W.w, out=out, bias=W.bias, residual=residual)
        if out_f32:
            o = torch.empty(x.shape[0], W.out_features, dtype=torch.float32, device=x.device)
            return native.gemm_bf16(x, W.w, bias=W.bias, residual=residual, out_f32=o)
        return native.gemm_bf16(x, W.w, out=out, bias=W.bias, residual=residual)
    # CPU statement
    if W.fp8:
        xq = x if isinstance(x, QTensor) else QTensor(*ref.quant_fp8(x))
        y = ref.gemm_fp8(xq.q, xq.s, W.wq, W.ws, W.bias, residual, torch.float32 if out_f32 else torch.bfloat16)
    else:
        y = ref.gemm(x, W.w, W.bias, residual, torch.float32 if out_f32 else x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def norm(x, w, eps, residual=None, beta=None, layernorm=False, quant_for: Optional[LinearWeight] = None):
    """Returns the normalised activations in the form the consuming linear wants (QTensor for FP8
    weights on CUDA). ``residual`` (if given) is updated in place with residual + x."""
    want_q = quant_for is not None and quant_for.fp8 and x.shape[-1] % 128 == 0
    if x.is_cuda:
        if want_q:
            _, q, s = native.norm(x, w, eps, residual=residual, beta=beta, layernorm=layernorm, quant=True,
                                  want_out=False)
            return QTensor(q, s)
        return native.norm(x, w, eps, residual=residual, beta=beta, layernorm=layernorm)
    y, new_res = ref.norm(x, w, eps, residual, beta, layernorm)
    if residual is not None:
        residual.copy_(new_res)
    return QTensor(*ref.quant_fp8(y)) if want_q else y


def act_mul(x, kind="silu", gated=True, quant_for: Optional[LinearWeight] = None):
    inter = x.shape[-1] // 2 if gated else x.shape[-1]
    want_q = quant_for is not None and quant_for.fp8 and inter % 128 == 0
    if x.is_cuda:
        if want_q:
            _, q, s = native.act_mul(x, kind, gated, quant=True, want_out=False)
            return QTensor(q, s)
        return native.act_mul(x, kind, gated)
    y = ref.act_mul(x, kind, gated)
    return QTensor(*ref.quant_fp8(y)) if want_q else y


def embedding(ids, table, vocab_lo=0, vocab_hi=None, positions=None, pos_table=None, scale=1.0):
    if table.is_cuda:
        return native.embedding(ids, table, vocab_lo=vocab_lo, vocab_hi=vocab_hi, positions=positions,
                                pos_table=pos_table, scale=scale)
    return ref.embedding(ids, table, vocab_lo, vocab_hi, positions, pos_table, scale)


def gather_rows(x, idx):
    if x.is_cuda:
        return native.gather_rows(x, idx)
    return x[idx.long()]


def add(a, b=None, bias=None):
    if a.is_cuda:
        return native.add(a, b, bias)
    y = a.float()
    if b is not None:
        y = y + b.float()
    if bias is not None:
        y = y + bias.float()
    return y.to(a.dtype)


def rope_kv_append(qkv, positions, slots, cos_sin, cache_layer, block_tokens, Hq, Hkv, D, rot_dim, neox=True,
                   mrope_sections=None, k_scale=1.0, v_scale=1.0, apply_rope=True):
    if qkv.is_cuda:
        native.rope_kv_append(qkv, positions, slots, cos_sin, cache_layer,
                              cache_layer.stride(0) if cache_layer is not None else 0, block_tokens, Hq, Hkv, D,
                              rot_dim, neox, mrope_sections, k_scale, v_scale, apply_rope)
    else:
        ref.rope_kv_append(qkv, positions, slots, cos_sin, cache_layer, block_tokens, Hq, Hkv, D, rot_dim, neox,
                           mrope_sections, k_scale, v_scale, apply_rope)


# ------------------------------------------------------------------------------- 32-bit residual stream
@dataclass
class NormParams:
    """Weight and optional bias of a norm over ``size`` real columns (stored padded with zeros to a multiple of 8).
    ``groups`` > 1: root-mean-square norm of each of that many parts of equal size."""
    w: torch.Tensor
    b: Optional[torch.Tensor]
    size: int
    eps: float
    rms: bool = False
    groups: int = 1


def embed_pair(ids, prev, table, pair, scale, buckets=0, mul_prev=0, mul_cur=0, copy=None, vocab=None):
    """fp32 rows: scaled token embedding plus, with a ``pair`` table, the row (prev * mul_prev + id * mul_cur) mod buckets
    of it (row ``buckets`` where prev < 0: the first token of a sequence). ``copy`` receives the rows in the table's type."""
    if table.is_cuda:
        return native.embed_pair(ids, prev, table, pair, scale, buckets, mul_prev, mul_cur, copy, vocab)
    x = ref.embed_pair(ids, prev, table, pair, scale, buckets, mul_prev, mul_cur)
    if copy is not None:
        copy.copy_(x)
    return x


@dataclass
class ExpertSum:
    """A sublayer's result that is still spread over expert outputs: row t is the sum over k of w[t, k] * y[dst_row[t, k]]
    (negative rows: left out), plus w[t, K] * shared[t], or plus shared[t] where w has K columns."""
    y: torch.Tensor
    dst_row: torch.Tensor                 # [T, K] int32
    w: torch.Tensor                       # [T, K] or [T, K + 1] fp32
    shared: Optional[torch.Tensor] = None

    @property
    def dtype(self):
        return self.y.dtype


def stream_norm(x, norm: NormParams, dtype, rows=None, scale=1.0):
    """norm of the fp32 residual stream (of its ``rows``) times ``scale`` as the next linear's operand."""
    if x.is_cuda:
        z = torch.empty(rows.numel() if rows is not None else x.shape[0], x.shape[1], dtype=dtype, device=x.device)
        native.residual_norm(x, norm.size, norm.eps, w2=norm.w, b2=norm.b, z=z, rows=rows, rms=norm.rms,
                             groups=norm.groups, z_scale=scale)
        return z
    return (ref.stream_norm(x[rows.long()] if rows is not None else x, norm) * scale).to(dtype)


def stream_enter(x, add, vec, then: NormParams, dtype, inplace=True):
    """x + add + vec (fp32 rows or None, one row) and the following norm of the sum: (x, normed)."""
    if x.is_cuda:
        z = torch.empty(x.shape, dtype=dtype, device=x.device)
        out = x if inplace else torch.empty_like(x)
        native.residual_norm(x, then.size, then.eps, x_out=out, w2=then.w, b2=then.b, z=z, rms=then.rms, groups=then.groups, add=add,
                             vec=vec)
        return out, z
    out = x + vec.float() if add is None else x + add + vec.float()
    if inplace:
        out = x.copy_(out)
    return out, ref.stream_norm(out, then).to(dtype)


def stream_copy(x, out):
    """The fp32 stream's rows in the type of ``out`` (a strided view is fine)."""
    if x.is_cuda:
        native.residual_norm(x, x.shape[1], 0.0, z=out)
    else:
        out.copy_(x)


def stream_add(x, y, post: Optional[NormParams], scale, then: Optional[NormParams] = None, copy=None, inplace=True, alpha=1.0,
               add=None, vec=None):
    """x + alpha * scale * norm(y; post) + add + vec (``scale``: per column, ``alpha``: one number, ``add``: fp32 rows, ``vec``: one
    row) on the fp32 residual stream, fused with what reads the sum next: ``then`` (the following norm, returned in y's type) or
    ``copy`` (a buffer that receives the sum in its own type). ``y`` may be an :class:`ExpertSum`. Returns (x, normed or None);
    ``inplace`` updates x."""
    if x.is_cuda:
        experts = (y.dst_row, y.w, y.shared) if isinstance(y, ExpertSum) else None
        z = torch.empty(x.shape, dtype=y.dtype, device=x.device) if then is not None else copy
        out = x if inplace else torch.empty_like(x)
        size, eps, rms = (post.size, post.eps, post.rms) if post is not None else (
            (then.size, then.eps, then.rms) if then is not None else (x.shape[1], 0.0, False))
        native.residual_norm(x, size, eps, y=y.y if experts else y, w1=post.w if post else None, b1=post.b if post else None, ls=scale,
                             x_out=out, w2=then.w if then else None, b2=then.b if then else None, z=z, rms=rms, alpha=alpha,
                             groups=then.groups if then else 1, add=add, vec=vec, experts=experts)
        return out, (z if then is not None else None)
    dtype = y.dtype
    if isinstance(y, ExpertSum):
        y = ref.expert_sum(y.y, y.dst_row, y.w, y.shared)
    a = ref.stream_norm(y, post) if post is not None else y.float()
    if scale is not None:
        a = a * scale.float()
    if alpha != 1.0:
        a = a * alpha
    if add is not None:
        a = a + add
    if vec is not None:
        a = a + vec.float()
    out = x.add_(a) if inplace else x + a
    if copy is not None:
        copy.copy_(out)
    return out, (ref.stream_norm(out, then).to(dtype) if then is not None else None)


def embed_normed(ids, positions, table, pos_table, scale, norm: NormParams, vocab):
    """fp32 rows norm(table[id] * scale + pos_table[position]) (root mean square)."""
    if table.is_cuda:
        return native.embed_normed(ids, positions, table, pos_table, norm.w, norm.size, scale, norm.eps, vocab)
    return ref.stream_norm(table[ids.long()].float() * scale + pos_table[positions.long()].float(), norm)


def token_shift(h, mu, ring, step):
    """h_t + (h_(t-1) - h_t) * mu over a step's rows; ``ring`` [slots, 2, W]: the last rows of earlier steps (position p in row p
    mod 2)."""
    if h.is_cuda:
        return native.token_shift(h, mu, ring, step.cu_q, step.kv_lens, step.state_slots, max(step.max_q_len, 1))
    return ref.token_shift(h, mu, ring, step.cu_q, step.kv_lens, step.state_slots)


def gated_norm(y, w, eps, heads, real, parts, z=None, g=None, factor=1.0, out=None):
    """factor * norm(y * silu(z)) * w * sigmoid(g), the root mean square taken over each of ``parts`` equal parts of a row of
    ``heads`` heads of ``real`` columns (padded to y's width)."""
    if y.is_cuda:
        return native.gated_norm(y, w, y.shape[1] // heads, real, parts, eps, z, g, factor, out)
    v = ref.gated_norm(y, w, y.shape[1] // heads, real, parts, eps, z, g, factor)
    return v if out is None else out.copy_(v)


def panel_append(k, step, cache, block_tokens):
    """Columns k [T, heads * size] of a projection into the paged panel ``cache`` [blocks, heads, block tokens, size]."""
    if k.is_cuda:
        return native.panel_append(k, step.slots, cache, block_tokens)
    on = step.slots >= 0
    slots = step.slots[on].long()
    cache[slots // block_tokens, :, slots % block_tokens] = k[on].unflatten(1, (cache.shape[1], -1))


def softcap(z, cap):
    """cap * tanh(z / cap); fp32 rows are overwritten on the GPU."""
    return native.softcap(z, cap) if z.is_cuda else cap * torch.tanh(z / cap)


@dataclass
class ShortConv:
    """Causal convolution per channel with the inputs that earlier steps left: ``w`` [taps, C] (the last row is the current
    token's), ``ring`` [slots, taps, C] inside the state records (the input of position p in row p mod taps)."""
    w: torch.Tensor
    bias: Optional[torch.Tensor]
    ring: torch.Tensor


def _recurrence(x, conv: ShortConv, step, run):
    """Several-token sequences of a step (convolution, then scan), then its single-token ones (one fused step): ``run`` gets the
    rows' range, the convolved rows or None, and cu_q, kv_lens and state slots of its sequences."""
    nm, tm = step.num_multi, step.num_multi_tokens
    if nm:
        cu, kv, slots = step.cu_q[:nm + 1], step.kv_lens[:nm], step.state_slots[:nm]
        run(slice(0, tm), native.causal_conv(x[:tm], conv, cu, kv, slots, step.max_q_len), cu, kv, slots)
    if step.num_single:
        run(slice(tm, None), None, None, step.kv_lens[nm:], step.state_slots[nm:])


def state_space(x, conv: ShortConv, dt, dt_bias, A, D, state, groups, step):
    """y_t = S_t^T C_t + D x_t with S_t = exp(-A dt_t) S_(t-1) + dt_t B_t x_t^T per head, dt = softplus(dt + dt_bias), over a
    step's rows. x [T, heads * P + 2 * groups * N]: raw x | B | C, which pass the short convolution and silu first. ``state``
    [slots, heads, P, N] (fp32)."""
    n, H, P, N = state.shape
    y = torch.empty(x.shape[0], H * P, dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        return y.copy_(ref.state_space(x, conv, dt, dt_bias, A, D, state, groups, step))
    _recurrence(x, conv, step, lambda r, c, cu, kv, slots: native.state_space(
        x[r], conv, c, dt[r], dt_bias, A, D, y[r], state, groups, cu, kv, slots))
    return y


def delta_rule(x, conv: ShortConv, beta, decay, decay_bias, A, state, groups, q_scale, step):
    """Gated delta rule over a step's rows: per head S' = diag(g) S, u = beta (v - S'^T k), S = S' + k u^T, o = S^T q, with q and k
    unit vectors (q times ``q_scale``), beta = sigmoid(beta) and g = exp(-A softplus(decay + decay_bias)) per key channel. x [T,
    2 * groups * K + heads * V]: raw q | k | v, which pass the short convolution and silu first. ``state`` [slots, heads, V, K]."""
    n, H, V, _ = state.shape
    o = torch.empty(x.shape[0], H * V, dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        return o.copy_(ref.delta_rule(x, conv, beta, decay, decay_bias, A, state, groups, q_scale, step))
    _recurrence(x, conv, step, lambda r, c, cu, kv, slots: native.delta_rule(
        x[r], conv, c, beta[r], decay[r], decay_bias, A, o[r], state, groups, q_scale, cu, kv, slots))
    return o


def glu_clamp(x, limit, alpha=1.702, offset=1.0):
    """min(gate, limit) * sigmoid(alpha * gate) * (clamp(up, -limit, limit) + offset) of packed gate | up columns."""
    if x.is_cuda:
        return native.glu_clamp(x, limit, alpha, offset)
    return ref.glu_clamp(x, limit, alpha, offset)


def xielu(x, pos, neg, lin=0.5):
    """pos x^2 + lin x above zero, neg (exp(x) - 1 - x) + lin x below."""
    return native.xielu(x, pos, neg, lin) if x.is_cuda else ref.xielu(x, pos, neg, lin)


def gated_recurrence(y, W, state, block_tokens, step, offset=0.5):
    """S_t = (1 - gate) S_(t-1) + gate * cand with gate = sigmoid(z) and cand = u + offset (u >= 0) or sigmoid(u), out =
    S_t * silu(g), over a step's new rows; y [T, 3 W] holds z | u | g. ``state`` [blocks, W] (fp32, part of the cache's
    block records): a block's row is the state after the last of its tokens computed so far."""
    z, u, g = y[:, :W], y[:, W:2 * W], y[:, 2 * W:]
    if not y.is_cuda:
        return ref.gated_recurrence(z, u, g, state, block_tokens, step.block_table, step.cu_q, step.kv_lens, offset)
    out = torch.empty(y.shape[0], W, dtype=y.dtype, device=y.device)
    nm, ns, tm = step.num_multi, step.num_single, step.num_multi_tokens
    if nm:
        native.gated_recurrence(z, u, g, out, state, block_tokens, step.block_table, step.cu_q, step.kv_lens[:nm], offset)
    if ns:
        native.gated_recurrence(z[tm:], u[tm:], g[tm:], out[tm:], state, block_tokens, step.block_table[nm:], None,
                                step.kv_lens[nm:], offset, slots=step.slots[tm:])
    return out


# ------------------------------------------------------------------------------- latent attention
def bmm(a, w, out, gate=None):
    """out[b] = a[b] w[b]^T (times sigmoid(gate[b])) over (strided) views a [B, M, K], w [B, N, K], out and gate [B, M, N]."""
    if not a.is_cuda:
        y = torch.matmul(a.float(), w.float().transpose(1, 2))
        return out.copy_(y if gate is None else y * torch.sigmoid(gate.float()))
    return (native.gemm_f32_batched if a.dtype == torch.float32 else native.gemm_bf16_batched)(a, w, out, gate)


def latent_append(q, nope, kv, norm: Optional[NormParams], step, cos_sin, cache, block_tokens):
    """Packed query rows [T, G, DK] whose rotary columns (the last ones) are filled with the rotated queries' (q: [T, G, nope
    + rotary], rows may be part of wider ones), and the append of the normed latents and the rotated key of ``kv`` [T, DK]
    to the panel ``cache`` [blocks, block tokens, DK]. ``kv`` None: the latents are another layer's, nothing is appended."""
    T, G = q.shape[:2]
    qfull = torch.empty(T, G, cache.shape[2], dtype=q.dtype, device=q.device)
    w, eps, rank = (norm.w, norm.eps, norm.size) if kv is not None else (None, 0.0, cache.shape[2] - (q.shape[2] - nope))
    if q.is_cuda:
        native.mla_rope_append(q, nope, kv, w, eps, step.positions, step.slots, cos_sin, qfull, cache, block_tokens, G, rank)
    else:
        ref.latent_append(q, nope, kv, w, eps, rank, step.positions, step.slots, cos_sin, qfull, cache, block_tokens)
    return qfull


def latent_norms(q, kv, q_norm: NormParams, kv_norm: NormParams, step, cache, block_tokens):
    """Normed query latents, and the append of the normed key/value latents to the panel ``cache`` [blocks, block tokens, rank];
    q, kv: column ranges of one projection's rows."""
    fn = native.latent_norms if q.is_cuda else ref.latent_norms
    return fn(q, kv, q_norm.w, kv_norm.w, q_norm.eps, q_norm.size, kv_norm.size, step.slots, cache, block_tokens)


def latent_attention(qfull, cache, dv, block_tokens, step, scale, window=0, sinks=None, gate=None):
    """Absorbed attention of packed query rows [T, G, DK] against the latent panel [blocks, block tokens, DK], values = the
    first ``dv`` columns of its rows: [T, G, dv]. ``sinks`` [G]: logits in the denominator only, ``gate`` [T, G]: a head's output
    is multiplied by its sigmoid. The tensor-core kernel serves bf16 rows up to 576 / 512 columns over
    blocks of 8 to 256 (a power of two) tokens, the 32-bit one the rest."""
    T, G, dk = qfull.shape
    if not qfull.is_cuda:
        return ref.mla_attention(qfull, cache, step.block_table, step.cu_q, step.kv_lens, scale, dv, window, sinks, gate).to(qfull.dtype)
    out = torch.empty(T, G, dv, dtype=qfull.dtype, device=qfull.device)
    B, mq = step.num_multi + step.num_single, max(step.max_q_len, 1)
    if qfull.dtype == torch.bfloat16:
        seen = min(step.max_kv_len, window + 64) if window > 0 else step.max_kv_len
        n = native.mla_splits(B, mq, seen, halves=(dv + 255) // 256) if step.num_multi == 0 else 1
        if native.mla_attention(qfull, out, cache, block_tokens, step.block_table, step.cu_q, step.kv_lens, B, mq, scale, n, window,
                                sinks, gate):
            return out
    panel = cache.unsqueeze(1)                           # one key/value head shared by all query heads
    native.attention_f32(qfull, G * dk, out.view(T, G * dv), panel, panel[..., :dv], block_tokens, step.block_table, step.cu_q,
                         step.kv_lens, B, mq, G, 1, scale, window, sinks=sinks, gate=gate)
    return out


def qkv_rope_append(qkv, positions, slots, cos_sin, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim):
    """Partial rotation of q and k and append of k, v to separate paged panels (key and value sizes may differ)."""
    fn = native.qkv_rope_append if qkv.is_cuda else ref.qkv_rope_append
    fn(qkv, positions, slots, cos_sin, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim)


def qkv_norm_rope_append(qkv, step, cos_sin, q_norm: NormParams, k_norm: NormParams, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim,
                         sums=None):
    """Norms over all of q and all of k, partial rotation of neighbouring pairs, append of k and v to paged panels. ``sums`` [T, 2]:
    sums of squares of the whole rows where ``qkv`` holds this rank's heads only (the norms' sizes are those of the whole)."""
    fn = native.qkv_norm_rope_append if qkv.is_cuda else ref.qkv_norm_rope_append
    fn(qkv, step.positions, step.slots, cos_sin, q_norm.w, k_norm.w, q_norm.eps, q_norm.size, k_norm.size, k_cache, v_cache, block_tokens,
       Hq, Hkv, rot_dim, sums)


def moe_route(logits, K, **kw):
    """(ids [T, K] int32, weights fp32) by rows of router logits; options as in native.moe_route."""
    if logits.is_cuda:
        return native.moe_route(logits, K, **kw)
    ids, w = ref.moe_route(logits, K, **kw)
    return ids.to(torch.int32), w


def refit_stream_rows(x, pos, emb):
    """Rows of the residual stream replaced by given embeddings (real columns only)."""
    if x.is_cuda:
        native.refit_rows_f32(x, pos, emb.contiguous())
    else:
        x[pos.long(), :emb.shape[1]] = emb.float()


def panel_attention(qkv, k_cache, v_cache, block_tokens, step, Hq, Hkv, scale, window=0, keep=0, sinks=None, weights=None, out=None):
    """Attention of a step's new rows (multi-token sequences first, then single-token ones; the queries are the leading columns of
    ``qkv``) against separate K and V panels, with an optional sliding window (``keep`` first tokens stay visible) and per-head
    sink logits, or with the unnormalised ``weights`` of a :class:`SigmoidWeights`."""
    D, Dv = k_cache.shape[-1], v_cache.shape[-1]
    T = qkv.shape[0]
    if out is None:
        out = torch.empty(T, Hq * Dv, dtype=qkv.dtype, device=qkv.device)
    if not qkv.is_cuda:
        out.copy_(ref.panel_attention(qkv[:, :Hq * D], k_cache, v_cache, step.block_table, step.cu_q, step.kv_lens, Hq, Hkv, scale,
                                      window, keep, sinks, weights))
        return out
    if qkv.dtype == torch.float32:
        native.attention_f32(qkv, qkv.stride(0), out, k_cache, v_cache, block_tokens, step.block_table, step.cu_q, step.kv_lens,
                             step.num_multi + step.num_single, max(step.max_q_len, 1), Hq, Hkv, scale, window, keep, sinks, weights=weights)
        return out
    nm, ns, tm = step.num_multi, step.num_single, step.num_multi_tokens
    if nm:
        native.paged_prefill(qkv, qkv.stride(0), out, k_cache, k_cache.stride(0), block_tokens, step.block_table, step.cu_q,
                             step.kv_lens, nm, step.max_q_len, Hq, Hkv, D, scale, v_cache=v_cache, window=window, keep=keep,
                             sinks=sinks, weights=weights)
    if ns:
        seen = min(step.max_kv_len, window + keep + 128) if window > 0 else step.max_kv_len
        # keys that are the values take half of the shared memory
        n = decode_splits(ns, Hkv * ((Hq // Hkv + 15) // 16), seen, ctas_per_sm=4 if k_cache.data_ptr() == v_cache.data_ptr() else 2)
        po = pml = None
        if n > 1:
            po = torch.empty(ns * Hq * n * Dv, dtype=torch.float32, device=qkv.device)
            pml = torch.empty(ns * Hq * n * 2, dtype=torch.float32, device=qkv.device)
        native.paged_decode(qkv[tm:], qkv.stride(0), out[tm:], k_cache, k_cache.stride(0), block_tokens, step.block_table[nm:],
                            step.kv_lens[nm:], ns, Hq, Hkv, D, scale, num_splits=n, part_o=po, part_ml=pml, v_cache=v_cache,
                            window=window, keep=keep, sinks=sinks, weights=weights.rows(tm) if weights is not None else None)
    return out


def decode_splits(batch: int, hkv: int, max_kv_len: int, sms: int = 148, ctas_per_sm: int = 2) -> int:
    """Split-KV factor of the decode attention kernel. One CTA serves one (sequence, kv head, split) and two CTAs
    fit an SM (shared memory), so the time is about waves x (64-token tiles per split + a fixed set-up cost of about
    two tiles); the factor minimising that is chosen, with at least two tiles per split."""
    import os
    forced = int(os.environ.get("KSANA_DECODE_SPLITS", "0"))
    tiles = max(1, (max_kv_len + 63) // 64)
    most = max(1, min(32, tiles // 2))
    if forced > 0:
        return min(forced, most)
    slots = sms * ctas_per_sm
    best, best_cost = 1, None
    for n in range(1, most + 1):
        waves = (batch * hkv * n + slots - 1) // slots
        cost = waves * ((tiles + n - 1) // n + 2)
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return best


def paged_attention(qkv, out, cache_layer, block_tokens, block_table, cu_q, kv_lens, num_multi, num_single,
                    num_multi_tokens, max_q_len, Hq, Hkv, D, scale, alibi=None, k_scale=1.0, v_scale=1.0,
                    num_splits=1, workspace=None, quant_for: Optional[LinearWeight] = None):
    """Attention of this step's new tokens (rows of ``qkv``: multi-token sequences first, then one row per
    single-token sequence) against the paged cache, which already holds their K/V. ``out`` None allocates the
    result; with ``quant_for`` (the FP8 linear that consumes it) a pure decode step returns the QTensor that linear
    wants, quantised inside the attention kernels."""
    T = qkv.shape[0]
    if qkv.is_cuda and quant_for is not None and quant_for.fp8 and num_multi == 0 and num_single and D == 128 and out is None:
        po, pml = workspace if workspace is not None else (None, None)
        if num_splits > 1 and po is None:
            po = torch.empty(num_single * Hq * num_splits * D, dtype=torch.float32, device=qkv.device)
            pml = torch.empty(num_single * Hq * num_splits * 2, dtype=torch.float32, device=qkv.device)
        oq = torch.empty(T, Hq * D, dtype=torch.float8_e4m3fn, device=qkv.device)
        osc = torch.empty(Hq, max(4, (T + 3) // 4 * 4), dtype=torch.float32, device=qkv.device)
        native.paged_decode(qkv, qkv.stride(0), None, cache_layer, cache_layer.stride(0), block_tokens, block_table,
                            kv_lens, num_single, Hq, Hkv, D, scale, alibi, k_scale, v_scale, num_splits, po, pml,
                            out_q=oq, out_scale=osc)
        return QTensor(oq, osc)
    if out is None:
        out = torch.empty(T, Hq * D, dtype=qkv.dtype, device=qkv.device)
    if qkv.is_cuda:
        if num_multi:
            native.paged_prefill(qkv, qkv.stride(0), out, cache_layer, cache_layer.stride(0), block_tokens, block_table,
                                 cu_q, kv_lens, num_multi, max_q_len, Hq, Hkv, D, scale, alibi, k_scale, v_scale)
        if num_single:
            po, pml = workspace if workspace is not None else (None, None)
            if num_splits > 1 and po is None:
                po = torch.empty(num_single * Hq * num_splits * D, dtype=torch.float32, device=qkv.device)
                pml = torch.empty(num_single * Hq * num_splits * 2, dtype=torch.float32, device=qkv.device)
            native.paged_decode(qkv[num_multi_tokens:], qkv.stride(0), out[num_multi_tokens:], cache_layer,
                                cache_layer.stride(0), block_tokens, block_table[num_multi:], kv_lens[num_multi:],
                                num_single, Hq, Hkv, D, scale, alibi, k_scale, v_scale, num_splits, po, pml)
        return out
    q = qkv[:, : Hq * D]
    o = ref.paged_attention(q, cache_layer, block_table, cu_q, kv_lens, Hq, Hkv, D, scale, alibi, k_scale, v_scale)
    out.copy_(o)
    return out
