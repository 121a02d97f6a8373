"""Rasizen: a pre-norm decoder with a 32-bit residual stream that mixes two kinds of layers: latent attention (absorbed
form) with a sliding window and an output gate, where a layer may read another layer's latents, and a gated recurrence
that is linear in its state (the gates do not see it). Norms take the root mean square of each of several equal parts of a row, the
residual additions have a common factor, the feed-forwards are plain with a piecewise unit, any layer may lack one.

The step functions, the block pool, the scheduler and the sampler are the ones of every other family. A cache block is one
record with, per layer that owns latents, a panel of [latent | rotated key] rows, and per recurrent layer one fp32 row: the
state after the last of the block's tokens that has been computed. Blocks are therefore self-contained: prefix sharing,
forks, swaps and recomputation act on them as on a pure attention model's. Per sublayer:

  attention    [q | latent, rotary key | gate] GEMM -> latent norm + rotations + append -> q W_uk -> attention over the
               latent rows -> W_uv with the output gate in its epilogue -> output GEMM -> [scaled residual add, next norm] in one kernel
  recurrence   [z | x | g] GEMM -> scan with gates, states and output gate in one kernel -> output GEMM -> same kernel
  feed-forward up GEMM -> unit -> down GEMM -> same kernel

Tensor parallelism: attention heads, recurrence channels, feed-forward columns and the vocabulary are split; the latents
and their cache are replicated.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from ..config import GatedRecurrenceSpec, LatentAttentionSpec, LayerSpec, ModelConfig
from ..ops import dispatch as ops
from ..ops.dispatch import LinearWeight, NormParams
from ..utils import nvtx
from .common import RecordLayout, StepInput
from .stream import StreamLoader, StreamModel, pad8, pad_to

CANDIDATE_OFFSET = 0.5            # candidate of the recurrence: u + 1/2 from zero on, sigmoid(u) below
UNIT_LINEAR = 0.5                 # linear part of the feed-forward's unit


@dataclass
class HybridLayer:
    spec: LayerSpec
    norm1: NormParams
    w_in: LinearWeight                         # all projections of the mixer's input, packed by rows
    o_proj: LinearWeight
    heads: int = 0                             # of this rank (attention)
    channels: int = 0                          # of this rank, padded (recurrence)
    latent_norm: Optional[NormParams] = None   # absent where the latents are another layer's
    uk_t: Optional[torch.Tensor] = None        # [heads, rank, dim]: W_uk as the operand of the absorbing product
    uv: Optional[torch.Tensor] = None          # [heads, vdim, rank]
    norm2: Optional[NormParams] = None
    up: Optional[LinearWeight] = None
    down: Optional[LinearWeight] = None
    unit: Optional[tuple] = None               # (quadratic factor above zero, exponential factor below)


class RasizenModel(StreamModel):
    moves_blocks = False

    def __init__(self, cfg: ModelConfig, *a, **kw):
        super().__init__(cfg, *a, **kw)
        self.carries_state = any(isinstance(s.mixer, GatedRecurrenceSpec) for s in cfg.layer_specs)
        self.tables = [self.rotation_table(s.mixer.rotary) if isinstance(s.mixer, LatentAttentionSpec) else None for s in cfg.layer_specs]

    # ------------------------------------------------------------------ cache
    def allocate_kv_cache(self, num_blocks: int, block_tokens: int, dtype=None):
        """[blocks, record]: latent panels [block tokens, latent + rotary] and fp32 state rows, layer by layer."""
        self.check_cache_dtype(dtype)
        self.block_tokens = block_tokens
        self.layout = RecordLayout(self.dtype)
        index = []
        for lw in self.layers:
            m = lw.spec.mixer
            if isinstance(m, GatedRecurrenceSpec):
                index.append(self.layout.add((lw.channels,), torch.float32))
            elif m.kv_from is None:
                index.append(self.layout.add((block_tokens, pad8(m.kv_rank) + pad8(m.rot_dim))))
            else:
                index.append(index[m.kv_from])
        self.kv_cache = torch.zeros(num_blocks, self.layout.record, dtype=self.dtype, device=self.device)
        self.panels = [self.layout.view(self.kv_cache, i) for i in index]
        return self.kv_cache

    # ------------------------------------------------------------------ blocks
    def attention(self, i: int, lw: HybridLayer, xn: torch.Tensor, step: StepInput) -> torch.Tensor:
        m: LatentAttentionSpec = lw.spec.mixer
        T, H, dim, rank = xn.shape[0], lw.heads, pad8(m.dim), pad8(m.kv_rank)
        y = ops.linear(xn, lw.w_in)
        nq, ng = H * (dim + pad8(m.rot_dim)), H * pad8(m.vdim)
        q, g = y[:, :nq].unflatten(1, (H, -1)), y[:, y.shape[1] - ng:]
        kv = y[:, nq:y.shape[1] - ng] if lw.latent_norm is not None else None
        cache = self.panels[i]
        qfull = ops.latent_append(q, dim, kv, lw.latent_norm, step, self.tables[i], cache, self.block_tokens)
        ops.bmm(q[..., :dim].transpose(0, 1), lw.uk_t, qfull[..., :rank].transpose(0, 1))
        o_lat = ops.latent_attention(qfull, cache, rank, self.block_tokens, step, m.scale, m.window)
        o = torch.empty(T, H, pad8(m.vdim), dtype=y.dtype, device=y.device)
        ops.bmm(o_lat.transpose(0, 1), lw.uv, o.transpose(0, 1), gate=g.unflatten(1, (H, -1)).transpose(0, 1))
        return o.view(T, ng)

    def recurrence(self, i: int, lw: HybridLayer, xn: torch.Tensor, step: StepInput) -> torch.Tensor:
        return ops.gated_recurrence(ops.linear(xn, lw.w_in), lw.channels, self.panels[i], self.block_tokens, step, CANDIDATE_OFFSET)

    def mlp(self, lw: HybridLayer, xn: torch.Tensor) -> torch.Tensor:
        return ops.xielu(ops.linear(xn, lw.up), *lw.unit, UNIT_LINEAR)

    def forward_layers(self, step: StepInput, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        x = self.embed_tokens(step)
        xn = ops.stream_norm(x, self.layers[0].norm1, self.dtype)
        alpha = self.cfg.residual_mult
        for i, lw in enumerate(self.layers):
            then = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else None
            mixer = self.recurrence if isinstance(lw.spec.mixer, GatedRecurrenceSpec) else self.attention
            with nvtx.annotate(mixer.__name__):
                y = self.project(mixer(i, lw, xn, step), lw.o_proj)
            x, xn = ops.stream_add(x, y, None, None, lw.norm2 if lw.up is not None else then, alpha=alpha)
            if lw.up is not None:
                with nvtx.annotate("mlp"):
                    y = self.project(self.mlp(lw, xn), lw.down)
                x, xn = ops.stream_add(x, y, None, None, then, alpha=alpha)
            if self.stream_hook is not None:
                self.stream_hook(i, x)
        return x

    def weight_bytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size()
        for lw in self.layers:
            n += sum(w.nbytes() for w in (lw.w_in, lw.o_proj, lw.up, lw.down) if w is not None)
            n += sum(t.numel() * t.element_size() for t in (lw.uk_t, lw.uv) if t is not None)
        return n


# ------------------------------------------------------------------------------------- loading
def _softplus(x: float) -> float:
    return max(x, 0.0) + math.log1p(math.exp(-abs(x)))


def build_rasizen(cfg: ModelConfig, source, tp_rank=0, tp_size=1, comm=None, device="cpu", dtype=torch.bfloat16, quant=None,
                  layer_range=None, max_positions=None) -> RasizenModel:
    if layer_range is not None and tuple(layer_range) != (0, cfg.num_layers - 1):
        raise ValueError("rasizen: layers may read another layer's latents, pipeline stages are not supported")
    for s in cfg.layer_specs:
        if isinstance(s.mixer, LatentAttentionSpec) and s.mixer.heads % tp_size:
            raise ValueError(f"rasizen: {s.mixer.heads} heads cannot be split over {tp_size} ranks")
    m = RasizenModel(cfg, tp_rank, tp_size, comm, device, dtype, max_positions)
    ld = StreamLoader(m, source, quant)
    W, WP = cfg.hidden_size, m.width

    def norm(name, n=W, groups=cfg.norm_groups):
        return NormParams(ld.param(ld.get(name, (n,), "ones"), pad8(n)), None, n, cfg.rms_norm_eps, rms=True, groups=groups)

    ld.vocabulary()
    for i, spec in enumerate(cfg.layer_specs):
        p, a = f"l{i}.", spec.mixer
        x = p + "mix."
        n1 = norm(p + "norm1")
        if isinstance(a, GatedRecurrenceSpec):
            n = ld.shard(a.width)
            z, u, g = (ld.split_rows(x + s, a.width) for s in ("z", "x", "g"))
            bz, bu = (ld.rows(pad_to(ld.get(x + s, (a.width,), "zeros"), n * tp_size)) for s in ("z.b", "x.b"))
            lw = HybridLayer(spec, n1, ld.linear(torch.cat([z, u, g], 0), torch.cat([bz, bu, torch.zeros_like(bz)], 0)),
                             ld.linear(ld.split_cols(x + "o", a.width)), channels=n)
        else:
            H, d, r, v, k = a.heads, pad8(a.dim), pad8(a.rot_dim), pad8(a.vdim), pad8(a.kv_rank)
            q = ld.get(x + "q", (H * (a.dim + a.rot_dim), W)).reshape(H, a.dim + a.rot_dim, W)
            q = torch.cat([pad_to(q[:, :a.dim], H, d, WP), pad_to(q[:, a.dim:], H, r, WP)], 1)
            rows = [ld.rows(q).reshape(-1, WP)]
            latent_norm = None
            if a.kv_from is None:
                dkv = ld.get(x + "dkv", (a.kv_rank + a.rot_dim, W))
                rows += [pad_to(dkv[:a.kv_rank], k, WP), pad_to(dkv[a.kv_rank:], r, WP)]
                latent_norm = norm(x + "dkv.norm", a.kv_rank, 1)
            rows.append(ld.rows(pad_to(ld.get(x + "g", (H * a.vdim, W)).reshape(H, a.vdim, W), H, v, WP)).reshape(-1, WP))
            uk = ld.rows(pad_to(ld.get(x + "uk", (H * a.dim, a.kv_rank)).reshape(H, a.dim, a.kv_rank), H, d, k))
            uv = ld.rows(pad_to(ld.get(x + "uv", (H * a.vdim, a.kv_rank)).reshape(H, a.vdim, a.kv_rank), H, v, k))
            o = ld.cols(pad_to(ld.get(x + "o", (W, H * a.vdim)).reshape(W, H, a.vdim), WP, H, v))
            lw = HybridLayer(spec, n1, ld.linear(torch.cat(rows, 0)), ld.linear(o.reshape(WP, -1)), heads=H // tp_size,
                             latent_norm=latent_norm, uk_t=ld.param(uk.transpose(1, 2), H // tp_size, k, d),
                             uv=ld.param(uv, H // tp_size, v, k))
        if spec.mlp is not None:
            ff = spec.mlp.size
            lw.norm2 = norm(p + "norm2")
            lw.up, lw.down = ld.linear(ld.split_rows(p + "mlp.up", ff)), ld.linear(ld.split_cols(p + "mlp.down", ff))
            above, below = (float(t) for t in ld.get(p + "mlp.act", (2,)).float().cpu())
            lw.unit = (_softplus(above), UNIT_LINEAR + _softplus(below))
        m.layers.append(lw)
    m.final = norm("final.norm")
    return m
