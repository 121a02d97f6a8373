"""Lenolix: a decoder with a 32-bit residual stream and norms on both sides of every sublayer, a hashed embedding of
token pairs, sliding-window attention with kept first tokens and per-head sink logits, clamped gated feed-forwards,
layer scale, and a run of layers that is repeated with the same weights (a cache per pass) and re-fed with the
embedding output before every pass.

The step functions, the paged cache, the scheduler and the sampler are the ones of every other family; this file
describes the layers in terms of the shared ops. Per sublayer:

  norm (fused into the previous sublayer's add) -> QKV GEMM -> rotation + paged append -> attention -> output GEMM
  -> [norm, layer scale, residual add, next norm] in one kernel -> gate|up GEMM -> clamped unit -> down GEMM -> same kernel

The residual stream, the padding of odd sizes and the loading helpers are those of models/stream.py. Tensor parallelism:
query and key/value heads, feed-forward columns and the vocabulary are split; the partial sums of the output and down
projections are added across ranks before the norm that follows them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..config import AttentionSpec, LayerSpec, ModelConfig
from ..ops import dispatch as ops
from ..ops.dispatch import LinearWeight, NormParams
from ..utils import nvtx
from .common import PanelLayout, StepInput
from .stream import LayerRun, StreamLoader, StreamModel, layer_runs, pad8, pad_to, rerotate_panel

MAX_HEAD = 256                    # largest head size of the attention kernels


@dataclass
class SandwichLayer:
    spec: LayerSpec
    heads: int                    # of this rank
    kv_heads: int
    norm1: NormParams
    norm1b: NormParams
    qkv: LinearWeight
    o_proj: LinearWeight
    sinks: Optional[torch.Tensor]
    ls1: torch.Tensor
    norm2: Optional[NormParams] = None
    norm2b: Optional[NormParams] = None
    ls2: Optional[torch.Tensor] = None
    gate_up: Optional[LinearWeight] = None
    down: Optional[LinearWeight] = None
    moe: Optional[object] = None


class LenolixModel(StreamModel):
    def __init__(self, cfg: ModelConfig, *a, **kw):
        super().__init__(cfg, *a, **kw)
        self.needs_prev_ids = cfg.pair_embedding is not None
        self.runs = layer_runs(cfg)
        self.pair: Optional[torch.Tensor] = None
        self.loop_in: List[LinearWeight] = []            # one per pass: shared weight, the pass's step vector as bias
        self.rotary = {i: self.rotation_table(s.mixer.rotary) for i, s in enumerate(cfg.layer_specs) if s.mixer.rotary is not None}

    # ------------------------------------------------------------------ KV cache
    def allocate_kv_cache(self, num_blocks: int, block_tokens: int, dtype=None):
        """[blocks, record]: the K and V panels of every layer run, one after the other (sizes differ by layer)."""
        self.check_cache_dtype(dtype)
        self.block_tokens = block_tokens
        shapes = []
        for run in self.runs:
            m, lw = self.cfg.layer_specs[run.layer].mixer, self.layers[run.layer]
            shapes.append((lw.kv_heads, pad8(m.dim), pad8(m.vdim)))
        self.layout = PanelLayout(shapes, block_tokens)
        self.kv_cache = torch.zeros(num_blocks, self.layout.record, dtype=self.dtype, device=self.device)
        self.panels = [self.layout.views(self.kv_cache, i) for i in range(len(self.runs))]
        return self.kv_cache

    def rerotate_blocks(self, triples) -> None:
        """Copies that landed at another position (flexible cache): every run's keys are turned by the position delta."""
        for run, (k, _) in zip(self.runs, self.panels):
            table = self.rotary.get(run.layer)
            if table is not None:
                rerotate_panel(k, triples, table)

    # ------------------------------------------------------------------ blocks
    def embed_tokens(self, step: StepInput, copy=None) -> torch.Tensor:
        p = self.cfg.pair_embedding
        return super().embed_tokens(step, copy, self.pair, (p.buckets, p.mul_prev, p.mul_cur) if p is not None else (0, 0, 0))

    def attention(self, run: LayerRun, lw: SandwichLayer, xn: torch.Tensor, step: StepInput) -> torch.Tensor:
        m: AttentionSpec = lw.spec.mixer
        k, v = self.panels[run.cache]
        table = self.rotary.get(run.layer)
        qkv = ops.linear(xn, lw.qkv)
        ops.qkv_rope_append(qkv, step.positions, step.slots, table, k, v, self.block_tokens, lw.heads, lw.kv_heads,
                            m.rotary.dims if m.rotary is not None else 0)
        return ops.panel_attention(qkv, k, v, self.block_tokens, step, lw.heads, lw.kv_heads, m.scale, m.window, m.keep_first,
                                   lw.sinks)

    def mlp(self, lw: SandwichLayer, xn: torch.Tensor) -> torch.Tensor:
        s = lw.spec.mlp
        return ops.glu_clamp(ops.linear(xn, lw.gate_up), s.limit, s.alpha, s.offset)

    def forward_layers(self, step: StepInput, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        T, W = step.input_ids.shape[0], self.width
        # operand of the loop's entry projection: [stream | embedding output]
        pair = torch.empty(T, 2 * W, dtype=self.dtype, device=self.device) if self.loop_in else None
        x = self.embed_tokens(step, copy=pair[:, W:] if pair is not None else None)
        xn = None                                        # the stream after the next sublayer's norm, once computed
        for r, run in enumerate(self.runs):
            lw = self.layers[run.layer]
            if run.enter is not None:
                if r == 0:
                    ops.stream_copy(x, pair[:, :W])
                x = ops.linear(pair, self.loop_in[run.enter], out_f32=True)
                xn = None
            if xn is None:
                xn = ops.stream_norm(x, lw.norm1, self.dtype)
            nxt = self.runs[r + 1] if r + 1 < len(self.runs) else None
            copy = pair[:, :W] if nxt is not None and nxt.enter is not None else None
            then = self.layers[nxt.layer].norm1 if nxt is not None and copy is None else None
            with nvtx.annotate("attention"):
                y = self.project(self.attention(run, lw, xn, step), lw.o_proj)
            if lw.gate_up is None:                       # a layer without a feed-forward
                x, xn = ops.stream_add(x, y, lw.norm1b, lw.ls1, then, copy)
            else:
                x, xn = ops.stream_add(x, y, lw.norm1b, lw.ls1, lw.norm2)
                with nvtx.annotate("mlp"):
                    y = self.project(self.mlp(lw, xn), lw.down)
                x, xn = ops.stream_add(x, y, lw.norm2b, lw.ls2, then, copy)
            if self.stream_hook is not None:
                self.stream_hook(r, x)
        return x

    def weight_bytes(self) -> int:
        extra = [t for t in (self.pair, self.loop_in[0].w if self.loop_in else None) if t is not None]
        return super().weight_bytes() + sum(t.numel() * t.element_size() for t in extra)


# ------------------------------------------------------------------------------------- loading
def build_lenolix(cfg: ModelConfig, source, tp_rank=0, tp_size=1, comm=None, device="cpu", dtype=torch.bfloat16, quant=None,
                  layer_range=None, max_positions=None) -> LenolixModel:
    if layer_range is not None and tuple(layer_range) != (0, cfg.num_layers - 1):
        raise ValueError("lenolix: repeated layers need the embedding output, pipeline stages are not supported")
    for s in cfg.layer_specs:
        if s.mixer.heads % tp_size or (s.mixer.kv_heads % tp_size and tp_size % s.mixer.kv_heads):
            raise ValueError(f"lenolix: {s.mixer.heads} / {s.mixer.kv_heads} heads cannot be split over {tp_size} ranks")
        if torch.device(device).type == "cuda" and max(s.mixer.dim, s.mixer.vdim) > MAX_HEAD:
            raise ValueError(f"lenolix: head sizes above {MAX_HEAD} are not supported")
    m = LenolixModel(cfg, tp_rank, tp_size, comm, device, dtype, max_positions)
    ld = StreamLoader(m, source, quant)
    get, param, linear, rows, cols = ld.get, ld.param, ld.linear, ld.rows, ld.cols
    W, WP = cfg.hidden_size, m.width

    def norm(name):
        return NormParams(param(get(name, (W,), "ones"), WP), param(get(name + ".b", (W,), "zeros"), WP), W, cfg.rms_norm_eps)

    ld.vocabulary()
    if cfg.pair_embedding is not None:
        m.pair = param(get("bigram", (cfg.pair_embedding.buckets + 1, W)), cfg.pair_embedding.buckets + 1, WP)
    if cfg.loop is not None:
        w_in = param(pad_to(get("loop.in", (W, 2 * W)).reshape(W, 2, W), WP, 2, WP).reshape(WP, 2 * WP))
        steps = param(get("loop.step", (cfg.loop.times, W)), cfg.loop.times, WP)
        m.loop_in = [LinearWeight(w=w_in, bias=steps[t]) for t in range(cfg.loop.times)]
    for i, spec in enumerate(cfg.layer_specs):
        p, a = f"l{i}.", spec.mixer
        D, DV = pad8(a.dim), pad8(a.vdim)
        q = rows(pad_to(get(p + "mix.q", (a.heads * a.dim, W)).reshape(a.heads, a.dim, W), a.heads, D, WP))
        k = ld.kv_heads(pad_to(get(p + "mix.k", (a.kv_heads * a.dim, W)).reshape(a.kv_heads, a.dim, W), a.kv_heads, D, WP))
        v = ld.kv_heads(pad_to(get(p + "mix.v", (a.kv_heads * a.vdim, W)).reshape(a.kv_heads, a.vdim, W), a.kv_heads, DV, WP))
        o = cols(pad_to(get(p + "mix.o", (W, a.heads * a.vdim)).reshape(W, a.heads, a.vdim), WP, a.heads, DV))
        sinks = get(p + "mix.sink", (a.heads,))[tp_rank * q.shape[0]:(tp_rank + 1) * q.shape[0]] if a.sink else None
        lw = SandwichLayer(spec, q.shape[0], k.shape[0], norm(p + "norm1"), norm(p + "norm1b"),
                           linear(torch.cat([t.reshape(-1, WP) for t in (q, k, v)], 0)), linear(o.reshape(WP, -1)),
                           sinks.to(device=device, dtype=torch.float32).contiguous() if sinks is not None else None,
                           param(get(p + "ls1", (W,), "ones"), WP))
        if spec.mlp is not None:
            gate, up = (ld.split_rows(p + "mlp." + s, spec.mlp.size) for s in ("gate", "up"))
            down = ld.split_cols(p + "mlp.down", spec.mlp.size)
            lw.norm2, lw.norm2b, lw.ls2 = norm(p + "norm2"), norm(p + "norm2b"), param(get(p + "ls2", (W,), "ones"), WP)
            lw.gate_up, lw.down = linear(torch.cat([gate, up], 0)), linear(down)
        m.layers.append(lw)
    m.final = norm("final.norm")
    return m
