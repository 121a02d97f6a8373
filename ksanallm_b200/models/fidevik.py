"""Fidevik: a pre-norm decoder with a 32-bit residual stream and two kinds of mixer, in any order: grouped-query attention
whose queries and keys are normed over the whole projection and partly rotated (neighbouring pairs), and latent attention
without positions, with normed query and key/value latents, a sink logit and an output gate per head. A layer's feed-forward is
dense, a mixture of experts with grouped sigmoid routing and a gated shared expert, or absent. A run of layers repeats with
the same weights (a cache per pass); a step vector, and from the second pass on the embedding output, is added to the stream
before each pass.

The step functions, the block pool, the scheduler and the sampler are the ones of every other family. A cache block is one
record with a K and a V panel per run of an attention layer and a panel of latent rows per run of a latent one. Per sublayer:

  attention         QKV GEMM -> norms + rotation + paged append -> attention -> output GEMM -> [add, next norm] in one kernel
  latent attention  [query latent | latent | gate] GEMM -> both norms + paged append -> query GEMM -> q W_uk -> attention over
                    the latent rows (sink and gate in its epilogue) -> W_uv -> output GEMM -> same kernel
  dense             gate|up GEMM -> unit -> down GEMM -> same kernel
  experts           [router | shared gate] GEMM (fp32 result) -> choice -> grouped GEMMs; shared expert -> the weighted sum of the
                    experts' and the shared expert's outputs inside the same kernel

The additions in front of a pass ride in the kernel that ends the sublayer before it. Tensor parallelism: heads, feed-forward
and expert columns and the vocabulary are split, latents and their cache are replicated; the sums of squares of queries and
keys are added over the ranks.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..config import AttentionSpec, LatentAttentionSpec, LayerSpec, ModelConfig, MoeSpec
from ..ops import dispatch as ops
from ..ops.dispatch import ExpertSum, LinearWeight, NormParams
from ..utils import nvtx
from .common import RecordLayout, StepInput
from .moe import expert_outputs
from .stream import LayerRun, StreamLoader, StreamModel, layer_runs, pad8, pad_to, rerotate_panel

MAX_HEAD = 256                    # largest head size of the attention kernels


@dataclass
class ExpertWeights:
    router: LinearWeight                       # router rows, then the shared expert's gate
    correction: torch.Tensor                   # [E] fp32
    w13: torch.Tensor                          # [E * 2I, W]: gate rows, then up rows of every expert
    w2: torch.Tensor                           # [E * W, I]
    inter: int
    shared_gate_up: Optional[LinearWeight] = None
    shared_down: Optional[LinearWeight] = None

    def nbytes(self) -> int:
        n = sum(t.numel() * t.element_size() for t in (self.correction, self.w13, self.w2))
        return n + sum(w.nbytes() for w in (self.router, self.shared_gate_up, self.shared_down) if w is not None)


@dataclass
class MixedLayer:
    spec: LayerSpec
    norm1: NormParams
    w_in: LinearWeight                         # all projections of the mixer's input, packed by rows
    o_proj: LinearWeight
    heads: int                                 # of this rank
    kv_heads: int = 0
    q_norm: Optional[NormParams] = None        # of the whole query projection, or of the query latent
    k_norm: Optional[NormParams] = None        # of the whole key projection, or of the key/value latent
    uq: Optional[LinearWeight] = None
    uk_t: Optional[torch.Tensor] = None        # [heads, rank, dim]: W_uk as the operand of the absorbing product
    uv: Optional[torch.Tensor] = None          # [heads, vdim, rank]
    sinks: Optional[torch.Tensor] = None       # [heads] fp32
    norm2: Optional[NormParams] = None
    gate_up: Optional[LinearWeight] = None
    down: Optional[LinearWeight] = None
    experts: Optional[ExpertWeights] = None


class FidevikModel(StreamModel):
    def __init__(self, cfg: ModelConfig, *a, **kw):
        super().__init__(cfg, *a, **kw)
        self.runs = layer_runs(cfg)
        self.pass_steps: Optional[torch.Tensor] = None       # [passes, width]
        self.rotary = {i: self.rotation_table(s.mixer.rotary) for i, s in enumerate(cfg.layer_specs) if s.mixer.rotary is not None}

    # ------------------------------------------------------------------ cache
    def allocate_kv_cache(self, num_blocks: int, block_tokens: int, dtype=None):
        """[blocks, record]: the panels of every layer run, one after the other."""
        self.check_cache_dtype(dtype)
        self.block_tokens = block_tokens
        self.layout = RecordLayout(self.dtype)
        index = []
        for run in self.runs:
            lw = self.layers[run.layer]
            m = lw.spec.mixer
            if isinstance(m, LatentAttentionSpec):
                index.append((self.layout.add((block_tokens, pad8(m.kv_rank))),))
            else:
                index.append(tuple(self.layout.add((lw.kv_heads, block_tokens, pad8(n))) for n in (m.dim, m.vdim)))
        self.kv_cache = torch.zeros(num_blocks, self.layout.record, dtype=self.dtype, device=self.device)
        self.panels = [tuple(self.layout.view(self.kv_cache, i) for i in group) for group in index]
        return self.kv_cache

    def rerotate_blocks(self, triples) -> None:
        """Copies that landed at another position (flexible cache): rotated keys are turned, latents have no position."""
        for run, panels in zip(self.runs, self.panels):
            table = self.rotary.get(run.layer)
            if table is not None:
                rerotate_panel(panels[0], triples, table, interleaved=True)

    # ------------------------------------------------------------------ blocks
    def attention(self, run: LayerRun, lw: MixedLayer, xn: torch.Tensor, step: StepInput) -> torch.Tensor:
        m: AttentionSpec = lw.spec.mixer
        k, v = self.panels[run.cache]
        qkv = ops.linear(xn, lw.w_in)
        ops.qkv_norm_rope_append(qkv, step, self.rotary.get(run.layer), lw.q_norm, lw.k_norm, k, v, self.block_tokens, lw.heads, lw.kv_heads,
                                 m.rotary.dims if m.rotary is not None else 0, self._square_sums(qkv, lw, m) if self.tp_size > 1 else None)
        return ops.panel_attention(qkv, k, v, self.block_tokens, step, lw.heads, lw.kv_heads, m.scale)

    def _square_sums(self, qkv: torch.Tensor, lw: MixedLayer, m: AttentionSpec) -> torch.Tensor:
        """Sums of squares of the whole q and k rows, of which this rank holds some heads (key heads may be on several ranks)."""
        D = pad8(m.dim)
        nq, nk = lw.heads * D, lw.kv_heads * D
        copies = lw.kv_heads * self.tp_size // m.kv_heads
        parts = [qkv[:, :nq].float().pow(2).sum(1), qkv[:, nq:nq + nk].float().pow(2).sum(1) / copies]
        return self.comm.all_reduce(torch.stack(parts, 1).contiguous())

    def latent_attention(self, run: LayerRun, lw: MixedLayer, xn: torch.Tensor, step: StepInput) -> torch.Tensor:
        m: LatentAttentionSpec = lw.spec.mixer
        T, H, rank, nq = xn.shape[0], lw.heads, pad8(m.kv_rank), pad8(m.q_rank)
        cache, = self.panels[run.cache]
        y = ops.linear(xn, lw.w_in)
        c_q = ops.latent_norms(y[:, :nq], y[:, nq:nq + rank], lw.q_norm, lw.k_norm, step, cache, self.block_tokens)
        q = ops.linear(c_q, lw.uq).unflatten(1, (H, -1))
        q_lat = torch.empty(T, H, rank, dtype=y.dtype, device=y.device)
        ops.bmm(q.transpose(0, 1), lw.uk_t, q_lat.transpose(0, 1))
        o_lat = ops.latent_attention(q_lat, cache, rank, self.block_tokens, step, m.scale, m.window, lw.sinks,
                                     y[:, nq + rank:nq + rank + H])
        o = torch.empty(T, H, pad8(m.vdim), dtype=y.dtype, device=y.device)
        ops.bmm(o_lat.transpose(0, 1), lw.uv, o.transpose(0, 1))
        return o.view(T, -1)

    def mixture(self, lw: MixedLayer, xn: torch.Tensor):
        """The experts' outputs with their weights, still to be summed; under tensor parallelism the summed rows."""
        s: MoeSpec = lw.spec.mlp
        e, r = lw.experts, s.router
        ids, w = ops.moe_route(ops.linear(xn, e.router, out_f32=True), r.top, scoring=r.scoring, renorm=r.renorm, scale=r.scale,
                               bias=e.correction, n_group=r.groups, topk_group=r.keep_groups, E=r.experts,
                               gate_col=r.experts if s.shared else -1)
        y, dst_row = expert_outputs(xn, ids, e.w13, e.w2, e.inter, s.expert.act)
        shared = None
        if s.shared:
            shared = ops.linear(ops.act_mul(ops.linear(xn, e.shared_gate_up), s.shared.act), e.shared_down)
        y = ExpertSum(y, dst_row, w, shared)
        if self.tp_size > 1:
            part = torch.zeros(xn.shape, dtype=torch.float32, device=xn.device)
            y = self.comm.all_reduce(ops.stream_add(part, y, None, None)[0].to(xn.dtype))
        return y

    def mlp(self, lw: MixedLayer, xn: torch.Tensor):
        if lw.experts is not None:
            return self.mixture(lw, xn)
        return self.project(ops.act_mul(ops.linear(xn, lw.gate_up), lw.spec.mlp.act), lw.down)

    def _opening(self, run: Optional[LayerRun], first: torch.Tensor):
        """(embedding output or None, step vector or None): what is added to the stream right before ``run``."""
        if run is None or run.enter is None:
            return None, None
        return first if run.enter > 0 else None, self.pass_steps[run.enter]

    def _enter(self, x, run: LayerRun, first: torch.Tensor, keep: bool):
        add, vec = self._opening(run, first)
        norm1 = self.layers[run.layer].norm1
        if vec is None:
            return x, ops.stream_norm(x, norm1, self.dtype)
        return ops.stream_enter(x, add, vec, norm1, self.dtype, inplace=not (keep and x is first))

    def forward_layers(self, step: StepInput, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        first = x = self.embed_tokens(step)
        keep = any((run.enter or 0) > 0 for run in self.runs)            # the embedding output is needed again
        x, xn = self._enter(x, self.runs[0], first, keep)
        for r, run in enumerate(self.runs):
            lw = self.layers[run.layer]
            nxt = self.runs[r + 1] if r + 1 < len(self.runs) else None
            fused = nxt is not None and self.stream_hook is None
            then = self.layers[nxt.layer].norm1 if fused else None
            add, vec = self._opening(nxt if fused else None, first)
            mixer = self.latent_attention if isinstance(lw.spec.mixer, LatentAttentionSpec) else self.attention
            with nvtx.annotate(mixer.__name__):
                y = self.project(mixer(run, lw, xn, step), lw.o_proj)
            inplace = not (keep and x is first)
            if lw.norm2 is None:                                         # a layer without a feed-forward
                x, xn = ops.stream_add(x, y, None, None, then, inplace=inplace, add=add, vec=vec)
            else:
                x, xn = ops.stream_add(x, y, None, None, lw.norm2, inplace=inplace)
                with nvtx.annotate("mlp"):
                    y = self.mlp(lw, xn)
                x, xn = ops.stream_add(x, y, None, None, then, add=add, vec=vec)
            if self.stream_hook is not None:
                self.stream_hook(r, x)
                if nxt is not None:
                    x, xn = self._enter(x, nxt, first, keep)
        return x

    def weight_bytes(self) -> int:
        n = sum(t.numel() * t.element_size() for t in (self.embed, self.lm_head.w))
        for lw in self.layers:
            n += sum(w.nbytes() for w in (lw.w_in, lw.o_proj, lw.uq, lw.gate_up, lw.down, lw.experts) if w is not None)
            n += sum(t.numel() * t.element_size() for t in (lw.uk_t, lw.uv) if t is not None)
        return n


# ------------------------------------------------------------------------------------- loading
def _check_sizes(cfg: ModelConfig, tp_size: int, device) -> None:
    for s in cfg.layer_specs:
        a = s.mixer
        if isinstance(a, LatentAttentionSpec):
            if a.heads % tp_size:
                raise ValueError(f"fidevik: {a.heads} heads cannot be split over {tp_size} ranks")
        else:
            if a.heads % tp_size or (a.kv_heads % tp_size and tp_size % a.kv_heads):
                raise ValueError(f"fidevik: {a.heads} / {a.kv_heads} heads cannot be split over {tp_size} ranks")
            if torch.device(device).type == "cuda" and max(a.dim, a.vdim) > MAX_HEAD:
                raise ValueError(f"fidevik: head sizes above {MAX_HEAD} are not supported")


def build_fidevik(cfg: ModelConfig, source, tp_rank=0, tp_size=1, comm=None, device="cpu", dtype=torch.bfloat16, quant=None,
                  layer_range=None, max_positions=None) -> FidevikModel:
    if layer_range is not None and tuple(layer_range) != (0, cfg.num_layers - 1):
        raise ValueError("fidevik: repeated layers need the embedding output, pipeline stages are not supported")
    _check_sizes(cfg, tp_size, device)
    m = FidevikModel(cfg, tp_rank, tp_size, comm, device, dtype, max_positions)
    ld = StreamLoader(m, source, quant)
    get, rows, cols, linear = ld.get, ld.rows, ld.cols, ld.linear
    W, WP, eps = cfg.hidden_size, m.width, cfg.rms_norm_eps

    def norm(name):
        return NormParams(ld.param(get(name, (W,), "ones"), WP), ld.param(get(name + ".b", (W,), "zeros"), WP), W, eps)

    def latent_norm(name, n):
        return NormParams(ld.param(get(name, (n,), "ones"), pad8(n)), None, n, eps, rms=True)

    def head_norm(name, heads, dim, share):
        """Norm over a whole projection of ``heads`` heads, of whose weights this rank needs its own heads'."""
        w = share(pad_to(get(name, (heads * dim,), "ones").reshape(heads, dim), heads, pad8(dim)))
        return NormParams(ld.param(w.reshape(-1), w.numel()), None, heads * dim, eps, rms=True)

    def by_head(name, heads, dim, width=W, padded=WP):
        return pad_to(get(name, (heads * dim, width)).reshape(heads, dim, width), heads, pad8(dim), padded)

    def flat(*parts):
        return torch.cat([t.reshape(-1, t.shape[-1]) for t in parts], 0)

    def out_proj(x, a):
        o = cols(pad_to(get(x + "o", (W, a.heads * a.vdim)).reshape(W, a.heads, a.vdim), WP, a.heads, pad8(a.vdim)))
        return linear(o.reshape(WP, -1))

    def attention(spec, x, n1):
        a: AttentionSpec = spec.mixer
        q, k, v = by_head(x + "q", a.heads, a.dim), by_head(x + "k", a.kv_heads, a.dim), by_head(x + "v", a.kv_heads, a.vdim)
        q, k, v = rows(q), ld.kv_heads(k), ld.kv_heads(v)
        return MixedLayer(spec, n1, linear(flat(q, k, v)), out_proj(x, a), q.shape[0], k.shape[0],
                          head_norm(x + "q.norm", a.heads, a.dim, rows), head_norm(x + "k.norm", a.kv_heads, a.dim, ld.kv_heads))

    def latent_attention(spec, x, n1):
        a: LatentAttentionSpec = spec.mixer
        H, r, qr = a.heads // tp_size, pad8(a.kv_rank), pad8(a.q_rank)
        w_in = flat(pad_to(get(x + "dq", (a.q_rank, W)), qr, WP), pad_to(get(x + "dkv", (a.kv_rank, W)), r, WP),
                    pad_to(rows(get(x + "g", (a.heads, W))), pad8(H), WP))
        uk, uv = (rows(by_head(x + s, a.heads, n, a.kv_rank, r)) for s, n in (("uk", a.dim), ("uv", a.vdim)))
        return MixedLayer(spec, n1, linear(w_in), out_proj(x, a), H,
                          q_norm=latent_norm(x + "dq.norm", a.q_rank), k_norm=latent_norm(x + "dkv.norm", a.kv_rank),
                          uq=linear(flat(rows(by_head(x + "uq", a.heads, a.dim, a.q_rank, qr)))),
                          uk_t=ld.param(uk.transpose(1, 2), H, r, pad8(a.dim)), uv=ld.param(uv, H, pad8(a.vdim), r),
                          sinks=rows(get(x + "sink", (a.heads,))).to(device=m.device, dtype=torch.float32).contiguous())

    def gate_up(x, size):
        return torch.cat([ld.split_rows(x + "gate", size), ld.split_rows(x + "up", size)], 0)

    def experts(s: MoeSpec, x):
        E, size = s.router.experts, s.expert.size
        router = [get(x + "router", (E, W))] + ([get(x + "shared.sg", (1, W))] if s.shared else [])
        # expert by expert into place: a whole stack and its parts never exist at the same time
        n = ld.shard(size)
        w13, w2 = torch.empty(E, 2 * n, WP, dtype=dtype, device=m.device), torch.empty(E, WP, n, dtype=dtype, device=m.device)
        for i in range(E):
            w13[i], w2[i] = gate_up(f"{x}e{i}.", size), ld.split_cols(f"{x}e{i}.down", size)
        e = ExpertWeights(LinearWeight(w=ld.param(flat(*router), pad8(E + len(router) - 1), WP)),
                          get(x + "correction", (E,), "zeros").to(device=m.device, dtype=torch.float32).contiguous(),
                          w13.view(-1, WP), w2.view(-1, n), n)
        if s.shared:
            e.shared_gate_up = linear(gate_up(x + "shared.", s.shared.size))
            e.shared_down = linear(ld.split_cols(x + "shared.down", s.shared.size))
        return e

    ld.vocabulary()
    if cfg.loop is not None:
        m.pass_steps = ld.param(get("loop.step", (cfg.loop.times, W)), cfg.loop.times, WP)
    for i, spec in enumerate(cfg.layer_specs):
        p = f"l{i}."
        build = latent_attention if isinstance(spec.mixer, LatentAttentionSpec) else attention
        lw = build(spec, p + "mix.", norm(p + "norm1"))
        if spec.mlp is not None:
            lw.norm2 = norm(p + "norm2")
            if isinstance(spec.mlp, MoeSpec):
                lw.experts = experts(spec.mlp, p + "mlp.")
            else:
                lw.gate_up, lw.down = linear(gate_up(p + "mlp.", spec.mlp.size)), linear(ld.split_cols(p + "mlp.down", spec.mlp.size))
        m.layers.append(lw)
    m.final = norm("final.norm")
    return m
