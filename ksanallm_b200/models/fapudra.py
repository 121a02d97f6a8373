"""Fapudra: a decoder with a 32-bit residual stream whose layers add a mixer and a mixture of experts side by side (one norm, both
read it; the mixer reads it shifted towards the previous token). A mixer is a selective state space, or sigmoid attention over
a window with kept first tokens next to a gated delta rule. Learned positions at the input, soft-capped logits.

The step functions, the block pool, the scheduler and the sampler are the ones of every other family. A cache block is one
record with a K panel per attention (the values are the keys). What the recurrences carry lives in a state slot per sequence: one
record with, per layer, the last normed row (token shift) in a ring of two, the last inputs of the short convolution in a ring,
and the fp32 state matrices. Per layer:

  token shift    one kernel
  state space    [z | x | B | C | dt] GEMM -> convolution -> scan (decode: both in one kernel) -> gated norm -> output GEMM
  parallel       [q | k | attention gate | q k v | beta | decay, gate latents] GEMM -> append -> attention with its gate in the epilogue;
                 [decay | gate] GEMM -> convolution -> scan (decode: one kernel) -> norm with the gate; one output GEMM for both halves
  experts        router GEMM (fp32 result) -> choice -> grouped GEMMs
  sum            the weighted sum of the experts' outputs, the mixer's result, the residual add and the next norm in one kernel
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..config import AttentionSpec, DeltaRuleSpec, LayerSpec, ModelConfig, MoeSpec, ParallelSpec, StateSpaceSpec
from ..ops import dispatch as ops
from ..ops.dispatch import ExpertSum, LinearWeight, NormParams, ShortConv, SigmoidWeights
from ..utils import nvtx
from .common import RecordLayout, StepInput
from .moe import expert_outputs
from .stream import StreamLoader, StreamModel, distance_biases, pad8, pad_to

MAX_HEAD = 256                    # largest head size of the attention kernels
MAX_KEYS = 256                    # largest key dimension of a recurrent state
MAX_TAPS = 16                     # of a short convolution


@dataclass
class RecurrentWeights:
    conv_w: torch.Tensor                       # [taps, channels]
    conv_b: Optional[torch.Tensor]
    A: torch.Tensor                            # fp32, per head: exp(A_log)
    bias: torch.Tensor                         # fp32: of the step sizes (per head) or of the decays (per head and key channel)
    norm: torch.Tensor                         # of the output, all columns
    D: Optional[torch.Tensor] = None           # fp32, per head
    low_rank: Optional[LinearWeight] = None    # [decay latent | gate latent] -> [decay | gate]


@dataclass
class ParallelLayer:
    spec: LayerSpec
    norm1: NormParams
    shift: torch.Tensor
    w_in: LinearWeight                         # all projections of the mixer's input, packed by rows
    o_proj: LinearWeight
    rec: RecurrentWeights
    columns: list                              # where the parts of w_in's result start, and its width
    biases: Optional[torch.Tensor] = None      # [heads, distances] fp32
    router: Optional[LinearWeight] = None
    w13: Optional[torch.Tensor] = None         # [E * 2I, W]: gate rows, then up rows of every expert
    w2: Optional[torch.Tensor] = None          # [E * W, I]
    inter: int = 0


class FapudraModel(StreamModel):
    needs_state_slots = True
    moves_blocks = False

    def __init__(self, cfg: ModelConfig, *a, **kw):
        super().__init__(cfg, *a, **kw)
        self.embed_norm: Optional[NormParams] = None
        self.state_layout: Optional[RecordLayout] = None

    # ------------------------------------------------------------------ cache and state
    def allocate_kv_cache(self, num_blocks: int, block_tokens: int, dtype=None):
        """[blocks, record]: the K panel of every attention, one after the other."""
        self.check_cache_dtype(dtype)
        self.block_tokens = block_tokens
        self.layout = RecordLayout(self.dtype)
        index = {}
        for i, lw in enumerate(self.layers):
            if isinstance(lw.spec.mixer, ParallelSpec):
                a = lw.spec.mixer.attention
                index[i] = self.layout.add((a.kv_heads, block_tokens, pad8(a.dim)))
        # a model without attention has nothing to cache, but its tokens are counted in blocks all the same
        self.kv_cache = torch.zeros(num_blocks, max(self.layout.record, 16 // self.dtype.itemsize), dtype=self.dtype, device=self.device)
        self.panels = {i: self.layout.view(self.kv_cache, k) for i, k in index.items()}
        return self.kv_cache

    def _lay_out_state(self):
        self.state_layout, self._state_index = RecordLayout(torch.float32), []
        for lw in self.layers:
            m = lw.spec.mixer
            heads, rows, keys = (m.heads, m.vdim, m.state) if isinstance(m, StateSpaceSpec) else \
                (m.recurrence.heads, m.recurrence.vdim, m.recurrence.dim)
            self._state_index.append((self.state_layout.add((2, self.width), self.dtype),
                                      self.state_layout.add(tuple(lw.rec.conv_w.shape), self.dtype),
                                      self.state_layout.add((heads, pad8(rows), pad8(keys)))))

    def state_bytes(self) -> int:
        if self.state_layout is None:
            self._lay_out_state()
        return self.state_layout.record * 4

    def allocate_state(self, num_slots: int) -> None:
        self.state = torch.zeros(num_slots, self.state_bytes() // 4, dtype=torch.float32, device=self.device)
        self.slots = [tuple(self.state_layout.view(self.state, k) for k in group) for group in self._state_index]

    # ------------------------------------------------------------------ blocks
    def embed_tokens(self, step: StepInput, **_) -> torch.Tensor:
        x = ops.embed_normed(step.input_ids, step.positions, self.embed, self.pos_embed, self.cfg.emb_scale, self.embed_norm,
                             self.cfg.vocab_size)
        if step.refit_positions is not None and step.refit_positions.numel() > 0:
            ops.refit_stream_rows(x, step.refit_positions, step.refit_embeddings)
        return x

    def state_space(self, i: int, lw: ParallelLayer, m: torch.Tensor, step: StepInput) -> torch.Tensor:
        s: StateSpaceSpec = lw.spec.mixer
        r, (_, ring, state) = lw.rec, self.slots[i]
        y = ops.linear(m, lw.w_in)
        x, dt, _ = lw.columns
        out = ops.state_space(y[:, x:dt], ShortConv(r.conv_w, r.conv_b, ring), y[:, dt:], r.bias, r.A, r.D, state, s.groups, step)
        return ops.gated_norm(out, r.norm, self.cfg.rms_norm_eps, s.heads, s.vdim, s.norm_groups, z=y[:, :x])

    def parallel(self, i: int, lw: ParallelLayer, m: torch.Tensor, step: StepInput) -> torch.Tensor:
        s: ParallelSpec = lw.spec.mixer
        a, d = s.attention, s.recurrence
        k_at, g_at, x_at, beta_at, low_at, end = lw.columns
        y = ops.linear(m, lw.w_in)
        out = torch.empty(y.shape[0], k_at + d.heads * pad8(d.vdim), dtype=y.dtype, device=y.device)
        cache = self.panels[i]
        ops.panel_append(y[:, k_at:g_at], step, cache, self.block_tokens)
        ops.panel_attention(y, cache, cache, self.block_tokens, step, a.heads, a.kv_heads, a.scale, a.window, a.keep_first,
                            weights=SigmoidWeights(lw.biases, y[:, g_at:x_at], s.attention_scale), out=out[:, :k_at])
        r, (_, ring, state) = lw.rec, self.slots[i]
        low = ops.linear(y[:, low_at:end], r.low_rank)
        dk = d.heads * pad8(d.dim)
        o = ops.delta_rule(y[:, x_at:beta_at], ShortConv(r.conv_w, None, ring), y[:, beta_at:], low[:, :dk], r.bias, r.A, state,
                           d.kv_heads, d.dim ** -0.5, step)
        ops.gated_norm(o, r.norm, self.cfg.rms_norm_eps, d.heads, d.vdim, d.heads, g=low[:, dk:], factor=s.recurrence_scale,
                       out=out[:, k_at:])
        return out

    def mixture(self, lw: ParallelLayer, h: torch.Tensor, beside: torch.Tensor) -> ExpertSum:
        """The experts' outputs with their weights and the mixer's result, still to be summed."""
        s: MoeSpec = lw.spec.mlp
        r = s.router
        ids, w = ops.moe_route(ops.linear(h, lw.router, out_f32=True), r.top, scoring=r.scoring, renorm=r.renorm, scale=r.scale,
                               n_group=r.groups, topk_group=r.keep_groups, E=r.experts, group_top=r.group_top)
        y, dst_row = expert_outputs(h, ids, lw.w13, lw.w2, lw.inter, s.expert)
        return ExpertSum(y, dst_row, w, beside)

    def forward_layers(self, step: StepInput, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        x = self.embed_tokens(step)
        h = ops.stream_norm(x, self.layers[0].norm1, self.dtype)
        for i, lw in enumerate(self.layers):
            then = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else None
            mixer = self.parallel if isinstance(lw.spec.mixer, ParallelSpec) else self.state_space
            m = ops.token_shift(h, lw.shift, self.slots[i][0], step)
            with nvtx.annotate(mixer.__name__):
                y = ops.linear(mixer(i, lw, m, step), lw.o_proj)
            if lw.router is not None:
                with nvtx.annotate("experts"):
                    y = self.mixture(lw, h, y)
            x, h = ops.stream_add(x, y, None, None, then)
            if self.stream_hook is not None:
                self.stream_hook(i, x)
        return x

    def weight_bytes(self) -> int:
        n = sum(t.numel() * t.element_size() for t in (self.embed, self.pos_embed, self.lm_head.w))
        for lw in self.layers:
            n += sum(w.nbytes() for w in (lw.w_in, lw.o_proj, lw.rec.low_rank, lw.router) if w is not None)
            n += sum(t.numel() * t.element_size() for t in (lw.w13, lw.w2) if t is not None)
        return n


# ------------------------------------------------------------------------------------- loading
def _check_sizes(cfg: ModelConfig, tp_size: int, device) -> None:
    if tp_size > 1:
        raise ValueError("fapudra: the states of its recurrences are not split over tensor-parallel ranks")
    for s in cfg.layer_specs:
        a = s.mixer
        keys, taps = (a.state, a.taps) if isinstance(a, StateSpaceSpec) else (a.recurrence.dim, a.recurrence.taps)
        if torch.device(device).type == "cuda":
            if keys > MAX_KEYS or taps > MAX_TAPS:
                raise ValueError(f"fapudra: recurrent keys above {MAX_KEYS} and convolutions above {MAX_TAPS} taps are not supported")
            if isinstance(a, ParallelSpec) and a.attention.dim > MAX_HEAD:
                raise ValueError(f"fapudra: head sizes above {MAX_HEAD} are not supported")


def _starts(*sizes):
    out = [0]
    for n in sizes:
        out.append(out[-1] + n)
    return out


def build_fapudra(cfg: ModelConfig, source, tp_rank=0, tp_size=1, comm=None, device="cpu", dtype=torch.bfloat16, quant=None,
                  layer_range=None, max_positions=None) -> FapudraModel:
    if layer_range is not None and tuple(layer_range) != (0, cfg.num_layers - 1):
        raise ValueError("fapudra: pipeline stages are not supported")
    _check_sizes(cfg, tp_size, device)
    m = FapudraModel(cfg, tp_rank, tp_size, comm, device, dtype, max_positions)
    ld = StreamLoader(m, source, quant)
    get, param, linear = ld.get, ld.param, ld.linear
    W, WP = cfg.hidden_size, m.width

    def norm(name):
        """One number for all columns."""
        return NormParams(param(get(name, (), "ones").reshape(1).expand(W), WP), None, W, cfg.rms_norm_eps, rms=True)

    def heads(t, n, real):
        """[n * real, ...] -> [n * padded, ...]"""
        return pad_to(t.reshape(n, real, *t.shape[1:]), n, pad8(real), *t.shape[1:]).flatten(0, 1)

    def rows(name, n, real):
        """A projection of the input to ``n`` heads, padded."""
        return pad_to(heads(get(name, (n * real, W)), n, real), n * pad8(real), WP)

    def plain(t, n):
        return pad_to(t, pad8(n), WP)

    def a_log(name, n):
        return ld.f32(get(name, (n,), "zeros")).exp()

    def out_cols(name, n, real):
        return pad_to(heads(get(name, (W, n * real)).t(), n, real).t(), WP, n * pad8(real))

    def taps(*parts):
        """Convolution weights by tap: [taps, channels]."""
        t = torch.cat(parts, 0).t()
        return param(t, *t.shape)

    def state_space(spec, x, n1, shift):
        s: StateSpaceSpec = spec.mixer
        H, P, N, G = s.heads, s.vdim, s.state, s.groups
        sizes = [H * P, H * P, G * N, G * N]
        w = get(x + "in", (sum(sizes) + H, W)).split(sizes + [H])
        lay = ((H, P), (H, P), (G, N), (G, N))
        w_in = [pad_to(heads(t, *hp), hp[0] * pad8(hp[1]), WP) for t, hp in zip(w, lay)] + [plain(w[4], H)]
        c = get(x + "conv", (sum(sizes[1:]), s.taps)).split(sizes[1:])
        b = get(x + "conv.b", (sum(sizes[1:]),), "zeros").split(sizes[1:])
        bias = torch.cat([heads(t, *hp) for t, hp in zip(b, lay[1:])])
        rec = RecurrentWeights(taps(*[heads(t, *hp) for t, hp in zip(c, lay[1:])]), param(bias, bias.numel()),
                               a_log(x + "A_log", H), ld.f32(get(x + "dt_bias", (H,), "zeros")),
                               param(heads(get(x + "norm", (H * P,), "ones"), H, P), H * pad8(P)),
                               D=ld.f32(get(x + "D", (H,), "ones")))
        z = H * pad8(P)
        return ParallelLayer(spec, n1, shift, linear(torch.cat(w_in)), linear(out_cols(x + "o", H, P)), rec,
                             [z, z + bias.numel(), z + bias.numel() + pad8(H)])

    def parallel(spec, x, n1, shift):
        s: ParallelSpec = spec.mixer
        a: AttentionSpec = s.attention
        d: DeltaRuleSpec = s.recurrence
        le, ri = x + "left.", x + "right."
        H, G, dim = a.heads, a.kv_heads, a.dim
        proj = [rows(le + "q", H, dim), rows(le + "k", G, dim), rows(le + "g", H, dim)]
        bias = [heads(get(le + "q.b", (H * dim,), "zeros"), H, dim), heads(get(le + "k.b", (G * dim,), "zeros"), G, dim)]
        qkv = (("q", d.kv_heads, d.dim), ("k", d.kv_heads, d.dim), ("v", d.heads, d.vdim))
        conv = [rows(ri + n, h, r) for n, h, r in qkv]
        low = [ld.shape(ri + n, (d.vdim, W))[0] for n in ("a1", "g1")]           # sizes of the latents: the tensors'
        latents = [plain(get(ri + n, (r, W)), r) for n, r in zip(("a1", "g1"), low)]
        beta = plain(get(ri + "b", (d.heads, W)), d.heads)
        parts = proj + [torch.cat(conv), beta, torch.cat(latents)]
        w_in = torch.cat(parts)
        starts = _starts(*(t.shape[0] for t in parts))
        b = pad_to(torch.cat(bias).float(), w_in.shape[0])
        # [decay latent | gate latent] -> [decay | gate]: one product with a block-diagonal weight
        up = [pad_to(heads(get(ri + n, (d.heads * r, k)), d.heads, r), d.heads * pad8(r), pad8(k))
              for n, r, k in zip(("a2", "g2"), (d.dim, d.vdim), low)]
        rec = RecurrentWeights(taps(*[heads(get(f"{ri}{n}.conv", (h * r, d.taps)), h, r) for n, h, r in qkv]), None,
                               a_log(ri + "A_log", d.heads),
                               ld.f32(heads(get(ri + "dt_bias", (d.heads * d.dim,), "zeros"), d.heads, d.dim)),
                               param(pad_to(get(ri + "norm", (d.vdim,), "ones"), pad8(d.vdim)).repeat(d.heads), d.heads * pad8(d.vdim)),
                               low_rank=linear(torch.block_diag(*up)))
        rel = get(le + "rel", ld.shape(le + "rel", (32, H)))
        biases = distance_biases(ld.f32(rel), a.bias_far) + ld.f32(get(le + "pb", (H,), "zeros"))[:, None]
        return ParallelLayer(spec, n1, shift, linear(w_in, b),
                             linear(torch.cat([out_cols(le + "o", H, dim), out_cols(ri + "o", d.heads, d.vdim)], 1)), rec, starts[1:],
                             biases=biases.contiguous())

    def experts(lw, s: MoeSpec, x):
        E, size = s.router.experts, s.expert.size
        lw.inter = n = pad8(size)
        lw.router = LinearWeight(w=param(get(x + "router", (E, W)), pad8(E), WP))
        # expert by expert into place: a whole stack and its parts never exist at the same time
        w13, w2 = torch.empty(E, 2 * n, WP, dtype=dtype, device=m.device), torch.empty(E, WP, n, dtype=dtype, device=m.device)
        for e in range(E):
            for at, part in ((0, "gate"), (n, "up")):
                w13[e, at:at + n] = pad_to(get(f"{x}e{e}.{part}", (size, W)), n, WP)
            w2[e] = pad_to(get(f"{x}e{e}.down", (W, size)), WP, n)
        lw.w13, lw.w2 = w13.view(-1, WP), w2.view(-1, n)

    ld.vocabulary()
    positions = min(cfg.max_token_len, max_positions or cfg.max_token_len)
    m.pos_embed = param(get("pos", (cfg.max_position_embeddings, W))[:positions], positions, WP)
    m.embed_norm = norm("embed.norm")
    for i, spec in enumerate(cfg.layer_specs):
        p = f"l{i}."
        build = parallel if isinstance(spec.mixer, ParallelSpec) else state_space
        lw = build(spec, p + "mix.", norm(p + "norm1"), param(get(p + "shift", (W,), "zeros"), WP))
        if spec.mlp is not None:
            experts(lw, spec.mlp, p + "mlp.")
        m.layers.append(lw)
    m.final = norm("final.norm")
    return m
