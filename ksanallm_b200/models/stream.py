"""Base of the families with a 32-bit residual stream whose layers are configured one by one (``ModelConfig.layer_specs``):
padded stream rows, per-layer rotation tables, layers that run several times, row-parallel projections, the final norm over
the rows that need logits, and the loading helpers.

Sizes that are not multiples of 8 are padded with zeros when the weights are loaded (rows of the residual stream, head
sizes, feed-forward widths, vocabulary), so the kernels always see 16-byte vectors; norms count the real columns only.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List, Optional

import torch
import torch.nn.functional as F

from ..config import ModelConfig, RotarySpec
from ..ops import dispatch as ops
from ..ops import native
from ..ops import reference as ref
from ..ops.dispatch import LinearWeight, NormParams
from .common import CommonModel, StepInput


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def pad_to(t: torch.Tensor, *sizes: int) -> torch.Tensor:
    """Zero-pads every dimension of ``t`` to ``sizes``."""
    spec = []
    for have, want in zip(reversed(t.shape), reversed(sizes)):
        spec += [0, want - have]
    return F.pad(t, spec) if any(spec) else t


@dataclass
class LayerRun:
    layer: int
    cache: int                    # cache layer of this run
    enter: Optional[int] = None   # number of the loop pass that starts right before this run


def layer_runs(cfg: ModelConfig) -> List[LayerRun]:
    order, n, loop = [], len(cfg.layer_specs), cfg.loop
    if loop is None:
        order = [(i, None) for i in range(n)]
    else:
        order = [(i, None) for i in range(loop.start)]
        for t in range(loop.times):
            order += [(i, t if i == loop.start else None) for i in range(loop.start, loop.stop)]
        order += [(i, None) for i in range(loop.stop, n)]
    return [LayerRun(i, c, enter) for c, (i, enter) in enumerate(order)]


def distance_biases(rel: torch.Tensor, far: int) -> torch.Tensor:
    """[heads, n] biases by distance from a table [buckets, heads]: the first half of the buckets are single distances, the
    others grow logarithmically up to ``far``; distances from n - 1 on have the last one's bias."""
    count = rel.shape[0]
    half = count // 2

    def bucket(n):
        if n < half:
            return n
        if half == 0 or far <= half:
            return count - 1
        return min(count - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (count - half)))

    index = torch.tensor([bucket(n) for n in range(max(far, half) + 1)], device=rel.device)
    return rel.float()[index].t().contiguous()


def rerotate_panel(k: torch.Tensor, triples, table: torch.Tensor, interleaved: bool = False) -> None:
    """Turns the keys of copied blocks (``triples``: source, destination, position delta) of a panel [blocks, heads, block
    tokens, size] by the position delta."""
    dims = table.shape[1]
    if k.is_cuda and k.dtype == torch.bfloat16:
        t3 = torch.as_tensor(triples, dtype=torch.int32).contiguous().to(k.device)
        native.rerotate_panel(k, t3, table, dims, neox=not interleaved)
        return
    for _, dst, delta in triples:
        delta = int(delta)
        if delta:
            cos, sin = table[abs(delta)].chunk(2)
            sin = sin if delta > 0 else -sin
            r = k[int(dst), ..., :dims].float()
            u, v = (r[..., 0::2], r[..., 1::2]) if interleaved else r.chunk(2, dim=-1)
            turned = (u * cos - v * sin, v * cos + u * sin)
            k[int(dst), ..., :dims] = (torch.stack(turned, -1).flatten(-2) if interleaved else torch.cat(turned, -1)).to(k.dtype)


class StreamModel(CommonModel):
    stream_hook = None                                   # debugging: called with (run, stream) after every layer run

    def __init__(self, cfg: ModelConfig, tp_rank=0, tp_size=1, comm=None, device="cpu", dtype=torch.bfloat16, max_positions=None):
        super().__init__(cfg, tp_rank, tp_size, comm, device, dtype)
        self.width = pad8(cfg.hidden_size)
        self.final: Optional[NormParams] = None
        self._tables, self._positions = {}, max_positions or min(cfg.max_token_len, 1 << 15)

    def rotation_table(self, r: RotarySpec) -> torch.Tensor:
        """cos | sin table of a rotation, shared by the layers with equal rotations."""
        key = (r.dims, r.base, tuple(sorted((r.scaling or {}).items())))
        if key not in self._tables:
            self._tables[key] = ref.build_cos_sin_cache(r.dims, self._positions, r.base, r.scaling, self.device)
        return self._tables[key]

    def check_cache_dtype(self, dtype) -> None:
        if dtype is not None and dtype != self.dtype:
            raise ValueError(f"{self.cfg.model_type}: the KV cache has the activations' type ({self.dtype}), not {dtype}")

    def embed_tokens(self, step: StepInput, copy=None, pair=None, hashed=(0, 0, 0)) -> torch.Tensor:
        """The fp32 embedding output; ``copy`` receives it in the activations' type. ``pair``: table of hashed token pairs
        that is added."""
        refit = step.refit_positions is not None and step.refit_positions.numel() > 0
        x = ops.embed_pair(step.input_ids, step.prev_ids, self.embed, pair, self.cfg.emb_scale, *hashed,
                           copy=None if refit else copy, vocab=self.cfg.vocab_size)
        if refit:
            ops.refit_stream_rows(x, step.refit_positions, step.refit_embeddings)
            if copy is not None:
                ops.stream_copy(x, copy)
        return x

    def project(self, a: torch.Tensor, w: LinearWeight) -> torch.Tensor:
        """Row-parallel output projection: the sublayer's full result."""
        y = ops.linear(a, w)
        return self.comm.all_reduce(y) if self.tp_size > 1 else y

    def forward(self, step: StepInput, hidden_in: Optional[torch.Tensor] = None):
        return self.lm_head_forward(self.forward_layers(step), step)

    def lm_head_forward(self, x: torch.Tensor, step: StepInput):
        # the factor of the logits goes into their GEMM's operand
        scale = self.cfg.logit_scale
        if step.want_hidden:
            self.step_hidden, self.step_normed = x, ops.stream_norm(x, self.final, self.dtype, scale=scale)
        return self.logits_or_candidates(ops.stream_norm(x, self.final, self.dtype, rows=step.logits_rows, scale=scale), step)


class StreamLoader:
    """Reads, checks, pads and converts the tensors of a :class:`StreamModel`."""

    def __init__(self, model: StreamModel, source, quant=None):
        self.m, self.source, self.quant = model, source, quant

    def get(self, name, shape, kind="normal"):
        t = self.source.get(name, shape, device=self.m.device, kind=kind)
        if tuple(t.shape) != tuple(shape):
            raise ValueError(f"{name}: shape {tuple(t.shape)} in the checkpoint, {tuple(shape)} by the configuration")
        return t

    def shape(self, name, default):
        """Shape of a tensor whose sizes the configuration does not give (``default``: where the source makes up its tensors)."""
        from .weights import RandomSource
        return tuple(default) if isinstance(self.source, RandomSource) else tuple(self.source.get(name, None, device="cpu").shape)

    def f32(self, t):
        return t.to(device=self.m.device, dtype=torch.float32).contiguous()

    def param(self, t, *sizes):
        return pad_to(t, *sizes).to(device=self.m.device, dtype=self.m.dtype).contiguous()

    def linear(self, t, bias=None):
        from .weights import _make_linear
        return _make_linear(t.contiguous(), bias, self.m.device, self.m.dtype, self.quant)

    def rows(self, t):
        """This rank's share of the rows (their number divides by the ranks)."""
        from .weights import _rows
        return _rows(t, self.m.tp_rank, self.m.tp_size)

    def cols(self, t):
        from .weights import _cols
        return _cols(t, self.m.tp_rank, self.m.tp_size)

    def shard(self, n: int) -> int:
        """Padded share of ``n`` columns or channels that are split over the ranks."""
        return pad8((n + self.m.tp_size - 1) // self.m.tp_size)

    def split_rows(self, name, n: int) -> torch.Tensor:
        """This rank's rows of a projection of the stream to ``n`` columns that are split over the ranks, padded."""
        return self.rows(pad_to(self.get(name, (n, self.m.cfg.hidden_size)), self.shard(n) * self.m.tp_size, self.m.width))

    def split_cols(self, name, n: int) -> torch.Tensor:
        """This rank's columns of a projection of ``n`` split columns to the stream, padded."""
        return self.cols(pad_to(self.get(name, (self.m.cfg.hidden_size, n)), self.m.width, self.shard(n) * self.m.tp_size))

    def kv_heads(self, t: torch.Tensor) -> torch.Tensor:
        """This rank's key/value heads of ``t`` [heads, ...]: its share of them, or the one that it shares with other ranks."""
        from .weights import _rows
        rep = max(1, self.m.tp_size // t.shape[0])
        return _rows(t, self.m.tp_rank // rep, self.m.tp_size // rep)

    def vocabulary(self) -> None:
        """Embedding table, and the output projection (this rank's rows): the tensor ``head``, or the table again."""
        m, cfg = self.m, self.m.cfg
        full = (cfg.vocab_size, cfg.hidden_size)
        m.embed = self.param(self.get("embed", full), pad8(cfg.vocab_size), m.width)
        vs = (cfg.vocab_size + m.tp_size - 1) // m.tp_size
        head = m.embed if cfg.tie_word_embeddings else self.get("head", full)
        tied = cfg.tie_word_embeddings and m.tp_size == 1
        m.lm_head = LinearWeight(w=head if tied else self.param(self.rows(head[:cfg.vocab_size]), pad8(vs), m.width))
        m.vocab_shard = vs
