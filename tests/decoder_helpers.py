"""Drivers shared by the tests of the families whose layers are configured one by one: building a model and an engine from
a config.json dict and a dict of weights, running given tokens through the engine in arbitrary portions and batches,
error measures."""
import copy
import json
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from ksanallm_b200.config import EngineConfig, model_config_from_hf
from ksanallm_b200.models.weights import DictSource, build_model
from ksanallm_b200.ops import native
from ksanallm_b200.runtime.engine import LLMEngine
from ksanallm_b200.utils import native_engine as ne

gpu = pytest.mark.gpu
# where the same test runs: the plain statements of the ops, and the kernels in both precisions
PLACES = [pytest.param("cpu", torch.float32, id="cpu-f32"), pytest.param("cuda", torch.float32, id="gpu-f32", marks=gpu),
          pytest.param("cuda", torch.bfloat16, id="gpu-bf16", marks=gpu)]


def save_checkpoint(path, c, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(c, f)
    save_file({k: v.bfloat16().contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))


def build(c, w, device, dtype, max_positions=512):
    return build_model(model_config_from_hf(copy.deepcopy(c)), DictSource(w, c["architecture"].lower()), device=device, dtype=dtype,
                       max_positions=max_positions)


def engine(c, w, device, dtype, blocks=64, max_len=None, host_blocks=0, block_tokens=16, graphs=False, **sched):
    model = build(c, w, device, dtype)
    ec = EngineConfig()
    ec.block_manager.block_token_num = block_tokens
    ec.batch_scheduler.max_batch_size = 8
    ec.batch_scheduler.max_token_len = max_len or min(blocks * block_tokens, 512)
    ec.global_.enable_cuda_graph = graphs
    for k, v in sched.items():
        setattr(ec.batch_scheduler, k, v)
    return LLMEngine(model, model.cfg, ec, num_blocks=blocks, num_host_blocks=host_blocks)


def tokens(c, n, seed=0):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


@torch.inference_mode()
def run_portions(eng, toks, sizes):
    """Logits of every position of one request that arrives in portions of the given sizes (the last one repeats)."""
    sid, out, at, k = eng.open_given(), [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(eng.step_given([(sid, toks[at:at + n], list(range(n)))]).float().cpu())
        at, k = at + n, k + 1
    eng.close_given(sid)
    return torch.cat(out)


def error(got, want):
    """Largest error of a row: root mean square over the vocabulary, means taken off, relative to the rows' spread."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float(d.pow(2).mean(-1).sqrt().max() / scale)


LIMIT = {torch.float32: 3e-5, torch.bfloat16: 0.1}


def check(got, want, dtype, device):
    if device == "cuda":
        native.check_err_flag("cuda")
    assert torch.isfinite(got).all()
    e = error(got, want)
    assert e < LIMIT[dtype], e


@torch.inference_mode()
def run_batch(eng, requests, seed, slots=4):
    """Feeds requests (token lists) in random portions, up to ``slots`` live at a time; a request may pause. Returns the
    logits of every position per request."""
    rng = np.random.default_rng(seed)
    waiting, live, out = list(range(len(requests))), {}, {i: [] for i in range(len(requests))}
    at = {i: 0 for i in out}
    while waiting or live:
        while waiting and len(live) < slots:
            i = waiting.pop(0)
            live[i] = eng.open_given()
        entries, who = [], []
        for i in rng.permutation(sorted(live)).tolist():
            if len(live) > 1 and rng.random() < 0.2:
                continue
            left = len(requests[i]) - at[i]
            n = min(left, 1 if rng.random() < 0.5 else int(rng.integers(2, 40)))
            entries.append((live[i], requests[i][at[i]:at[i] + n], list(range(n))))
            who.append((i, n))
        if not entries:
            continue
        logits, k = eng.step_given(entries).float().cpu(), 0
        for i, n in who:
            out[i].append(logits[k:k + n])
            k, at[i] = k + n, at[i] + n
            if at[i] == len(requests[i]):
                eng.close_given(live.pop(i))
    return [torch.cat(out[i]) for i in range(len(requests))]


def greedy(n):
    s = ne.SamplingConfig()
    s.max_new_tokens, s.ignore_eos, s.topk = n, True, 1
    return s


def greedy_within_rounding(logits, out, dtype):
    """Every token of ``out`` is the best one of its row of ``logits`` (within rounding)."""
    spread = float(logits.std())
    for row, tok in zip(logits, out):
        assert float(row.max() - row[tok]) <= (1e-3 if dtype == torch.float32 else 0.12) * spread


# ------------------------------------------------------------------------------------------------ single ops
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}
rand = lambda seed, *s: torch.randn(*s, generator=torch.Generator().manual_seed(seed)).bfloat16().float()  # noqa: E731
pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))  # noqa: E731
up8 = lambda n: (n + 7) // 8 * 8  # noqa: E731


def close(got, want, dtype, scale=None):
    got, want = got.float().cpu(), want.float()
    s = scale if scale is not None else max(1.0, float(want.abs().max()))
    assert torch.isfinite(got).all()
    assert float((got - want).abs().max()) <= TOL[dtype] * s, float((got - want).abs().max()) / s


def make_step(lens, tables, bt, device):
    """Step of sequences (cached, new), multi-token ones first; ``tables``: block ids (of bt tokens) per sequence."""
    news = [n for _, n in lens]
    cu = torch.tensor([0] + news).cumsum(0).to(torch.int32)
    multi = sum(n > 1 for n in news)
    width = max(len(t) for t in tables) + 1
    table = torch.tensor([list(t) + [0] * (width - len(t)) for t in tables], dtype=torch.int32)
    kv = torch.tensor([p + n for p, n in lens], dtype=torch.int32)
    slots = torch.tensor([tables[s][t // bt] * bt + t % bt for s, (p, n) in enumerate(lens) for t in range(p, p + n)], dtype=torch.int32)
    return SimpleNamespace(slots=slots.to(device), block_table=table.to(device), cu_q=cu.to(device), kv_lens=kv.to(device), num_multi=multi,
                           num_single=len(news) - multi, num_multi_tokens=int(cu[multi]), max_q_len=max(news), max_kv_len=int(kv.max()))
