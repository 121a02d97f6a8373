"""Trace replay: feeds given token ids through the engine's step function and writes logits (nothing is sampled).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` names the requests of the step with their next tokens (a request is admitted at its first entry) and the
places among them whose logits are wanted; all entries run as one batch. ``end`` lists the requests that are finished
after the step. The wanted logits go to ``DIR/<step>.f32`` (little-endian fp32, [wanted, vocab], in the order of the
entries); after every step the line ``done <step>`` is printed. ``--max-tokens``: the most tokens that live requests
hold at any time; the block pool is made for that many.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4                      # requests live at any time


def make_llm(model_dir: str, dtype: str, max_tokens: int, device: str):
    import torch

    from .config import EngineConfig
    from .llm import LLM
    if device == "cuda" and not torch.cuda.is_available():
        raise RuntimeError("no CUDA device")
    ec = EngineConfig()
    ec.model_dir = model_dir
    bt = ec.block_manager.block_token_num
    ec.batch_scheduler.max_batch_size = MAX_LIVE
    ec.batch_scheduler.preempt_mode = 1                              # no host pool: nothing is ever preempted here
    blocks = max((max_tokens + bt - 1) // bt, 1)
    ec.batch_scheduler.max_token_len = blocks * bt
    ec.block_manager.device_blocks_num = blocks
    # fp32 mode: no reduced-precision matrix products anywhere
    torch.backends.cuda.matmul.allow_tf32 = torch.backends.cudnn.allow_tf32 = False
    return LLM(ec, device=device, dtype={"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype])


def replay(llm, lines, out_dir: str, report) -> None:
    """Runs the steps of ``lines`` (JSON texts) and calls ``report(step)`` after each."""
    import numpy as np

    from .ops import native
    engine, live = llm.engine, {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_given()
            entries.append((live[e["id"]], e["tokens"], e["want"]))
        if entries:
            logits = engine.step_given(entries)
            if logits.shape[0]:
                rows = logits.float().cpu().numpy().astype("<f4", copy=False)
                part = os.path.join(out_dir, f".{step['step']}.part")
                np.ascontiguousarray(rows).tofile(part)
                os.replace(part, os.path.join(out_dir, f"{step['step']}.f32"))
            if logits.is_cuda:
                native.check_err_flag(logits.device)
        for name in step.get("end", []):
            engine.close_given(live.pop(name))
        report(step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens held by live requests at any time")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: the plain PyTorch statements of the ops (tests)")
    a = ap.parse_args(argv)
    from . import build
    from .config import load_model_config
    cfg = load_model_config(a.model)
    if a.dtype == "float32" and a.device == "cuda" and cfg.layer_specs is None:
        print(f"model type {cfg.model_type} is not served in float32", file=sys.stderr)
        return 3
    build.ensure_built(only=build.FAMILY_KERNELS.get(cfg.model_type))
    import torch
    with torch.inference_mode():
        llm = make_llm(a.model, a.dtype, a.max_tokens, a.device)

        def report(step):
            print(f"done {step}", flush=True)

        replay(llm, sys.stdin, a.out, report)
    llm.shutdown()
    return 0
