"""ctypes bindings to ``libksana_kernels.so`` (the hand-written sm_100a kernels).

Every wrapper takes torch CUDA tensors, passes raw pointers plus the current CUDA stream and
raises if the native library is missing or a launch is rejected, so a GPU box can never fall
back silently to PyTorch ops.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from pathlib import Path
from typing import Optional

import torch

_LIB = None
_LIB_PATH = Path(__file__).resolve().parent.parent / "lib" / "libksana_kernels.so"

vp, i32, i64, f32 = C.c_void_p, C.c_int, C.c_longlong, C.c_float

_SIGS = {
    "ksana_gemm_bf16": [vp, i32, vp, i32, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp],
    "ksana_gemm_pair": [i32, vp, i32, vp, i32, vp, i32, vp, vp, i32, vp, vp, i32, i32, i32, i32, vp, i32, i32, vp, vp],
    "ksana_gemm_nvfp4": [vp, i32, vp, i32, vp, vp, i32, vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp],
    "ksana_gemm_bf16_batched": [vp, i64, i64, vp, i64, i64, vp, i64, i64, i32, i32, i32, i32, vp, i64, i64, vp, vp],
    "ksana_gemm_grouped_nvfp4": [vp, i32, vp, i32, vp, vp, i32, vp, i32, vp, vp, i32, i32, i32, i32, i32, vp, i32, vp, vp],
    "ksana_quant_nvfp4": [vp, i32, vp, i32, vp, i32, vp, i32, i32, vp],
    "ksana_gemm_mxfp8": [vp, i32, vp, i32, vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, vp, i32, i32, vp,
                         vp],
    "ksana_gemm_bf16_tall": [vp, i32, vp, i32, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, vp, vp],
    "ksana_gemm_mxfp8_tall": [vp, i32, vp, i32, vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, vp, i32, i32, vp,
                              vp],
    "ksana_gemm_mxfp8_pair": [vp, i32, vp, i32, vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, vp, i32, i32, vp, vp],
    "ksana_gemm_fp8_block": [vp, i32, vp, i32, vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp],
    "ksana_gemm_smallm": [i32, vp, i32, vp, i32, vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, vp, i64, vp, i32,
                          vp, vp],
    "ksana_gemm_grouped": [i32, vp, i32, vp, i32, vp, i32, vp, vp, i32, i32, i32, i32, i32, vp, vp, i32, vp, vp],
    "ksana_moe_route": [vp, i32, vp, vp, vp, i32, i32, i32, i32, i32, i32, f32, i32, i32, i32, i32, vp],
    "ksana_moe_align": [vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
    "ksana_moe_permute": [vp, vp, vp, i32, i32, i32, i32, vp, vp],
    "ksana_moe_combine": [vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
    "ksana_gemm_smallm_push": [i32, vp, i32, vp, i32, vp, i32, vp, i32, vp, i32, i32, i32, vp, i64, vp, i32, vp, i32, vp, vp],
    "ksana_gemm_smallm_push_signal": [i32, vp, i32, vp, i32, vp, i32, vp, i32, vp, i32, i32, i32, vp, i64, vp, i32, vp, i32,
                                      vp, vp, vp, vp, vp],
    "ksana_gemm_fp8_block_push": [vp, i32, vp, i32, vp, i32, vp, i32, vp, i32, i32, i32, i32, vp, i32, i32, vp, vp],
    "ksana_gemm_bf16_push": [vp, i32, vp, i32, i32, vp, i32, i32, i32, i32, vp, i32, i32, vp, vp],
    "ksana_reduce_norm": [vp, vp, i32, i32, vp, i64, i64, i32, i32, i32, i32, vp, vp, vp, f32, i32, vp, vp, vp, i32, i32,
                          i64, i64, i64, i64, C.c_ulonglong, vp, vp],
    "ksana_comm_barrier": [vp, vp, i32, i32, vp, vp, vp],
    "ksana_allreduce_pull": [vp, vp, i32, i32, vp, i64, vp, vp, i64, vp, vp],
    "ksana_allreduce_nvls": [vp, vp, i32, i32, vp, C.c_ulonglong, i64, vp, vp, i64, vp, vp],
    "ksana_allgather_pull": [vp, vp, i32, i32, vp, i64, vp, i32, i32, i32, i32, vp, vp],
    "ksana_norm": [vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, f32, i32, vp],
    "ksana_act_mul": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp],
    "ksana_act_mul_f32": [vp, vp, i32, i32, i32, i32, i32, vp],
    "ksana_quant_fp8": [vp, vp, vp, i32, i32, i32, i32, vp],
    "ksana_embedding": [vp, vp, vp, vp, vp, i32, i32, i32, i32, f32, vp],
    "ksana_gather_rows": [vp, vp, vp, i32, i32, i32, vp, vp],
    "ksana_refit_rows": [vp, vp, vp, i32, i32, vp],
    "ksana_rope_kv_append": [vp, vp, i32, vp, vp, vp, i64, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, f32, f32,
                             i32, vp],
    "ksana_copy_blocks": [vp, vp, i32, i64, i32, vp, vp],
    "ksana_swap_blocks": [vp, vp, vp, i32, i64, i32, i32, i32, vp, vp],
    "ksana_add": [vp, vp, vp, vp, i64, i32, vp],
    "ksana_patch_ids": [vp, vp, vp, vp, i32, i32, i32, vp, vp],
    "ksana_smallm_estimate": [i32, i32, i32, i32, vp],
    "ksana_absmax_scale": [vp, i32, i32, i64, f32, f32, vp, vp, vp],
    "ksana_rerotate_blocks": [vp, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32, i32, i64, vp, vp],
    "ksana_embed_pair": [vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i64, i64, i64, f32, i32, vp, vp],
    "ksana_residual_norm": [vp, i32, vp, i32, vp, i32, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, f32, i32, i32, f32, i32, vp, vp, f32,
                            vp, vp, i32, i32, i32, vp, i32, vp, vp],
    "ksana_glu_clamp": [vp, vp, i32, i32, i32, f32, f32, f32, vp, i32, vp],
    "ksana_embed_normed": [vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, f32, f32, i32, vp, vp],
    "ksana_token_shift": [vp, i64, vp, vp, i64, vp, i64, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
    "ksana_gated_norm": [vp, i64, vp, i64, vp, i64, vp, vp, i64, i32, i32, i32, i32, i32, f32, f32, i32, vp],
    "ksana_panel_append": [vp, i64, vp, vp, i64, i32, i32, i32, i32, i32, i32, vp, vp],
    "ksana_softcap": [vp, i64, i32, i32, f32, vp],
    "ksana_causal_conv": [vp, i64, vp, vp, vp, i64, i32, i32, vp, i64, vp, vp, vp, i32, i32, i32, i32, vp, vp],
    "ksana_state_space": [vp, i64, vp, vp, vp, i64, i32, vp, i64, vp, i64, vp, vp, vp, vp, i64, vp, i64, vp, vp, vp, i32, i32, i32, i32,
                          i32, i32, i32, vp, vp],
    "ksana_delta_rule": [vp, i64, vp, vp, i64, i32, vp, i64, vp, i64, vp, i64, vp, vp, vp, i64, vp, i64, vp, vp, vp, i32, i32, i32, i32,
                         i32, i32, f32, i32, vp, vp],
    "ksana_xielu": [vp, i32, vp, i32, i32, i32, f32, f32, f32, i32, vp],
    "ksana_gated_recurrence": [vp, vp, vp, i64, vp, i64, vp, i64, i32, i32, vp, i32, vp, vp, vp, i32, i32, f32, i32, vp, vp],
    "ksana_gemm_f32_batched": [vp, i32, i64, vp, i32, i64, vp, i32, i64, i32, i32, i32, i32, vp, i32, i64, vp],
    "ksana_qkv_rope_append": [vp, vp, vp, vp, i32, vp, vp, i64, i32, i32, i32, i32, i32, i32, i32, i32, i32, vp, vp],
    "ksana_qkv_norm_rope_append": [vp, vp, vp, vp, i32, vp, vp, f32, i32, i32, vp, vp, vp, i64, i32, i32, i32, i32, i32, i32, i32, i32,
                                   i32, vp, vp],
    "ksana_latent_norms": [vp, vp, i64, vp, vp, f32, vp, i32, i32, vp, vp, i64, i32, i64, i32, i32, vp, vp],
    "ksana_gemm_grouped_f32": [vp, i32, vp, i32, vp, i32, i32, i32, i32, i32, vp, vp],
    "ksana_refit_rows_f32": [vp, i32, vp, vp, i32, i32, i32, vp, vp],
    "ksana_gemm_f32": [vp, i32, vp, i32, vp, i32, vp, vp, i32, i32, i32, i32, vp],
    "ksana_attention_f32": [vp, i64, vp, i64, vp, vp, i32, i64, i32, i32, vp, i32, vp, vp, vp, vp, i64, i32, f32, vp, i32, i32, i32, i32,
                            i32, i32, i32, i32, i32, f32, i32, vp, vp],
    "ksana_cast_f32": [vp, vp, i64, vp],
    "ksana_paged_prefill_tc": [vp, i64, i64, vp, i64, vp, vp, i64, i32, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32,
                               i32, i32, f32, i32, vp, i32, vp, i64, f32, vp, vp],
    "ksana_paged_prefill": [vp, i64, vp, i64, vp, vp, i64, i32, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32,
                            f32, i32, f32, f32, i32, vp, i32, vp, i64, f32, vp, vp],
    "ksana_paged_decode": [vp, i64, vp, i64, vp, vp, i64, i32, vp, i32, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, i32,
                           f32, f32, i32, vp, vp, i32, vp, vp, i32, vp, i32, vp, i64, f32, vp, vp],
    "ksana_mla_attention": [vp, i64, vp, i64, vp, i64, i32, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp, i64, f32, i32, i32, vp,
                            vp, vp, vp],
    "ksana_mla_rope_append": [vp, i64, i32, vp, i64, vp, f32, vp, vp, vp, vp, vp, i64, i32, i32, i32, i32, i32, i32, i64, i32, vp, vp],
    "ksana_gemm_smallm_w4": [vp, i32, vp, vp, vp, i32, vp, i32, vp, vp, i32, i32, i32, i32, vp, i64, vp, i32, vp, vp],
    "ksana_w4_gemv": [vp, i64, vp, vp, vp, vp, vp, i64, vp, i64, i32, i32, i32, i32, vp],
    "ksana_w4_dequant": [vp, vp, vp, vp, i64, i32, i32, i32, vp],
    "ksana_sample": [vp, i64, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp, i32, i32, vp],
    "ksana_sample_merged": [vp, i64, vp, i64, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp, i32, i32, vp],
    "ksana_shard_topk": [vp, i64, vp, i32, i32, i32, i32, vp, vp, vp],
    "ksana_repetition_penalty": [vp, i64, vp, vp, vp, vp, i32, i32, vp],
    "ksana_ban_tokens": [vp, i64, vp, vp, vp, i32, i32, vp],
}

_launches = 0


def launch_count() -> int:
    """Number of native kernel launches issued through this module (bench accounting)."""
    return _launches


def available() -> bool:
    return _LIB_PATH.exists()


_recorder = None
_recorded_tensors: list = []              # arguments seen while recording: their memory is not given to anyone else


class _RecordingLib:
    """Stand-in for the library handle while a launch recorder is installed: every entry point called through it
    is appended to the recorder as (name, function, arguments) before it runs."""

    def __init__(self, real, rec):
        self._real, self._rec = real, rec

    def __getattr__(self, name):
        fn = getattr(self._real, name)
        rec = self._rec

        def call(*args):
            rec.append((name, fn, args))
            return fn(*args)
        return call


class recording:
    """Context manager: collects every native launch issued inside it into ``calls`` (used by the step breakdown
    in benchmarks/step_breakdown.py, which replays subsets of a step's launches in graphs of their own)."""

    def __init__(self, calls: list):
        self.calls = calls

    def __enter__(self):
        global _recorder
        _recorder = self.calls
        _recorded_tensors.clear()
        return self.calls

    def __exit__(self, *exc):
        global _recorder
        _recorder = None
        self.tensors = list(_recorded_tensors)
        _recorded_tensors.clear()
        return False


def lib():
    if _recorder is not None:
        return _RecordingLib(_load(), _recorder)
    return _load()


def _load():
    global _LIB
    if _LIB is None:
        if not _LIB_PATH.exists():
            raise RuntimeError(
                f"native kernel library {_LIB_PATH} is missing: run `python -m ksanallm_b200.build` "
                "(CUDA tensors are never served by a PyTorch fallback)")
        _LIB = C.CDLL(str(_LIB_PATH))
        for name, sig in _SIGS.items():
            fn = getattr(_LIB, name, None)
            if fn is not None:
                fn.argtypes = sig
                fn.restype = C.c_int
    return _LIB


def _p(t: Optional[torch.Tensor]):
    if t is None:
        return None
    if _recorder is not None:
        _recorded_tensors.append(t)
    return t.data_ptr()


def _st():
    return torch.cuda.current_stream().cuda_stream


def _check(rc: int, name: str):
    global _launches
    _launches += 1
    if rc != 0:
        raise RuntimeError(f"{name} rejected its arguments or failed to launch (code {rc})")


_err_flags = {}


def err_flag(device) -> torch.Tensor:
    """Per-device int32 word that kernels with bounded waits set when a wait gave up."""
    d = torch.device(device)
    key = (d.type, d.index or 0)
    if key not in _err_flags:
        _err_flags[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _err_flags[key]


def describe_err_code(code: int) -> str:
    if code >= 1000000:
        names = {11: "block-table entry", 12: "sequence row range", 13: "position", 14: "cache slot", 15: "expert id",
                 16: "expert destination row", 17: "gather row index"}
        return (f"a kernel skipped an out-of-range {names.get(code // 1000000, 'index')} "
                f"(value mod 1e6 = {code % 1000000}); the step's results are invalid")
    what = {2: "a tensor-core GEMM gave up waiting for its operands", 3: "a wait for a peer GPU's flag ran out",
            4: "an attention kernel gave up waiting for its K/V tiles"}.get(code, "a device-side bounded wait timed out")
    return f"{what} (kernel reported error status {code})"


def clear_err_flag(device) -> None:
    with torch.inference_mode():              # the word may have been created inside the engine's inference mode
        err_flag(device).zero_()


def check_err_flag(device) -> None:
    """Reads the device error word (synchronises the stream); raises and clears it when a kernel reported."""
    code = int(err_flag(device).item())
    if code != 0:
        clear_err_flag(device)
        raise RuntimeError(describe_err_code(code))


# ------------------------------------------------------------------------------------- GEMM
import os as _os

SMALL_M_FP8 = int(_os.environ.get("KSANA_SKINNY_MAX_M", "32"))   # FP8: rows up to which the skinny stream-K kernel always runs
SMALL_M_BF16 = 128                 # bf16: no per-K-block promotion, the skinny kernel wins up to a full token tile
_SCRATCH_BYTES = 64 << 20
_COUNTERS = 4096
_workspaces = {}


def gemm_workspace(device):
    """Per-device scratch for tiles whose K range is cut across CTAs (fp32 partial tiles) and the tile
    arrival counters (zeroed once; the kernel leaves them zero). Launches that share it must be
    ordered on one stream. ``splits`` of the GEMM wrappers: 0 = automatic, > 0 = number of persistent
    CTAs, < 0 = force the skinny kernel for M up to 128."""
    key = torch.device(device).index or 0
    if key not in _workspaces:
        _workspaces[key] = (torch.empty(_SCRATCH_BYTES // 4, dtype=torch.float32, device=device),
                            torch.zeros(_COUNTERS, dtype=torch.int32, device=device))
    return _workspaces[key]


def _gemm_smallm(kind, x, xs, w, ws, out, out_f32, bias, residual, M, N, K, splits):
    dst = out if out_f32 is None else out_f32
    scratch, counters = gemm_workspace(x.device)
    rc = lib().ksana_gemm_smallm(kind, _p(x), x.stride(0), _p(xs), xs.stride(0) if xs is not None else 0, _p(w),
                                 w.stride(0), _p(ws), _p(out) if out_f32 is None else None, _p(out_f32), dst.stride(0),
                                 _p(bias), _p(residual), residual.stride(0) if residual is not None else 0, M, N, K,
                                 max(splits, 0), _p(scratch), scratch.numel() * 4, _p(counters), counters.numel(),
                                 _p(err_flag(x.device)), _st())
    _check(rc, "ksana_gemm_smallm")
    return dst


PAIR_MIN_M = 0                     # CTA-pair (cta_group::2) kernel from this many rows; 0 disables it


def gemm_pair(kind, x, xs, w, ws, out, bias=None, residual=None, push=None, push_n=0, push_rows=0):
    """CTA-pair tcgen05 GEMM (256 x 256 tiles over two SMs). kind 0: bf16, 1: block-scaled FP8. bf16 output only."""
    M, K = x.shape
    N = w.shape[0]
    rc = lib().ksana_gemm_pair(kind, _p(x), x.stride(0), _p(xs), xs.stride(0) if xs is not None else 0, _p(w),
                               w.stride(0), _p(ws), _p(out), out.stride(0) if out is not None else N, _p(bias),
                               _p(residual), residual.stride(0) if residual is not None else 0, M, N, K, push, push_n,
                               push_rows, _p(err_flag(x.device)), _st())
    _check(rc, "ksana_gemm_pair")
    return out


BF16_TALL_MIN_M = 0                # 256 x 256-tile bf16 kernel from this many rows; 0 disables it


def gemm_bf16_tall(x, w, out=None, bias=None, residual=None, out_f32=None, max_ctas=0):
    """bf16 GEMM with 256 x 256 tiles per CTA (two 128-row MMAs share every weight tile)."""
    M, K = x.shape
    N = w.shape[0]
    dst = out if out_f32 is None else out_f32
    rc = lib().ksana_gemm_bf16_tall(_p(x), x.stride(0), _p(w), w.stride(0), _p(out) if out_f32 is None else None,
                                    _p(out_f32), dst.stride(0), _p(bias), _p(residual),
                                    residual.stride(0) if residual is not None else 0, M, N, K, max_ctas,
                                    _p(err_flag(x.device)), _st())
    _check(rc, "ksana_gemm_bf16_tall")
    return dst


def _pair_ok(M, N, K, kind, bn, out_f32, max_ctas):
    return (PAIR_MIN_M > 0 and M >= PAIR_MIN_M and bn == 0 and max_ctas == 0 and out_f32 is None and N % 8 == 0
            and N >= 256 and K % (128 if kind else 8) == 0)


def gemm_bf16(x, w, out=None, bias=None, residual=None, out_f32=None, bn=0, max_ctas=0, splits=0):
    """out[M,N] = x[M,K] @ w[N,K]^T (+bias)(+residual). bf16 in, bf16 (or fp32) out."""
    M, K = x.shape
    N = w.shape[0]
    assert x.stride(1) == 1 and w.stride(1) == 1 and w.shape[1] == K
    if out is None and out_f32 is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    dst = out if out_f32 is None else out_f32
    if (M <= SMALL_M_BF16 or splits < 0) and M <= 128 and bn == 0 and K % 8 == 0:
        return _gemm_smallm(0, x, None, w, None, out, out_f32, bias, residual, M, N, K, splits)
    if (BF16_TALL_MIN_M > 0 and M >= BF16_TALL_MIN_M and bn == 0 and splits == 0 and N % 8 == 0 and K % 8 == 0
            and ((M + 255) // 256) * ((N + 255) // 256) >= 148):
        return gemm_bf16_tall(x, w, out, bias, residual, out_f32, max_ctas)
    if _pair_ok(M, N, K, 0, bn, out_f32, max_ctas):
        return gemm_pair(0, x, None, w, None, out, bias, residual)
    rc = lib().ksana_gemm_bf16(_p(x), x.stride(0), _p(w), w.stride(0), _p(out) if out_f32 is None else None,
                               _p(out_f32), dst.stride(0), _p(bias), _p(residual),
                               residual.stride(0) if residual is not None else 0, M, N, K, bn, max_ctas,
                               _p(err_flag(x.device)), _st())
    _check(rc, "ksana_gemm_bf16")
    return dst


MX_MIN_M = 33                      # hardware-scaled kernel from this many rows (below: the skinny stream-K kernel)


def gemm_mxfp8(xq, xs, wq, ws, out=None, bias=None, residual=None, out_f32=None, bn=0, max_ctas=0, push=None,
               push_n=0, push_rows=0, ldd=None):
    """FP8 GEMM whose power-of-two scales are applied by the tensor cores (tcgen05 block_scale MMA)."""
    M, K = xq.shape
    N = wq.shape[0]
    dst = out if out_f32 is None else out_f32
    rc = lib().ksana_gemm_mxfp8(_p(xq), xq.stride(0), _p(xs), xs.stride(0), _p(wq), wq.stride(0), _p(ws),
                                _p(out) if out_f32 is None else None, _p(out_f32),
                                dst.stride(0) if dst is not None else ldd, _p(bias), _p(residual),
                                residual.stride(0) if residual is not None else 0, M, N, K, bn, max_ctas, push, push_n,
                                push_rows, _p(err_flag(xq.device)), _st())
    _check(rc, "ksana_gemm_mxfp8")
    return dst


MX_TALL_MIN_M = 512                # 256 x 224-tile hardware-scaled kernel from this many rows (measured faster); 0 disables it


def _tall_wins(M, N, K, max_ctas=0, sms=148):
    """256 x 224 tiles against 128 x 256 tiles for one problem, from measured behaviour: the tall tile does 1.75
    times the MMA work at about 1.18 times the rate but cannot overlap its accumulator drain (about three K
    blocks of time per tile), so it needs a long K and a tile count that fills its last wave."""
    if K < 4096:
        return False
    ctas = min(sms, max_ctas) if max_ctas > 0 else sms
    kb = K // 128
    t_tall = ((M + 255) // 256) * ((N + 223) // 224)
    t_std = ((M + 127) // 128) * ((N + 255) // 256)
    if t_tall < ctas:
        return False
    tall = -(-t_tall // ctas) * (1.75 * kb + 3.0) / 1.18
    std = -(-t_std // ctas) * (kb + 0.5)
    return tall < std


def gemm_mxfp8_tall(xq, xs, wq, ws, out=None, bias=None, residual=None, out_f32=None, max_ctas=0, push=None, push_n=0,
                    push_rows=0, ldd=None):
    """Hardware-scaled FP8 GEMM with 256 x 224 tiles per CTA (less operand traffic per MMA than 128 x 256)."""
    M, K = xq.shape
    N = wq.shape[0]
    dst = out if out_f32 is None else out_f32
    rc = lib().ksana_gemm_mxfp8_tall(_p(xq), xq.stride(0), _p(xs), xs.stride(0), _p(wq), wq.stride(0), _p(ws),
                                     _p(out) if out_f32 is None else None, _p(out_f32),
                                     dst.stride(0) if dst is not None else ldd, _p(bias), _p(residual),
                                     residual.stride(0) if residual is not None else 0, M, N, K, max_ctas, push, push_n,
                                     push_rows, _p(err_flag(xq.device)), _st())
    _check(rc, "ksana_gemm_mxfp8_tall")
    return dst


MX_PAIR_MIN_M = 0                  # CTA-pair hardware-scaled kernel from this many rows; 0 disables it


def gemm_mxfp8_pair(xq, xs, wq, ws, out=None, bias=None, residual=None, out_f32=None, push=None, push_n=0, push_rows=0,
                    ldd=None):
    """Hardware-scaled FP8 GEMM on CTA pairs (256 x 256 tiles over two SMs, tcgen05 cta_group::2 block_scale MMA)."""
    M, K = xq.shape
    N = wq.shape[0]
    dst = out if out_f32 is None else out_f32
    rc = lib().ksana_gemm_mxfp8_pair(_p(xq), xq.stride(0), _p(xs), xs.stride(0), _p(wq), wq.stride(0), _p(ws),
                                     _p(out) if out_f32 is None else None, _p(out_f32),
                                     dst.stride(0) if dst is not None else ldd, _p(bias), _p(residual),
                                     residual.stride(0) if residual is not None else 0, M, N, K, push, push_n,
                                     push_rows, _p(err_flag(xq.device)), _st())
    _check(rc, "ksana_gemm_mxfp8_pair")
    return dst


def _skinny_wins_mx(M, N, K, sms=148):
    """Rows 33..128 with tensor-core-applied scales: skinny stream-K kernel or tiled kernel, from their measured
    behaviour in CUDA graphs of decode steps (microseconds). Tiled: about 6.5 + 0.37 per 128-deep K block and wave of
    128 x 128 tiles (0.69 with 128 x 256 tiles); one CTA walks the whole K range of its tile, so few tiles leave
    SMs idle. Skinny: the (tile, K block) units are spread evenly over the SMs at about 0.62 per K block and CTA for 64
    rows (0.9 for 128), plus a higher fixed cost and the cross-CTA reduction of cut tiles."""
    kb = K // 128
    t128 = (N + 127) // 128
    t256 = (N + 255) // 256
    if t256 >= 100:
        tiled = 6.5 + -(-t256 // sms) * kb * 0.69
    else:
        tiled = 6.5 + -(-t128 // sms) * kb * 0.37
    units = t128 * kb
    ctas = min(sms, max(1, units // 4))
    per_cta = -(-units // ctas)
    pieces = -(-kb // max(1, per_cta)) + 1 if per_cta < kb else 1
    skinny = 11.5 + 0.15 * pieces + per_cta * (0.62 if M <= 64 else 0.9)
    return skinny < tiled


def gemm_fp8(xq, xs, wq, ws, out=None, bias=None, residual=None, out_f32=None, bn=0, max_ctas=0, splits=0,
             hw_scale=False):
    """Block-scaled FP8 GEMM. xq [M,K] e4m3, xs [K/128, ld] fp32; wq [N,K] e4m3, ws [ceil(N/128), K/128] fp32.
    hw_scale: every scale is a power of two, so the tensor cores may apply them (large-M path)."""
    M, K = xq.shape
    N = wq.shape[0]
    if out is None and out_f32 is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=xq.device)
    dst = out if out_f32 is None else out_f32
    if hw_scale:
        # power-of-two scales: both kernels let the tensor cores apply them. Skinny stream-K kernel for decode-sized
        # M and wherever the tiled kernel would leave most SMs idle; tiled kernel otherwise (256-wide tiles when
        # they fill the SMs).
        t256 = ((M + 127) // 128) * ((N + 255) // 256)
        skinny = M <= SMALL_M_FP8 or (M <= 128 and _skinny_wins_mx(M, N, K))
        if (skinny or splits != 0) and M <= 128 and bn == 0:
            return _gemm_smallm(2, xq, xs, wq, ws, out, out_f32, bias, residual, M, N, K, splits)
        if MX_TALL_MIN_M > 0 and M >= MX_TALL_MIN_M and bn == 0 and _tall_wins(M, N, K, max_ctas):
            return gemm_mxfp8_tall(xq, xs, wq, ws, out, bias, residual, out_f32, max_ctas)
        if MX_PAIR_MIN_M > 0 and M >= MX_PAIR_MIN_M and bn == 0 and max_ctas == 0 and t256 >= 148:
            return gemm_mxfp8_pair(xq, xs, wq, ws, out, bias, residual, out_f32)
        if bn == 0 or bn >= 128:
            return gemm_mxfp8(xq, xs, wq, ws, out, bias, residual, out_f32, bn or (256 if t256 >= 100 else 128),
                              max_ctas)
    skinny = M <= SMALL_M_FP8 or (M <= 64 and K >= 16384 and N <= 16384)
    if (skinny or splits < 0) and M <= 128 and bn == 0:
        return _gemm_smallm(1, xq, xs, wq, ws, out, out_f32, bias, residual, M, N, K, splits)
    if bn == 0 and M <= 128:
        bn = 128 if N >= 10240 else 64     # decode-sized rows on the tiled kernel: measured best tile widths
    rc = lib().ksana_gemm_fp8_block(_p(xq), xq.stride(0), _p(xs), xs.stride(0), _p(wq), wq.stride(0), _p(ws),
                                    _p(out) if out_f32 is None else None, _p(out_f32), dst.stride(0), _p(bias),
                                    _p(residual), residual.stride(0) if residual is not None else 0, M, N, K, bn,
                                    max_ctas, _p(err_flag(xq.device)), _st())
    _check(rc, "ksana_gemm_fp8_block")
    return dst


_absmax_acc = {}


def absmax_scale(x, divisor: float, floor: float = 1e-12):
    """max(|x|) / divisor (at least ``floor``) of a bf16 matrix as an fp32 scalar tensor on the device: the tensor
    scale of an NVFP4 activation, without a host round trip or a widened copy of ``x``."""
    rows, cols = x.shape
    key = (x.device.type, x.device.index)
    acc = _absmax_acc.get(key)
    if acc is None:
        acc = _absmax_acc[key] = torch.zeros(1, dtype=torch.int32, device=x.device)
    scale = torch.empty((), dtype=torch.float32, device=x.device)
    _check(lib().ksana_absmax_scale(_p(x), rows, cols, x.stride(0), float(divisor), float(floor), _p(acc), _p(scale),
                                    _st()), "ksana_absmax_scale")
    return scale


def quant_nvfp4(x, tensor_scale):
    """bf16 [M, K] -> (packed e2m1 [M, K/2] uint8, e4m3 block scales [M, K/16], tensor_scale). K % 16 == 0.
    ``tensor_scale``: fp32 scalar tensor on the device (calibrated or amax / (448 * 6))."""
    M, K = x.shape
    q = torch.empty(M, K // 2, dtype=torch.uint8, device=x.device)
    bs = torch.empty(M, K // 16, dtype=torch.float8_e4m3fn, device=x.device)
    _check(lib().ksana_quant_nvfp4(_p(x), x.stride(0), _p(q), q.stride(0), _p(bs), bs.stride(0), _p(tensor_scale), M, K,
                                   _st()), "ksana_quant_nvfp4")
    return q, bs, tensor_scale


def gemm_nvfp4(aq, a_bs, a_ts, wq, w_bs, w_ts, out=None, bias=None, residual=None, out_f32=None, bn=0, max_ctas=0):
    """NVFP4 x NVFP4 GEMM (e2m1 values, e4m3 scales per 16 elements, fp32 tensor scales) on the block-scaled tensor
    cores. aq [M, K/2], wq [N, K/2] packed bytes; K % 256 == 0."""
    M, N, K = aq.shape[0], wq.shape[0], aq.shape[1] * 2
    if out is None and out_f32 is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=aq.device)
    dst = out if out_f32 is None else out_f32
    rc = lib().ksana_gemm_nvfp4(_p(aq), aq.stride(0), _p(a_bs), a_bs.stride(0), _p(a_ts), _p(wq), wq.stride(0), _p(w_bs),
                                w_bs.stride(0), _p(w_ts), _p(out) if out_f32 is None else None, _p(out_f32),
                                dst.stride(0), _p(bias), _p(residual), residual.stride(0) if residual is not None else 0,
                                M, N, K, bn, max_ctas, _p(err_flag(aq.device)), _st())
    _check(rc, "ksana_gemm_nvfp4")
    return dst


def _gate_args(gate, out):
    if gate is None:
        return None, 0, 0
    assert gate.shape == out.shape and gate.dtype == out.dtype and gate.stride(2) == 1
    return _p(gate), gate.stride(1), gate.stride(0)


def gemm_bf16_batched(a, w, out, gate=None):
    """out[b] = a[b] @ w[b]^T for every b: a [B, M, K], w [B, N, K], out [B, M, N], bf16 views with unit stride in the
    last dimension and any (16-byte aligned) strides in the others, e.g. head-interleaved activations
    ``x.view(T, H, D).transpose(0, 1)``. One launch of the tcgen05 GEMM over all batch entries' tiles. ``gate`` [B, M, N]:
    the result is multiplied with sigmoid(gate) before it is stored."""
    B, M, K = a.shape
    N = w.shape[1]
    assert w.shape[0] == B and w.shape[2] == K and tuple(out.shape) == (B, M, N)
    assert a.stride(2) == 1 and w.stride(2) == 1 and out.stride(2) == 1
    rc = lib().ksana_gemm_bf16_batched(_p(a), a.stride(1), a.stride(0), _p(w), w.stride(1), w.stride(0), _p(out),
                                       out.stride(1), out.stride(0), B, M, N, K, *_gate_args(gate, out), _p(err_flag(a.device)), _st())
    _check(rc, "ksana_gemm_bf16_batched")
    return out


def gemm_grouped_nvfp4(aq, a_bs, a_ts, wq, w_bs, w_ts, tile_expert, E, N, out=None, bn=0):
    """Expert-major NVFP4 rows ``aq`` [cap, K/2] (128-row tiles, one expert each, ``tile_expert`` < 0: unused) times
    the experts' stacked NVFP4 matrices ``wq`` [E * N, K/2] with block scales ``w_bs`` [E * N, K/16] and one tensor
    scale per expert ``w_ts`` [E]. Rows of unused tiles are left untouched."""
    cap, K = aq.shape[0], aq.shape[1] * 2
    if out is None:
        out = torch.zeros(cap, N, dtype=torch.bfloat16, device=aq.device)
    rc = lib().ksana_gemm_grouped_nvfp4(_p(aq), aq.stride(0), _p(a_bs), a_bs.stride(0), _p(a_ts), _p(wq), wq.stride(0),
                                        _p(w_bs), w_bs.stride(0), _p(w_ts), _p(out), out.stride(0), cap, N, K, E,
                                        _p(tile_expert), bn, _p(err_flag(aq.device)), _st())
    _check(rc, "ksana_gemm_grouped_nvfp4")
    return out


W4_TENSOR_CORE = True        # rows 3..128: expand-in-kernel + tcgen05 (the CUDA-core GEMV is compute bound beyond 2 rows)
W4_GEMV_MAX_M = 32          # up to this many rows the 4-bit weights are streamed by the GEMV kernel (8 rows per pass)
_w4_scratch = {}


def linear_w4(x, q4, scale, zs, out=None, bias=None, residual=None):
    """y = x W^T (+bias, +residual) for 4-bit group-quantised W (see csrc/kernels/w4a16.cu)."""
    M, K = x.shape
    N = q4.shape[0]
    g = K // scale.shape[1]
    if out is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    if W4_TENSOR_CORE and 2 < M <= 128 and g % 64 == 0 and K % 64 == 0:
        # weight stream on the tensor cores: four warps expand the packed tiles to bf16 in shared memory, the rest is
        # the stream-K skinny GEMM
        scratch, counters = gemm_workspace(x.device)
        rc = lib().ksana_gemm_smallm_w4(_p(x), x.stride(0), _p(q4), _p(scale), _p(zs), g, _p(out), out.stride(0), _p(bias),
                                        _p(residual), residual.stride(0) if residual is not None else 0, M, N, K,
                                        _p(scratch), scratch.numel() * 4, _p(counters), counters.numel(),
                                        _p(err_flag(x.device)), _st())
        _check(rc, "ksana_gemm_smallm_w4")
        return out
    if M <= W4_GEMV_MAX_M:
        rc = lib().ksana_w4_gemv(_p(x), x.stride(0), _p(q4), _p(scale), _p(zs), _p(bias), _p(residual),
                                 residual.stride(0) if residual is not None else 0, _p(out), out.stride(0), M, N, K, g, _st())
        _check(rc, "ksana_w4_gemv")
        return out
    # compute-bound: expand once into a per-device scratch matrix shared by all layers, then the tcgen05 bf16 GEMM
    key = (x.device.index or 0)
    buf = _w4_scratch.get(key)
    if buf is None or buf.numel() < N * K:
        buf = torch.empty(N * K, dtype=torch.bfloat16, device=x.device)
        _w4_scratch[key] = buf
    w = buf[: N * K].view(N, K)
    _check(lib().ksana_w4_dequant(_p(q4), _p(scale), _p(zs), _p(w), K, N, K, g, _st()), "ksana_w4_dequant")
    return gemm_bf16(x, w, out=out, bias=bias, residual=residual)


def quant_fp8(x, q=None, s=None):
    M, K = x.shape
    if q is None:
        q = torch.empty(M, K, dtype=torch.float8_e4m3fn, device=x.device)
    if s is None:
        s = torch.empty(K // 128, max(4, (M + 3) // 4 * 4), dtype=torch.float32, device=x.device)
    _check(lib().ksana_quant_fp8(_p(x), _p(q), _p(s), s.stride(0), M, K, x.stride(0), _st()), "ksana_quant_fp8")
    return q, s


# -------------------------------------------------------------------------------- elementwise
def norm(x, w, eps, residual=None, beta=None, out=None, layernorm=False, quant=False, q=None, s=None,
         want_out=True):
    """y = norm(x (+residual, updated in place)) * w (+beta); optionally also the FP8 operand of y."""
    M, H = x.shape
    if want_out and out is None:
        out = torch.empty(M, H, dtype=torch.bfloat16, device=x.device)
    if quant:
        if q is None:
            q = torch.empty(M, H, dtype=torch.float8_e4m3fn, device=x.device)
        if s is None:
            s = torch.empty(H // 128, max(4, (M + 3) // 4 * 4), dtype=torch.float32, device=x.device)
    rc = lib().ksana_norm(_p(x), _p(residual), _p(w), _p(beta), _p(out) if want_out else None, _p(q) if quant else None,
                          _p(s) if quant else None, s.stride(0) if quant else 0, M, H, float(eps), int(layernorm),
                          _st())
    _check(rc, "ksana_norm")
    return (out, q, s) if quant else out


_ACTS = {"silu": 0, "swiglu": 0, "gelu": 1, "gelu_new": 1, "gelu_pytorch_tanh": 1, "relu": 2}


def act_mul(x, act="silu", gated=True, out=None, quant=False, q=None, s=None, want_out=True, tile_rows=None):
    """``tile_rows``: of every 128 rows only so many hold anything (expert-major rows); the others are skipped."""
    M = x.shape[0]
    inter = x.shape[1] // 2 if gated else x.shape[1]
    if x.dtype == torch.float32:
        out = torch.empty(M, inter, dtype=x.dtype, device=x.device)
        _check(lib().ksana_act_mul_f32(_p(x), _p(out), M, inter, x.stride(0), _ACTS[act], int(gated), _st()), "ksana_act_mul_f32")
        return out
    if want_out and out is None:
        out = torch.empty(M, inter, dtype=torch.bfloat16, device=x.device)
    if quant:
        if q is None:
            q = torch.empty(M, inter, dtype=torch.float8_e4m3fn, device=x.device)
        if s is None:
            s = torch.empty(inter // 128, max(4, (M + 3) // 4 * 4), dtype=torch.float32, device=x.device)
    rc = lib().ksana_act_mul(_p(x), _p(out) if want_out else None, _p(q) if quant else None, _p(s) if quant else None,
                             s.stride(0) if quant else 0, M, inter, x.stride(0), _ACTS[act], int(gated), _p(tile_rows), _st())
    _check(rc, "ksana_act_mul")
    return (out, q, s) if quant else out


def embedding(ids, table, out=None, vocab_lo=0, vocab_hi=None, positions=None, pos_table=None, scale=1.0):
    T, H = ids.numel(), table.shape[1]
    if out is None:
        out = torch.empty(T, H, dtype=torch.bfloat16, device=table.device)
    hi = vocab_lo + table.shape[0] if vocab_hi is None else vocab_hi
    rc = lib().ksana_embedding(_p(ids), _p(table), _p(positions), _p(pos_table), _p(out), T, H, vocab_lo, hi,
                               float(scale), _st())
    _check(rc, "ksana_embedding")
    return out


def gather_rows(x, idx, out=None):
    R, H = idx.numel(), x.shape[1]
    if out is None:
        out = torch.empty(R, H, dtype=torch.bfloat16, device=x.device)
    _check(lib().ksana_gather_rows(_p(x), _p(idx), _p(out), R, H, int(x.shape[0]), _p(err_flag(x.device)), _st()),
           "ksana_gather_rows")
    return out


def refit_rows(hidden, pos, emb):
    _check(lib().ksana_refit_rows(_p(hidden), _p(pos), _p(emb), pos.numel(), hidden.shape[1], _st()),
           "ksana_refit_rows")


def patch_ids(ids, rows, src, prev_tokens):
    """ids[rows[i]] = prev_tokens[src[i]] on the device (all int32)."""
    _check(lib().ksana_patch_ids(_p(ids), _p(rows), _p(src), _p(prev_tokens), rows.numel(), ids.numel(),
                                 prev_tokens.numel(), _p(err_flag(ids.device)), _st()), "ksana_patch_ids")


def rerotate_blocks(cache, triples, cos_sin, rot_dim, neox):
    """Rotate the K rows of the destination blocks of ``triples`` (int32 [n, 3] on the device: source block,
    destination block, position delta) by their position deltas, in place. ``cache``: [blocks, layers, 2, kv heads,
    block tokens, head dim], bf16 or e4m3; ``cos_sin``: [max_pos, rot_dim] fp32."""
    nb, layers, _, hkv, bt, D = cache.shape
    _check(lib().ksana_rerotate_blocks(_p(cache), _p(triples), triples.shape[0], _p(cos_sin), cos_sin.shape[0], layers,
                                       hkv, bt, D, rot_dim, int(bool(neox)), cache.element_size(), nb, 0,
                                       _p(err_flag(cache.device)), _st()), "ksana_rerotate_blocks")


def rerotate_panel(k_panel, triples, cos_sin, rot_dim, neox=True):
    """:func:`rerotate_blocks` for one layer whose K panels [blocks, kv heads, block tokens, head dim] (bf16) sit inside
    larger block records."""
    nb, hkv, bt, D = k_panel.shape
    _check(lib().ksana_rerotate_blocks(_p(k_panel), _p(triples), triples.shape[0], _p(cos_sin), cos_sin.shape[0], 1, hkv, bt, D,
                                       rot_dim, int(bool(neox)), k_panel.element_size(), nb, int(k_panel.stride(0)),
                                       _p(err_flag(k_panel.device)), _st()), "ksana_rerotate_blocks")


def add(a, b=None, bias=None, out=None):
    if out is None:
        out = torch.empty_like(a)
    H = a.shape[-1]
    _check(lib().ksana_add(_p(a), _p(b), _p(bias), _p(out), a.numel() // H, H, _st()), "ksana_add")
    return out


def cast_f32(x, out=None):
    if out is None:
        out = torch.empty(x.shape, dtype=torch.float32, device=x.device)
    _check(lib().ksana_cast_f32(_p(x), _p(out), x.numel(), _st()), "ksana_cast_f32")
    return out


# -------------------------------------------------------------------------- 32-bit residual stream
def gemm_f32(x, w, out=None, bias=None, residual=None):
    """out[M,N] = x[M,K] @ w[N,K]^T (+bias)(+residual), everything fp32 on the CUDA cores."""
    M, K = x.shape
    N = w.shape[0]
    assert x.dtype == w.dtype == torch.float32 and x.stride(1) == 1 and w.stride(1) == 1 and w.shape[1] == K
    if out is None:
        out = torch.empty(M, N, dtype=torch.float32, device=x.device)
    _check(lib().ksana_gemm_f32(_p(x), x.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), _p(bias), _p(residual),
                                residual.stride(0) if residual is not None else 0, M, N, K, _st()), "ksana_gemm_f32")
    return out


def embed_pair(ids, prev, table, pair, scale, buckets=0, mul_prev=0, mul_cur=0, copy=None, vocab=None):
    """fp32 rows table[id] * scale (+ the pair table's row of (previous id, id)); ``copy``: the same rows in the table's
    type (a strided view is fine)."""
    T, H = ids.numel(), table.shape[1]
    x = torch.empty(T, H, dtype=torch.float32, device=table.device)
    _check(lib().ksana_embed_pair(_p(ids), _p(prev), _p(table), _p(pair), _p(x), _p(copy), copy.stride(0) if copy is not None else 0,
                                  T, H, vocab or table.shape[0], buckets, mul_prev, mul_cur, float(scale),
                                  int(table.dtype == torch.float32), _p(err_flag(table.device)), _st()), "ksana_embed_pair")
    return x


def residual_norm(x, H, eps, y=None, w1=None, b1=None, ls=None, x_out=None, w2=None, b2=None, z=None, rows=None, rms=False,
                  alpha=1.0, groups=1, add=None, vec=None, z_scale=1.0, experts=None):
    """One pass over rows of the fp32 stream ``x`` (``H`` real columns, padded to a multiple of 8):
    x' = x + alpha * ls * norm(y; w1, b1) + add + vec, stored to ``x_out``; z = z_scale * norm(x'; w2, b2), or a copy of x'
    without ``w2``. Parts whose arguments are None are left out; ``rows`` gathers stream rows. ``groups`` > 1: the stream's
    norm (RMS, without ``w1``) is taken for each of that many equal parts of a row. ``add``: fp32 rows like x, ``vec``: one
    row of the activations' type. ``experts`` = (dst_row [M, K], weights [M, K or K + 1], shared or None): y are expert outputs
    and a row's addend is the sum of weights[k] * y[dst_row[k]] (+ weights[K] * shared)."""
    M = rows.numel() if rows is not None else x.shape[0]
    t = z if z is not None else y if y is not None else vec
    dst_row, w, shared = experts if experts is not None else (None, None, None)
    top = dst_row.numel() // max(M, 1) if dst_row is not None else 0
    assert add is None or (add.dtype == torch.float32 and add.stride(0) == x.stride(0))
    _check(lib().ksana_residual_norm(_p(x), x.stride(0), _p(rows), x.shape[0], _p(y), y.stride(0) if y is not None else 0, _p(w1),
                                     _p(b1), _p(ls), _p(x_out), _p(w2), _p(b2), _p(z), z.stride(0) if z is not None else 0, M, H,
                                     float(eps), int(rms), int(t is None or t.dtype == torch.float32), float(alpha), int(groups),
                                     _p(add), _p(vec), float(z_scale), _p(dst_row), _p(w), w.stride(0) if w is not None else 0, top,
                                     y.shape[0] if dst_row is not None else 0, _p(shared),
                                     shared.stride(0) if shared is not None else 0, _p(err_flag(x.device)), _st()),
           "ksana_residual_norm")


def glu_clamp(x, limit, alpha, offset, tile_rows=None):
    """``tile_rows``: of every 128 rows only so many hold anything; the others are skipped."""
    M, I = x.shape[0], x.shape[1] // 2
    out = torch.empty(M, I, dtype=x.dtype, device=x.device)
    _check(lib().ksana_glu_clamp(_p(x), _p(out), M, I, x.stride(0), float(limit), float(alpha), float(offset),
                                 _p(tile_rows), int(x.dtype == torch.float32), _st()), "ksana_glu_clamp")
    return out


def xielu(x, pos, neg, lin, out=None):
    M, I = x.shape
    if out is None:
        out = torch.empty(M, I, dtype=x.dtype, device=x.device)
    _check(lib().ksana_xielu(_p(x), x.stride(0), _p(out), out.stride(0), M, I, float(pos), float(neg), float(lin),
                             int(x.dtype == torch.float32), _st()), "ksana_xielu")
    return out


def gated_recurrence(z, u, g, out, state, block_tokens, block_table, cu_q, kv_lens, offset, slots=None):
    """Recurrence over the new tokens of ``kv_lens.numel()`` sequences; z, u, g: column ranges [T, W] of one projection's
    rows, ``state``: [blocks, W] fp32 rows inside the cache's block records. ``slots``: every sequence has one row, with
    this cache slot."""
    assert z.stride() == u.stride() == g.stride() and z.dtype == u.dtype == g.dtype == out.dtype and z.stride(1) == 1
    assert state.dtype == torch.float32 and state.stride(1) == 1
    _check(lib().ksana_gated_recurrence(_p(z), _p(u), _p(g), z.stride(0), _p(out), out.stride(0), _p(state), state.stride(0),
                                        block_tokens, state.shape[0], _p(block_table), block_table.stride(0), _p(cu_q), _p(kv_lens),
                                        _p(slots), kv_lens.numel(), z.shape[1], float(offset), int(z.dtype == torch.float32),
                                        _p(err_flag(z.device)), _st()), "ksana_gated_recurrence")


def embed_normed(ids, positions, table, pos_table, norm_w, real, scale, eps, vocab):
    """fp32 rows: root-mean-square norm (``real`` columns) of table[id] * scale + pos_table[position]."""
    T, H = ids.numel(), table.shape[1]
    x = torch.empty(T, H, dtype=torch.float32, device=table.device)
    _check(lib().ksana_embed_normed(_p(ids), _p(positions), _p(table), _p(pos_table), _p(norm_w), _p(x), T, H, real, vocab,
                                    pos_table.shape[0], float(scale), float(eps), int(table.dtype == torch.float32),
                                    _p(err_flag(table.device)), _st()), "ksana_embed_normed")
    return x


def token_shift(h, mu, ring, cu_q, kv_lens, slots, max_q, out=None):
    """h + (previous row - h) * mu; ``ring`` [slots, 2, W] (inside the state records) holds the rows of earlier steps."""
    T, W = h.shape
    if out is None:
        out = torch.empty(T, W, dtype=h.dtype, device=h.device)
    assert ring.dtype == mu.dtype == h.dtype and ring.stride(2) == 1 and ring.stride(1) == W and ring.shape[1] == 2
    _check(lib().ksana_token_shift(_p(h), h.stride(0), _p(mu), _p(out), out.stride(0), _p(ring), ring.stride(0), _p(cu_q), _p(kv_lens),
                                   _p(slots), ring.shape[0], kv_lens.numel(), max_q, W, int(h.dtype == torch.float32),
                                   _p(err_flag(h.device)), _st()), "ksana_token_shift")
    return out


def gated_norm(y, w, pad, real, parts, eps, z=None, g=None, factor=1.0, out=None):
    """factor * norm(y * silu(z)) * w * sigmoid(g) with the root mean square of each of ``parts`` equal parts of a row; the row is
    heads of ``pad`` columns, of which ``real`` count."""
    T, C = y.shape
    if out is None:
        out = torch.empty(T, C, dtype=y.dtype, device=y.device)
    assert w.dtype == y.dtype and w.numel() == C
    ld = lambda t: t.stride(0) if t is not None else 0  # noqa: E731
    _check(lib().ksana_gated_norm(_p(y), y.stride(0), _p(z), ld(z), _p(g), ld(g), _p(w), _p(out), out.stride(0), T, C, pad, real, parts,
                                  float(eps), float(factor), int(y.dtype == torch.float32), _st()), "ksana_gated_norm")
    return out


def panel_append(k, slots, cache, block_tokens):
    """Columns k [T, heads * size] of a projection to the paged panel ``cache`` [blocks, heads, block tokens, size]."""
    _check(lib().ksana_panel_append(_p(k), k.stride(0), _p(slots), _p(cache), cache.stride(0), block_tokens, cache.shape[0],
                                    cache.shape[1], cache.shape[3], k.shape[0], int(k.dtype == torch.float32), _p(err_flag(k.device)),
                                    _st()), "ksana_panel_append")


def softcap(z, cap):
    """cap * tanh(z / cap) of fp32 rows, in place."""
    assert z.dtype == torch.float32 and z.stride(1) == 1
    _check(lib().ksana_softcap(_p(z), z.stride(0), z.shape[0], z.shape[1], float(cap), _st()), "ksana_softcap")
    return z


def _conv_args(x, conv):
    ring, w = conv.ring, conv.w
    assert x.stride(1) == 1 and w.dtype == x.dtype == ring.dtype and w.is_contiguous() and ring.stride(2) == 1
    assert ring.shape[1:] == w.shape and ring.stride(1) == w.shape[1] == x.shape[1]
    return _p(x), x.stride(0), _p(w), conv.bias, _p(ring), ring.stride(0), w.shape[0]


def causal_conv(x, conv, cu_q, kv_lens, slots, max_q):
    """silu(conv(x) + bias) over the new rows x [T, C] of sequences of any number of new tokens; ``conv``: a
    :class:`ksanallm_b200.ops.dispatch.ShortConv`."""
    px, ld, w, bias, ring, rs, taps = _conv_args(x, conv)
    out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    _check(lib().ksana_causal_conv(px, ld, w, _p(bias), ring, rs, taps, x.shape[1], _p(out), out.stride(0), _p(cu_q), _p(kv_lens),
                                   _p(slots), conv.ring.shape[0], kv_lens.numel(), max_q, int(x.dtype == torch.float32),
                                   _p(err_flag(x.device)), _st()), "ksana_causal_conv")
    return out


def state_space(x, conv, c, dt, dt_bias, A, D, y, state, G, cu_q, kv_lens, slots):
    """State-space recurrence: a scan over convolved rows ``c`` (``cu_q`` given), or one token per sequence straight from the raw
    rows ``x``. ``state`` [slots, heads, columns, keys] fp32 inside the state records; y [T, heads * columns] receives the result."""
    px, ld, w, bias, ring, rs, taps = _conv_args(x, conv)
    n, H, P, N = state.shape
    assert state.dtype == torch.float32 and state[0].is_contiguous() and dt.stride(1) == y.stride(1) == 1
    _check(lib().ksana_state_space(px, ld, w, _p(bias), ring, rs, taps, _p(c), c.stride(0) if c is not None else 0, _p(dt), dt.stride(0),
                                   _p(dt_bias), _p(A), _p(D), _p(y), y.stride(0), _p(state), state.stride(0), _p(cu_q), _p(kv_lens),
                                   _p(slots), n, kv_lens.numel(), H, G, P, N, int(x.dtype == torch.float32), _p(err_flag(x.device)),
                                   _st()), "ksana_state_space")


def delta_rule(x, conv, c, beta, decay, decay_bias, A, o, state, G, q_scale, cu_q, kv_lens, slots):
    """Gated delta rule, forms as in :func:`state_space`; ``state`` [slots, heads, value size, key size]."""
    px, ld, w, bias, ring, rs, taps = _conv_args(x, conv)
    assert bias is None
    n, H, V, Kd = state.shape
    assert state.dtype == torch.float32 and state[0].is_contiguous() and beta.stride(1) == decay.stride(1) == o.stride(1) == 1
    _check(lib().ksana_delta_rule(px, ld, w, ring, rs, taps, _p(c), c.stride(0) if c is not None else 0, _p(beta), beta.stride(0),
                                  _p(decay), decay.stride(0), _p(decay_bias), _p(A), _p(o), o.stride(0), _p(state), state.stride(0),
                                  _p(cu_q), _p(kv_lens), _p(slots), n, kv_lens.numel(), H, G, Kd, V, float(q_scale),
                                  int(x.dtype == torch.float32), _p(err_flag(x.device)), _st()), "ksana_delta_rule")


def gemm_f32_batched(a, w, out, gate=None):
    """:func:`gemm_bf16_batched` in fp32 on the CUDA cores."""
    B, M, K = a.shape
    N = w.shape[1]
    assert w.shape[0] == B and w.shape[2] == K and tuple(out.shape) == (B, M, N)
    assert a.stride(2) == 1 and w.stride(2) == 1 and out.stride(2) == 1
    _check(lib().ksana_gemm_f32_batched(_p(a), a.stride(1), a.stride(0), _p(w), w.stride(1), w.stride(0), _p(out), out.stride(1),
                                        out.stride(0), B, M, N, K, *_gate_args(gate, out), _st()), "ksana_gemm_f32_batched")
    return out


def refit_rows_f32(x, pos, emb):
    _check(lib().ksana_refit_rows_f32(_p(x), x.stride(0), _p(pos), _p(emb), pos.numel(), emb.shape[1], x.shape[0],
                                      _p(err_flag(x.device)), _st()), "ksana_refit_rows_f32")


# ---------------------------------------------------------------------------- attention path
def rope_kv_append(qkv, positions, slots, cos_sin, cache_layer, block_stride, block_tokens, Hq, Hkv, D, rot_dim,
                   neox=True, mrope_sections=None, k_scale=1.0, v_scale=1.0, apply_rope=True):
    """In-place RoPE on q,k of qkv [T,(Hq+2Hkv)*D] and append of k,v into the layer's paged cache."""
    T = qkv.shape[0]
    fp8 = cache_layer is not None and cache_layer.dtype != torch.bfloat16
    pos_stride, s0, s1 = 0, 0, 0
    if mrope_sections is not None:
        pos_stride = positions.stride(0)
        s0, s1 = mrope_sections[0], mrope_sections[0] + mrope_sections[1]
    rc = lib().ksana_rope_kv_append(_p(qkv), _p(positions), pos_stride, _p(slots), _p(cos_sin), _p(cache_layer),
                                    block_stride, block_tokens, T, Hq, Hkv, D, rot_dim, int(neox), s0, s1, int(fp8),
                                    float(k_scale), float(v_scale), int(apply_rope), _st())
    _check(rc, "ksana_rope_kv_append")


PREFILL_TC = True                  # prefill attention on tcgen05 where the kernel covers the configuration


def _panels(cache_layer, v_cache, D):
    """(K panel of block 0, V panel of block 0, V head size) as addresses: from one interleaved layer tensor
    [blocks, 2, kv heads, block tokens, D], or from separate K and V panel views [blocks, kv heads, block tokens, size]."""
    if v_cache is not None:
        return cache_layer.data_ptr(), v_cache.data_ptr(), int(v_cache.shape[-1])
    return cache_layer.data_ptr(), cache_layer.data_ptr() + cache_layer.stride(1) * cache_layer.element_size(), D


@dataclass
class SigmoidWeights:
    """Attention whose weights are sigmoid(score + bias[head, distance]), not normalised over keys. ``bias`` [heads, n] fp32:
    distances from n - 1 on have the last value. ``gate`` [rows, heads * value size]: outputs are multiplied by its sigmoid and
    by ``factor``."""
    bias: torch.Tensor
    gate: Optional[torch.Tensor] = None
    factor: float = 1.0

    def rows(self, first: int) -> "SigmoidWeights":
        return SigmoidWeights(self.bias, self.gate[first:] if self.gate is not None else None, self.factor)


def _sigmoid_args(weights: Optional[SigmoidWeights]):
    if weights is None:
        return None, 0, None, 0, 1.0
    b, g = weights.bias, weights.gate
    assert b.dtype == torch.float32 and b.is_contiguous() and (g is None or g.stride(1) == 1) and (g is not None or weights.factor == 1.0)
    return _p(b), b.shape[1], _p(g), g.stride(0) if g is not None else 0, float(weights.factor)


def paged_prefill(q, q_stride, out, cache_layer, block_stride, block_tokens, block_table, cu_q, kv_lens, B, max_q_len,
                  Hq, Hkv, D, scale, alibi=None, k_scale=1.0, v_scale=1.0, v_cache=None, window=0, keep=0, sinks=None,
                  weights=None):
    """``v_cache``: V panels of their own (``cache_layer`` then holds the K panels). ``window`` > 0: position i sees j <= i
    with i - j < window or j < keep. ``sinks``: fp32 [Hq] logits in the softmax denominator. ``weights``: see
    :class:`SigmoidWeights`."""
    fp8 = cache_layer.dtype != torch.bfloat16
    kc, vc, Dv = _panels(cache_layer, v_cache, D)
    nblocks = int(cache_layer.shape[0])
    if PREFILL_TC and not fp8 and max(D, Dv) <= 128:
        # tcgen05 kernel (head sizes up to 128, bf16 cache, groups of up to 128 heads); -100 = configuration not covered
        rc = lib().ksana_paged_prefill_tc(_p(q), q_stride, q.shape[0], _p(out), out.stride(0), kc, vc, block_stride,
                                          block_tokens, _p(block_table), block_table.stride(0), _p(cu_q), _p(kv_lens),
                                          _p(alibi), _p(sinks), B, max_q_len, Hq, Hkv, D, Dv, window, keep, float(scale),
                                          nblocks, *_sigmoid_args(weights), _p(err_flag(q.device)), _st())
        if rc != -100:
            _check(rc, "ksana_paged_prefill_tc")
            return
    rc = lib().ksana_paged_prefill(_p(q), q_stride, _p(out), out.stride(0), kc, vc, block_stride, block_tokens,
                                   _p(block_table), block_table.stride(0), _p(cu_q), _p(kv_lens), _p(alibi), _p(sinks), B,
                                   max_q_len, Hq, Hkv, D, Dv, window, keep, float(scale), int(fp8), float(k_scale),
                                   float(v_scale), nblocks, *_sigmoid_args(weights), _p(err_flag(q.device)), _st())
    _check(rc, "ksana_paged_prefill")


def paged_decode(q, q_stride, out, cache_layer, block_stride, block_tokens, block_table, kv_lens, B, Hq, Hkv, D, scale,
                 alibi=None, k_scale=1.0, v_scale=1.0, num_splits=1, part_o=None, part_ml=None, out_q=None,
                 out_scale=None, v_cache=None, window=0, keep=0, sinks=None, weights=None):
    """``out_q`` / ``out_scale`` (head dim 128): the output also (or, with ``out`` None, only) as the FP8 operand of the
    next GEMM: e4m3 [B, Hq * D] and scales [Hq, ld]. ``v_cache`` / ``window`` / ``keep`` / ``sinks`` / ``weights``: see
    :func:`paged_prefill`."""
    fp8 = cache_layer.dtype != torch.bfloat16
    kc, vc, Dv = _panels(cache_layer, v_cache, D)
    rc = lib().ksana_paged_decode(_p(q), q_stride, _p(out), out.stride(0) if out is not None else Hq * Dv, kc, vc,
                                  block_stride, block_tokens, _p(block_table), block_table.stride(0), _p(kv_lens), _p(alibi),
                                  _p(sinks), B, Hq, Hkv, D, Dv, window, keep, float(scale), int(fp8), float(k_scale),
                                  float(v_scale), num_splits, _p(part_o), _p(part_ml), int(cache_layer.shape[0]), _p(out_q),
                                  _p(out_scale), out_scale.stride(0) if out_scale is not None else 0, *_sigmoid_args(weights),
                                  _p(err_flag(q.device)), _st())
    _check(rc, "ksana_paged_decode")


def attention_f32(q, q_stride, out, k_cache, v_cache, block_tokens, block_table, cu_q, kv_lens, B, max_q_len, Hq, Hkv, scale,
                  window=0, keep=0, sinks=None, gate=None, weights=None):
    """All of a step's new rows (any lengths) against K and V panels, in 32-bit arithmetic throughout (bf16 storage is fine).
    ``v_cache`` may be a column range of ``k_cache``. ``gate`` [rows, heads]: outputs are multiplied by its sigmoid.
    ``weights``: see :class:`SigmoidWeights`."""
    assert gate is None or (gate.dtype == q.dtype and gate.stride(1) == 1 and weights is None)
    bias, bias_len, wide, wide_ld, factor = _sigmoid_args(weights)
    rc = lib().ksana_attention_f32(_p(q), q_stride, _p(out), out.stride(0), _p(k_cache), _p(v_cache), v_cache.stride(-2),
                                   k_cache.stride(0), block_tokens, k_cache.shape[0], _p(block_table), block_table.stride(0),
                                   _p(cu_q), _p(kv_lens), _p(sinks), _p(gate) if wide is None else wide,
                                   gate.stride(0) if gate is not None else wide_ld, int(wide is not None), factor, bias, bias_len, B,
                                   max_q_len, Hq, Hkv, k_cache.shape[-1], v_cache.shape[-1], window, keep, float(scale),
                                   int(q.dtype == torch.float32), _p(err_flag(q.device)), _st())
    _check(rc, "ksana_attention_f32")


def qkv_rope_append(qkv, positions, slots, cos_sin, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim):
    """Rotation (halves) of the first ``rot_dim`` dimensions of q (in place) and k, and append of k and v to their paged
    panels [blocks, kv heads, block tokens, size]."""
    T = qkv.shape[0]
    rc = lib().ksana_qkv_rope_append(_p(qkv), _p(positions), _p(slots), _p(cos_sin), cos_sin.shape[0] if cos_sin is not None else 0,
                                     _p(k_cache), _p(v_cache), k_cache.stride(0), block_tokens, k_cache.shape[0], T, Hq, Hkv,
                                     k_cache.shape[-1], v_cache.shape[-1], rot_dim, int(qkv.dtype == torch.float32),
                                     _p(err_flag(qkv.device)), _st())
    _check(rc, "ksana_qkv_rope_append")


def qkv_norm_rope_append(qkv, positions, slots, cos_sin, qw, kw, eps, nq, nk, k_cache, v_cache, block_tokens, Hq, Hkv, rot_dim,
                         sums=None):
    """Root-mean-square norms over all of q (``nq`` real columns) and all of k (``nk``) of a row, rotation of the pairs (2i,
    2i + 1) of the first ``rot_dim`` dimensions of every head, q in place, k and v to their paged panels. ``sums`` [T, 2]: sums of
    squares of the whole rows where ``qkv`` holds a part of them."""
    T = qkv.shape[0]
    assert sums is None or (sums.dtype == torch.float32 and sums.is_contiguous())
    rc = lib().ksana_qkv_norm_rope_append(
        _p(qkv), _p(positions), _p(slots), _p(cos_sin), cos_sin.shape[0] if cos_sin is not None else 0, _p(qw), _p(kw), float(eps), nq, nk,
        _p(sums), _p(k_cache), _p(v_cache), k_cache.stride(0), block_tokens, k_cache.shape[0], T, Hq, Hkv, k_cache.shape[-1],
        v_cache.shape[-1], rot_dim, int(qkv.dtype == torch.float32), _p(err_flag(qkv.device)), _st())
    _check(rc, "ksana_qkv_norm_rope_append")


def latent_norms(q, kv, q_w, kv_w, eps, q_rank, kv_rank, slots, cache, block_tokens):
    """Root-mean-square norms of the query latents ``q`` [T, q_rank padded] (returned) and of the key/value latents ``kv`` [T,
    kv_rank padded] (into the paged panel ``cache`` [blocks, block tokens, kv_rank padded]); both are column ranges of the same
    rows."""
    T = q.shape[0]
    assert q.stride() == kv.stride() and q.stride(1) == 1 and cache.stride(1) == cache.shape[2] == kv.shape[1]
    out = torch.empty(T, q.shape[1], dtype=q.dtype, device=q.device)
    _check(lib().ksana_latent_norms(_p(q), _p(kv), q.stride(0), _p(q_w), _p(kv_w), float(eps), _p(out), q_rank, kv_rank, _p(slots),
                                    _p(cache), cache.stride(0), block_tokens, int(cache.shape[0]) * block_tokens, T,
                                    int(q.dtype == torch.float32), _p(err_flag(q.device)), _st()), "ksana_latent_norms")
    return out


def mla_rope_append(q, nope, kv, norm_w, eps, positions, slots, cos_sin, qfull, cache, block_tokens, G, rank):
    """Latent RMS norm + rotary key rotation + append to the paged latent panel ``cache`` [blocks, block tokens, DK], and
    rotation of the queries' rotary parts into ``qfull`` [T, G, DK] (its leading columns are filled by the caller). q: [T,
    G * (nope + rotary)], kv: [T, DK] or None (queries only: the latents are another layer's). ``rank``: real latent
    size; latent and rotary columns are padded to multiples of 8 with zeros."""
    T = q.shape[0]
    _check(lib().ksana_mla_rope_append(
        _p(q), q.stride(0), nope, _p(kv), kv.stride(0) if kv is not None else 0, _p(norm_w), float(eps), _p(positions), _p(slots),
        _p(cos_sin), _p(qfull), _p(cache), cache.stride(0), block_tokens, T, G, rank, int(cos_sin.shape[1]), int(cos_sin.shape[0]),
        int(cache.shape[0]) * block_tokens, int(q.dtype == torch.float32), _p(err_flag(q.device)), _st()), "ksana_mla_rope_append")


def mla_splits(num_seqs: int, max_q_len: int, max_kv: int, sms: int = 148, halves: int = 2) -> int:
    """KV splits for the latent-attention kernel: only pure decode steps split; the count minimises the number of
    CTA waves times the tiles per CTA, and a split never holds fewer than 4 tiles of 64 tokens."""
    if max_q_len != 1 or num_seqs <= 0:
        return 1
    tiles = max(1, (max_kv + 63) // 64)
    most = max(1, min(32, tiles // 4))
    best, best_cost = 1, None
    for n in range(1, most + 1):
        waves = (halves * num_seqs * n + sms - 1) // sms       # one CTA per SM and output half of a sequence
        cost = waves * ((tiles + n - 1) // n + 2)              # tile times of the longest CTA chain (+ set-up)
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return best


def mla_attention(qfull, out, cache, block_tokens, block_table, cu_q, kv_lens, B, max_q_len, scale, nsplit=1, window=0,
                  sinks=None, gate=None) -> bool:
    """Absorbed multi-head latent attention on tcgen05 (see csrc/kernels/mla_attention.cu). qfull [T, G, DK], cache: latent
    panel [blocks, block tokens, DK], out [T, G, DV] (values are the leading DV columns of the cache rows). ``sinks`` [G]: logits
    that only enter the denominator, ``gate`` [T, G]: outputs are multiplied by its sigmoid. Returns False when the kernel does
    not cover the configuration."""
    assert gate is None or (gate.dtype == torch.bfloat16 and gate.stride(1) == 1)
    assert sinks is None or sinks.dtype == torch.float32
    T, G, dk = qfull.shape
    dv = out.shape[2]
    assert qfull.is_contiguous() and out.stride(2) == 1 and out.stride(1) == dv and cache.stride(1) == dk == cache.shape[2]
    po = pml = None
    if nsplit > 1:
        po = torch.empty(nsplit * T * G * dv, dtype=torch.float32, device=qfull.device)
        pml = torch.empty(nsplit * T * G * 2, dtype=torch.float32, device=qfull.device)
    rc = lib().ksana_mla_attention(_p(qfull), T, _p(out), out.stride(0), _p(cache), cache.stride(0), block_tokens, _p(block_table),
                                   block_table.stride(0), _p(cu_q), _p(kv_lens), B, max_q_len, G, dk, dv, window, _p(sinks), _p(gate),
                                   gate.stride(0) if gate is not None else 0, float(scale), int(cache.shape[0]), nsplit, _p(po), _p(pml), _p(err_flag(qfull.device)), _st())
    if rc == -100:
        return False
    _check(rc, "ksana_mla_attention")
    return True


def copy_blocks(cache, pairs, block_bytes):
    """pairs: int32 [n, 2] (source block, destination block) on the device; ids outside the cache are skipped and
    recorded in the error word."""
    _check(lib().ksana_copy_blocks(_p(cache), _p(pairs), pairs.numel() // 2, block_bytes, int(cache.shape[0]),
                                   _p(err_flag(cache.device)), _st()), "ksana_copy_blocks")


def swap_blocks(cache, host_pool, pairs, block_bytes, to_host: bool):
    """Whole cache blocks between the device cache and the pinned host block pool, one launch per list. ``pairs``:
    int32 [n, 2] (device block, host block) on the device; ``host_pool``: pinned uint8 [host_blocks, block_bytes]
    (the kernel reads / writes it over PCIe, no staging copy). Bad ids are skipped and recorded in the error word."""
    _check(lib().ksana_swap_blocks(_p(cache), host_pool.data_ptr(), _p(pairs), pairs.numel() // 2, block_bytes,
                                   0 if to_host else 1, int(cache.shape[0]), int(host_pool.shape[0]),
                                   _p(err_flag(cache.device)), _st()), "ksana_swap_blocks")


# ----------------------------------------------------------------------------------- sampler
def sample(logits, temperature, top_k, top_p, seeds, steps, out_tokens, row_idx=None, num_logprobs=0, lp_ids=None,
           lp_vals=None):
    B = out_tokens.numel()
    rc = lib().ksana_sample(_p(logits), logits.stride(0), _p(row_idx), _p(temperature), _p(top_k), _p(top_p),
                            _p(seeds), _p(steps), _p(out_tokens), num_logprobs, _p(lp_ids), _p(lp_vals), B,
                            logits.shape[1], _st())
    _check(rc, "ksana_sample")


def sample_merged(cand_vals, cand_ids, temperature, top_k, top_p, seeds, steps, out_tokens, num_logprobs=0, lp_ids=None,
                  lp_vals=None):
    """The sampler over candidate lists gathered from the vocabulary shards: cand_vals [B, C] fp32 logits and
    cand_ids [B, C] int32 token ids of the same columns."""
    B = out_tokens.numel()
    rc = lib().ksana_sample_merged(_p(cand_vals), cand_vals.stride(0), _p(cand_ids), cand_ids.stride(0), None,
                                   _p(temperature), _p(top_k), _p(top_p), _p(seeds), _p(steps), _p(out_tokens),
                                   num_logprobs, _p(lp_ids), _p(lp_vals), B, cand_vals.shape[1], _st())
    _check(rc, "ksana_sample_merged")


def shard_topk(logits, vocab, k, idx_offset, out_vals, out_ids):
    """This vocabulary shard's k largest logits per row and their token ids (column + idx_offset):
    out_vals fp32 [B, k], out_ids int32 [B, k], sorted by value (descending) then id."""
    B = logits.shape[0]
    rc = lib().ksana_shard_topk(_p(logits), logits.stride(0), None, B, vocab, k, idx_offset, _p(out_vals), _p(out_ids),
                                _st())
    _check(rc, "ksana_shard_topk")


def repetition_penalty(logits, offsets, ids, penalty, row_idx=None):
    B = penalty.numel()
    rc = lib().ksana_repetition_penalty(_p(logits), logits.stride(0), _p(row_idx), _p(offsets), _p(ids), _p(penalty),
                                        B, logits.shape[1], _st())
    _check(rc, "ksana_repetition_penalty")


def ban_tokens(logits, offsets, ids, row_idx=None):
    B = offsets.numel() - 1
    rc = lib().ksana_ban_tokens(_p(logits), logits.stride(0), _p(row_idx), _p(offsets), _p(ids), B, logits.shape[1],
                                _st())
    _check(rc, "ksana_ban_tokens")


# --------------------------------------------------------------------------- mixture of experts
def gemm_grouped(a, w, tile_expert, E, N, out=None, a_scale=None, w_scale=None, bn=0, tile_rows=None):
    """Expert-major rows of ``a`` [cap, K] (128-row tiles, one expert each) times stacked W [E*N, K]. ``tile_rows``: rows of every
    tile that hold anything; the others need not be stored (worth it where tiles are mostly empty; with full ones, reading the counts
    only sets the CTAs apart that share operand tiles in L2, up to twice the time)."""
    cap, K = a.shape
    if cap > 191 * E:                  # more than 64 rows per expert on average
        tile_rows = None
    if a.dtype == torch.float32:
        out = torch.empty(cap, N, dtype=a.dtype, device=a.device)
        _check(lib().ksana_gemm_grouped_f32(_p(a), a.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), cap, N, K, E,
                                            _p(tile_expert), _st()), "ksana_gemm_grouped_f32")
        return out
    kind = 0 if a_scale is None else 1
    if out is None:
        out = torch.empty(cap, N, dtype=torch.bfloat16, device=a.device)
    rc = lib().ksana_gemm_grouped(kind, _p(a), a.stride(0), _p(a_scale), a_scale.stride(0) if a_scale is not None else 0,
                                  _p(w), w.stride(0), _p(w_scale), _p(out), out.stride(0), cap, N, K, E,
                                  _p(tile_expert), _p(tile_rows), bn, _p(err_flag(a.device)), _st())
    _check(rc, "ksana_gemm_grouped")
    return out


def moe_route(logits, K, scoring="softmax", renorm=True, scale=1.0, bias=None, n_group=1, topk_group=1, E=None, gate_col=-1,
              group_top=2):
    """Expert choice by rows of router logits (the first ``E`` columns of fp32 rows): (ids [T, K] int32, weights fp32 [T, K], or
    [T, K + 1] with ``gate_col``: the sigmoid of that column comes last). A group's score is the sum of its two largest choice
    scores, or with ``group_top`` 1 its largest."""
    T, E = logits.shape[0], logits.shape[1] if E is None else E
    ids = torch.empty(T, K, dtype=torch.int32, device=logits.device)
    w = torch.empty(T, K + (gate_col >= 0), dtype=torch.float32, device=logits.device)
    rc = lib().ksana_moe_route(_p(logits), logits.stride(0), _p(bias), _p(ids), _p(w), w.stride(0), T, E, K,
                               0 if scoring == "softmax" else 1, int(renorm), float(scale), n_group, topk_group, group_top, gate_col, _st())
    _check(rc, "ksana_moe_route")
    return ids, w


def moe_align(topk_ids, E, expert_lo=0, expert_hi=None):
    """(destination row of every (token, choice), expert of every 128-row tile, row offsets of the experts, padded row count,
    capacity in rows, rows of every tile that hold a token)."""
    TK = topk_ids.numel()
    hi = E if expert_hi is None else expert_hi
    max_tiles = (TK + (hi - expert_lo) * 127 + 127) // 128
    dev = topk_ids.device
    dst_row = torch.empty(TK, dtype=torch.int32, device=dev)
    tile_expert = torch.empty(max_tiles, dtype=torch.int32, device=dev)
    tile_rows = torch.empty_like(tile_expert)
    offsets = torch.empty(E + 1, dtype=torch.int32, device=dev)
    total = torch.empty(1, dtype=torch.int32, device=dev)
    rc = lib().ksana_moe_align(_p(topk_ids), _p(dst_row), _p(tile_expert), _p(tile_rows), _p(offsets), _p(total), TK, E, max_tiles,
                               expert_lo, hi, _p(err_flag(dev)), _st())
    _check(rc, "ksana_moe_align")
    return dst_row, tile_expert, offsets, total, max_tiles * 128, tile_rows


def moe_permute(x, dst_row, K, cap, zero=False):
    """``zero``: padding rows are zero instead of undefined (for consumers that reduce over the whole tensor)."""
    T, H = x.shape
    perm = (torch.zeros if zero else torch.empty)(cap, H, dtype=x.dtype, device=x.device)
    units = H * x.element_size() // 2                                        # the kernel moves 16-bit units
    _check(lib().ksana_moe_permute(_p(x), _p(dst_row), _p(perm), T, K, units, cap, _p(err_flag(x.device)), _st()),
           "ksana_moe_permute")
    return perm


def moe_combine(y, dst_row, topk_w, out, K, accumulate):
    T, H = out.shape
    _check(lib().ksana_moe_combine(_p(y), _p(dst_row), _p(topk_w), _p(out), T, K, H, int(accumulate), int(y.shape[0]),
                                   _p(err_flag(out.device)), _st()), "ksana_moe_combine")
    return out
