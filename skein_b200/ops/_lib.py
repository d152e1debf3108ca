"""ctypes binding of libskein_kernels.so (the hand-written sm_100a kernels).

The library is plain C ABI: raw device pointers plus a CUDA stream handle. It is loaded lazily;
on a machine with a GPU a missing library is an error (there is no silent fallback to PyTorch on
the device path), on a CPU-only machine the operators in this package use their PyTorch reference
implementations instead.
"""
from __future__ import annotations

import ctypes as C
from pathlib import Path

import torch

MAX_PEERS = 8
MAX_GROUPS = 64

_LIB = None
_LIB_PATH = Path(__file__).resolve().parent.parent / "_native" / "libskein_kernels.so"


class GemmParams(C.Structure):
    """Mirror of SkeinGemmParams in csrc/kernels/gemm_ws.cuh (same field order)."""

    _fields_ = [
        ("W", C.c_void_p), ("X", C.c_void_p), ("out", C.c_void_p), ("residual", C.c_void_p),
        ("group_off", C.c_void_p), ("group_cnt", C.c_void_p),
        ("workspace", C.c_void_p), ("counters", C.c_void_p), ("status", C.c_void_p),
        ("w_scale", C.c_void_p), ("x_scale", C.c_void_p),
        ("peer_flag", C.c_void_p * MAX_PEERS),
        ("epoch", C.c_void_p), ("done_counter", C.c_void_p),
        ("n_peers", C.c_int32), ("G", C.c_int32), ("F", C.c_int32), ("K", C.c_int32),
        ("w_rows_per_group", C.c_int32), ("up_row_off", C.c_int32), ("x_rows", C.c_int32),
        ("t_static", C.c_int32), ("n_tile", C.c_int32), ("ldo", C.c_int32), ("out_col0", C.c_int32),
        ("mode", C.c_int32), ("fp8", C.c_int32), ("stages", C.c_int32), ("grid", C.c_int32),
        ("wait_budget_ms", C.c_int32), ("w_packed", C.c_int32), ("line_cut_only", C.c_int32),
        ("x_ld", C.c_int32), ("x_group_cols", C.c_int32), ("out_group_cols", C.c_int32), ("glu", C.c_int32),
        ("glu_limit", C.c_float), ("glu_slope", C.c_float), ("out_f32", C.c_int32), ("gate_ld", C.c_int32),
        ("gate", C.c_void_p), ("relu2_cols", C.c_int32), ("pad", C.c_int32),
    ]


class RecParams(C.Structure):
    """Mirror of SkeinRecParams in csrc/kernels/recurrent.cuh (same field order)."""

    _fields_ = [(n, C.c_void_p) for n in ("row", "out", "state", "tail", "conv_w", "conv_b", "neg_decay", "decay", "dt_bias", "skip", "step",
                                          "positions", "slots", "status")] + [("ld", C.c_int64)] + [
        (n, C.c_int32) for n in ("kind", "H", "G", "D", "V", "taps", "C", "q_col", "k_col", "v_col", "a_col", "b_col", "num_slots")]


class RecGate(C.Structure):
    """Mirror of SkeinRecGate in csrc/kernels/recurrent.cuh (same field order)."""

    _fields_ = [("norm", C.c_void_p), ("out", C.c_void_p), ("gate", C.c_void_p), ("out_ld", C.c_int64), ("gate_ld", C.c_int64),
                ("sigmoid", C.c_int32), ("eps", C.c_float), ("scale", C.c_float), ("pad", C.c_int32)]


class RecChunk(C.Structure):
    """Mirror of SkeinRecChunk in csrc/kernels/recurrent.cuh (same field order)."""

    _fields_ = [(n, C.c_void_p) for n in ("seq_of_token", "q_start", "q_len", "qkv", "gates", "unit", "chunk_mat")] + [
        ("qkv_ld", C.c_int64), ("v_off", C.c_int32), ("max_q_len", C.c_int32)]


class RouteRule(C.Structure):
    """Mirror of SkeinRouteRule in csrc/kernels/route.cuh (same field order)."""

    _fields_ = [(n, C.c_int32) for n in ("n_groups", "keep", "score", "group_best", "renorm")] + [("scale", C.c_float)]


class AttnRule(C.Structure):
    """Mirror of SkeinAttnRule in csrc/kernels/attn_rule.cuh (same field order)."""

    _fields_ = [("lam", C.c_void_p), ("gate", C.c_void_p), ("sinks", C.c_void_p), ("gate_ld", C.c_int64)] + [
        (n, C.c_int32) for n in ("window", "chunk", "sink", "maps", "keep_first")] + [(n, C.c_float) for n in ("softcap", "scale", "out_scale", "eps")] + [
        ("pad", C.c_int32)]


class HeadExtras(C.Structure):
    """Mirror of SkeinHeadExtras in csrc/kernels/attn_rule.cuh (same field order)."""

    _fields_ = [(n, C.c_void_p) for n in ("q_bias", "k_bias", "v_bias", "q_norm", "k_norm", "mix", "v_first", "v_keep")]


class DepthNormParams(C.Structure):
    """Mirror of SkeinDepthNormParams in csrc/kernels/prenorm.cu (same field order)."""

    _fields_ = [(n, C.c_void_p) for n in ("terms", "weights", "x_out", "gain", "act_out", "shift", "state", "positions", "slots", "seq_of_token",
                                          "q_start", "q_len", "status")] + [("term_stride", C.c_int64)] + [
        (n, C.c_int32) for n in ("n_terms", "T", "C", "groups", "num_slots")] + [("eps", C.c_float)]


class ScanParams(C.Structure):
    """Mirror of SkeinScanParams in csrc/kernels/selective.cu (same field order)."""

    _fields_ = [(n, C.c_void_p) for n in ("x", "xc", "proj", "dt", "z", "out", "state", "tail", "conv_w", "conv_b", "dt_bias", "neg_a", "skip",
                                          "positions", "slots", "seq_of_token", "q_start", "q_len", "status")] + [
        (n, C.c_int64) for n in ("x_ld", "proj_ld", "out_ld")] + [(n, C.c_int32) for n in ("I", "N", "taps", "b_col", "c_col", "num_slots")]


byref = C.byref


def lib_path() -> Path:
    return _LIB_PATH


def available() -> bool:
    return _LIB_PATH.exists()


def _sig(lib, name, restype, argtypes):
    # a library built for one architecture holds that architecture's kernels only (_build.py): calling an absent one raises
    # AttributeError naming it
    if not hasattr(lib, name):
        return None
    fn = getattr(lib, name)
    fn.restype = restype
    fn.argtypes = argtypes
    return fn


def lib():
    """Load the kernel library (once). Raises if it has not been built."""
    global _LIB
    if _LIB is not None:
        return _LIB
    if not _LIB_PATH.exists():
        raise RuntimeError(
            f"{_LIB_PATH} is missing: build it with `python -m skein_b200._build` "
            "(the CUDA path has no PyTorch fallback)")
    L = C.CDLL(str(_LIB_PATH), mode=C.RTLD_GLOBAL)
    vp, i32, i64, f32 = C.c_void_p, C.c_int, C.c_longlong, C.c_float
    _sig(L, "skein_gemm_ws", i32, [C.POINTER(GemmParams), vp])
    _sig(L, "skein_gemm_ws_workspace_bytes", i64, [C.POINTER(GemmParams)])
    _sig(L, "skein_sm_count", i32, [])
    _sig(L, "skein_reduce_residual_rmsnorm", i32,
         [vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, i64, i32, i32, i32, i32, f32, i32, vp, i32, i32, vp, vp, vp])
    _sig(L, "skein_reduce_norm_route", i32,
         [vp, vp, vp, vp, vp, vp, vp, vp, i64, i32, i32, i32, f32, i32, vp, i32, i32, i32, i32, vp, vp, vp, vp, vp, vp,
          vp, vp, i32, vp, vp, vp])
    _sig(L, "skein_rope_kv_append", i32,
         [vp, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, i32, vp, vp])
    _sig(L, "skein_embed_gather", i32, [vp, vp, vp, i32, i32, i32, i32, vp])
    _sig(L, "skein_gather_rows", i32, [vp, vp, vp, i32, i32, vp, vp])
    _sig(L, "skein_attn_decode_workspace_floats", i64, [i32, i32, i32])
    _sig(L, "skein_attn_decode", i32,
         [vp, i64, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, f32, vp])
    _sig(L, "skein_attn_decode_mma", i32,
         [vp, i64, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, f32, vp])
    _sig(L, "skein_attn_decode_rope_mma", i32,
         [vp, i64, vp, vp, vp, vp, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, f32, vp])
    _sig(L, "skein_attn_prefill", i32,
         [vp, i64, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, f32, vp])
    _sig(L, "skein_attn_decode_tc", i32,
         [vp, i64, vp, vp, vp, vp, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, vp])
    _sig(L, "skein_attn_prefill_tc", i32,
         [vp, i64, i64, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, f32, vp])
    _sig(L, "skein_router_topk", i32, [vp, vp, i32, i32, i32, i32, vp, vp, vp, vp, vp, vp, vp, i32, i32, vp, vp])
    _sig(L, "skein_router_plan", i32, [vp, i32, i32, i32, vp, vp, vp, vp, i32, i32, vp])
    _sig(L, "skein_sample_argmax", i32, [vp, i64, i32, i32, i32, vp, vp, vp])
    _sig(L, "skein_merge_candidates", i32, [vp, vp, i32, i32, i32, vp, vp, vp, i32, vp, vp])
    _sig(L, "skein_sample_topk_topp", i32, [vp, i64, i32, i32, vp, vp, vp, vp, vp, i32, vp, vp])
    _sig(L, "skein_quant_fp8_block128", i32, [vp, vp, vp, i64, i32, vp])
    _sig(L, "skein_dequant_fp8_block128_t", i32, [vp, vp, vp, i64, i32, vp])
    _sig(L, "skein_advance_decode_state", i32, [vp, vp, vp, vp, i32, vp, vp])
    pvp = C.POINTER(C.c_void_p)
    _sig(L, "skein_ep_dispatch_pull", i32, [pvp, pvp, i32, i32, i32, i32, i32, i32, i32, vp, vp, vp, i32, vp, vp, vp, vp, vp, vp, vp])
    _sig(L, "skein_ipc_alloc", i32, [pvp, i64])
    _sig(L, "skein_ipc_free", i32, [vp])
    _sig(L, "skein_ipc_get_handle", i32, [vp, C.c_char_p])
    _sig(L, "skein_ipc_open", i32, [C.c_char_p, pvp])
    _sig(L, "skein_ipc_close", i32, [vp])
    _sig(L, "skein_ipc_handle_bytes", i32, [])
    _sig(L, "skein_publish_rows", i32, [vp, i64, vp, pvp, i32, vp, vp, vp])
    _sig(L, "skein_pull_collective", i32, [i32, pvp, i32, i32, i64, vp, vp, vp, vp, i32, vp])
    _sig(L, "skein_argmax_push", i32, [vp, i64, i32, i32, i32, pvp, pvp, pvp, i32, vp, vp, vp])
    _sig(L, "skein_copy_pages", i32, [vp, vp, vp, vp, i32, i64, vp])
    _sig(L, "skein_wait_flag", i32, [vp, i32, i32, vp, vp])
    _sig(L, "skein_gemm_simt", i32, [C.POINTER(GemmParams), i32, i32, vp])
    _sig(L, "skein_gemm_small", i32, [vp, i64, vp, vp, i64, vp, i32, i32, i32, i32, vp])
    _sig(L, "skein_embed_f32", i32, [vp, vp, vp, i32, i32, i32, i32, vp])
    _sig(L, "skein_conv_input", i32, [vp, vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, i32, vp])
    _sig(L, "skein_post_norm", i32, [vp, vp, vp, vp, vp, vp, vp, vp, f32, f32, i32, i32, i32, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, vp])
    _sig(L, "skein_post_norm_route", i32,
         [vp, vp, vp, vp, f32, f32, i32, i32, vp, i32, i32, i32, i32, vp, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp])
    _sig(L, "skein_poly_norm", i32, [vp, vp, vp, i32, i32, f32, i32, vp])
    rule = C.POINTER(RouteRule)
    _sig(L, "skein_route_grouped", i32, [vp, i32, i32, i32, rule, vp, vp, vp, vp, vp, vp, vp])
    _sig(L, "skein_norm_route", i32, [vp, vp, vp, f32, i32, i32, vp, i32, i32, rule, vp, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp])
    _sig(L, "skein_add_norm", i32, [vp, vp, vp, vp, i32, vp, vp, vp, vp, i32, i32, f32, i32, vp])
    _sig(L, "skein_latent_append", i32,
         [vp, i32, i32, vp, i32, vp, i32, i32, vp, i32, vp, vp, vp, i32, vp, i32, i32, vp, vp, vp, vp, vp, vp, i32, i32, i32, f32, i32, vp, i32, vp])
    _sig(L, "skein_rope_rows", i32, [vp, i64, vp, vp, i32, i32, i32, i32, i32, vp, i32, vp])
    _sig(L, "skein_latent_gather", i32, [vp, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, i32, vp])
    _sig(L, "skein_latent_attn_rows", i32,
         [vp, vp, i64, vp, i32, vp, vp, vp, i32, vp, i32, i32, vp, i32, i32, i32, i32, i32, f32, vp, vp, i32, vp])
    _sig(L, "skein_latent_attn_decode", i32,
         [vp, vp, i64, vp, i32, vp, vp, vp, i32, vp, i32, i32, vp, i32, i32, i32, i32, i32, f32, vp, i32, i32, vp, vp])
    _sig(L, "skein_latent_attn_prefill", i32,
         [vp, i64, i32, vp, i32, vp, i32, vp, i32, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, f32, vp, vp])
    _sig(L, "skein_residual_tanh", i32, [vp, vp, i32, vp, vp, vp, vp, vp, vp, i64, i32, i32, i32, vp])
    _sig(L, "skein_gated_norm", i32, [vp, vp, i64, vp, i32, vp, i64, i32, i32, i32, i32, i32, f32, f32, i32, vp])
    _sig(L, "skein_window_append", i32,
         [vp, vp, vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, f32, i32, vp])
    _sig(L, "skein_head_append", i32,
         [vp, vp, vp, i64, vp, vp, vp, vp, vp, vp, C.POINTER(HeadExtras), i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, f32, i32,
          vp])
    _sig(L, "skein_depth_norm", i32, [C.POINTER(DepthNormParams), i32, vp])
    arule = C.POINTER(AttnRule)
    _sig(L, "skein_window_attn_rows", i32, [vp, i64, vp, vp, vp, vp, vp, i64, vp, i32, i32, i32, i32, i32, i32, i32, i32, arule, i32, vp])
    _sig(L, "skein_attn_decode_window", i32,
         [vp, i64, vp, vp, vp, vp, i64, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, arule, vp])
    _sig(L, "skein_attn_prefill_window", i32,
         [vp, i64, i64, vp, vp, vp, vp, vp, vp, i64, vp, i32, i32, i32, i32, i32, i32, i32, i32, arule, vp])
    scanp = C.POINTER(ScanParams)
    _sig(L, "skein_short_conv", i32, [scanp, i32, i32, i32, vp])
    _sig(L, "skein_scan_step", i32, [scanp, i32, i32, vp])
    _sig(L, "skein_scan_rows", i32, [scanp, i32, i32, vp])
    rec, chunk = C.POINTER(RecParams), C.POINTER(RecChunk)
    _sig(L, "skein_rec_step", i32, [rec, C.POINTER(RecGate), i32, i32, vp])
    _sig(L, "skein_rec_step_gates", i32, [rec])
    _sig(L, "skein_rec_prep", i32, [rec, chunk, i32, i32, vp])
    _sig(L, "skein_rec_scan", i32, [rec, chunk, i32, i32, vp])
    _sig(L, "skein_rec_tc", i32, [rec, chunk, i32, i32, vp])
    _sig(L, "skein_rec_tc_scratch_bytes", i64, [rec, i32, i32])
    _sig(L, "skein_rec_channel", i32, [rec, chunk, i32, i32, vp])
    _sig(L, "skein_rec_channel_scratch_bytes", i64, [rec, i32, i32])
    _sig(L, "skein_rec_tail", i32, [rec, chunk, i32, i32, vp])
    for name, rt, at in _OPTIONAL:
        if hasattr(L, name):
            _sig(L, name, rt, at)
    _LIB = L
    return L


# Entry points that newer builds add; bound when present.
_OPTIONAL: list = []


def register_optional(name, restype, argtypes):
    _OPTIONAL.append((name, restype, argtypes))
    if _LIB is not None and hasattr(_LIB, name):
        _sig(_LIB, name, restype, argtypes)


def ptr(t) -> int | None:
    """Device (or host) address of a tensor, None for None."""
    return None if t is None else t.data_ptr()


def stream_ptr() -> int:
    return torch.cuda.current_stream().cuda_stream


def check(rc: int, what: str) -> None:
    if rc != 0:
        raise RuntimeError(f"{what} failed with code {rc}")


# launch counter: every kernel launched through this package increments it (bench.py reports it)
_launches = 0


def count_launch(n: int = 1) -> None:
    global _launches
    _launches += n


def launches() -> int:
    return _launches
