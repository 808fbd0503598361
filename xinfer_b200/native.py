"""Loads the two native libraries (building them at first use) and declares their C signatures.

There is no fallback: if the kernels cannot be built or loaded the engine raises.
"""
from __future__ import annotations

import ctypes
import threading
from ctypes import (POINTER, c_char_p, c_float, c_int, c_int32, c_longlong, c_void_p)

_lock = threading.Lock()
_host = None
_kernels = None

_I32P = POINTER(c_int32)
_I64P = POINTER(c_longlong)


def host_lib():
    """Host runtime: cache manager, scheduler, step metadata assembly (no CUDA needed)."""
    global _host
    with _lock:
        if _host is None:
            from .csrc.build import build_host
            lib = ctypes.CDLL(build_host())
            _declare_host(lib)
            _host = lib
    return _host


def kernels_lib():
    """CUDA kernels for sm_100a."""
    global _kernels
    with _lock:
        if _kernels is None:
            from .csrc.build import build_kernels
            lib = ctypes.CDLL(build_kernels())
            _declare_kernels(lib)
            _kernels = lib
    return _kernels


def _sig(lib, name, restype, argtypes):
    fn = getattr(lib, name)
    fn.restype = restype
    fn.argtypes = argtypes


def _declare_host(lib):
    _sig(lib, "xb_cm_create", c_void_p, [c_int, POINTER(c_int), POINTER(c_int), POINTER(c_int), POINTER(c_int), c_int])
    _sig(lib, "xb_cm_destroy", None, [c_void_p])
    for name in ("xb_cm_open", "xb_cm_live_requests"):
        _sig(lib, name, c_int, [c_void_p])
    for name in ("xb_cm_close", "xb_cm_is_live", "xb_cm_length", "xb_cm_free_pages"):
        _sig(lib, name, c_int, [c_void_p, c_int])
    for name in ("xb_cm_can_extend", "xb_cm_extend", "xb_cm_advance", "xb_cm_table_size"):
        _sig(lib, name, c_int, [c_void_p, c_int, c_int])
    _sig(lib, "xb_cm_copy_table", c_int, [c_void_p, c_int, c_int, _I32P, c_int])
    _sig(lib, "xb_cm_consistent", c_int, [c_void_p, c_char_p, c_int])
    _sig(lib, "xb_attn_prefill_work", c_longlong,
         [c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_longlong, c_void_p])
    _sig(lib, "xb_cm_log_freed", None, [c_void_p, c_int])
    _sig(lib, "xb_cm_drain_freed", c_int, [c_void_p, c_void_p, c_void_p, c_int])
    _sig(lib, "xb_assemble", c_longlong,
         [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int,
          c_void_p, c_void_p, c_longlong, c_void_p])
    _sig(lib, "xb_sched_create", c_void_p, [c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_int])
    _sig(lib, "xb_sched_destroy", None, [c_void_p])
    _sig(lib, "xb_sched_add", c_int, [c_void_p, c_longlong, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p, c_int])
    _sig(lib, "xb_sched_abort", c_int, [c_void_p, c_longlong])
    _sig(lib, "xb_sched_schedule", c_int,
         [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p])
    _sig(lib, "xb_sched_commit", None, [c_void_p, c_void_p, c_int])
    _sig(lib, "xb_sched_schedule_ahead", c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p])
    _sig(lib, "xb_sched_fail_steps", c_int, [c_void_p])
    _sig(lib, "xb_sched_drain_finished", c_int, [c_void_p, c_void_p, c_int])
    for name in ("xb_sched_num_waiting", "xb_sched_num_running", "xb_sched_preemptions"):
        _sig(lib, name, c_int, [c_void_p])
    for name in ("xb_sched_finish_reason", "xb_sched_output_length", "xb_sched_prompt_length",
                 "xb_sched_num_drawn", "xb_sched_release"):
        _sig(lib, name, c_int, [c_void_p, c_longlong])
    _sig(lib, "xb_sched_copy_output", c_int, [c_void_p, c_longlong, c_void_p, c_int])
    _sig(lib, "xb_sched_copy_tail", c_int, [c_void_p, c_longlong, c_void_p, c_int])


def _declare_kernels(lib):
    P, I, F, L = c_void_p, c_int, c_float, c_longlong
    _sig(lib, "xb_embedding", I, [I, P, P, P, P, I, I, I, I, F, P, P])
    _sig(lib, "xb_logits_post", I, [P, L, F, F, P])
    _sig(lib, "xb_rmsnorm", I, [I, P, P, P, P, P, P, I, I, I, F, F, P, P])
    _sig(lib, "xb_add", I, [I, P, P, P, L, F, P])
    _sig(lib, "xb_gemm_plain", I, [I, I, I, P, P, P, I, I, I, P])
    _sig(lib, "xb_rope_table", I, [P, P, P, I, I, P])
    _sig(lib, "xb_qk_norm_rope_write", I,
         [I, P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, F, I, P, P])
    _sig(lib, "xb_attention_plain", I,
         [I, P, P, L, L, P, P, I, I, P, P, P, P, I, I, I, I, I, I, I, I, I, I, F, F, F, I, L, F, P, P])
    _sig(lib, "xb_swiglu", I, [I, P, P, I, I, I, F, F, P])
    _sig(lib, "xb_widen_bf16", I, [P, P, L, P])
    _sig(lib, "xb_sample", I, [P, P, P, P, I, I, I, I, P, P, P])
    _sig(lib, "xb_sample_scratch_bytes", c_longlong, [I])
    _sig(lib, "xb_sample_params_size", I, [])
    _sig(lib, "xb_rmsnorm_bf16", I, [P, P, P, P, P, P, I, I, I, F, F, P, P])
    _sig(lib, "xb_swiglu_bf16", I, [P, P, I, I, I, F, F, P])
    _sig(lib, "xb_qk_norm_rope_write_bf16", I,
         [P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, F, I, P, P])
    _sig(lib, "xb_swiglu_rows_bf16", I, [P, P, I, I, I, F, F, P])
    _sig(lib, "xb_attn_prefill_tc", I, [P, P, P, P, P, P, P, I, I, I, I, I, I, L, I, I, I, I, F, F, F, P, F, P, I, P, P])
    _sig(lib, "xb_gemm_skinny_tc", I, [P, I, P, P, I, I, I, I, P, P])
    _sig(lib, "xb_gemm_skinny_swiglu", I, [P, P, P, I, I, I, I, P, P])
    _sig(lib, "xb_gemm_skinny_qkv", I,
         [P, P, P, P, P, I, I, I, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, P])
    _sig(lib, "xb_attn_prefill_bf16", I, [P, P, P, P, P, P, I, P, I, I, I, I, I, I, I, F, I, I, I, I, P, P])
    _sig(lib, "xb_attn_decode_bf16", I,
         [P, P, P, P, P, P, P, P, P, I, P, I, I, I, I, I, I, I, F, I, I, I, I, I, P, P, P])
    _sig(lib, "xb_attn_decode_plan_size", c_longlong, [I, I, I])
    _sig(lib, "xb_attn_decode_plan", I, [P, P, P, P, I, I, I, I, I, I, I, I, I, P, P])
    _sig(lib, "xb_embedding_f32", I, [I, P, P, P, P, I, I, I, I, F, P, P])
    _sig(lib, "xb_rmsnorm_f32", I, [I, I, P, P, P, P, P, P, I, I, I, F, F, P, P])
    _sig(lib, "xb_add_f32", I, [I, P, P, P, L, F, P])
    _sig(lib, "xb_qkv_prepare", I, 
         [I, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, I, F, I, F, P, F, I, L, L, P, I, P, P, P, I, F, P, P])
    _sig(lib, "xb_rms_chain", I, [I, I, P, P, P, P, P, P, P, P, I, I, I, F, F, F, F, F, P, P])
    _sig(lib, "xb_dual_rms_sum", I, [I, P, P, P, P, P, I, I, F, F, F, F, P])
    _sig(lib, "xb_add_bias", I, [I, P, P, I, I, P])
    _sig(lib, "xb_swiglu_bias", I, [I, I, P, P, P, I, I, I, P])
    _sig(lib, "xb_embed_sum", I, [I, P, P, P, P, P, P, I, P, P, P, P, P, I, I, I, I, L, L, I, F, P, P])
    _sig(lib, "xb_prev_store", I, [P, P, P, I, P, P, I, P])
    _sig(lib, "xb_token_gate", I, [I, P, P, P, I, I, P, P, I, P, I, I, I, P, P])
    _sig(lib, "xb_conv_silu", I, [I, P, P, L, I, P, P, P, P, P, P, I, I, I, P])
    _sig(lib, "xb_conv_state", I, [I, P, P, L, I, P, P, I, I, I, P])
    _sig(lib, "xb_selective_scan", I, [P, P, I, P, L, I, P, P, P, P, P, P, I, I, I, I, I, P])
    _sig(lib, "xb_delta_rule", I, [P, P, I, P, L, I, P, L, P, P, P, P, P, I, I, I, I, I, F, P])
    _sig(lib, "xb_linear_scan", I, [P, P, L, P, P, P, P, I, I, I, I, F, P])
    _sig(lib, "xb_low_rank_decay", I, [P, P, L, P, P, I, I, I, F, P])
    _sig(lib, "xb_stream_conv", I, [I, P, P, P, P, P, P, P, P, P, P, I, I, I, F, F, F, I, P])
    _sig(lib, "xb_gated_head_norm", I, [I, P, P, P, L, I, P, I, I, I, I, F, I, P, L, F, P])
    _sig(lib, "xb_matrix_memory", I, [P, P, P, L, I, P, P, F, P, P, P, P, P, P, I, I, I, I, F, F, P])
    _sig(lib, "xb_stream_mix", I, [I, I, P, P, P, L, L, P, P, P, P, P, P, I, I, I, I, F, F, P, P])
    _sig(lib, "xb_dyt_norm", I, [I, I, I, P, P, P, P, P, P, P, P, F, P, P, P, I, I, I, P, P])
    _sig(lib, "xb_latent_prepare", I,
         [I, P, P, P, L, I, I, P, L, L, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, F, I, P, I, I, P, P, P])
    _sig(lib, "xb_attn_latent_mma_takes", I, [I, I])
    _sig(lib, "xb_attn_latent_mma", I, [P, P, P, P, P, I, P, I, I, I, I, I, I, I, I, F, P, I, I, P, P, P, P])
    _sig(lib, "xb_gate_sigmoid", I, [I, P, P, L, L, P, L, I, I, I, I, P])
    _sig(lib, "xb_gemm_batched_plain", I, [I, P, P, P, I, I, I, I, L, L, L, L, L, L, L, P])
    _sig(lib, "xb_attn_talking_tile", I, [I, I, I, I])
    _sig(lib, "xb_attn_talking", I, [I, P, I, P, P, P, P, P, P, I, P, I, I, I, I, I, I, I, I, I, F, I, F, I, I, P, P, P, P])
    _sig(lib, "xb_attn_talking_mma_tile", I, [I, I, I, I, I])
    _sig(lib, "xb_attn_talking_mma", I, [P, I, P, P, P, P, P, P, I, P, I, I, I, I, I, I, I, I, I, F, I, F, I, I, P, P, P, P])
    _sig(lib, "xb_gated_scan", I, [I, P, I, P, P, P, P, P, P, P, I, I, I, F, I, P, P])
    _sig(lib, "xb_polynorm", I, [I, P, P, P, I, I, F, P])
    _sig(lib, "xb_expert_route", I, [P, P, P, P, P, P, I, P, I, I, I, I, P, P])
    _sig(lib, "xb_expert_gemm", I, [I, I, P, P, P, P, P, I, I, I, I, I, I, I, L, L, I, F, F, P])
    _sig(lib, "xb_expert_select_gate", I, [I, P, P, P, P, P, I, P, I, I, I, I, I, I, P, P, I, F, F, P, P])
    _sig(lib, "xb_expert_gemm_mma", I, [I, P, P, P, P, P, I, I, I, I, I, I, I, L, L, I, F, F, P])
    _sig(lib, "xb_expert_gather", I, [I, P, P, P, P, I, I, I, I, P])
    _sig(lib, "xb_expert_combine", I, [I, P, P, P, I, I, I, P, P, P, P])
    _sig(lib, "xb_expert_router", I, [I, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, F, P])
    _sig(lib, "xb_attn_decode_tc", I,
         [P, P, P, P, P, P, P, P, I, I, I, I, I, I, L, I, I, I, F, F, F, P, F, I, I, I, I, P, I, P, P])
