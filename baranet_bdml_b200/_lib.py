"""ctypes binding of libbn_attn.so (the C ABI declared in include/bn_attn.h).

There is no fallback: if the library is missing, or a call returns a non-zero
status, a RuntimeError is raised — the reference's own error convention
(src/utils/check_error.cuh:8-14 turns every failure into std::runtime_error,
which pybind11 surfaces as RuntimeError).
"""
from __future__ import annotations

import ctypes as C
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
# BN_ATTN_LIB names another build of the same library (e.g. an instrumented one)
LIB_PATH = os.environ.get("BN_ATTN_LIB") or os.path.join(_HERE, "libbn_attn.so")

BN_OK, BN_ERR_INVALID_ARG, BN_ERR_UNSUPPORTED, BN_ERR_CUDA, BN_ERR_ARCH, BN_ERR_TIMEOUT, BN_ERR_WORKSPACE = range(7)
BN_HEADS_COLLAPSED, BN_HEADS_PER_HEAD = 0, 1
BN_PAGE_TOKENS = 16
BN_ACT_NONE, BN_ACT_SILU, BN_ACT_GELU_TANH, BN_ACT_RELU2 = range(4)

_i, _i64, _f, _p, _sz = C.c_int, C.c_int64, C.c_float, C.c_void_p, C.c_size_t

# name -> (restype, argtypes); mirrors include/bn_attn.h one to one
SIGNATURES = {
    "bn_last_error": (C.c_char_p, []),
    "bn_version": (_i, []),
    "bn_mm_f32": (_i, [_p, _i64, _i64, _p, _i64, _i64, _p, _i64, _i64, _i, _i, _i, _p]),
    "bn_rope_f32": (_i, [_p, _i64, _i64, _p, _i64, _i64, _i, _i, _i, _f, _i, _p]),
    "bn_embedding_gather_f32": (_i, [_p, _i64, _p, _p, _i64, _i, _i, _i, _p, _p]),
    "bn_argmax_rows_f32": (_i, [_p, _i64, _i64, _p, _i, _i, _p]),
    "bn_add_rmsnorm_bf16": (_i, [_p, _p, _p, _p, _p, _i, _i, _f, _p]),
    "bn_gemm_bf16_nt": (_i, [_p, _p, _p, _i, _i, _i, _p, _p]),
    "bn_gemm_bf16_nt_small_m_workspace_bytes": (_sz, [_i, _i, _i]),
    "bn_gemm_bf16_nt_small_m": (_i, [_p, _p, _p, _i, _i, _i, _p, _sz, _p, _p]),
    "bn_gemm_bf16_nt_skinny": (_i, [_p, _p, _i, _i, _i, _p, _i, _p, _i, _p, _p]),
    "bn_gemm_swiglu_bf16_nt_skinny": (_i, [_p, _p, _p, _p, _i, _i, _i, _p]),
    "bn_gemm_qkv_append_bf16_skinny": (_i, [_p, _p, _i, _i, _i, _i, _i, _p, _p, _i64, _p, _i, _p, _p, _f, _p]),
    "bn_gemm_swiglu_bf16_nt": (_i, [_p, _p, _p, _i, _i, _i, _p, _p]),
    "bn_rmsnorm_f32": (_i, [_p, _i64, _i64, _p, _i64, _p, _i64, _i64, _i, _i, _f, _p]),
    "bn_add_rmsnorm_f32": (_i, [_p, _i64, _i64, _p, _i64, _i64, _p, _i64, _p, _i64, _i64, _p, _i64, _i64, _i, _i, _f,
                                _p]),
    "bn_attn_prefill_f32": (_i, [_p, _i64, _i64, _p, _i64, _i64, _p, _i64, _i64, _p, _i64, _i64,
                                 _i, _i, _i, _i, _f, _f, _i, _i, _i, _i, _p]),
    "bn_attn_prefill_bf16_workspace_bytes": (_sz, [_i, _i, _i, _i, _i]),
    "bn_attn_prefill_bf16": (_i, [_p, _p, _p, _p, _p, _i, _i, _i, _i, _i, _f, _f, _i, _i, _i, _p, _sz, _p]),
    "bn_attn_prefill_bf16_table": (_i, [_i, _i, _i, _i, _f, _i, _p, _sz, _p]),
    "bn_gemm_qkv_rope_bf16": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _i, _i, _i, _p, _sz, _p, _i64, _p, _i, _p, _p]),
    "bn_kv_append": (_i, [_p, _i64, _p, _i, _p, _p, _i, _p, _p, _i64, _i, _i, _i, _f, _p]),
    "bn_attn_decode_workspace_bytes": (_sz, [_i, _i, _i, _i, _i, _i]),
    "bn_attn_decode_paged": (_i, [_p, _p, _i64, _p, _i, _p, _p, _p, _p, _p, _i, _i, _i, _i, _f, _f, _i, _i, _i,
                                  _p, _sz, _p]),
    "bn_attn_decode_paged_static": (_i, [_p, _p, _i64, _p, _i, _p, _p, _p, _p, _p, _i, _i, _i, _i, _f, _f, _i, _i, _p]),
    "bn_attn_decode_paged_static_status": (_i, [_p]),
    "bn_attn_lse_combine": (_i, [_p, _p, _i, _i64, _i, _p, _p, _p, _p]),
    "bn_attn_lse_combine_strided": (_i, [_p, _i64, _p, _i64, _i, _i64, _i, _p, _p, _p, _p]),
    "bn_workspace_status": (_i, [_p, _p]),
    "bn_selftest_wait_timeout": (_i, [_p, C.c_uint, _p]),
    "bn_exchange_create": (_i, [_i, _i, _i, _i, C.POINTER(_p)]),
    "bn_exchange_ipc_handle": (_i, [_p, _p]),
    "bn_exchange_open_peers": (_i, [_p, _p, _i]),
    "bn_exchange_combine": (_i, [_p, _p, _p, _p, C.c_uint, _p]),
    "bn_exchange_status": (_i, [_p, _p]),
    "bn_exchange_destroy": (None, [_p]),
    "bn_gemm_glu_bf16_nt": (_i, [_p, _p, _p, _i, _i, _i, _i, _p, _p]),
    "bn_gemm_bf16_nt_f32": (_i, [_p, _p, _p, _i, _i, _i, _p, _p]),
    "bn_gemm_act_mul_bf16_nt": (_i, [_p, _p, _p, _i64, _p, _i, _i, _i, _i, _p, _p]),
    "bn_gemm_bf16_nt_small_m_f32": (_i, [_p, _p, _p, _i, _i, _i, _p, _sz, _p, _p]),
    "bn_gemm_act_mul_bf16_nt_small_m": (_i, [_p, _p, _p, _i64, _p, _i, _i, _i, _i, _p, _sz, _p, _p]),
    "bn_gemm_glu_bf16_nt_skinny": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _p]),
    "bn_gemm_bf16_nt_skinny_f32": (_i, [_p, _p, _i, _i, _i, _p, _p]),
    "bn_gemm_act_mul_bf16_nt_skinny": (_i, [_p, _p, _p, _i64, _p, _i, _i, _i, _i, _p]),
    "bn_act_mul_f32": (_i, [_p, _i64, _p, _i64, _p, _i64, _i, _i, _i, _p]),
    "bn_embedding_gather_bf16": (_i, [_p, _i64, _p, _p, _i64, _p, _i64, _i, _i, _i, _p, _p]),
    "bn_residual_norm": (_i, [_p, _p, _i64, _i, _p, _f, _p, _p, _p, _i64, _i, _p, _p, _p, _i64, _i, _i, _i, _i, _f,
                              _p]),
    "bn_latent_prep": (_i, [_p, _i64, _p, _p, _f, _p, _p, _p, _i, _i, _i, _i, _i, _p, _i64, _p, _p, _i, _i, _p, _i,
                            _i, _p]),
    "bn_latent_gather": (_i, [_p, _i, _i, _i, _p, _p, _i, _i, _p, _p, _i, _i, _p]),
    "bn_rope_heads": (_i, [_p, _i64, _i, _i, _i, _i, _i, _p, _p, _i, _p]),
    "bn_attn_window": (_i, [_p, _i64, _p, _p, _i64, _p, _i64, _p, _i64, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _p,
                            _i, _p]),
    "bn_latent_absorb_q": (_i, [_p, _i64, _p, _p, _p, _p, _i, _i, _i, _i, _i, _i, _p]),
    "bn_latent_decode_splits": (_i, [_i, _i, _i, _i, _i, _i]),
    "bn_latent_decode": (_i, [_p, _p, _i, _i, _p, _p, _p, _p, _i, _i, _i, _i, _i, _i, _f, _i, _p]),
    "bn_latent_expand_out": (_i, [_p, _p, _i, _p, _p, _i64, _i, _i, _i, _i, _i, _p]),
    "bn_mamba2_conv": (_i, [_p, _i64, _p, _p, _p, _p, _p, _p, _p, _i, _i, _i, _i, _i, _i, _i, _p, _i64, _p, _p, _i,
                            _p]),
    "bn_ssm_scan": (_i, [_p, _i64, _p, _p, _p, _p, _p, _i, _i, _i, _i, _i, _i, _p, _i64, _i, _p]),
    "bn_mamba2_step": (_i, [_p, _i64, _p, _p, _p, _p, _p, _p, _p, _p, _p, _i, _i, _i, _i, _i, _i, _p, _i, _p]),
    "bn_gemm_bias_act_bf16_nt": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _p, _p]),
    "bn_gemm_bias_act_bf16_nt_small_m": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _p, _sz, _p, _p]),
    "bn_gemm_bias_act_bf16_nt_skinny": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _p]),
    "bn_bias_act_f32": (_i, [_p, _i64, _p, _i, _i, _i, _p]),
    "bn_hyper_norm": (_i, [_p, _i, _i, _p, _p, _p, _p, _i64, _p, _p, _p, _p, _i64, _i, _i, _i, _f, _p]),
    "bn_kv_prep": (_i, [_p, _p, _i64, _p, _i64, _f, _p, _p, _i, _i, _i, _i, _i, _i, _f, _p, _p, _i, _i, _p, _p, _i, _i, _i, _p]),
    "bn_kv_gather": (_i, [_p, _p, _i, _i, _i, _i, _i, _p, _p, _i, _i, _p, _p, _i, _i, _p]),
    "bn_attn_chunked": (_i, [_p, _i64, _p, _i64, _p, _i64, _p, _i64, _p, _i64, _i, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _f,
                             _f, _p, _i, _p]),
    "bn_gqa_step_splits": (_i, [_i, _i, _i, _i, _i, _i, _i]),
    "bn_gqa_step": (_i, [_p, _p, _p, _p, _i64, _p, _i64, _f, _p, _p, _i, _i, _i, _p, _p, _p, _p, _i, _p, _i64, _i, _i, _i, _i, _i,
                         _i, _f, _f, _p, _i, _p]),
    "bn_gated_group_norm": (_i, [_p, _i64, _i, _p, _i64, _p, _p, _i64, _i, _i, _i, _f, _i, _p]),
}

_lib = None


def load() -> C.CDLL:
    """Loads the CUDA library; raises if it has not been built."""
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise RuntimeError(
                f"{LIB_PATH} is missing: build it with `python -m baranet_bdml_b200.build` "
                "(there is no CPU fallback for the attention kernels)")
        _bind(LIB_PATH, whole=True)
    return _lib


def load_family(family: str) -> C.CDLL:
    """Loads what a model family launches, compiling it first where the checkout has no current build."""
    if _lib is None:
        from . import build
        path = os.environ.get("BN_ATTN_LIB") or build.build_for(family)
        _bind(path, whole=path in (LIB_PATH, build.LIB))
    return _lib


def _bind(path: str, whole: bool) -> None:
    global _lib
    lib = C.CDLL(path)
    for name, (res, args) in SIGNATURES.items():
        if not whole and not hasattr(lib, name):
            continue                      # a family's library exports what that family calls
        fn = getattr(lib, name)
        fn.restype = res
        fn.argtypes = args
    _lib = lib


def last_error() -> str:
    return load().bn_last_error().decode()


def check(status: int) -> None:
    if status != BN_OK:
        raise RuntimeError(f"bn_attn status {status}: {last_error()}")
