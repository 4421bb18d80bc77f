"""ctypes bindings of the C ABIs declared in include/fa_b200.h and include/fa_b200_hybrid.h.

The libraries are loaded from the package directory, each when an operator of it is first used.  There is no
fallback: if a library is missing, the use of any of its operators raises, with the build command in the message.
"""
from __future__ import annotations

import ctypes
import os

from .build import HYBRID_LIB_PATH, LIB_PATH

_c = ctypes
_vp, _i, _i64, _sz = _c.c_void_p, _c.c_int, _c.c_int64, _c.c_size_t

# name -> (restype, argtypes); every symbol include/fa_b200.h declares
SIGNATURES = {
    "fa_version": (_i, []),
    "fa_last_error": (_c.c_char_p, []),
    "fa_decode_workspace_bytes": (_sz, [_i, _i, _i, _i]),
    "fa_decode_workspace_init": (_i, [_vp, _sz, _vp]),
    "fa_decode_status": (_i, [_vp, _vp, _c.POINTER(_i)]),
    "fa_decode_set_tuning": (_i, [_i, _i, _i]),
    "fa_paged_decode_gqa_f16": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i64, _i, _i64, _vp, _sz, _vp]),
    "fa_paged_decode_gqa_f16_out_bf16": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i64, _i, _i64, _vp, _sz, _vp]),
    "fa_paged_decode_gqa_f16_static_scratch": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i64, _i, _i64, _vp]),
    "fa_decode_gqa_f16": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _vp, _sz, _vp]),
    "fa_decode_sliding_window_gqa_f16": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _vp, _sz, _vp]),
    "fa_decode_int8_kv_cache_gqa": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp, _sz, _vp]),
    "fa_decode_varlen_f16": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp, _sz, _vp]),
    "fa_decode_int8_gqa": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp, _vp, _sz, _vp]),
    "fa_rope_append_paged_f16": (_i, [_vp] * 12 + [_i, _i, _i, _i, _i, _i, _i64, _i, _vp]),
    "fa_add_rmsnorm_bf16": (_i, [_vp, _vp, _vp, _vp, _i64, _i, _c.c_float, _vp]),
    "fa_qk_norm_split_f16": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i64, _i, _i, _i, _c.c_float, _vp]),
    "fa_qkv_rope_append_f16": (_i, [_vp] * 13 + [_i, _i, _i, _i, _i, _c.c_float, _i64, _i, _vp]),
    "fa_silu_mul_bf16": (_i, [_vp, _vp, _i64, _i, _vp]),
    "fa_half_to_bf16": (_i, [_vp, _vp, _i64, _vp]),
    "fa_peer_alloc": (_i, [_sz, _c.POINTER(_vp), _c.POINTER(_vp), _c.POINTER(_vp), _vp, _vp]),
    "fa_peer_open": (_i, [_vp, _c.POINTER(_vp)]),
    "fa_peer_close": (_i, [_vp]),
    "fa_peer_free": (_i, [_vp, _vp, _vp]),
    "fa_peer_allreduce_sum_bf16": (_i, [_c.POINTER(_vp), _c.POINTER(_vp), _vp, _i, _i, _i64, _i64, _vp]),
    "fa_peer_allreduce_add_rmsnorm_bf16": (_i, [_c.POINTER(_vp), _c.POINTER(_vp), _vp, _i, _i, _i64, _i64, _i64, _i64,
                                                _i, _vp, _c.c_float, _vp]),
    "fa_peer_allgather": (_i, [_c.POINTER(_vp), _c.POINTER(_vp), _vp, _i, _i, _vp, _i64, _i64, _vp]),
    "fa_peer_status": (_i, [_vp, _vp, _c.POINTER(_i)]),
    "fa_peer_reset": (_i, [_vp, _vp, _vp]),
    "fa_peer_set_max_polls": (_i, [_c.c_uint]),
    "fa_prefill_set_impl": (_i, [_i]),
    "fa_prefill_status": (_i, [_vp, _c.POINTER(_i), _i]),
    "fa_prefill_dense_f16": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp]),
    "fa_prefill_varlen_f16": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i64, _i, _i, _i, _i, _i, _vp]),
    "fa_prefill_varlen_f16_out_bf16": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i64, _i, _i, _i, _i, _i, _vp]),
    "fa_paged_decode_gqa_bf16": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i64, _i, _i64, _vp, _sz, _vp]),
    "fa_decode_gqa_bf16": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _vp, _sz, _vp]),
    "fa_prefill_dense_bf16": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp]),
    "fa_prefill_varlen_bf16": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i64, _i, _i, _i, _i, _i, _vp]),
    "fa_rope_append_paged_bf16": (_i, [_vp] * 12 + [_i, _i, _i, _i, _i, _i, _i64, _i, _vp]),
    "fa_qkv_rope_append_bf16": (_i, [_vp] * 13 + [_i, _i, _i, _i, _i, _c.c_float, _i64, _i, _vp]),
}

# every symbol include/fa_b200_hybrid.h declares
_f = _c.c_float
HYBRID_SIGNATURES = {
    "fah_last_error": (_c.c_char_p, []),
    "fah_residual_norm": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _vp, _vp, _i64, _i, _f, _i, _vp]),
    "fah_gated_norm": (_i, [_vp, _vp, _i64, _vp, _vp, _i64, _i, _f, _i, _vp]),
    "fah_clamped_glu": (_i, [_vp, _vp, _i64, _i, _f, _f, _f, _i, _vp]),
    "fah_side_gate": (_i, [_vp, _vp, _vp, _i, _i64, _i, _vp, _i64, _i, _i, _vp]),
    "fah_lightning_workspace": (_sz, [_i] * 6),
    "fah_lightning": (_i, [_vp, _i64] + [_i] * 6 + [_vp, _vp, _i, _vp, _vp, _vp, _i, _i, _i64, _vp, _vp, _sz, _vp, _i, _vp]),
    "fah_latent_prep": (_i, [_vp, _i64] + [_i] * 6 + [_vp, _vp, _f] + [_vp] * 6 + [_i, _i, _vp, _i, _i, _vp, _vp, _i64, _vp, _i, _vp]),
    "fah_rotate_heads": (_i, [_vp, _vp, _vp, _i64, _i, _i, _i, _i, _i, _vp]),
    "fah_latent_attention_workspace": (_sz, [_i, _i, _i, _i64, _i]),
    "fah_latent_attention": (_i, [_vp, _vp, _i, _i, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _vp, _vp, _vp, _i64, _i, _i, _i, _f, _vp,
                                  _i64, _vp, _sz, _vp, _i, _vp]),
    "fah_latent_prefill": (_i, [_vp, _vp, _vp, _vp, _i64, _vp, _vp, _i, _i, _i64, _i64, _i, _i, _i, _i, _f, _vp, _vp, _vp]),
    "fah_latent_prefill_supported": (_i, [_i, _i, _i, _f, _i]),
    "fah_latent_gather": (_i, [_vp, _i, _i, _vp, _i, _i, _vp, _i64, _i, _i, _vp, _vp, _vp, _i, _vp]),
}

_lib = None
_hybrid_lib = None


def _open(path: str, signatures) -> ctypes.CDLL:
    if not os.path.exists(path):
        raise RuntimeError(
            f"{path} is missing: the CUDA library has not been built. "
            "Run `python -m flash_attn_v100_b200.build` (needs nvcc); there is no CPU fallback.")
    lib = ctypes.CDLL(path)
    for name, (res, args) in signatures.items():
        fn = getattr(lib, name)  # AttributeError if the symbol is not exported
        fn.restype = res
        fn.argtypes = args
    return lib


def load() -> ctypes.CDLL:
    global _lib
    if _lib is None:
        _lib = _open(LIB_PATH, SIGNATURES)
    return _lib


def load_hybrid() -> ctypes.CDLL:
    global _hybrid_lib
    if _hybrid_lib is None:
        _hybrid_lib = _open(HYBRID_LIB_PATH, HYBRID_SIGNATURES)
    return _hybrid_lib


def last_error() -> str:
    return load().fa_last_error().decode("utf-8", "replace")


def check(rc: int) -> None:
    if rc != 0:
        raise RuntimeError(last_error() or f"fa_b200 call failed with status {rc}")


def check_hybrid(rc: int) -> None:
    if rc != 0:
        raise RuntimeError(load_hybrid().fah_last_error().decode("utf-8", "replace") or
                           f"fa_b200_hybrid call failed with status {rc}")
