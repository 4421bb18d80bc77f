"""ctypes bindings of the C ABIs declared in include/fa_b200.h, fa_b200_rows.h, fa_b200_hybrid.h and fa_b200_mixers.h.

The libraries are loaded from the package directory, each when an operator of it is first used.  There is no
fallback: if a library is missing, the use of any of its operators raises, with the build command in the message.
"""
from __future__ import annotations

import ctypes
import os

from .build import LIBRARIES

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

_f = _c.c_float

# every symbol include/fa_b200_rows.h declares
class ResidualNorm(_c.Structure):
    """FarResidualNorm"""
    _fields_ = [("x", _vp), ("delta", _vp), ("delta_w", _vp), ("embed", _vp), ("tokens", _vp), ("embed_mode", _i), ("vocab", _i),
                ("embed_scale", _f), ("eps", _f), ("more", _vp * 2), ("more_rows", _vp * 2), ("more_n", _i * 2), ("w", _vp), ("w2", _vp),
                ("out", _vp), ("out2", _vp), ("rows", _i64), ("cols", _i), ("dtype", _i)]


ROWS_SIGNATURES = {
    "far_last_error": (_c.c_char_p, []),
    "far_residual_norm": (_i, [_c.POINTER(ResidualNorm), _vp]),
    "far_gated_norm": (_i, [_vp, _vp, _i64, _vp, _vp, _i64, _i64, _i, _i, _i, _f, _i, _vp]),
    "far_gelu": (_i, [_vp, _i64, _vp, _i64, _i64, _i, _i, _vp]),
    "far_bigram_rows": (_i, [_vp] * 5 + [_i, _i, _i64, _i64, _i64, _i64, _vp, _vp, _vp]),
    "far_clamped_glu": (_i, [_vp, _vp, _i64, _i, _f, _f, _f, _i, _vp]),
    "far_side_gate": (_i, [_vp, _vp, _vp, _i, _i64, _i, _vp, _i64, _i, _i, _vp]),
}

# every symbol include/fa_b200_hybrid.h declares
HYBRID_SIGNATURES = {
    "fah_last_error": (_c.c_char_p, []),
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

# every symbol include/fa_b200_mixers.h declares
class Recurrence(_c.Structure):
    """FamRecurrence"""
    _fields_ = [("x", _vp), ("stride", _i64), ("total", _i64), ("off_q", _i), ("off_k", _i), ("off_v", _i), ("heads", _i), ("groups", _i), ("dk", _i),
                ("dv", _i), ("n_slots", _i), ("n_seq", _i), ("max_len", _i), ("dtype", _i), ("q_scale", _f), ("norm_eps", _f), ("la", _vp), ("b", _vp),
                ("floor", _vp), ("n0", _vp), ("skip", _vp), ("norm", _vp), ("state", _vp), ("slots", _vp), ("starts", _vp), ("cu_seqlens", _vp),
                ("out", _vp), ("workspace", _vp), ("workspace_bytes", _i64), ("status", _vp)]


class Pages(_c.Structure):
    """FamPages"""
    _fields_ = [("k_pool", _vp), ("v_pool", _vp), ("block_table", _vp), ("tok_seq", _vp), ("positions", _vp), ("n_blocks", _i), ("max_blocks", _i),
                ("n_seq", _i), ("heads", _i), ("kv_heads", _i), ("dim", _i), ("vdim", _i), ("dtype", _i), ("rows", _i64), ("status", _vp)]


_rec, _pg = _c.POINTER(Recurrence), _c.POINTER(Pages)
MIXERS_SIGNATURES = {
    "fam_last_error": (_c.c_char_p, []),
    "fam_recurrence_workspace": (_sz, [_rec]),
    "fam_recurrence": (_i, [_rec, _vp]),
    "fam_max_gates": (_i, [_vp, _i64, _i, _i, _i, _vp, _vp, _f, _vp, _vp, _vp, _i, _i, _vp, _vp, _vp, _i, _i64, _vp, _vp, _vp, _vp, _i, _vp]),
    "fam_step_gates": (_i, [_vp, _i64, _i, _i, _vp, _vp, _i64, _vp, _vp, _i, _vp]),
    "fam_conv_silu": (_i, [_vp, _i64, _i, _i, _i, _vp, _vp, _vp, _i] + [_vp] * 5 + [_i, _i64, _vp, _vp, _i, _vp]),
    "fam_recurrence_step_supported": (_i, [_i, _i]),
    "fam_max_gate_step": (_i, [_rec, _i, _i, _vp, _vp, _f, _vp, _vp]),
    "fam_ssd_step": (_i, [_rec, _i, _vp, _vp, _vp, _vp, _vp, _i, _vp]),
    "fam_kv_prep": (_i, [_pg, _vp, _i64, _i, _i, _i, _vp, _vp, _f, _vp, _i64, _f, _vp, _vp, _vp, _vp]),
    "fam_kv_attention_workspace": (_sz, [_pg, _i]),
    "fam_kv_attention": (_i, [_pg, _vp, _vp, _vp, _i64, _i, _f, _vp, _i64, _vp, _sz, _vp]),
    "fam_kv_gather": (_i, [_pg, _vp, _vp, _vp, _i, _i64, _vp, _vp, _vp]),
    "fam_kv_prefill_supported": (_i, [_i, _i, _i, _i, _f, _i]),
    "fam_kv_prefill": (_i, [_vp] * 5 + [_i, _i, _i64, _i64, _i, _i, _i, _i, _f, _vp, _vp, _i64, _vp, _i64, _vp, _vp]),
}

_libs = {}
_ABIS = {"attention": (SIGNATURES, "fa"), "rows": (ROWS_SIGNATURES, "far"), "hybrid": (HYBRID_SIGNATURES, "fah"),
         "mixers": (MIXERS_SIGNATURES, "fam")}


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


def library(name: str) -> ctypes.CDLL:
    """One of build.LIBRARIES, loaded when it is first asked for."""
    if name not in _libs:
        _libs[name] = _open(LIBRARIES[name][0], _ABIS[name][0])
    return _libs[name]


def load() -> ctypes.CDLL:
    return library("attention")


def last_error(name: str = "attention") -> str:
    return getattr(library(name), _ABIS[name][1] + "_last_error")().decode("utf-8", "replace")


def check(rc: int, name: str = "attention") -> None:
    if rc != 0:
        raise RuntimeError(last_error(name) or f"a call of the {name} library failed with status {rc}")
