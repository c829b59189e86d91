"""ctypes binding of the kernel libraries — the only route from Python to the kernels.

There is deliberately no fallback: if the shared library is missing or a call returns a
non-zero status, a RuntimeError is raised.
"""
from __future__ import annotations

import ctypes
import os
import re

from .build import LIB_PATH, library_path

NB_F32, NB_F16, NB_BF16 = 0, 1, 2

_INCLUDE = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "include")
_HEADERS = {"packed": "nativebit_b200.h", "layered": "nativebit_b200_layered.h"}
_lib = None
_layered = None

_c = ctypes
_SIGNATURES = {
    "nb_version": (_c.c_int, []),
    "nb_status_string": (_c.c_char_p, [_c.c_int]),
    "nb_last_cuda_error": (_c.c_char_p, []),
    "nb_selftest_tables": (_c.c_int, []),
    "nb_unpack": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int64, _c.c_void_p, _c.c_void_p]),
    "nb_pack": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int64, _c.c_void_p, _c.c_void_p]),
    "nb_dequant": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int64, _c.c_int64,
                              _c.c_void_p, _c.c_int, _c.c_void_p]),
    "nb_quantize": (_c.c_int, [_c.c_void_p, _c.c_int64, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p]),
    "nb_gemv_workspace_bytes": (_c.c_size_t, [_c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int]),
    "nb_prefill_workspace_bytes": (_c.c_size_t, [_c.c_int, _c.c_int, _c.c_int]),
    "nb_gemm_prefill": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                   _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_size_t, _c.c_void_p]),
    "nb_prefill_fused_workspace_bytes": (_c.c_size_t, [_c.c_int, _c.c_int, _c.c_int]),
    "nb_gemm_prefill_fused": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p,
                                         _c.c_int, _c.c_void_p, _c.c_size_t, _c.c_void_p]),
    "nb_gemm_bf16": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p,
                                _c.c_void_p]),
    "nb_add_rmsnorm": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_float, _c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p]),
    "nb_rope_kv_write": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p,
                                    _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_void_p]),
    "nb_decode_attention": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                       _c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p]),
    "nb_decode_attention_rope": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_int,
                                            _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p]),
    "nb_silu_mul": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p]),
    "nb_lm_head_scratch_bytes": (_c.c_size_t, []),
    "nb_lm_head": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_float, _c.c_void_p, _c.c_int, _c.c_int, _c.c_float,
                              _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_void_p]),
    "nb_prefill_attention": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_int,
                                        _c.c_void_p, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p]),
    "nb_allreduce_buffer_bytes": (_c.c_size_t, [_c.c_int, _c.c_int]),
    "nb_allreduce": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_uint32,
                                _c.c_void_p, _c.c_void_p]),
    "nb_embed_rows": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p]),
    "nb_softcap_argmax": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_float, _c.c_void_p, _c.c_void_p, _c.c_void_p,
                                     _c.c_void_p]),
    "nb_gemv_fused": (_c.c_int, [_c.c_int, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_float, _c.c_void_p, _c.c_int, _c.c_void_p,
                                 _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p,
                                 _c.c_size_t, _c.c_void_p]),
    "nb_exchange_buffer_bytes": (_c.c_size_t, [_c.c_int, _c.c_int]),
    "nb_exchange_init": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int]),
    "nb_gemv_tp": (_c.c_int, [_c.c_int, _c.c_void_p, _c.c_void_p, _c.c_void_p, _c.c_float, _c.c_void_p, _c.c_int, _c.c_void_p,
                              _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p,
                              _c.c_size_t, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_uint32, _c.c_void_p]),
    "nb_exchange_gather": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_uint32, _c.c_void_p,
                                      _c.c_void_p]),
    "nb_gemv_static": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int,
                                  _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p]),
    "nb_gemv_static_status": (_c.c_int, [_c.c_void_p, _c.c_int]),
    "nb_gemv_ordered": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int,
                                   _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_size_t, _c.c_void_p]),
    "nb_stream_packed_bytes": (_c.c_size_t, [_c.c_int, _c.c_int, _c.c_int]),
    "nb_stream_pack": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p,
                                  _c.c_void_p]),
    "nb_stream_state_bytes": (_c.c_size_t, []),
    "nb_stream_max_ops": (_c.c_int, []),
    "nb_stream_ctas": (_c.c_int, []),
    "nb_stream_slots": (_c.c_int, [_c.c_int, _c.c_int, _c.c_int]),
    "nb_stream_run": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_uint32, _c.c_void_p]),
    "nb_gemv_stream": (_c.c_int, [_c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_float, _c.c_void_p, _c.c_void_p,
                                  _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p]),
    "nb_gemv_stream_max_rows": (_c.c_int, [_c.c_int, _c.c_int]),
    "nb_gemv_stream_rows": (_c.c_int, [_c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_float, _c.c_void_p, _c.c_void_p,
                                       _c.c_int, _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p]),
    "nb_group_plan_bytes": (_c.c_size_t, [_c.c_void_p, _c.c_int]),
    "nb_group_max_items": (_c.c_int, []),
    "nb_group_build": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_size_t]),
    "nb_group_run": (_c.c_int, [_c.c_void_p, _c.c_void_p, _c.c_void_p]),
    "nb_gemv_plan": (_c.c_int, [_c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_void_p]),
    "nb_gemv": (_c.c_int, [_c.c_void_p, _c.c_int, _c.c_int, _c.c_void_p, _c.c_void_p, _c.c_int, _c.c_int, _c.c_int,
                           _c.c_int, _c.c_int, _c.c_void_p, _c.c_int, _c.c_void_p, _c.c_size_t, _c.c_void_p]),
}


_P, _I, _F = _c.c_void_p, _c.c_int, _c.c_float


def _struct(name: str, pointers: str, floats: str, ints: str):
    """An argument block of nativebit_b200_layered.h: pointers first, then floats, then ints."""
    fields = [(n, _P) for n in pointers.split()] + [(n, _F) for n in floats.split()] + [(n, _I) for n in ints.split()]
    return type(name, (_c.Structure,), {"_fields_": fields})


MatvecArgs = _struct("MatvecArgs", "w bias y x delta delta_w x_out norm_w", "eps alpha limit", "N K ldw act norm")
StreamArgs = _struct("StreamArgs", "x x_out y0 w0 y1 w1 coef norm_w", "eps", "streams C y_norm norm")
LatentPrepareArgs = _struct("LatentPrepareArgs", "a cq cache q_norm kv_norm cos2 sin2", "eps",
                            "dtype B T lda q_off q_rank ldcq kv_off rank rot ctx ldc pos0")
LatentAttentionArgs = _struct("LatentAttentionArgs", "q kv cache gate out cos2 sin2", "scale",
                              "dtype B T H dim rot vdim rank ctx ldc ldq ldkv v_off kv_rows kv_pos0 ldg ldo pos0 window")
LatentDecodeArgs = _struct("LatentDecodeArgs", "q a cache uk uv kv_norm cos2 sin2 pos out", "scale eps",
                           "cache_dtype B H dim rot vdim rank ctx ldc ldq lda kv_off g_off ldu ldo window")
GlaArgs = _struct("GlaArgs", "p out state a2 a2_b norm_w lower", "tau eps",
                  "kind dtype B T H dim vdim ldp q_off k_off v_off g_off a_off a_rank lda2 lds ldo")
TalkAttentionArgs = _struct("TalkAttentionArgs", "q cache gate out penalty talk", "scale softcap",
                            "dtype B T H G dim vdim ctx ldc v_off ldq ldg ldo pos0 window n_pen")
TalkDecodeArgs = _struct("TalkDecodeArgs", "p cache penalty talk pos out", "scale softcap",
                         "cache_dtype B H G dim vdim ctx ldc v_off ldp q_off k_off g_off ldo window n_pen")

_LAYERED_SIGNATURES = {
    "nb_embed_scaled": (_I, [_P, _P, _I, _I, _I, _F, _I, _P, _P]),
    "nb_residual_norm": (_I, [_P, _P, _P, _P, _I, _F, _P, _I, _I, _I, _I, _P]),
    "nb_stream_norm": (_I, [_c.POINTER(StreamArgs), _P, _I, _I, _I, _P]),
    "nb_linear_bf16": (_I, [_P, _I, _P, _I, _P, _I, _F, _F, _I, _I, _I, _P, _I, _I, _P, _P]),
    "nb_linear_f32": (_I, [_P, _I, _P, _I, _P, _I, _F, _F, _I, _I, _I, _P, _I, _P]),
    "nb_matvec_bf16": (_I, [_c.POINTER(MatvecArgs), _P]),
    "nb_matvec_streams": (_I, [_c.POINTER(MatvecArgs), _c.POINTER(StreamArgs), _P]),
    "nb_matvec_pair": (_I, [_c.POINTER(MatvecArgs), _c.POINTER(MatvecArgs), _P]),
    "nb_latent_prepare": (_I, [_c.POINTER(LatentPrepareArgs), _P]),
    "nb_latent_attention": (_I, [_c.POINTER(LatentAttentionArgs), _P]),
    "nb_latent_decode": (_I, [_c.POINTER(LatentDecodeArgs), _P]),
    "nb_gla_workspace_bytes": (_c.c_size_t, [_I, _I, _I, _I, _I]),
    "nb_gla_prefill": (_I, [_c.POINTER(GlaArgs), _P, _c.c_size_t, _P]),
    "nb_gla_decode": (_I, [_c.POINTER(GlaArgs), _P]),
    "nb_cache_append": (_I, [_P, _I, _I, _I, _P, _I, _I, _I, _I, _I, _I, _P]),
    "nb_talk_attention_workspace_bytes": (_c.c_size_t, [_I, _I, _I, _I, _I, _I]),
    "nb_talk_attention": (_I, [_c.POINTER(TalkAttentionArgs), _P, _c.c_size_t, _P]),
    "nb_talk_decode": (_I, [_c.POINTER(TalkDecodeArgs), _P]),
    "nb_argmax": (_I, [_P, _I, _I, _P, _P, _P]),
}


def declared_symbols(which: str = "packed") -> list[str]:
    """Names of the functions a public header declares."""
    text = open(os.path.join(_INCLUDE, _HEADERS[which])).read()
    text = re.sub(r"/\*.*?\*/", "", text, flags=re.S)
    return sorted(set(re.findall(r"\b(nb_[a-z0-9_]+)\s*\(", text)))


def _open(path: str, signatures: dict) -> ctypes.CDLL:
    if not os.path.exists(path):
        raise RuntimeError(
            f"{path} is missing: build it with `python -m nativebit_b200.build` "
            "(nativebit_b200 has no fallback path)")
    handle = ctypes.CDLL(path)
    for name, (res, args) in signatures.items():
        fn = getattr(handle, name)
        fn.restype, fn.argtypes = res, args
    return handle


def lib() -> ctypes.CDLL:
    """The packed-model kernels (include/nativebit_b200.h)."""
    global _lib
    if _lib is None:
        _lib = _open(LIB_PATH, _SIGNATURES)
    return _lib


def layered_lib() -> ctypes.CDLL:
    """The layered-model kernels (include/nativebit_b200_layered.h)."""
    global _layered
    if _layered is None:
        common = {n: _SIGNATURES[n] for n in ("nb_status_string", "nb_last_cuda_error")}
        _layered = _open(library_path("layered"), {**_LAYERED_SIGNATURES, **common})
    return _layered


def check(status: int, what: str, handle: ctypes.CDLL | None = None) -> None:
    if status != 0:
        l = handle or lib()
        msg = l.nb_status_string(status).decode()
        cuda = l.nb_last_cuda_error().decode()
        raise RuntimeError(f"{what} failed: status {status} ({msg})" + (f" [{cuda}]" if cuda and status == 5 else ""))
