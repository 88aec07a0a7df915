"""ctypes binding of libdejavu_b200.so (declared in include/dejavu_b200.h), libdejavu_b200_hybrid.so
(include/dejavu_b200_hybrid.h) and libdejavu_b200_routed.so (include/dejavu_b200_routed.h).

The libraries are the only compute path of this package: if one is missing the import of any operator
raises, there is no PyTorch or CPU fallback.
"""
from __future__ import annotations

import ctypes as C
from pathlib import Path

PKG = Path(__file__).resolve().parent
LIB_PATH = PKG / "libdejavu_b200.so"
HYBRID_LIB_PATH = PKG / "libdejavu_b200_hybrid.so"
ROUTED_LIB_PATH = PKG / "libdejavu_b200_routed.so"

OK, ERR_INVALID, ERR_UNSUPPORTED, ERR_CUDA, ERR_SCRATCH, ERR_TIMEOUT = 0, -1, -2, -3, -4, -5
ACT = {"id": 0, "relu": 1, "gelu": 2, "gelu_approx": 3, "squared_relu": 4, "softcap": 5, "clamped_glu": 6, "silu_glu": 7}
DTYPE_F16, DTYPE_BF16, DTYPE_F32 = 0, 1, 2
MAX_BATCH = 32
KV_WINDOW = 16
EXCHANGE_REFILL = 1
ATTN_STATE_HDR = 8


class DejavuKernelError(RuntimeError):
    """A C-ABI call returned a negative status."""

    def __init__(self, fn: str, status: int, message: str):
        super().__init__(f"{fn} failed with status {status}: {message}")
        self.status = status


_vp, _i, _ll, _sz, _f = C.c_void_p, C.c_int, C.c_longlong, C.c_size_t, C.c_float

# name -> (restype, argtypes); mirrors include/dejavu_b200.h one to one
SIGNATURES = {
    "djv_version": (_i, []),
    "djv_last_error": (C.c_char_p, []),
    "djv_status_string": (C.c_char_p, [_i]),
    "djv_launch_count": (C.c_ulonglong, []),
    "djv_gather_gemv": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _ll, _i, _i, _vp]),
    "djv_gather_transposed_gemv_scratch_bytes": (_sz, [_i, _i, _i]),
    "djv_gather_transposed_gemv": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _ll, _i, _vp, _sz, _vp]),
    "djv_gather_transposed_gemv_static": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _ll, _i, _vp]),
    "djv_mlp_sparse": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _ll, _ll, _i, _vp, _sz, _vp]),
    "djv_topk": (_i, [_vp, _vp, _vp, _i, _i, _i, _vp]),
    "djv_qkv_proj_sparse": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp]),
    "djv_out_proj_sparse": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp]),
    "djv_k_cache_copy_sparse": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _ll, _ll, _vp]),
    "djv_v_cache_copy_sparse": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _ll, _ll, _vp]),
    "djv_attn_state_reset": (_i, [_vp, _i, _i, _vp]),
    "djv_attn_step_scratch_bytes": (_sz, [_i, _i, _i]),
    "djv_attn_step": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _f, _vp, _sz, _vp]),
    "djv_attn_step_project": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp]),
    "djv_topk_attn_prep": (_i, [_vp, _vp, _i, _i, _i, _vp, _i, _vp]),
    "djv_attn_step_attend": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _f, _vp, _sz, _vp]),
    "djv_attn_step_project_batch": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp]),
    "djv_attn_step_attend_batch": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _f, _vp, _sz, _vp]),
    "djv_attn_step_finish": (_i, [_vp, _i, _vp]),
    "djv_decode_attn_scratch_bytes": (_sz, [_i, _i, _i, _i]),
    "djv_decode_attn": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _f, _vp, _sz, _vp]),
    "djv_add_layernorm": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _f, _vp]),
    "djv_ipc_alloc": (_i, [_sz, C.POINTER(_vp)]),
    "djv_ipc_free": (_i, [_vp]),
    "djv_ipc_get_handle": (_i, [_vp, C.c_char_p]),
    "djv_ipc_open": (_i, [C.c_char_p, C.POINTER(_vp)]),
    "djv_ipc_close": (_i, [_vp]),
    "djv_comm_buffer_bytes": (_sz, [_i, _sz]),
    "djv_comm_create": (_i, [C.POINTER(_vp), _i, _i, C.POINTER(_vp), _sz]),
    "djv_gather_transposed_gemv_push": (_i, [_vp, _i, _vp, _vp, _vp, _vp, _i, _i, _i, _ll, _i, _vp, _sz, _vp]),
    "djv_out_proj_sparse_push": (_i, [_vp, _i, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp]),
    "djv_comm_end_step": (_i, [_vp, _i, _vp]),
    "djv_prefetch_rows_l2": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _ll, _ll, _vp]),
    "djv_prefetch_segments_l2": (_i, [_vp, _vp, _i, _i, _i, _ll, _i, _vp]),
    "djv_mlp_sparse_fused_supported": (_i, [_i, _i, _i]),
    "djv_mlp_sparse_fused_single_batch": (_i, [_i, _i, _i]),
    "djv_mlp_sparse_fused_scratch_bytes": (_sz, [_i, _i, _i]),
    "djv_mlp_ring_timeouts": (C.c_uint, []),
    "djv_mlp_ring_bad_indices": (C.c_uint, []),
    "djv_mlp_sparse_fused": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _ll, _ll, _i, _vp, _sz, _vp]),
    "djv_mlp_sparse_fused_exchange": (_i, [_vp, _i, _i, _i, _vp, _vp, _vp, _vp, _vp, _f, _vp, _vp, _vp, _vp, _vp,
                                           _i, _i, _i, _i, _ll, _ll, _i, _vp, _sz, _vp]),
    "djv_set_early_weight_prefetch": (None, [_i]),
    "djv_set_programmatic_launch": (None, [_i]),
    "djv_batch_sum": (_i, [_vp, _vp, _i, _i, _vp]),
    "djv_comm_destroy": (_i, [_vp]),
    "djv_comm_status": (_i, [_vp]),
    "djv_allreduce_add_layernorm": (_i, [_vp, _i, _i, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _f, _vp]),
}

# functions every library has (each keeps its own error message, launch counter and launch mode)
_PLUMBING = ("djv_version", "djv_last_error", "djv_status_string", "djv_launch_count", "djv_set_early_weight_prefetch",
             "djv_set_programmatic_launch")

# mirrors include/dejavu_b200_hybrid.h one to one
HYBRID_SIGNATURES = {
    "djv_hyper_step": (_i, [_i, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _f, _vp, _vp, _vp, _i, _i, _i, _i, _vp]),
    "djv_dense_gemv": (_i, [_i, _i, _vp, _vp, _vp, _i, _i, _i, _ll, _i, _f, _vp]),
    "djv_residual_step": (_i, [_i, _vp, _vp, _vp, _vp, _vp, _vp, _i, _vp, _vp, _f, _f, _vp, _vp, _vp, _i, _i, _i, _vp]),
    "djv_glu": (_i, [_i, _vp, _vp, _ll, _i, _i, _f, _vp]),
    "djv_softcap": (_i, [_vp, _ll, _f, _vp]),
    "djv_rotary": (_i, [_i, _vp, _ll, _vp, _f, _vp, _i, _i, _i, _i, _i, _i, _vp]),
    "djv_window_attn": (_i, [_i, _vp, _vp, _ll, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _f, _vp]),
    "djv_window_store": (_i, [_i, _vp, _vp, _vp, _ll, _vp, _i, _i, _i, _i, _i, _i, _i, _vp]),
    "djv_window_attn_decode": (_i, [_i, _vp, _vp, _ll, _vp, _vp, _vp, _vp, _f, _i, _vp, _i, _i, _i, _i, _i, _i, _i, _f,
                                    _vp]),
    "djv_window_timeouts": (C.c_uint, []),
    "djv_gla_scratch_bytes": (_sz, [_i, _i, _i, _i, _i, _i]),
    "djv_gla_prefill": (_i, [_i, _vp, _vp, _ll, _vp, _vp, _i, _f, _vp, _f, _f, _vp, _vp, _i, _i, _i, _i, _i, _vp, _sz,
                             _vp]),
    "djv_gla_decode": (_i, [_i, _vp, _vp, _ll, _vp, _vp, _i, _f, _vp, _f, _f, _vp, _vp, _i, _i, _i, _i, _vp]),
}

# mirrors include/dejavu_b200_routed.h one to one
ROUTED_SIGNATURES = {
    "djv_mlstm_state_floats": (_i, [_i, _i]),
    "djv_mlstm_scratch_bytes": (_sz, [_i, _i, _i, _i, _i, _i]),
    "djv_mlstm_prefill": (_i, [_i, _vp, _vp, _ll, _vp, _ll, _vp, _vp, _f, _vp, _f, _f, _vp, _vp, _i, _i, _i, _i, _i, _vp,
                               _sz, _vp]),
    "djv_mlstm_decode": (_i, [_i, _vp, _vp, _ll, _vp, _ll, _vp, _vp, _f, _vp, _f, _f, _vp, _vp, _i, _i, _i, _i, _vp]),
    "djv_mlstm_timeouts": (C.c_uint, []),
    "djv_latent_rows": (_i, [_i, _vp, _vp, _ll, _vp, _vp, _f, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _vp]),
    "djv_latent_attn": (_i, [_i, _vp, _vp, _ll, _vp, _ll, _vp, _ll, _vp, _ll, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _f,
                             _vp]),
    "djv_latent_scratch_floats": (_sz, [_i, _i, _i, _i]),
    "djv_latent_decode": (_i, [_i, _vp, _vp, _vp, _sz, _vp, _ll, _vp, _vp, _vp, _f, _vp, _vp, _vp, _ll, _vp, _i, _i, _i, _i,
                               _i, _i, _i, _i, _f, _i, _vp]),
    "djv_moe_route": (_i, [_i, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _vp]),
    "djv_moe_grouped": (_i, [_i, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp]),
    "djv_moe_decode": (_i, [_i, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _vp]),
    "djv_moe_timeouts": (C.c_uint, []),
}

# functions of the hybrid header that the routed library has as well
SHARED = ("djv_hyper_step", "djv_residual_step", "djv_dense_gemv", "djv_glu", "djv_softcap", "djv_rotary",
          "djv_window_timeouts")

_lib = None
_hybrid = None
_routed = None


def _open(path, signatures) -> C.CDLL:
    if not path.exists():
        raise ImportError(
            f"{path} is missing: build it with `python -m dejavu_b200.build` "
            "(there is no fallback path)"
        )
    lib = C.CDLL(str(path))
    for name, (res, args) in signatures.items():
        fn = getattr(lib, name)
        fn.restype = res
        fn.argtypes = args
    return lib


def load() -> C.CDLL:
    """Loads the sparse path's shared library (once). Raises if it has not been built."""
    global _lib
    if _lib is None:
        _lib = _open(LIB_PATH, SIGNATURES)
    return _lib


def load_hybrid() -> C.CDLL:
    """Loads the hybrid decoders' shared library (once). Raises if it has not been built."""
    global _hybrid
    if _hybrid is None:
        _hybrid = _open(HYBRID_LIB_PATH, {**HYBRID_SIGNATURES, **{n: SIGNATURES[n] for n in _PLUMBING}})
    return _hybrid


def load_routed() -> C.CDLL:
    """Loads the shared library of the routed decoders (once). Raises if it has not been built."""
    global _routed
    if _routed is None:
        own = {**ROUTED_SIGNATURES, **{n: HYBRID_SIGNATURES[n] for n in SHARED}}
        _routed = _open(ROUTED_LIB_PATH, {**own, **{n: SIGNATURES[n] for n in _PLUMBING}})
    return _routed


def _library_of(fn_name: str) -> C.CDLL:
    if fn_name in ROUTED_SIGNATURES:
        return load_routed()
    if fn_name in SHARED and _hybrid is None and (_routed is not None or not HYBRID_LIB_PATH.exists()):
        return load_routed()
    return load_hybrid() if fn_name in HYBRID_SIGNATURES else load()


def check(fn_name: str, status: int, lib=None) -> None:
    if status != OK:
        msg = (lib or load()).djv_last_error().decode(errors="replace")
        raise DejavuKernelError(fn_name, status, msg)


def call(fn_name: str, *args) -> None:
    lib = _library_of(fn_name)
    check(fn_name, getattr(lib, fn_name)(*args), lib)


def launch_count() -> int:
    """Kernels launched by the loaded libraries since load."""
    return sum(int(lib.djv_launch_count()) for lib in (_lib, _hybrid, _routed) if lib is not None)
