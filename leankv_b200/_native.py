"""ctypes bindings of ``libleankv_b200.so`` and ``libleankv_mixers.so`` (the C ABI declared in
``include/leankv_b200.h`` and ``include/leankv_mixers.h``).

There is no CPU or PyTorch fallback behind these calls: if the library is missing or a
kernel reports an error, a ``RuntimeError`` is raised.
"""

from __future__ import annotations

import ctypes
import os
from ctypes import (POINTER, Structure, c_char_p, c_float, c_int, c_int32, c_longlong, c_size_t,
                    c_uint8, c_ulonglong, c_void_p)

_PKG_DIR = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_PKG_DIR, "libleankv_b200.so")
MIXERS_PATH = os.path.join(_PKG_DIR, "libleankv_mixers.so")

MAX_SEGMENTS = 4
TQ_PAGE_TOKENS = 16
TQ_DIM = 128
TQ_CHUNK_BYTES = 800
ATTN_EARLY_FETCH = 1


class Segments(Structure):
    """Mirror of ``leankv_segments_t``."""

    _fields_ = [
        ("n_segments", c_int),
        ("seg_end", c_int * MAX_SEGMENTS),
        ("threshold", c_float * MAX_SEGMENTS),
    ]


MAX_RANKS = 8


class Xchg(Structure):
    """Mirror of ``leankv_xchg_t``."""

    _fields_ = [
        ("world", c_int), ("rank", c_int),
        ("n_slots", c_int), ("max_cols", c_int),
        ("max_wait_iters", c_int),
        ("recv", c_void_p * MAX_RANKS),
        ("epoch", c_void_p),
        ("status", c_void_p),
    ]


# name -> (restype, argtypes); every symbol the header declares appears here.
SIGNATURES = {
    "leankv_strerror": (c_char_p, [c_int]),
    "leankv_abi_version": (c_int, []),
    "leankv_last_cuda_error": (c_char_p, []),
    "leankv_sparse_gemv_workspace_bytes": (c_size_t, [c_int, c_int]),
    "leankv_sparse_gemv_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float,
                                       c_void_p, c_void_p, c_void_p, c_size_t, c_void_p, c_void_p]),
    "leankv_sparse_gemv_seg_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int,
                                           POINTER(Segments), c_void_p, c_void_p, c_void_p,
                                           c_size_t, c_void_p, c_void_p]),
    "leankv_sparse_gemv_rmsnorm_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_int, c_int,
                                               POINTER(Segments), c_void_p, c_void_p, c_size_t, c_void_p,
                                               c_void_p]),
    "leankv_sparse_swiglu_rmsnorm_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_void_p,
                                                 c_int, c_int, c_float, c_float, c_void_p, c_size_t,
                                                 c_void_p, c_void_p]),
    "leankv_sparse_gemv_f16_static": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p]),
    "leankv_sparse_swiglu_workspace_bytes": (c_size_t, [c_int, c_int]),
    "leankv_sparse_swiglu_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                         c_float, c_float, c_void_p, c_size_t, c_void_p, c_void_p]),
    "leankv_tq_packed_len": (c_int, [c_int, c_int]),
    "leankv_tq_quantize": (c_int, [c_void_p, c_int, c_longlong, c_int, c_int, c_void_p, c_void_p,
                                   c_void_p, c_void_p, c_void_p]),
    "leankv_tq_dequantize": (c_int, [c_void_p, c_void_p, c_longlong, c_int, c_int, c_void_p,
                                     c_void_p, c_void_p, c_int, c_void_p]),
    "leankv_tq_pool_bytes": (c_size_t, [c_int, c_int]),
    "leankv_tq_pool_append": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p,
                                      c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
                                      c_void_p]),
    "leankv_tq_band_stats": (c_int, [POINTER(c_ulonglong), c_int]),
    "leankv_tq_pool_unpack": (c_int, [c_void_p, c_int, c_int, c_void_p, c_int, c_int, c_void_p,
                                      c_void_p, c_void_p]),
    "leankv_tq_decode_attn_workspace_bytes": (c_size_t, [c_int, c_int, c_int, c_int]),
    "leankv_tq_decode_attn": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_int,
                                      c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                      c_void_p, c_float, c_void_p, c_size_t, c_void_p]),
    "leankv_tq_decode_attn_rotated": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_int,
                                              c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                              c_float, c_void_p, c_size_t, c_int, c_void_p]),
    "leankv_decode_qkv_post": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                       c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "leankv_tq_decode_attn_status": (c_int, [c_void_p, POINTER(c_int)]),
    "leankv_tq_prefill_attn_workspace_bytes": (c_size_t, [c_int, c_int, c_int, c_int]),
    "leankv_tq_prefill_attn": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_int,
                                       c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_size_t,
                                       c_void_p]),
    "leankv_rmsnorm_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_float, c_void_p]),
    "leankv_decode_begin": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "leankv_rope_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                                c_void_p]),
    "leankv_decode_end": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p]),
    "leankv_decode_end_sharded": (c_int, [c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                          c_int, c_void_p]),
    "leankv_tq_append_status": (c_int, [POINTER(c_int)]),
    "leankv_xchg_recv_bytes": (c_size_t, [c_int, c_int, c_int]),
    "leankv_xchg_advance": (c_int, [c_void_p, c_void_p]),
    "leankv_sparse_gemv_allreduce_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p,
                                                 c_void_p, c_size_t, c_void_p, c_void_p, c_int, c_void_p]),
    "leankv_ipc_alloc": (c_int, [c_size_t, POINTER(c_void_p), c_char_p]),
    "leankv_ipc_open": (c_int, [c_char_p, POINTER(c_void_p)]),
    "leankv_ipc_close": (c_int, [c_void_p]),
    "leankv_ipc_free": (c_int, [c_void_p]),
    "leankv_rmsnorm_rows_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p]),
    "leankv_batch_decode_begin": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p,
                                          c_int, c_void_p, c_void_p, c_void_p, c_void_p]),
    "leankv_batch_qkv_post": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                      c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "leankv_paged_table_step": (c_int, [c_int, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
                                        c_void_p, c_void_p, c_void_p, c_void_p, c_void_p]),
    "leankv_silu_mul_f16": (c_int, [c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "leankv_batch_decode_end": (c_int, [c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                        c_void_p]),
}


# ── libleankv_mixers.so ──────────────────────────────────────────────────────────────────────

DT_BF16, DT_F32 = 1, 2
MAX_MIX = 8
STATE_PARITY = 6         # state word that selects the half of a double-buffered previous-token vector


class DenseGemv(Structure):
    """Mirror of ``leankv_dense_gemv_t``."""

    _fields_ = [("w", c_void_p), ("x", c_void_p), ("y", c_void_p),
                ("dtype", c_int), ("rows", c_int), ("cols", c_int), ("gated", c_int),
                ("gain", c_void_p), ("eps", c_float),
                ("n_mix", c_int), ("mix_end", c_int * MAX_MIX), ("mu", c_void_p * MAX_MIX),
                ("prev", c_void_p), ("state", c_void_p),
                ("bias", c_void_p), ("bias_rows", c_int),
                ("scale", c_void_p), ("residual", c_void_p),
                ("gain_per_col", c_int), ("delta", c_void_p), ("post_gain", c_void_p), ("post_mult", c_float),
                ("x_out", c_void_p), ("group_rows", c_int), ("group_stride", c_int), ("softcap", c_float)]


class StreamNorm(Structure):
    """Mirror of ``leankv_stream_norm_t``."""

    _fields_ = [("x_in", c_void_p), ("x_out", c_void_p), ("delta", c_void_p), ("scale", c_void_p),
                ("gain", c_void_p), ("h", c_void_p), ("mixed", c_void_p), ("mu", c_void_p * MAX_MIX),
                ("prev_in", c_void_p), ("prev_out", c_void_p),
                ("dtype", c_int), ("delta_dtype", c_int), ("rows", c_int), ("width", c_int), ("n_mix", c_int),
                ("eps", c_float), ("gain_per_col", c_int), ("post_gain", c_void_p), ("post_mult", c_float)]


class WindowPool(Structure):
    """Mirror of ``leankv_window_pool_t``."""

    _fields_ = [("dtype", c_int), ("heads", c_int), ("kv_heads", c_int), ("dim", c_int), ("vdim", c_int),
                ("dim_pad", c_int), ("vdim_pad", c_int),
                ("size", c_int), ("pool", c_int), ("ring", c_int), ("max_blocks", c_int),
                ("scale", c_float),
                ("k_ring", c_void_p), ("v_ring", c_void_p), ("k_pool", c_void_p), ("v_pool", c_void_p),
                ("q_norm", c_void_p), ("k_norm", c_void_p), ("eps", c_float), ("talk", c_void_p)]


class TimeMix(Structure):
    """Mirror of ``leankv_time_mix_t``."""

    _fields_ = [("dtype", c_int), ("heads", c_int), ("dim", c_int),
                ("S", c_void_p), ("u", c_void_p), ("w0", c_void_p), ("norm", c_void_p), ("eps", c_float)]


class MixerStep(Structure):
    """Mirror of ``leankv_mixer_step_t``."""

    _fields_ = [("y", c_void_p), ("qkv_off", c_int), ("rkvg_off", c_int), ("w1_off", c_int), ("rank", c_int),
                ("w2", c_void_p), ("out", c_void_p), ("right_off", c_int),
                ("left_scale", c_float), ("right_scale", c_float), ("state", c_void_p), ("max_pos", c_int),
                ("ws", c_void_p), ("ws_bytes", c_size_t)]


class CausalAttn(Structure):
    """Mirror of ``leankv_causal_attn_t``."""

    _fields_ = [("dtype", c_int), ("heads", c_int), ("kv_heads", c_int),
                ("dim", c_int), ("shared_dim", c_int), ("vdim", c_int),
                ("dim_pad", c_int), ("shared_pad", c_int), ("vdim_pad", c_int),
                ("size", c_int), ("scale", c_float),
                ("k", c_void_p), ("v", c_void_p), ("k_base", c_int), ("k_ring", c_int), ("k_rows", c_int),
                ("shared", c_void_p), ("s_ring", c_int)]


class RowSegment(Structure):
    """Mirror of ``leankv_row_segment_t``."""

    _fields_ = [("src", c_void_p), ("ld", c_int), ("heads", c_int), ("head_stride", c_int), ("n", c_int),
                ("dst", c_void_p), ("dst_ld", c_int), ("dst_head_stride", c_int), ("n_pad", c_int), ("ring", c_int),
                ("gain", c_void_p), ("rot", c_int)]


MAX_ROW_SEGMENTS = 4


class PlaceRows(Structure):
    """Mirror of ``leankv_place_rows_t``."""

    _fields_ = [("dtype", c_int), ("rows", c_int), ("start", c_int), ("n_seg", c_int),
                ("seg", RowSegment * MAX_ROW_SEGMENTS), ("rate", c_void_p), ("eps", c_float)]


class CausalStep(Structure):
    """Mirror of ``leankv_causal_step_t``."""

    _fields_ = [("q", c_void_p), ("q_shared", c_void_p), ("k_new", c_void_p), ("shared_new", c_void_p),
                ("v_new", c_void_p), ("q_stride", c_int), ("qs_stride", c_int),
                ("k_gain", c_void_p), ("eps", c_float), ("rate", c_void_p), ("rot_own", c_int), ("rot_shared", c_int),
                ("gate", c_void_p), ("out", c_void_p), ("state", c_void_p), ("max_pos", c_int),
                ("ws", c_void_p), ("ws_bytes", c_size_t)]


MIXER_SIGNATURES = {
    "leankv_dense_gemv": (c_int, [POINTER(DenseGemv), c_void_p]),
    "leankv_embed_begin": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "leankv_greedy_end": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p]),
    "leankv_stream_norm": (c_int, [POINTER(StreamNorm), c_void_p]),
    "leankv_silu_mul": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "leankv_softcap": (c_int, [c_void_p, c_longlong, c_float, c_void_p]),
    "leankv_tanh_split": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "leankv_window_pool_append": (c_int, [POINTER(WindowPool), c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
                                          c_void_p]),
    "leankv_window_pool_workspace_bytes": (c_size_t, [POINTER(WindowPool), c_int, c_int]),
    "leankv_window_pool_attend": (c_int, [POINTER(WindowPool), c_void_p, c_void_p, c_int, c_float, c_int, c_int,
                                          c_void_p, c_size_t, c_void_p]),
    "leankv_time_mix_workspace_bytes": (c_size_t, [POINTER(TimeMix), c_int]),
    "leankv_time_mix_rows": (c_int, [POINTER(TimeMix), c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                     c_int, c_float, c_int, c_void_p, c_size_t, c_void_p]),
    "leankv_mixer_step_workspace_bytes": (c_size_t, [POINTER(WindowPool), c_int]),
    "leankv_mixer_step": (c_int, [POINTER(WindowPool), POINTER(TimeMix), POINTER(MixerStep), c_void_p]),
    "leankv_place_rows": (c_int, [POINTER(PlaceRows), c_void_p]),
    "leankv_causal_attend": (c_int, [POINTER(CausalAttn), c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int,
                                     c_void_p, c_void_p]),
    "leankv_causal_step_workspace_bytes": (c_size_t, [POINTER(CausalAttn), c_int]),
    "leankv_causal_step": (c_int, [POINTER(CausalAttn), POINTER(CausalStep), c_void_p]),
}
_COMMON = ("leankv_strerror", "leankv_last_cuda_error", "leankv_abi_version")     # capi.cu, in both libraries

_lib = None
_mixers = None


def _load(path: str, signatures: dict) -> ctypes.CDLL:
    if not os.path.exists(path):
        raise RuntimeError(
            f"{path} is missing: build it with `python -m leankv_b200.build` "
            "(leankv_b200 has no CPU or PyTorch fallback)")
    handle = ctypes.CDLL(path)
    for name, (restype, argtypes) in signatures.items():
        fn = getattr(handle, name)   # AttributeError if the build is stale
        fn.restype = restype
        fn.argtypes = argtypes
    return handle


def lib() -> ctypes.CDLL:
    """Load the shared library once; raise if it has not been built."""
    global _lib
    if _lib is None:
        _lib = _load(LIB_PATH, SIGNATURES)
    return _lib


def mixers() -> ctypes.CDLL:
    """The token-mixer library, loaded once."""
    global _mixers
    if _mixers is None:
        _mixers = _load(MIXERS_PATH, {**MIXER_SIGNATURES, **{n: SIGNATURES[n] for n in _COMMON}})
    return _mixers


def check(code: int, what: str, handle=None) -> None:
    """Raise ``RuntimeError`` for a negative status code (``handle``: the library that returned it)."""
    if code == 0:
        return
    handle = handle or lib()
    msg = handle.leankv_strerror(code).decode()
    if code == -4:
        msg += ": " + handle.leankv_last_cuda_error().decode()
    raise RuntimeError(f"{what} failed: {msg} (code {code})")


def ptr(t) -> int | None:
    """Device address of a torch tensor (None passes NULL)."""
    return None if t is None else t.data_ptr()


def current_stream() -> int:
    import torch

    return torch.cuda.current_stream().cuda_stream


def require_cuda(t, name: str) -> None:
    if not t.is_cuda:
        raise RuntimeError(
            f"{name} must be a CUDA tensor: leankv_b200 runs only on the GPU (no CPU fallback)")
