"""ctypes view of the C ABI declared in ``include/twm_dense.h``."""
from __future__ import annotations

import ctypes as C

from .build import build_library
from ._lib import TWM_FLAG_PDL, TWM_OK  # noqa: F401

TWM_DENSE_F32, TWM_DENSE_BF16 = 0, 2
MIX_SIGMOID, MIX_LATENT, MIX_GLA = 0, 1, 2
EPI_STORE, EPI_STORE_F32, EPI_GELU_GLU, EPI_RELU2 = 0, 1, 2, 3


class Layer(C.Structure):
    """``twm_dense_layer``."""
    _fields_ = [("mixer", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("dim_pad", C.c_int),
                ("vdim_pad", C.c_int), ("window", C.c_int), ("keep_first", C.c_int), ("ff_pad", C.c_int), ("scale", C.c_float),
                ("w_in", C.c_void_p), ("w_out", C.c_void_p), ("w_gate_up", C.c_void_p), ("w_down", C.c_void_p),
                ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("bias_table", C.c_void_p), ("shift", C.c_void_p),
                ("norm1", C.c_void_p), ("norm2", C.c_void_p), ("pre1", C.c_void_p), ("pre2", C.c_void_p), ("step", C.c_void_p),
                ("rank", C.c_int), ("rank_pad", C.c_int), ("rot_pad", C.c_int), ("w_expand", C.c_void_p), ("latent_norm", C.c_void_p),
                ("rot_table", C.c_void_p), ("latent_cache", C.c_void_p), ("inv_tau", C.c_float), ("w_decay", C.c_void_p),
                ("decay_bias", C.c_void_p), ("head_norm", C.c_void_p), ("gla_state", C.c_void_p),
                ("experts", C.c_int), ("top", C.c_int), ("groups", C.c_int), ("keep", C.c_int), ("w_router", C.c_void_p),
                ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("shift_state", C.c_void_p)]


class Model(C.Structure):
    """``twm_dense_model``."""
    _fields_ = [("dtype", C.c_int), ("width", C.c_int), ("width_pad", C.c_int), ("vocab", C.c_int), ("n_layers", C.c_int),
                ("bias_len", C.c_int), ("capacity", C.c_int), ("slots", C.c_int), ("eps", C.c_float), ("embed_scale", C.c_float),
                ("embed", C.c_void_p), ("pos_embed", C.c_void_p),
                ("head", C.c_void_p), ("final_norm", C.c_void_p), ("layers", C.POINTER(Layer))]


class Buffers(C.Structure):
    """``twm_dense_buffers``."""
    _fields_ = [("max_rows", C.c_int), ("max_want", C.c_int), ("meta", C.c_void_p), ("tokens", C.c_void_p), ("want", C.c_void_p),
                ("x0", C.c_void_p), ("x1", C.c_void_p), ("y", C.c_void_p), ("a", C.c_void_p), ("proj", C.c_void_p),
                ("att", C.c_void_p), ("act", C.c_void_p), ("vec", C.c_void_p), ("logits", C.c_void_p),
                ("max_keys", C.c_int), ("lat", C.c_void_p), ("kv", C.c_void_p), ("decay", C.c_void_p), ("chunk_state", C.c_void_p),
                ("mix", C.c_void_p), ("router_logits", C.c_void_p), ("route", C.c_void_p), ("route_weight", C.c_void_p),
                ("grouped", C.c_void_p), ("expert_out", C.c_void_p), ("max_slots", C.c_int)]


_P = C.c_void_p
_M, _B = C.POINTER(Model), C.POINTER(Buffers)
SIGNATURES = {
    "twm_dense_prefill": (C.c_int, [_M, _B, C.c_int, C.c_int, C.c_int, _P, C.c_int, _P]),
    "twm_dense_decode": (C.c_int, [_M, _B, C.c_int, C.c_int, _P]),
    "twm_dense_launches": (C.c_int, []),
    "twm_dense_set_step": (C.c_int, [_B, C.c_int, C.c_int, C.c_int, _P]),
    "twm_dense_argmax_scratch_bytes": (C.c_size_t, []),
    "twm_dense_argmax_advance": (C.c_int, [_B, C.c_int, C.c_int, _P, C.c_int, _P, C.c_size_t, C.c_int, _P]),
    "twm_dense_gemm": (C.c_int, [C.c_int, _P, C.c_int, _P, C.c_int, _P, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int,
                                 C.c_int, _P]),
    "twm_dense_route": (C.c_int, [_P, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, _P, _P, C.c_int, _P]),
    "twm_dense_grouped_gemm": (C.c_int, [C.c_int, _P, C.c_int, _P, C.c_int, _P, C.c_int, _P, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int,
                                         C.c_int, C.c_int, _P]),
    "twm_dense_gla": (C.c_int, [_M, C.c_int, _B, C.c_int, C.c_int, C.c_int, _P]),
    "twm_dense_attention": (C.c_int, [_M, C.c_int, _B, C.c_int, C.c_int, C.c_int, C.c_int, _P]),
    "twm_dense_device_error": (C.c_int, [_P, C.POINTER(C.c_uint)]),
    "twm_dense_status_string": (C.c_char_p, [C.c_int]),
    "twm_dense_last_error": (C.c_char_p, []),
}

_lib = None


def lib() -> C.CDLL:
    """Load ``libtwmdense.so``, compiling it first if it is missing or out of date."""
    global _lib
    if _lib is None:
        handle = C.CDLL(build_library("dense"))
        for name, (res, args) in SIGNATURES.items():
            fn = getattr(handle, name)
            fn.restype, fn.argtypes = res, args
        _lib = handle
    return _lib


class DenseError(RuntimeError):
    """A non-zero status of a ``twm_dense_*`` call."""

    def __init__(self, status: int, where: str):
        self.status = status
        super().__init__(f"{where}: {lib().twm_dense_status_string(status).decode()} [{lib().twm_dense_last_error().decode()}]")


def check(status: int, where: str) -> None:
    if status != TWM_OK:
        raise DenseError(status, where)


def device_error(stream: int = 0) -> int:
    """The sticky device error word (0 = none); reading clears it."""
    word = C.c_uint(0)
    lib().twm_dense_device_error(stream, C.byref(word))
    return int(word.value)
