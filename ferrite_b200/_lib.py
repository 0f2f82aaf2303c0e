"""ctypes binding of include/ferrite_b200.h.

The shared library is the product's only compute path: if it is missing this module raises (there is
no CPU or PyTorch fallback).  Build it with `python -m ferrite_b200.build` (needs nvcc).
"""
import ctypes
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "lib", "libferrite_b200.so")

BF16, FP32, INT32, BFP8, BFP4 = 0, 1, 2, 3, 4
DTYPES = {"bf16": BF16, "fp32": FP32, "int32": INT32, "bfp8": BFP8, "bfp4": BFP4}
EPI_NONE, EPI_SWIGLU, EPI_RESIDUAL = 0, 1, 2
LINEAR_AUTO, LINEAR_TCGEN05, LINEAR_GEMV, LINEAR_MMA, LINEAR_PERSISTENT, LINEAR_GEMV_STREAM = 0, 1, 2, 3, 4, 5  # fb_linear_prefer

_p, _i, _i64, _f, _sz = ctypes.c_void_p, ctypes.c_int, ctypes.c_int64, ctypes.c_float, ctypes.c_size_t

DENSE_NONE, DENSE_SILU, DENSE_GLU, DENSE_GATE, DENSE_DYT_ADD, DENSE_SWIGLU, DENSE_GEGLU, DENSE_RELU2 = 0, 1, 2, 3, 4, 5, 6, 7  # fb_dense_epilogue_kind


class DenseEpilogue(ctypes.Structure):
    """fb_dense_epilogue of include/ferrite_b200.h, field by field."""
    _fields_ = [("kind", _i), ("act_cols", _i64), ("limit", _f), ("slope", _f), ("gate", _p), ("ld_gate", _i64), ("residual", _p), ("ld_residual", _i64),
                ("alpha", _p), ("w", _p), ("b", _p), ("h_out", _p), ("ld_h", _i64), ("alpha2", _p), ("w2", _p), ("b2", _p), ("gate_bias", _p), ("up_bias", _p), ("row_scale", _p)]


class Heads(ctypes.Structure):
    """fb_heads, likewise."""
    _fields_ = [("heads", _i), ("kv_heads", _i), ("dim", _i), ("vdim", _i), ("bias", _p), ("q_norm", _p), ("k_norm", _p), ("eps", _f), ("first", _p), ("ld_first", _i64),
                ("first_bias", _p), ("share", _p), ("norm_all", _i), ("keys_are_values", _i), ("turned", _i), ("freq", _p), ("mag", _f), ("places", _p), ("taps", _i), ("conv", _p),
                ("state", _p), ("state_stride", _i64), ("sequences", _i), ("dead", _i), ("temp_coef", _f), ("temp_every", _f)]


class Router(ctypes.Structure):
    """fb_router, likewise."""
    _fields_ = [("n", _i), ("k", _i), ("identity", _i), ("bias", _p), ("scored", _i), ("scale", _f), ("as_scored", _i)]


class Branches(ctypes.Structure):
    """fb_branches, likewise."""
    _fields_ = [("x", _p), ("ld_x", _i64), ("mixer", _p), ("ld_mixer", _i64), ("mixer_scale", _p), ("other", _p), ("ld_other", _i64), ("other_scale", _p), ("chosen", _p),
                ("ld_chosen", _i64), ("slots", _p), ("weights", _p), ("k", _i), ("x_out", _p), ("ld_x_out", _i64), ("w", _p), ("plus", _f), ("eps", _f), ("h", _p), ("ld_h", _i64),
                ("mixer_bias", _p), ("own", _p), ("ld_own", _i64), ("gate", _p), ("ld_gate", _i64), ("gate_bias", _p), ("post", _p)]


class Conv(ctypes.Structure):
    """fb_conv, likewise."""
    _fields_ = [("cols", _i64), ("taps", _i), ("w", _p), ("bias", _p), ("in_bias", _p), ("silu", _i), ("places", _p), ("dead", _i), ("sequences", _i64), ("tokens", _i64), ("state", _p),
                ("state_stride", _i64)]


class Lru(ctypes.Structure):
    """fb_lru, likewise."""
    _fields_ = [("width", _i64), ("blocks", _i), ("lam", _p), ("rate", _f), ("gate_bias", _p), ("y_bias", _p), ("scale", _f), ("places", _p), ("dead", _i), ("sequences", _i64), ("tokens", _i64),
                ("state", _p), ("state_stride", _i64)]


# name -> (restype, argtypes); one entry per declaration in include/ferrite_b200.h
SIGNATURES = {
    "fb_version": (_i, []),
    "fb_last_error": (ctypes.c_char_p, []),
    "fb_status_word": (_i, []),
    "fb_packed_bytes": (_sz, [_i, _i64, _i64]),
    "fb_quantize": (_i, [_i, _p, _i64, _i64, _i64, _p, _p]),
    "fb_dequantize": (_i, [_i, _p, _i64, _i64, _i64, _p, _p]),
    "fb_unpack_fields": (_i, [_i, _p, _i64, _i64, _i64, _p, _p, _p, _p]),
    "fb_linear_workspace_bytes": (_sz, [_i64, _i64, _i64]),
    "fb_linear_prefer": (_i, [_i]),
    "fb_linear": (_i, [_i, _p, _i64, _i64, _i64, _p, _i64, _p, _i, _i64, _p, _f, _i, _p, _i64, _p, _sz, _p]),
    "fb_linear_chain_parts": (_i, [_i, _i64, _i64, _i64, _i]),
    "fb_linear_chained": (_i, [_i, _p, _i64, _i64, _i64, _p, _i64, _p, _i, _i64, _f, _i, _p, _i64, _p, _i, _p, _p, _i64, _p, _p, _sz, _p]),
    "fb_linear_indexed": (_i, [_i, _p, _i64, _i64, _i64, _i64, _p, _i64, _i, _p, _i, _i, _p, _i, _i64, _i64, _p, _f, _i, _p, _i64, _p, _p, _sz, _p]),
    "fb_gather_rows": (_i, [_p, _i64, _i64, _p, _i64, _p, _p]),
    "fb_put_rows": (_i, [_p, _i64, _i64, _i64, _p, _i64, _i64, _i64, _p, _i64, _i64, _i64, _i64, _i, _p]),
    "fb_rope_kv_write": (_i, [_p, _i64, _i64, _i, _i, _i, _p, _p, _i64, _i64, _p, _p, _p, _f, _p, _i64, _p, _i64, _i64, _p]),
    "fb_decode_attention_workspace_bytes": (_sz, [_i64, _i, _i, _i, _i64]),
    "fb_decode_attention": (_i, [_p, _i64, _i64, _i, _i, _i, _p, _i64, _i64, _p, _p, _i64, _i, _p, _i64, _p, _sz, _p]),
    "fb_decode_attention_static_max_bytes": (_sz, []),
    "fb_decode_attention_static": (_i, [_p, _i64, _i64, _i, _i, _i, _p, _i64, _i64, _p, _p, _i64, _i, _p, _i64, _p]),
    "fb_prefill_attention_workspace_bytes": (_sz, [_i64, _i, _i, _i64]),
    "fb_prefill_attention": (_i, [_i, _p, _i64, _i64, _i, _i, _i, _p, _i64, _i64, _i64, _p, _i64, _i, _p, _i64, _p, _sz, _p]),
    "fb_attend_workspace_bytes": (_sz, [_i64, _i64, _i, _i64]),
    "fb_attend": (_i, [_p, _i64, _i64, _i, _i64, _i64, _p, _p, _i64, _i64, _i64, _p, _i64, _i64, _i, _f, _p, _p, _sz, _p]),
    "fb_topk": (_i, [_i, _p, _i64, _i64, _i64, _i, _p, _p, _p, _p, _i64, _p]),
    "fb_touched": (_i, [_p, _p, _i64, _i, _i, _i, _p, _p, _p]),
    "fb_group": (_i, [_p, _i64, _i, _i, _p, _p, _p, _p]),
    "fb_elementwise": (_i, [_i, _p, _p, _i, _p, _p, _p, _p, _p, _i, _i64, _i64, _i64, _p]),
    "fb_reduce": (_i, [_i, _p, _p, _i, _i64, _i64, _i64, _i, _p, _p, _i, _p]),
    "fb_matmul": (_i, [_p, _p, _i, _p, _p, _i, _p, _p, _i, _i64, _i64, _i64, _i64, _p]),
    "fb_rmsnorm": (_i, [_p, _i64, _i64, _i64, _p, _f, _p, _i64, _p]),
    "fb_argmax": (_i, [_p, _i64, _i64, _i64, _p, _p, _p]),
    "fb_rope_kv_write_packed": (_i, [_i, _p, _i64, _i64, _i, _i, _i, _p, _p, _i64, _i64, _p, _p, _p, _f, _p, _i64, _p, _i64, _p]),
    "fb_decode_attention_packed": (_i, [_i, _p, _i64, _i64, _i, _i, _i, _p, _i64, _p, _p, _i64, _i, _p, _i64, _p, _sz, _p]),
    "fb_dense_supports": (_i, [_p, _i64, _i64, _p, _i64, _i64, _i64, _i64, _i]),
    "fb_dense": (_i, [_p, _i64, _i64, _i64, _i64, _p, _i64, _i64, _i64, _i64, _p, _i, _i64, _i64, _p, _i, _p]),
    "fb_latent_put": (_i, [_i, _p, _i64, _i64, _i, _i, _i, _i, _p, _p, _f, _p, _f, _p, _p, _i, _p, _i64, _i, _i, _p, _i64, _i64, _p, _i64, _p]),
    "fb_rotate_pairs": (_i, [_i, _p, _i64, _i, _i64, _i64, _i, _i, _p, _f, _p, _p, _i64, _i64, _p]),
    "fb_latent_attention_workspace_bytes": (_sz, [_i, _i64, _i, _i, _i, _i64, _i, _i]),
    "fb_latent_attention": (_i, [_i, _p, _i64, _i64, _i, _i, _i, _p, _i64, _p, _i64, _p, _i64, _i, _i, _f, _p, _p, _i64, _p, _sz, _p]),
    "fb_decay_scan": (_i, [_i, _p, _i64, _i, _i, _i, _p, _p, _i, _i64, _i64, _p, _i64, _p, _i64, _p]),
    "fb_selective_scan": (_i, [_i, _p, _i64, _i, _i, _i, _i, _p, _i64, _p, _p, _p, _p, _i, _i64, _i64, _p, _i64, _p, _i64, _p]),
    "fb_gated_rmsnorm": (_i, [_p, _i64, _i64, _i64, _i, _p, _i64, _i, _p, _f, _i, _i, _p, _i64, _p]),
    "fb_short_conv": (_i, [_p, _i, _p, _i64, _i, _p, _i64, _p]),
    "fb_lru_scan": (_i, [_p, _i, _p, _i64, _p, _i64, _i, _p, _i64, _p, _i64, _p]),
    "fb_dense_grouped": (_i, [_p, _i64, _i64, _i64, _i, _p, _i64, _i64, _i64, _i, _p, _p, _i64, _i, _p, _i, _i64, _p, _p]),
    "fb_route_tiles": (_i64, [_i64, _i, _i, _i, _i]),
    "fb_route": (_i, [_p, _p, _i64, _i64, _i, _i, _p, _p, _p, _p, _p, _p, _p]),
    "fb_spread_rows": (_i, [_p, _i64, _i64, _i64, _p, _i, _p, _i64, _p]),
    "fb_grouped_matmul": (_i, [_i, _p, _i64, _i64, _i, _i, _p, _p, _i, _i64, _i64, _p, _p, _i64, _i, _p, _i, _p, _i64, _p]),
    "fb_embed": (_i, [_i, _p, _i64, _i64, _p, _p, _i64, _p, _i64, _f, _p, _p]),
    "fb_heads_put": (_i, [_p, _i, _p, _i64, _i64, _p, _i, _p, _i64, _p, _i64, _i64, _p]),
    "fb_heads_attention": (_i, [_i, _p, _i64, _i64, _i, _i, _i, _i, _p, _i64, _i64, _p, _i64, _p, _i64, _i, _i, _i, _f, _f, _p, _p, _f, _i, _p, _i64, _p, _i64, _p]),
    "fb_add_norm": (_i, [_p, _i64, _i64, _i, _i, _p]),
    "fb_peer_reduce_add": (_i, [_p, _p, _i, _i, _p, _i64, _p, _p, _p]),
}


class FerriteError(RuntimeError):
    pass


_lib = None


def _left_out(name):
    def call(*_):
        raise ImportError(f"{LIB_PATH} was built without {name}: run `python -m ferrite_b200.build`")
    return call


def lib():
    """The loaded library (loads it on first use)."""
    global _lib
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise ImportError(f"{LIB_PATH} is not built: run `python -m ferrite_b200.build` (the CUDA library is the only compute path)")
        _lib = ctypes.CDLL(LIB_PATH)
        for name, (res, args) in SIGNATURES.items():
            fn = getattr(_lib, name, None)
            if fn is None:  # a library that was built for one model family: what it leaves out says so when it is called
                setattr(_lib, name, _left_out(name))
                continue
            fn.restype, fn.argtypes = res, args
    return _lib


_RAISES = {-1: AssertionError, -2: FerriteError, -3: TimeoutError, -4: MemoryError}


def check(status):
    """0 passes; a negative fb_status raises what ferrite raises for the same misuse: AssertionError for a
    bad shape or dtype, MemoryError, TimeoutError (ferrite/tensor.py asserts; ferrite/runtime.py:445,476)."""
    if status != 0:
        raise _RAISES.get(status, FerriteError)(lib().fb_last_error().decode())
