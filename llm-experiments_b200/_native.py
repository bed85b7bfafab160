"""ctypes binding of ``libb2kv.so``, the C-ABI CUDA library (declared in include/b2kv.h).

The library is the only compute path of this package.  If it is missing the import of
this module fails with instructions to build it: there is no CPU or PyTorch fallback.
"""
from __future__ import annotations

import ctypes
import pathlib

_PKG = pathlib.Path(__file__).resolve().parent
LIB_PATH = _PKG / "libb2kv.so"
SERVE_LIB_PATH = _PKG / "libb2kv_serve.so"  # the part models are served with (build.py --serve), where that is all there is

DTYPE_F32 = 0
DTYPE_BF16 = 1

ERR_BAD_ARG = -1
ERR_ALIGN = -2
ERR_UNSUPPORTED = -3
ERR_WORKSPACE = -4
ERR_CUDA = -5
ERR_STATIC_LIMIT = -6
STATIC_SCRATCH_BYTES = 32 << 20

DEV_STATUS_TEXT = {
    1: "a block-table entry points outside the pool",
    2: "an append position lies outside the cache",
    3: "a bounded wait on a barrier ran out",
    4: "a token id lies outside the embedding table",
}

_vp = ctypes.c_void_p
_i = ctypes.c_int
_i64 = ctypes.c_int64
_sz = ctypes.c_size_t

_f = ctypes.c_float

SEG_STORE, SEG_F32, SEG_GLU_SILU, SEG_GLU_CLAMP, SEG_RELU2, SEG_SOFTCAP, SEG_DECAY = 0, 1, 2, 3, 4, 5, 6
MAX_SEGMENTS = 3


class Segment(ctypes.Structure):
    """``b2kv_segment``: where a range of output columns of a linear layer goes."""

    _fields_ = [("out", _vp), ("ld", _i64), ("group", _i64), ("end", ctypes.c_int32), ("kind", ctypes.c_int32)]


class LinearArgs(ctypes.Structure):
    """``b2kv_linear_args``."""

    _fields_ = [("x", _vp), ("w", _vp), ("residual", _vp), ("bias", _vp), ("group_rows", _vp), ("ld_x", _i64), ("group_x", _i64),
                ("ld_w", _i64), ("group_w", _i64), ("ld_residual", _i64), ("seg", Segment * MAX_SEGMENTS),
                ("rows", ctypes.c_int32), ("K", ctypes.c_int32), ("N", ctypes.c_int32), ("groups", ctypes.c_int32),
                ("max_group_rows", ctypes.c_int32), ("n_seg", ctypes.c_int32), ("dtype", ctypes.c_int32),
                ("path", ctypes.c_int32), ("limit", _f)]


class GlaArgs(ctypes.Structure):
    """``b2kv_gla_args``."""

    _fields_ = [("y", _vp), ("alpha", _vp), ("norm", _vp), ("state", _vp), ("out", _vp), ("segments", _vp), ("row_pos", _vp), ("workspace", _vp),
                ("workspace_bytes", _sz),
                ("ld_y", _i64), ("ld_alpha", _i64), ("ld_out", _i64), ("q_col", ctypes.c_int32), ("k_col", ctypes.c_int32),
                ("v_col", ctypes.c_int32), ("g_col", ctypes.c_int32), ("H", ctypes.c_int32), ("dim", ctypes.c_int32),
                ("vdim", ctypes.c_int32), ("n_segments", ctypes.c_int32), ("max_n", ctypes.c_int32), ("rows", ctypes.c_int32),
                ("n_slots", ctypes.c_int32), ("dtype", ctypes.c_int32), ("path", ctypes.c_int32), ("q_scale", _f),
                ("eps", _f)]


# name -> (restype, argtypes); kept in the order of include/b2kv.h
SIGNATURES = {
    "b2kv_strerror": (ctypes.c_char_p, [_i]),
    "b2kv_last_cuda_error": (ctypes.c_char_p, []),
    "b2kv_version": (_i, []),
    "b2kv_append": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _vp]),
    "b2kv_append_paged": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i,
                               _vp, _vp]),
    "b2kv_append_rows_paged": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _vp]),
    "b2kv_advance_lengths": (_i, [_vp, _i, _i, _vp]),
    "b2kv_gather": (_i, [_vp, _vp, _vp, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp]),
    "b2kv_gather_paged": (_i, [_vp, _vp, _vp, _i, _vp, _i, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _vp]),
    "b2kv_decode_workspace_bytes": (_sz, [_i, _i, _i, _i, _i]),
    "b2kv_decode": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _sz, _vp, _vp]),
    "b2kv_decode_paged": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64,
                               _i, _vp, _sz, _vp, _vp]),
    "b2kv_decode_allgather": (_i, [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _sz, _vp, _vp,
                                   _vp, _vp, ctypes.c_uint32, _i, _i, _i, ctypes.c_uint32, _vp, _vp]),
    "b2kv_decode_partial": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _sz, _vp,
                                 _vp]),
    "b2kv_merge_partials": (_i, [_vp, _i, _i, _i, _i, _vp, _i, _vp]),
    "b2kv_decode_static": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _vp]),
    "b2kv_prefill": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i64, _i64, _i, _i, _i, _i, _i, _i, _vp, _vp]),
    "b2kv_prefill_workspace_bytes": (_sz, [_i, _i, _i, _i, _i]),
    "b2kv_prefill_ws": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i64, _i64, _i, _i, _i, _i, _i, _i, _vp, _sz,
                             _vp, _vp]),
    "b2kv_prefill_paged": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i64, _i64, _i, _i, _i, _i, _i,
                                _vp, _vp]),
    "b2kv_layernorm": (_i, [_vp, _vp, _vp, _vp, _i64, _i, ctypes.c_float, _vp]),
    "b2kv_layernorm_bf16": (_i, [_vp, _vp, _vp, _vp, _i64, _i, ctypes.c_float, _vp]),
    "b2kv_extract_last_tokens": (_i, [_vp, _vp, _i, _i, _i, _vp]),
    "b2kv_softmax": (_i, [_vp, _vp, _i64, _i, _vp]),
    "b2kv_argmax": (_i, [_vp, _vp, _i, _i, _vp]),
    "b2kv_extract_last_tokens_bf16": (_i, [_vp, _vp, _i, _i, _i, _vp]),
    "b2kv_argmax_bf16": (_i, [_vp, _vp, _i, _i, _vp]),
    "b2kv_embedding": (_i, [_vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _i, _i, _i, _vp, _vp]),
    "b2kv_qkv_append": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i, _vp, _vp]),
    "b2kv_matmul_rows": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp]),
    "b2kv_matmul": (_i, [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp, _vp]),
    "b2kv_embed_rows": (_i, [_vp, _vp, _vp, _vp, _f, _i, _i, _i, _i, _vp, _vp]),
    "b2kv_layernorm_rows": (_i, [_vp, _i64, _vp, _vp, _vp, _vp, _i64, _vp, _i64, _i, _i, _f, _i, _vp]),
    "b2kv_rmsnorm": (_i, [_vp, _i64, _vp, _vp, _f, _vp, _i64, _i, _i, _f, _i, _vp]),
    "b2kv_linear": (_i, [ctypes.POINTER(LinearArgs), _vp, _vp]),
    "b2kv_latent_append": (_i, [_vp, _i64, _i, _i, _i, _i, _vp, _i, _i, _vp, _f, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _vp, _vp]),
    "b2kv_latent_decode_workspace_bytes": (_sz, [_i, _i, _i, _i, _i]),
    "b2kv_latent_decode": (_i, [_vp, _vp, _i64, _i, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _f, _i, _i, _vp,
                                _sz, _vp, _vp]),
    "b2kv_latent_prefill_supported": (_i, [_i, _i, _i, _i, _i]),
    "b2kv_latent_prefill": (_i, [_vp, _i64, _vp, _vp, _i64, _vp, _i64, _vp, _i64, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _i,
                                 _vp, _vp]),
    "b2kv_gqa_append": (_i, [_vp, _i64, _i, _i, _i, _i, _vp, _vp, _f, _f, _i, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _vp, _vp]),
    "b2kv_gqa_decode_workspace_bytes": (_sz, [_i, _i, _i, _i, _i, _i]),
    "b2kv_gqa_decode": (_i, [_vp, _i64, _vp, _vp, _vp, _i64, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _f, _i, _i, _vp, _sz,
                             _vp, _vp]),
    "b2kv_gqa_prefill_supported": (_i, [_i, _i, _i]),
    "b2kv_gqa_prefill": (_i, [_vp, _i64, _vp, _vp, _i64, _vp, _i64, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _f, _i, _vp, _vp]),
    "b2kv_gla_workspace_bytes": (_sz, [_i, _i, _i, _i, _i, _i, _i]),
    "b2kv_gla": (_i, [ctypes.POINTER(GlaArgs), _vp, _vp]),
    "b2kv_route": (_i, [_vp, _i64, _i, _i, _i, _i, _i, _vp, _vp, _vp, _vp]),
    "b2kv_moe_plan": (_i, [_vp, _vp, _i, _i, _i, _vp, _vp, _vp, _i64, _vp, _i64, _i, _i, _vp]),
    "b2kv_moe_combine": (_i, [_vp, _i64, _vp, _i64, _vp, _vp, _i, _i, _i, _i, _vp]),
    "b2kv_tune": (_i, [ctypes.c_char_p, _i]),
}


class B2KVError(RuntimeError):
    """A C-ABI call returned a negative status."""

    def __init__(self, status: int, text: str):
        super().__init__(f"b2kv error {status}: {text}")
        self.status = status


def _not_built(name: str):
    def call(*_):
        raise ImportError(f"{name} is not part of {SERVE_LIB_PATH.name}; build the whole library with {_PKG.name}/build.py")

    return call


def _load() -> ctypes.CDLL:
    path = LIB_PATH if LIB_PATH.exists() or not SERVE_LIB_PATH.exists() else SERVE_LIB_PATH
    if not path.exists():
        raise ImportError(
            f"{LIB_PATH} is missing. Build the CUDA library first: "
            f"`python {_PKG.name}/build.py` (needs nvcc with sm_100a support). "
            "This package has no CPU fallback."
        )
    lib = ctypes.CDLL(str(path))
    for name, (restype, argtypes) in SIGNATURES.items():
        if path == SERVE_LIB_PATH and not hasattr(lib, name):
            setattr(lib, name, _not_built(name))
            continue
        fn = getattr(lib, name)  # AttributeError here means header and library disagree
        fn.restype = restype
        fn.argtypes = argtypes
    return lib


lib = _load()


def check(status: int) -> None:
    """Raise for a negative status of a C-ABI call."""
    if status == 0:
        return
    text = lib.b2kv_strerror(status).decode()
    if status == ERR_CUDA:
        text += ": " + lib.b2kv_last_cuda_error().decode()
    raise B2KVError(status, text)


def tune(name: str, value: int) -> None:
    check(lib.b2kv_tune(name.encode(), int(value)))
