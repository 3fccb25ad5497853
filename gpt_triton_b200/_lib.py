"""ctypes binding of libb200gpt.so (declared in include/b200_gpt.h).

There is no fallback: if the library is missing or a symbol cannot be bound, importing
the operators fails with an error that says how to build it.
"""

import ctypes
import os

import torch

from .build import LIB_PATH

F32, F16, BF16 = 0, 1, 2
_TORCH_TO_CODE = {torch.float32: F32, torch.float16: F16, torch.bfloat16: BF16}
CODE_TO_TORCH = {code: dtype for dtype, code in _TORCH_TO_CODE.items()}

c_i64, c_int, c_float, c_void_p, c_size_t = ctypes.c_int64, ctypes.c_int, ctypes.c_float, ctypes.c_void_p, ctypes.c_size_t
_p_i64 = ctypes.POINTER(ctypes.c_int64)



class LinearArgs(ctypes.Structure):
    """b200_linear_args of include/b200_gpt.h, field for field."""

    _fields_ = [("a", c_void_p), ("b", c_void_p), ("M", c_i64), ("N", c_i64), ("K", c_i64), ("lda", c_i64), ("ldb", c_i64),
                ("row_sumsq", c_void_p), ("row_sumsq_ld", c_i64), ("row_sumsq_cols", c_i64), ("out", c_void_p), ("ld_out", c_i64),
                ("act_split", c_i64), ("x", c_void_p), ("ld_x", c_i64), ("gain", c_void_p), ("gx", c_void_p), ("ld_gx", c_i64),
                ("sumsq_out", c_void_p), ("sumsq_out_ld", c_i64), ("status_word", c_void_p), ("op_dtype", c_int), ("out_dtype", c_int),
                ("row_sumsq_slices", c_int), ("act_lo", c_int), ("act_hi", c_int), ("eps", c_float), ("out_scale", c_float), ("bias", c_void_p), ("act_param", c_float),
                ("pair_limit", c_float), ("pair_alpha", c_float), ("pair_cols", c_i64)]


def _fields(text):
    """"type name name; type name" -> ctypes fields; ptr, i64, int and float."""
    kinds = {"ptr": c_void_p, "i64": c_i64, "int": c_int, "float": c_float}
    out = []
    for part in text.split(";"):
        kind, *names = part.split()
        out += [(n, kinds[kind]) for n in names]
    return out


class StreamArgs(ctypes.Structure):
    """b200_stream_args, field for field (as the classes below)."""

    _fields_ = _fields("ptr x y; i64 ld_y; ptr y_gain ids table; i64 V; ptr shift gain h; i64 ld_h T W; float table_scale eps; int keep dtype")


class RotaryArgs(ctypes.Structure):
    _fields_ = _fields("ptr rows; i64 ld off_k off_v; ptr q_weight k_weight freq k_rows; i64 ld_k; ptr v_rows; i64 ld_v; ptr k_cache v_cache pos_dev; "
                       "i64 B n q_heads kv_heads maps dim vdim rot_dims hist ring start; float eps; int dtype v_rows_dtype")


class PairAttentionArgs(ctypes.Structure):
    _fields_ = _fields("ptr q; i64 ld_q; ptr k; i64 k_batch k_head k_row; ptr v; i64 v_batch v_head v_row; ptr gate; i64 ld_gate; ptr lambda_ out; i64 ld_out; "
                       "ptr pos_dev; i64 B n hist ring heads kv_heads dim vdim window; float scale softcap eps out_scale; int dtype v_dtype; ptr workspace; "
                       "i64 workspace_bytes; ptr status_word")


class DeltaArgs(ctypes.Structure):
    _fields_ = _fields("ptr rows; i64 ld off_k off_v off_a off_b off_g; ptr conv_w conv_state; i64 conv_cols taps; ptr mixed; i64 ld_mixed; "
                       "ptr norms gates a_log dt_bias norm_w state y; i64 ld_y; ptr pos_dev; i64 B n start heads kv_heads dim vdim; "
                       "float eps unit_eps q_scale; int fresh dtype; ptr workspace; i64 workspace_bytes; ptr status_word")


# name -> (restype, argtypes); must list every function include/b200_gpt.h declares
SIGNATURES = {
    "b200_status_string": (ctypes.c_char_p, [c_int]),
    "b200_last_cuda_error": (ctypes.c_char_p, []),
    "b200_abi_version": (c_int, []),
    "b200_launch_count": (ctypes.c_uint64, []),
    "b200_embedding": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_i64, c_i64, c_i64, c_i64, c_i64, c_int, c_void_p, c_void_p]),
    "b200_embedding_ln_stats": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_i64, c_i64, c_i64, c_i64, c_i64, c_int, c_void_p, c_float, c_void_p, c_void_p,
                                        c_void_p]),
    "b200_row_ln_stats": (c_int, [c_void_p, c_void_p, c_void_p, c_i64, c_i64, c_float, c_int, c_void_p]),
    "b200_fold_layernorm": (c_int, [c_void_p] * 8 + [c_i64, c_i64, c_i64, c_int, c_void_p]),
    "b200_gemm_ln_workspace_bytes": (c_size_t, [c_i64, c_i64]),
    "b200_gemm_ln": (c_int, [c_void_p] * 5 + [c_i64] * 7 + [c_int, c_int, c_int] + [c_void_p] * 5 + [c_float, c_void_p, c_size_t, c_void_p, c_void_p]),
    "b200_layernorm": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_i64, c_i64, c_float, c_int, c_int, c_void_p]),
    "b200_pack_operand": (c_int, [c_void_p, c_void_p, c_i64, c_i64, c_i64, c_i64, c_int, c_int, c_int, c_void_p]),
    "b200_gemm": (c_int, [c_void_p] * 5 + [c_i64] * 7 + [c_int, c_int, c_int, c_void_p, c_void_p]),
    "b200_gemm_argmax_workspace_bytes": (c_size_t, [c_i64, c_i64]),
    "b200_gemm_argmax": (c_int, [c_void_p] * 5 + [c_i64] * 7 + [c_int, c_int, c_int, c_void_p, c_void_p, c_void_p, c_size_t, c_void_p, c_void_p]),
    "b200_gemm_rowstats": (c_int, [c_void_p] * 3 + [c_i64] * 5 + [c_int, c_int] + [c_void_p] * 5 + [c_size_t, c_void_p, c_void_p]),
    "b200_ffn_workspace_bytes": (c_size_t, [c_i64, c_i64, c_i64, c_int, c_int]),
    "b200_ffn": (c_int, [c_void_p] * 5 + [c_i64] * 4 + [c_int, c_int, c_int, c_void_p, c_size_t, c_void_p, c_void_p]),
    "b200_ffn_static_scratch": (c_int, [c_void_p] * 5 + [c_i64] * 4 + [c_int, c_int, c_int, c_void_p, c_void_p]),
    "b200_attention": (c_int, [c_void_p] * 4 + [c_i64] * 4 + [_p_i64] * 4 + [c_float, c_int, c_int, c_void_p, c_void_p]),
    "b200_embedding_at": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_i64, c_i64, c_i64, c_i64, c_i64, c_int, c_void_p, c_float, c_void_p, c_void_p,
                                  c_void_p, c_void_p]),
    "b200_kv_cache_fill": (c_int, [c_void_p, c_void_p, c_i64, c_i64, c_i64, c_i64, c_int, c_void_p]),
    "b200_attention_decode": (c_int, [c_void_p, c_void_p, c_void_p, c_i64, c_i64, c_i64, c_i64, c_float, c_int, c_void_p, c_void_p, c_void_p]),
    "b200_decode_append": (c_int, [c_void_p, c_void_p, c_i64, c_i64, c_i64, c_void_p, c_int, c_void_p, c_void_p, c_void_p]),
    "b200_sample_logits": (c_int, [c_void_p, c_i64, c_i64, c_i64, c_int, c_float, c_int, ctypes.c_uint64, c_void_p, c_void_p, c_void_p]),
    "b200_linear_slice_cols": (c_i64, [c_i64, c_int]),
    "b200_linear": (c_int, [ctypes.POINTER(LinearArgs), c_void_p]),
    "b200_embedding_rms": (c_int, [c_void_p] * 6 + [c_i64] * 4 + [c_int, c_void_p]),
    "b200_latent_append": (c_int, [c_void_p, c_i64, c_void_p, c_float, c_void_p, c_void_p] + [c_i64] * 6 + [c_void_p, c_int, c_void_p]),
    "b200_latent_gather": (c_int, [c_void_p, c_void_p] + [c_i64] * 6 + [c_int, c_void_p]),
    "b200_window_attention": (c_int, [c_void_p, c_i64] * 4 + [c_i64] * 7 + [c_float, c_void_p, c_int, c_void_p, c_void_p]),
    "b200_latent_decode_workspace_bytes": (c_size_t, [c_i64] * 4 + [c_int]),
    "b200_latent_decode": (c_int, [c_void_p, c_i64, c_void_p, c_void_p, c_void_p, c_void_p] + [c_i64] * 8 + [c_float, c_void_p, c_int, c_void_p, c_void_p,
                                                                                                        c_size_t, c_void_p]),
    "b200_decayed_attention_slices": (c_i64, [c_i64] * 4 + [c_int]),
    "b200_decayed_attention_workspace_bytes": (c_size_t, [c_i64] * 5 + [c_int]),
    "b200_decayed_attention": (c_int, [c_void_p] + [c_i64] * 4 + [c_void_p] * 3 + [c_int, c_void_p, c_i64, c_void_p] + [c_i64] * 6
                               + [c_int, c_void_p, c_size_t, c_void_p, c_void_p]),
    "b200_stream_update": (c_int, [ctypes.POINTER(StreamArgs), c_void_p]),
    "b200_gated_pairs": (c_int, [c_void_p, c_i64, c_void_p, c_i64, c_i64, c_i64, c_float, c_float, c_int, c_void_p]),
    "b200_rotary_append": (c_int, [ctypes.POINTER(RotaryArgs), c_void_p]),
    "b200_pair_attention_v_dtype": (c_int, [c_i64, c_i64, c_int]),
    "b200_pair_attention_workspace_bytes": (c_i64, [ctypes.POINTER(PairAttentionArgs)]),
    "b200_pair_attention": (c_int, [ctypes.POINTER(PairAttentionArgs), c_void_p]),
    "b200_delta_workspace_bytes": (c_i64, [ctypes.POINTER(DeltaArgs)]),
    "b200_delta": (c_int, [ctypes.POINTER(DeltaArgs), c_void_p]),
    "b200_selftest_bounded_wait": (c_int, [c_void_p, c_i64, c_void_p]),
}

_lib = None


class B200Error(RuntimeError):
    """A libb200gpt entry point returned a non-zero status."""


def load():
    """Load the shared library once and bind every declared symbol."""
    global _lib
    if _lib is not None:
        return _lib
    if not os.path.exists(LIB_PATH):
        raise ImportError(
            f"{LIB_PATH} is missing: the CUDA extension has not been built. "
            "Run `python -m gpt_triton_b200.build` (needs nvcc); there is no CPU or PyTorch fallback."
        )
    lib = ctypes.CDLL(LIB_PATH)
    for name, (res, args) in SIGNATURES.items():
        fn = getattr(lib, name)  # AttributeError if the library does not export it
        fn.restype = res
        fn.argtypes = args
    _lib = lib
    return lib


def dtype_code(dtype):
    try:
        return _TORCH_TO_CODE[dtype]
    except KeyError:
        raise TypeError(f"unsupported dtype {dtype}; expected float32, float16 or bfloat16") from None


def check(status, what):
    if status != 0:
        lib = load()
        msg = lib.b200_status_string(status).decode()
        if status == 3:
            msg += ": " + lib.b200_last_cuda_error().decode()
        raise B200Error(f"{what}: {msg} (status {status})")


def stream_ptr(device):
    return torch.cuda.current_stream(device).cuda_stream


def require_cuda(*tensors):
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise RuntimeError(
                "gpt_triton_b200 operators run only on CUDA tensors (sm_100a kernels); got a tensor on " + str(t.device)
            )
