"""ctypes binding of ``libtnsr_b200.so`` (the C ABI of include/tnsr_b200.h).

The library is built in-tree by ``python -m tnsr_b200.build`` and loaded from
``tnsr_b200/csrc``.  There is no fallback: if the shared library is missing the
import of anything that needs it raises.
"""
from __future__ import annotations

import ctypes as C
import os

HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(HERE, "csrc", "libtnsr_b200.so")

OK = 0
STATUS = {
    0: "OK", -1: "ERR_INVALID_ARGUMENT", -2: "ERR_CUDA", -3: "ERR_OUT_OF_MEMORY", -4: "ERR_CAPACITY",
    -5: "ERR_TOKEN_RANGE", -6: "ERR_FAILED_STATE", -7: "ERR_TIMEOUT", -8: "ERR_UNSUPPORTED", -9: "ERR_NO_DEVICE",
}
ACT = {"relu": 0, "gelu": 1, "swiglu": 2, "gelu_tanh": 3, "relu_squared": 4}
MIXER = {"attention": 0, "mamba2": 1, "attention+hgrn2": 2, "rglru": 3}
BLOCK = {"parallel": 0, "sequential": 1}
FEED_FORWARD = {"gelu_tanh": 0, "polynorm": 1, "experts": 2}
SCORE = {"softmax": 0, "sigmoid": 1}
ROTARY = {"interleaved": 0, "halves": 1}
DTYPE = {"f32": 0, "bf16": 1}
LOGITS = {"all": 0, "last": 1, "none": 2}
PREFILL = {"auto": 0, "scalar": 1}


class Config(C.Structure):
    _fields_ = [
        ("vocab_size", C.c_uint32), ("max_sequence_length", C.c_uint32), ("embed_dim", C.c_uint32),
        ("num_heads", C.c_uint32), ("feed_forward_dim", C.c_uint32), ("num_layers", C.c_uint32),
        ("layer_norm_epsilon", C.c_float), ("activation", C.c_uint32), ("weight_dtype", C.c_uint32),
        ("kv_dtype", C.c_uint32), ("batch", C.c_uint32), ("capacity", C.c_uint32), ("device", C.c_int32),
        ("logits_mode", C.c_uint32), ("prefill_mode", C.c_uint32), ("step_parts", C.c_uint32),
        ("kv_page_rows", C.c_uint32), ("kv_pool_pages", C.c_uint32), ("small_batch_mode", C.c_uint32),
    ]


class LayerDesc(C.Structure):
    _fields_ = [
        ("mixer", C.c_uint32), ("weights_of", C.c_int32), ("heads", C.c_uint32), ("vdim", C.c_uint32), ("conv_taps", C.c_uint32),
        ("feed_forward", C.c_uint32), ("kv_heads", C.c_uint32), ("dim", C.c_uint32), ("rotary_dims", C.c_uint32), ("rotary_layout", C.c_uint32),
        ("rotary_base", C.c_double), ("rotary_factor", C.c_double), ("rotary_low", C.c_double), ("rotary_high", C.c_double),
        ("rotary_original", C.c_double), ("score_scale", C.c_double), ("score_softcap", C.c_double), ("state", C.c_uint32),
        ("groups", C.c_uint32), ("norm_groups", C.c_uint32), ("block_form", C.c_uint32), ("feed_forward_kind", C.c_uint32),
        ("window", C.c_uint32), ("score_kind", C.c_uint32), ("rec_heads", C.c_uint32), ("rec_dim", C.c_uint32), ("rec_vdim", C.c_uint32),
        ("attention_gain", C.c_double), ("recurrent_gain", C.c_double), ("width", C.c_uint32), ("blocks", C.c_uint32),
        ("experts", C.c_uint32), ("identity_experts", C.c_uint32), ("top", C.c_uint32), ("pad0", C.c_uint32), ("router_scale", C.c_double),
    ]


class StackDesc(C.Structure):
    _fields_ = [("embedding_scale", C.c_double), ("norm_offset", C.c_double), ("layers", C.POINTER(LayerDesc)),
                ("num_layers", C.c_uint32)]


class Place(C.Structure):
    _fields_ = [("sessions", C.c_uint32), ("chunk", C.c_uint32), ("position", C.c_uint32), ("pad0", C.c_uint32),
                ("d_positions", C.c_void_p)]


class GroupedAttentionArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "k_cache", "v_cache", "gate", "out", "workspace", "d_status")] + [("workspace_bytes", C.c_uint64)] + \
        [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "capacity", "gate_ld", "out_ld", "out_cols")] + \
        [("scale", C.c_float), ("softcap", C.c_float), ("dtype", C.c_int32), ("engine", C.c_int32), ("head_bias", C.c_void_p),
         ("window", C.c_uint32), ("score_kind", C.c_uint32), ("gain", C.c_float), ("pad0", C.c_uint32)]


class RotaryArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "rotation", "q", "k_cache", "v_cache")] + \
        [(n, C.c_uint32) for n in ("ld", "heads", "kv_heads", "dim", "vdim", "rotary_dims", "rotary_layout", "capacity")] + \
        [("dtype", C.c_int32), ("pad0", C.c_uint32)]


class Hgrn2Args(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "v", "f", "f_bias", "lower", "norm_w", "state", "raw", "out")] + \
        [(n, C.c_uint32) for n in ("ld", "f_ld", "heads", "dim", "vdim", "out_ld", "out_cols")] + \
        [("eps", C.c_float), ("gain", C.c_float), ("dtype", C.c_int32), ("engine", C.c_int32), ("pad0", C.c_uint32)]


class RglruArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "gate_w", "conv_w", "conv_b", "r_bias", "i_bias", "lambda_", "ring", "state", "u", "gates", "out",
                                          "d_status")] + \
        [(n, C.c_uint32) for n in ("ld", "x_col", "width", "blocks", "taps", "out_ld", "out_cols")] + [("dtype", C.c_int32)]


class ExpertsArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("logits", "correction", "h", "up", "down", "x", "layer_scale", "norm_w", "norm_out", "workspace")] + \
        [("workspace_bytes", C.c_uint64)] + [(n, C.c_void_p) for n in ("chosen", "weights", "d_status")] + \
        [(n, C.c_uint32) for n in ("rows", "logits_ld", "d", "ff", "experts", "identity_experts", "top")] + \
        [("router_scale", C.c_float), ("norm_offset", C.c_float), ("eps", C.c_float), ("dtype", C.c_int32), ("engine", C.c_int32)]


class Mamba2Args(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "dt", "conv_w", "conv_b", "dt_bias", "a_log", "d_skip", "norm_w", "ring", "ssm", "xbc",
                                          "gated", "out")] + \
        [(n, C.c_uint32) for n in ("ld", "dt_ld", "heads", "vdim", "state", "groups", "norm_groups", "taps", "out_ld", "out_cols")] + \
        [("eps", C.c_float), ("dtype", C.c_int32), ("engine", C.c_int32), ("pad0", C.c_uint32)]


_vp, _u32, _u64, _i, _f = C.c_void_p, C.c_uint32, C.c_uint64, C.c_int, C.c_float
_fp, _u32p = C.POINTER(C.c_float), C.POINTER(C.c_uint32)

# name -> (restype, argtypes); one entry per declaration in include/tnsr_b200.h
SIGNATURES = {
    "tnsr_b200_version": (C.c_char_p, []),
    "tnsr_b200_device_count": (_i, []),
    "tnsr_b200_last_error": (C.c_char_p, [_vp]),
    "tnsr_b200_kernel_launches": (_u64, []),
    "tnsr_b200_set_gemm_engine": (_i, [_i]),
    "tnsr_b200_set_wait_limit_ns": (_i, [_u64]),
    "tnsr_b200_test_lose_gemm_stage": (_i, [_u32]),
    "tnsr_b200_decoder_create": (_i, [C.POINTER(Config), C.POINTER(_vp)]),
    "tnsr_b200_decoder_create_stack": (_i, [C.POINTER(Config), C.POINTER(StackDesc), C.POINTER(_vp)]),
    "tnsr_b200_decoder_destroy": (None, [_vp]),
    "tnsr_b200_decoder_param_count": (_u32, [_vp]),
    "tnsr_b200_decoder_param_elems": (_u64, [_vp, _u32]),
    "tnsr_b200_decoder_upload": (_i, [_vp, _u32, _fp, _u64]),
    "tnsr_b200_decoder_reset": (_i, [_vp]),
    "tnsr_b200_decoder_decode": (_i, [_vp, _u32p, _u32, _u32, _fp, _u32p]),
    "tnsr_b200_decoder_decode_ragged": (_i, [_vp, _u32p, _u32p, _fp, _u32p]),
    "tnsr_b200_decoder_decode_device": (_i, [_vp, _vp, _u32, _u32, _vp]),
    "tnsr_b200_decoder_synchronize": (_i, [_vp]),
    "tnsr_b200_decoder_stream": (_vp, [_vp]),
    "tnsr_b200_decoder_profile_attention": (_i, [_vp, _i]),
    "tnsr_b200_decoder_attention_profile": (_i, [_vp, C.POINTER(C.c_double), C.POINTER(C.c_uint64)]),
    "tnsr_b200_decoder_cache_count": (_u32, [_vp]),
    "tnsr_b200_decoder_cache_elems": (_u64, [_vp, _u32]),
    "tnsr_b200_decoder_read_cache": (_i, [_vp, _u32, _fp]),
    "tnsr_b200_decoder_write_cache": (_i, [_vp, _u32, _fp]),
    "tnsr_b200_embedding": (_i, [_vp, _vp, _vp, _vp, _u32, _u32, _u32, _u32, _u32, _i, _vp, _vp]),
    "tnsr_b200_layernorm": (_i, [_vp, _vp, _vp, _vp, _u32, _u32, _f, _i, _i, _vp]),
    "tnsr_b200_gemm_f32_strict": (_i, [_vp, _vp, _vp, _vp, _u32, _u32, _u32, _i, _vp]),
    "tnsr_b200_gemm_bf16": (_i, [_vp, _vp, _vp, _vp, _vp, _u32, _u32, _u32, _i, _i, _vp]),
    "tnsr_b200_gemm_workspace": (_u64, []),
    "tnsr_b200_gemm_bf16_ws": (_i, [_vp, _vp, _vp, _vp, _vp, _u32, _u32, _u32, _i, _i, _vp, _u64, _vp]),
    "tnsr_b200_transpose_bf16": (_i, [_vp, _vp, _u32, _u32, _vp]),
    "tnsr_b200_swiglu": (_i, [_vp, _vp, _vp, _u64, _vp]),
    "tnsr_b200_swiglu_mlp": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _u32, _u32, _u32, _vp]),
    "tnsr_b200_pack_gate_up": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _u32, _u32, _vp]),
    "tnsr_b200_decode_attention_workspace": (_u64, [_u32, _u32, _u32, _u32]),
    "tnsr_b200_decode_attention": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _u64, _u32, _u32, _u32, _u32, _vp]),
    "tnsr_b200_decode_attention_static": (_i, [_vp, _vp, _vp, _vp, _vp, _u32, _u32, _u32, _u32, _vp, _vp]),
    "tnsr_b200_prefill_attention": (_i, [_vp, _vp, _vp, _vp, _u32, _u32, _u32, _u32, _u32, _u32, _vp]),
    "tnsr_b200_argmax": (_i, [_vp, _vp, _u32, _u32, _vp]),
    "tnsr_b200_encoder_embed": (_i, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _u32, _u32, _u32, _u32, _u32, _vp, _vp]),
    "tnsr_b200_encoder_attention": (_i, [_vp, _vp, _vp, _u32, _vp, _vp, _u32, _u32, _u32, _u32, _vp]),
    "tnsr_b200_add_f32": (_i, [_vp, _vp, _vp, _u64, _vp]),
    "tnsr_b200_swiglu_f32": (_i, [_vp, _vp, _vp, _u64, _vp]),
    "tnsr_b200_rmsnorm": (_i, [_vp, _vp, _f, _vp, _u32, _u32, _f, _i, _vp]),
    "tnsr_b200_grouped_attention_workspace": (_u64, [_u32, _u32]),
    "tnsr_b200_grouped_attention": (_i, [C.POINTER(GroupedAttentionArgs), C.POINTER(Place), _vp]),
    "tnsr_b200_mamba2": (_i, [C.POINTER(Mamba2Args), C.POINTER(Place), _vp]),
    "tnsr_b200_rotary": (_i, [C.POINTER(RotaryArgs), C.POINTER(Place), _vp]),
    "tnsr_b200_hgrn2": (_i, [C.POINTER(Hgrn2Args), C.POINTER(Place), _vp]),
    "tnsr_b200_rglru": (_i, [C.POINTER(RglruArgs), C.POINTER(Place), _vp]),
    "tnsr_b200_polynorm": (_i, [_vp, _vp, _vp, _u32, _u32, _u32, _u32, _f, _i, _vp]),
    "tnsr_b200_gemm_grouped": (_i, [_vp, _vp, _vp, _vp, _u32, _u32, _u32, _u32, _i, _i, _i, _i, _vp, _vp]),
    "tnsr_b200_experts_workspace": (_u64, [_u32, _u32, _u32, _u32, _u32, _i]),
    "tnsr_b200_experts": (_i, [C.POINTER(ExpertsArgs), _vp]),
    "tnsr_b200_sample_top_k": (_i, [_vp, _vp, _u32, _u32, _f, _u32, _u64, _u32, _u32, _vp]),
    "tnsr_b200_decoder_set_sampler": (_i, [_vp, _f, _u32, _u64]),
    "tnsr_b200_decoder_release": (_i, [_vp, _u32]),
    "tnsr_b200_decoder_free_pages": (_u32, [_vp]),
}

_lib = None


def lib():
    """The loaded library; raises if it has not been built."""
    global _lib
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise RuntimeError(
                f"{LIB_PATH} is missing: build it with `python -m tnsr_b200.build` "
                "(nvcc, sm_100a). tnsr_b200 has no CPU or PyTorch fallback.")
        L = C.CDLL(LIB_PATH)
        for name, (res, args) in SIGNATURES.items():
            fn = getattr(L, name)
            fn.restype, fn.argtypes = res, args
        _lib = L
    return _lib


def last_error(handle=None) -> str:
    msg = lib().tnsr_b200_last_error(handle)
    return msg.decode("utf-8", "replace") if msg else ""


class NativeError(RuntimeError):
    def __init__(self, code: int, message: str):
        super().__init__(f"{STATUS.get(code, code)}: {message}")
        self.code = code
        self.message = message


def check(code: int, handle=None) -> None:
    if code != OK:
        raise NativeError(code, last_error(handle))
