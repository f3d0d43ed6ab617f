"""ctypes binding of the C-ABI libraries `libsocket_b200.so` (declared in `include/socket_b200.h`)
and `libsocket_b200_blocks.so` (`include/socket_b200_blocks.h`).  There is no fallback: if a library
is missing, calling one of its operators raises."""
from __future__ import annotations

import ctypes as C
import os

import torch

_PKG = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_PKG, "libsocket_b200.so")
BLOCKS_PATH = os.path.join(_PKG, "libsocket_b200_blocks.so")

SK_F32, SK_BF16, SK_F16 = 0, 1, 2
DTYPE_CODE = {torch.float32: SK_F32, torch.bfloat16: SK_BF16, torch.float16: SK_F16}

SK_DEV_POS_OUT_OF_RANGE = 1
SK_DEV_INDEX_OUT_OF_RANGE = 2
SK_DEV_WAIT_TIMEOUT = 4
SK_SPARSE_DECODE_STATIC_BYTES = 2 << 20


class SocketError(RuntimeError):
    """An entry point of the CUDA library returned a non-zero status."""


class DecodeParams(C.Structure):
    """Mirror of `sk_decode_params`."""
    _fields_ = [
        ("q", C.c_void_p), ("k_new", C.c_void_p), ("v_new", C.c_void_p), ("input_pos", C.c_void_p),
        ("planes", C.c_void_p), ("protos_T", C.c_void_p), ("temperature", C.c_float),
        ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("codes", C.c_void_p),
        ("v_norm", C.c_void_p), ("prefill_len", C.c_void_p),
        ("out", C.c_void_p), ("list", C.c_void_p), ("list_len", C.c_void_p),
        ("list_row_stride", C.c_int64),
        ("workspace", C.c_void_p), ("workspace_bytes", C.c_size_t), ("status", C.c_void_p),
        ("q_dtype", C.c_int), ("kv_dtype", C.c_int), ("plane_dtype", C.c_int),
        ("B", C.c_int), ("H", C.c_int), ("Hkv", C.c_int), ("D", C.c_int), ("L", C.c_int),
        ("P", C.c_int), ("R", C.c_int),
        ("Tcap", C.c_int64), ("T_max", C.c_int64), ("M", C.c_int64),
        ("sink", C.c_int), ("window", C.c_int), ("select_path", C.c_int),
    ]


_i, _i64, _p, _f, _sz = C.c_int, C.c_int64, C.c_void_p, C.c_float, C.c_size_t

# name -> (restype, argtypes); the order follows include/socket_b200.h
SIGNATURES = {
    "sk_abi_version": (_i, []),
    "sk_status_string": (C.c_char_p, [_i]),
    "sk_last_error": (C.c_char_p, []),
    "sk_hash_keys": (_i, [_p, _i, _i64, _p, _i, _i64, _i, _i, _i, _p, _i, _i64, _p]),
    "sk_kv_append": (_i, [_p, _p, _i, _p, _p, _i, _p, _p, _p, _p, _p, _p, _i, _i, _i, _i, _i64, _i, _i, _p]),
    "sk_hash_keys_tc_workspace_bytes": (_sz, [_i64]),
    "sk_hash_keys_tc": (_i, [_p, _i64, _p, _i64, _i, _i, _i, _p, _i64, _p, _p, _sz, _p, _p]),
    "sk_kv_append_tc_workspace_bytes": (_sz, [_i, _i, _i]),
    "sk_kv_append_tc": (_i, [_p, _p, _i, _p, _p, _i, _p, _p, _p, _p, _p, _p, _i, _i, _i, _i, _i64, _i, _i,
                             _p, _sz, _p]),
    "sk_rope_split": (_i, [_p, _i, _p, _i, _p, _i, _i, _i, _i, _i64, _p, _p, _p, _p, _p]),
    "sk_gemv_allreduce_buffer_bytes": (_sz, [_i, _i, _i]),
    "sk_gemv_allreduce": (_i, [_p, _p, _i64, _p, _p, _i, _i, _i, _i, _p, _i, _i, _i, _p, _p, _p]),
    "sk_lut_head_tile": (_i, [_i]),
    "sk_soft_hash": (_i, [_p, _i, _p, _i, _p, _f, _i, _i, _i, _i, _i, _i, _i, _p, _p, _p]),
    "sk_lut_from_probs": (_i, [_p, _i, _i, _i, _i, _i, _i, _p, _p]),
    "sk_score": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _i, _i64, _p, _i64, _p, _i64, _p, _p]),
    "sk_score_compat": (_i, [_p, _p, _p, _p, _p, _i, _i, _i, _i, _i64, _p]),
    "sk_list_len": (_i64, [_i64, _i, _i, _i64]),
    "sk_select_list": (_i, [_p, _i64, _p, _i64, _i64, _p, _i64, _i, _i, _i, _p, _i64, _p, _p, _p]),
    "sk_score_select_applicable": (_i, [_i, _i, _i, _i, _i, _i64, _i64]),
    "sk_score_select_workspace_bytes": (_sz, [_i, _i, _i, _i, _i64, _i64]),
    "sk_score_filter": (_i, [_p, _p, _p, _i, _i, _i, _i, _i, _i64, _p, _i64, _i64, _p, _sz, _p, _p]),
    "sk_select_candidates": (_i, [_p, _p, _p, _i, _i, _i, _i, _i, _i64, _p, _i64, _i64, _i, _i, _p, _i64, _p,
                                  _p, _sz, _p, _p]),
    "sk_score_select_list": (_i, [_p, _p, _p, _i, _i, _i, _i, _i, _i64, _p, _i64, _i64, _i, _i, _p, _i64, _p,
                                  _p, _sz, _p, _p]),
    "sk_packed_table_bytes": (_sz, [_i, _i, _i]),
    "sk_packed_applicable": (_i, [_i, _i, _i, _i, _i, _i64, _i64]),
    "sk_packed_preferred": (_i, [_i, _i, _i, _i, _i, _i64, _i64]),
    "sk_soft_hash_packed": (_i, [_p, _i, _p, _i, _p, _f, _i, _i, _i, _i, _i, _i, _i, _p, _p, _p]),
    "sk_score_select_packed": (_i, [_p, _p, _p, _p, _i, _i, _i, _i, _i, _i64, _p, _i64, _i64, _i, _i, _p, _i64,
                                    _p, _p, _sz, _p, _i, _p]),
    "sk_score_select_cluster_size": (_i, [_i, _i, _i, _i, _i, _i64, _i64]),
    "sk_score_select_cluster": (_i, [_p, _p, _p, _i, _i, _i, _i, _i, _i64, _p, _i64, _i64, _i, _i, _p, _i64, _p,
                                     _p, _p]),
    "sk_sparse_decode_workspace_bytes": (_sz, [_i, _i, _i, _i64]),
    "sk_sparse_decode": (_i, [_p, _i, _p, _p, _i, _i64, _i64, _i64, _p, _i64, _p, _i64, _p, _i, _i,
                              _i, _i, _i64, _p, _p, _sz, _p, _p]),
    "sk_sparse_decode_static": (_i, [_p, _i, _p, _p, _i, _i64, _i64, _i64, _p, _i64, _p, _i64, _p, _i, _i,
                                     _i, _i, _i64, _p, _p, _p]),
    "sk_decode_step_workspace_bytes": (_sz, [_i, _i, _i, _i, _i, _i, _i64, _i64, _i, _i]),
    "sk_decode_step_rescored_rows_offset": (_i64, [_i, _i, _i, _i, _i, _i, _i64, _i64, _i, _i]),
    "sk_decode_step": (_i, [C.POINTER(DecodeParams), _p]),
}


class ResidualParams(C.Structure):
    """Mirror of `sk_residual_params`."""
    _fields_ = [
        ("x", _p), ("y", _p), ("w_in", _p), ("x0", _p), ("w_out", _p), ("out", _p),
        ("rows", _i64), ("y_ld", _i64),
        ("width", _i), ("in_mode", _i), ("out_mode", _i), ("dtype", _i), ("y_dtype", _i), ("eps", _f),
    ]


class AttnParams(C.Structure):
    """Mirror of `sk_attn_params`."""
    _fields_ = [
        ("q", _p), ("k", _p), ("v", _p), ("out", _p), ("bias", _p), ("sink", _p), ("pos", _p), ("status", _p),
        ("workspace", _p), ("workspace_bytes", _sz),
        ("q_bs", _i64), ("q_ss", _i64), ("q_hs", _i64), ("k_bs", _i64), ("k_ts", _i64), ("k_hs", _i64),
        ("v_bs", _i64), ("v_ts", _i64), ("v_hs", _i64), ("o_bs", _i64), ("o_ss", _i64), ("o_hs", _i64),
        ("start", _i64), ("kv_start", _i64), ("kv_rows", _i64), ("bias_len", _i64),
        ("dtype", _i), ("B", _i), ("S", _i), ("H", _i), ("G", _i), ("dqk", _i), ("dv", _i), ("chunk", _i),
        ("window", _i), ("ring", _i), ("path", _i), ("scale", _f), ("softcap", _f),
    ]


class RotaryRowsParams(C.Structure):
    """Mirror of `sk_rotary_rows_params`."""
    _fields_ = [
        ("q_in", _p), ("k_in", _p), ("ring", _p), ("q_out", _p), ("rows_out", _p), ("angles", _p), ("pos", _p),
        ("status", _p), ("in_ld", _i64), ("start", _i64), ("n_pos", _i64), ("rows_cap", _i64), ("ring_rows", _i64),
        ("dtype", _i), ("B", _i), ("S", _i), ("H", _i), ("G", _i), ("dim", _i), ("rot_dims", _i), ("prev", _i),
    ]


class LatentParams(C.Structure):
    """Mirror of `sk_latent_params`."""
    _fields_ = [
        ("dkv", _p), ("q", _p), ("norm_w", _p), ("angles", _p), ("cache", _p), ("pos", _p), ("status", _p),
        ("dkv_ld", _i64), ("q_ld", _i64), ("cap", _i64), ("cache_ld", _i64), ("start", _i64),
        ("dtype", _i), ("B", _i), ("S", _i), ("H", _i), ("dim", _i), ("rot", _i), ("rot_dims", _i), ("rank", _i),
        ("eps", _f),
    ]


class SsmParams(C.Structure):
    """Mirror of `sk_ssm_params`."""
    _fields_ = [
        ("xbc_in", _p), ("dt_in", _p), ("conv_w", _p), ("conv_b", _p), ("conv_state", _p), ("xbc", _p), ("y", _p),
        ("dt_bias", _p), ("A_log", _p), ("D", _p), ("state", _p), ("pos", _p),
        ("workspace", _p), ("workspace_bytes", _sz), ("in_ld", _i64), ("xbc_ld", _i64), ("start", _i64),
        ("dtype", _i), ("B", _i), ("S", _i), ("H", _i), ("P", _i), ("N", _i), ("G", _i), ("taps", _i), ("path", _i),
    ]


class MlstmParams(C.Structure):
    """Mirror of `sk_mlstm_params`."""
    _fields_ = [
        ("q", _p), ("k", _p), ("v", _p), ("z", _p), ("norm_w", _p), ("gates", _p), ("i_bias", _p), ("f_bias", _p),
        ("S_state", _p), ("n_state", _p), ("m_state", _p), ("num", _p), ("den", _p), ("m_next", _p), ("out", _p),
        ("pos", _p), ("status", _p), ("workspace", _p), ("workspace_bytes", _sz), ("in_ld", _i64), ("gates_ld", _i64),
        ("out_ld", _i64), ("start", _i64), ("dtype", _i), ("B", _i), ("S", _i), ("H", _i), ("N", _i), ("P", _i),
        ("path", _i), ("cap", _f), ("q_scale", _f), ("eps", _f),
    ]


# the building-block library, in the order of include/socket_b200_blocks.h
BLOCK_SIGNATURES = {
    "skb_abi_version": (_i, []),
    "skb_status_string": (C.c_char_p, [_i]),
    "skb_last_error": (C.c_char_p, []),
    "skb_embed_rows": (_i, [_p, _p, _i, _i64, _i64, _i, _f, _p, _p, _p, _p]),
    "skb_residual_norm": (_i, [C.POINTER(ResidualParams), _p]),
    "skb_glu": (_i, [_p, _p, _i, _i64, _i, _i64, _i, _f, _f, _p, _i64, _p]),
    "skb_ring_append": (_i, [_p, _p, _i, _i, _i, _i64, _i64, _i64, _i64, _i, _i, _i, _i, _p, _i64, _p, _p, _p]),
    "skb_rotary_rows": (_i, [C.POINTER(RotaryRowsParams), _p]),
    "skb_attn_workspace_bytes": (_sz, [C.POINTER(AttnParams)]),
    "skb_attn": (_i, [C.POINTER(AttnParams), _p]),
    "skb_attn_path": (_i, [C.POINTER(AttnParams)]),
    "skb_latent_append": (_i, [C.POINTER(LatentParams), _p]),
    "skb_latent_absorb": (_i, [_p, _i64, _i, _p, _i64, _i, _i, _i, _i, _i, _p, _p]),
    "skb_latent_up": (_i, [_p, _i, _p, _i64, _i, _i, _i, _p, _p]),
    "skb_ssm_conv": (_i, [C.POINTER(SsmParams), _p]),
    "skb_ssm_workspace_bytes": (_sz, [C.POINTER(SsmParams)]),
    "skb_ssm_scan": (_i, [C.POINTER(SsmParams), _p]),
    "skb_ssm_path": (_i, [C.POINTER(SsmParams)]),
    "skb_mlstm_workspace_bytes": (_sz, [C.POINTER(MlstmParams)]),
    "skb_mlstm": (_i, [C.POINTER(MlstmParams), _p]),
    "skb_mlstm_path": (_i, [C.POINTER(MlstmParams)]),
    "skb_gated_group_norm": (_i, [_p, _p, _i64, _p, _i, _i64, _i, _i, _f, _p, _p]),
}

_handles = {}


def _load(path: str, library: str, signatures) -> C.CDLL:
    handle = _handles.get(path)
    if handle is None:
        if not os.path.exists(path):
            raise SocketError(f"{path} is missing: build it with `python -m socket_b200.build {library}` "
                              "(there is no fallback implementation)")
        handle = C.CDLL(path)
        for name, (res, args) in signatures.items():
            fn = getattr(handle, name)
            fn.restype = res
            fn.argtypes = args
        _handles[path] = handle
    return handle


def lib() -> C.CDLL:
    """The sparse-attention step's library.  Raises if it has not been built (`python -m socket_b200.build`)."""
    return _load(LIB_PATH, "step", SIGNATURES)


def blocks() -> C.CDLL:
    """The decoder building blocks' library."""
    return _load(BLOCKS_PATH, "blocks", BLOCK_SIGNATURES)


def check_blocks(status: int, what: str) -> None:
    if status != 0:
        l = blocks()
        raise SocketError(f"{what}: {l.skb_status_string(status).decode()} — {l.skb_last_error().decode()}")


def check(status: int, what: str) -> None:
    if status != 0:
        l = lib()
        raise SocketError(f"{what}: {l.sk_status_string(status).decode()} — {l.sk_last_error().decode()}")


def ptr(t) -> int:
    return 0 if t is None else t.data_ptr()


def stream_ptr(device=None) -> int:
    return torch.cuda.current_stream(device).cuda_stream


def dtype_code(t: torch.Tensor) -> int:
    try:
        return DTYPE_CODE[t.dtype]
    except KeyError:
        raise SocketError(f"unsupported dtype {t.dtype}") from None
