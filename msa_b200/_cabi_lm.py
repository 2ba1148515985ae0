"""ctypes binding of ``libmsa_b200_lm.so`` (declared in ``include/msa_b200_lm.h``): the kernels of the layered decoder
designs.  No fallback: a missing library or a failed call raises."""
from __future__ import annotations

import ctypes as C
import os

import torch

from ._cabi import MsaError, dtype_code, need_cuda, ptr, stream_ptr   # noqa: F401  (one set of helpers for both libraries)

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "libmsa_b200_lm.so")

EXPORTS = ["msa_lm_residual_norm", "msa_lm_embed", "msa_lm_silu_mul", "msa_lm_softcap", "msa_lm_tanh_split", "msa_lm_token_shift",
           "msa_lm_group_prep", "msa_lm_conv_store", "msa_lm_group_decode_supported", "msa_lm_group_decode", "msa_lm_wkv_decode",
           "msa_lm_wkv_scan", "msa_lm_wkv_chunk_supported", "msa_lm_wkv_chunk", "msa_lm_ssd_decode", "msa_lm_ssd_prep", "msa_lm_ssd_scan",
           "msa_lm_ssd_chunk_supported", "msa_lm_ssd_chunk", "msa_lm_part_norm", "msa_lm_latent_prep", "msa_lm_ring_store",
           "msa_lm_window_attn", "msa_lm_window_attn_tc_supported", "msa_lm_window_attn_tc", "msa_lm_latent_decode_supported", "msa_lm_latent_decode", "msa_lm_delta_decode", "msa_lm_delta_prep", "msa_lm_delta_prep_split", "msa_lm_delta_chunk_supported", "msa_lm_delta_chunk_workspace", "msa_lm_delta_chunk", "msa_lm_gather_rows", "msa_lm_delta_conv_store", "msa_lm_delta_scan",
           "msa_lm_delta_out", "msa_lm_moe_topk", "msa_lm_moe_sort", "msa_lm_moe_gemm", "msa_lm_moe_gemm_tc"]

vp, i32, i64, f32 = C.c_void_p, C.c_int32, C.c_int64, C.c_float


class AttnArgs(C.Structure):
    """``msa_lm_attn_args``."""
    _fields_ = [("qa", vp), ("qa_row", i64), ("qa_head", i64), ("qb", vp), ("qb_row", i64), ("qb_head", i64),
                ("ka", vp), ("ka_row", i64), ("ka_head", i64), ("kb", vp), ("kb_row", i64), ("kb_head", i64),
                ("v", vp), ("v_row", i64), ("v_head", i64), ("out", vp), ("out_row", i64), ("out_head", i64),
                ("gate", vp), ("gate_row", i64), ("slot", vp), ("start", vp), ("cu", vp), ("ctx_off", vp), ("ring_rows", i64),
                ("group", i32), ("sink", i32), ("seq0", i32), ("seq1", i32), ("max_len", i32), ("heads", i32), ("da", i32), ("db", i32), ("dv", i32),
                ("window", i32), ("qa_dtype", i32), ("out_dtype", i32), ("dtype", i32), ("scale", f32)]


class DeltaArgs(C.Structure):
    """``msa_lm_delta_args``."""
    _fields_ = [("proj", vp), ("proj_stride", i64), ("conv_w", vp), ("a_log", vp), ("dt_bias", vp), ("w_norm", vp),
                ("conv_state", vp), ("state", vp), ("pos", vp), ("tok_seq", vp), ("slot", vp), ("start", vp), ("cu", vp),
                ("n_tok", i32), ("n_seq", i32), ("n_decode", i32), ("heads", i32), ("kv_heads", i32), ("dim", i32),
                ("vdim", i32), ("taps", i32), ("eps", f32), ("dtype", i32)]


class EmbedArgs(C.Structure):
    """``msa_lm_embed_args``."""
    _fields_ = [("table", vp), ("token", vp), ("pair_table", vp), ("buckets", i64), ("mul_prev", i64), ("mul_cur", i64),
                ("last_token", vp), ("tok_seq", vp), ("slot", vp), ("start", vp), ("cu", vp), ("w_next", vp), ("w_next2", vp),
                ("x_out", vp), ("x_copy", vp), ("h_out", vp), ("h_out2", vp), ("cat0", vp), ("cat1", vp), ("cat_stride", i64),
                ("status", vp), ("n_rows", i32), ("width", i32), ("vocab", i32), ("eps", f32), ("dtype", i32)]


class GroupArgs(C.Structure):
    """``msa_lm_group_args``."""
    _fields_ = [("proj", vp), ("proj_stride", i64), ("conv_w", vp), ("inv_freq", vp), ("conv_state", vp), ("q_out", vp), ("ring", vp),
                ("ctx", vp), ("pos", vp), ("tok_seq", vp), ("slot", vp), ("start", vp), ("cu", vp), ("ctx_off", vp), ("old_off", vp),
                ("ring_rows", i64), ("heads", i32), ("kv_heads", i32), ("dim", i32), ("vdim", i32), ("rot", i32), ("taps", i32),
                ("q_pitch", i32), ("k_pitch", i32), ("v_pitch", i32), ("n_tok", i32), ("n_seq", i32), ("n_decode", i32), ("n_old", i32),
                ("window", i32), ("dtype", i32)]


class WkvArgs(C.Structure):
    """``msa_lm_wkv_args``."""
    _fields_ = [("r", vp), ("k", vp), ("v", vp), ("g", vp), ("row_stride", i64), ("decay", vp), ("w0", vp), ("u", vp), ("norm", vp),
                ("state", vp), ("tok_seq", vp), ("slot", vp), ("start", vp), ("cu", vp), ("n_tok", i32), ("n_seq", i32),
                ("n_decode", i32), ("heads", i32), ("dim", i32), ("eps", f32), ("dtype", i32)]


class SsdArgs(C.Structure):
    """``msa_lm_ssd_args``."""
    _fields_ = [("proj", vp), ("proj_stride", i64), ("conv_w", vp), ("conv_b", vp), ("dt_bias", vp), ("a_log", vp), ("d_skip", vp),
                ("conv_state", vp), ("state", vp), ("tok_seq", vp), ("slot", vp), ("start", vp), ("cu", vp), ("y", vp), ("n_tok", i32),
                ("n_seq", i32), ("n_decode", i32), ("heads", i32), ("vdim", i32), ("n_state", i32), ("groups", i32), ("taps", i32),
                ("dtype", i32)]


_lib = None


def lib() -> C.CDLL:
    global _lib
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise ImportError(f"{LIB_PATH} is missing: build it with `python -m msa_b200.build` (nvcc, sm_100a).  "
                              "msa_b200 has no CPU or PyTorch fallback.")
        l = C.CDLL(LIB_PATH)
        l.msa_last_error.restype = C.c_char_p
        dp, ap, wp, sp = C.POINTER(DeltaArgs), C.POINTER(AttnArgs), C.POINTER(WkvArgs), C.POINTER(SsdArgs)
        sig = {
            "msa_lm_residual_norm": [vp, i64, vp, i32, i64, vp, vp, i32, vp, vp, f32, vp, i32, i32, vp, vp, vp, i64, vp, vp, vp, i32, vp],
            "msa_lm_embed": [C.POINTER(EmbedArgs), vp],
            "msa_lm_silu_mul": [vp, i64, i32, i32, vp, i64, i32, vp],
            "msa_lm_softcap": [vp, i64, f32, vp],
            "msa_lm_tanh_split": [vp, i32, i32, i32, vp, i32, vp],
            "msa_lm_token_shift": [vp, vp, i32, i32, i32, vp, vp, vp, vp, vp, vp, i32, vp],
            "msa_lm_group_prep": [C.POINTER(GroupArgs), vp],
            "msa_lm_conv_store": [vp, i64, i32, i32, vp, vp, vp, vp, i32, i32, i32, vp],
            "msa_lm_group_decode_supported": [i32, i32],
            "msa_lm_group_decode": [vp, i64, vp, i64, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, i32, vp, i64, vp, i64, vp, vp, vp],
            "msa_lm_wkv_decode": [wp, vp, i64, vp],
            "msa_lm_wkv_scan": [wp, vp, vp, i64, vp],
            "msa_lm_wkv_chunk_supported": [i32],
            "msa_lm_wkv_chunk": [wp, vp, i32, vp, vp, i64, vp],
            "msa_lm_ssd_decode": [sp, vp],
            "msa_lm_ssd_prep": [sp, vp, vp, vp],
            "msa_lm_ssd_scan": [sp, vp, vp, vp],
            "msa_lm_ssd_chunk_supported": [i32, i32],
            "msa_lm_ssd_chunk": [sp, vp, vp, vp, i32, vp, vp, vp],
            "msa_lm_part_norm": [vp, i64, vp, i32, i32, i32, f32, vp, i64, i32, vp],
            "msa_lm_latent_prep": [vp, i64, vp, f32, vp, i32, i32, i32, i32, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32,
                                   i32, vp, i64, vp, i32, vp],
            "msa_lm_ring_store": [vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, vp, i64, i32, vp],
            "msa_lm_window_attn": [ap, vp],
            "msa_lm_window_attn_tc_supported": [i32, i32, i32],
            "msa_lm_window_attn_tc": [ap, i32, i32, i32, vp, vp],
            "msa_lm_latent_decode_supported": [i32, i32],
            "msa_lm_latent_decode": [vp, i64, i64, vp, i64, i64, vp, i64, vp, vp, i32, i32, i32, i32, i32, i32, f32, vp, vp, vp, vp, vp],
            "msa_lm_moe_gemm_tc": [vp, i64, i32, vp, vp, i32, vp, vp, i32, i32, i32, i32, f32, vp, i64, vp, vp],
            "msa_lm_delta_decode": [dp, vp, i64, vp],
            "msa_lm_delta_prep": [dp, vp, vp, vp, vp],
            "msa_lm_delta_conv_store": [dp, vp],
            "msa_lm_delta_scan": [dp, vp, vp, vp, vp, vp],
            "msa_lm_delta_out": [dp, vp, vp, i64, vp],
            "msa_lm_moe_topk": [vp, i64, vp, i32, i32, i32, vp, vp, vp],
            "msa_lm_moe_sort": [vp, i32, i32, i32, i32, vp, vp, vp, vp, i32, vp, vp],
            "msa_lm_gather_rows": [vp, i64, vp, i32, i32, vp, vp],
            "msa_lm_delta_prep_split": [dp, vp, vp, vp, vp],
            "msa_lm_delta_chunk_supported": [i32, i32, i32],
            "msa_lm_delta_chunk_workspace": [i32, i32],
            "msa_lm_delta_chunk": [dp, vp, vp, vp, vp, i32, i32, vp, vp, vp, i64, vp],
            "msa_lm_moe_gemm": [vp, i64, vp, vp, vp, vp, i32, i32, i32, i32, f32, vp, i64, i32, i32, vp],
        }
        for name in EXPORTS:
            getattr(l, name).argtypes = sig[name]
            getattr(l, name).restype = i64 if name.endswith("_workspace") else C.c_int
        _lib = l
    return _lib


launches = 0    # calls into the library since import (each is one kernel launch)


def call(name: str, *args) -> None:
    global launches
    rc = getattr(lib(), name)(*args)
    if rc != 0:
        raise MsaError(f"{name} failed ({rc}): {lib().msa_last_error().decode()}")
    launches += 1
