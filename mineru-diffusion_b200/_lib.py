"""ctypes binding of libmdb200.so (the declarations of include/mdb200.h).

There is no fallback: if the library is missing or a call fails, this raises.
"""
from __future__ import annotations

import ctypes as C
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "libmdb200.so")

_p = C.c_void_p
_i = C.c_int
_i64 = C.c_int64
_u32 = C.c_uint32
_f = C.c_float


def _struct(name, fields):
    return type(name, (C.Structure,), {"_fields_": fields})


# argument blocks of the fp32-residual decoders, field for field as in include/mdb200.h
Rows = _struct("Rows", [("x", _p), ("parts", _p), ("ld", _i64), ("part_stride", _i64), ("nparts", _i), ("col", _i)])
GemmArgs = _struct("GemmArgs", [
    ("dtype", _i), ("form", _i), ("act", _i), ("y_f32", _i), ("x", _p), ("w", _p), ("y", _p), ("ldx", _i64), ("ldy", _i64),
    ("m", _i), ("n", _i), ("k", _i), ("heads", _i), ("experts", _i), ("max_rows_per_expert", _i), ("tile_expert", _p),
    ("num_tiles", _p), ("act_from", _i)])
ResidualNormArgs = _struct("ResidualNormArgs", [
    ("dtype", _i), ("m", _i), ("width", _i), ("width_pad", _i), ("residual", _p), ("ids", _p), ("embed", _p), ("vocab", _i64),
    ("add", Rows * 2), ("moe_rows", _p), ("moe_ld", _i64), ("moe_slot", _p), ("moe_weight", _p), ("weight", _p), ("y", _p),
    ("ldy", _i64), ("embed_scale", _f), ("eps", _f), ("moe_top", _i), ("post", _i), ("weight2", _p), ("res_scale", _f)])
RmsSegment = _struct("RmsSegment", [
    ("src", Rows), ("weight", _p), ("out", _p), ("ld_out", _i64), ("slots", _p), ("num_slots", _i64), ("n", _i),
    ("n_pad", _i), ("eps", _f)])
GatedNormArgs = _struct("GatedNormArgs", [
    ("dtype", _i), ("m", _i), ("heads", _i), ("vdim", _i), ("o", _p), ("den", _p), ("gate", Rows), ("weight", _p), ("y", _p),
    ("ldy", _i64), ("weight_head_stride", _i), ("eps", _f)])
PartNormArgs = _struct("PartNormArgs", [(n, _i) for n in ("dtype", "m", "n", "parts", "gate_first")] + [
    ("out_scale", _f), ("eps", _f), ("o", _p), ("gate", Rows), ("weight", _p), ("y", _p), ("ldy", _i64)])
DecayPrepArgs = _struct("DecayPrepArgs", [(n, _i) for n in (
    "dtype", "m", "bs", "heads", "kv_heads", "dim", "dim_pad", "vdim", "taps", "channels", "shift_state",
    "for_chunks")] + [
    ("q", Rows), ("k", Rows), ("v", Rows), ("dt", Rows), ("conv", _p), ("conv_bias", _p), ("conv_state", _p),
    ("conv_slot_stride", _i64), ("num_slots", _i64), ("row_seq", _p), ("cu_q", _p), ("start", _p), ("state_slot", _p),
    ("a_log", _p), ("dt_bias", _p), ("decay_const", _p), ("q_out", _p), ("k_out", _p), ("v_out", _p), ("decay_out", _p),
    ("step_out", _p)])
RotaryCommitArgs = _struct("RotaryCommitArgs", [(n, _i) for n in (
    "dtype", "m", "heads", "kv_heads", "dim", "dim_pad", "rot_dims")] + [
    ("eps", _f), ("q", Rows), ("k", Rows), ("v", Rows), ("q_norm", _p), ("k_norm", _p), ("inv_freq", _p), ("row_pos", _p),
    ("slots", _p), ("num_slots", _i64), ("q_out", _p), ("k_cache", _p), ("v_cache", _p)])
WindowAttnArgs = _struct("WindowAttnArgs", [(n, _i) for n in (
    "dtype", "m", "bs", "heads", "kv_heads", "dim", "dim_pad", "window", "sink", "max_q", "nsplit")] + [
    ("scale", _f), ("out_scale", _f), ("q", _p), ("k_cache", _p), ("v_cache", _p), ("block_table", _p), ("row_seq", _p),
    ("row_pos", _p), ("cu_q", _p), ("start", _p), ("table_stride", _i), ("num_pages", _i), ("gate", Rows), ("out", _p),
    ("ld_out", _i64), ("workspace", _p), ("workspace_bytes", _i64)])
DeltaPrepArgs = _struct("DeltaPrepArgs", [(n, _i) for n in (
    "dtype", "m", "bs", "heads", "kv_heads", "dim", "dim_pad", "vdim", "taps", "channels", "shift_state", "copy_cols")] + [
    ("q", Rows), ("k", Rows), ("v", Rows), ("b", Rows), ("copy", Rows), ("copy_out", _p), ("copy_ld", _i64), ("conv_q", _p),
    ("conv_k", _p), ("conv_v", _p), ("conv_state", _p), ("conv_slot_stride", _i64), ("num_slots", _i64), ("row_seq", _p),
    ("cu_q", _p), ("start", _p), ("state_slot", _p), ("q_out", _p), ("k_out", _p), ("v_out", _p), ("beta_out", _p)])
DecayArgs = _struct("DecayArgs", [(n, _i) for n in ("m", "heads", "kv_heads", "dim", "dim_pad")] + [
    ("x", _p), ("ldx", _i64), ("a_log", _p), ("dt_bias", _p), ("q", _p), ("k", _p), ("beta", _p), ("g", _p), ("scalars", _p),
    ("row_seq", _p),
    ("cu_q", _p)])
MlstmPrepArgs = _struct("MlstmPrepArgs", [(n, _i) for n in ("dtype", "m", "heads", "dim", "dim_pad", "vdim")] + [
    ("q", Rows), ("k", Rows), ("v", Rows), ("i", Rows), ("f", Rows), ("bias_i", _p), ("bias_f", _p), ("q_out", _p),
    ("k_out", _p), ("v_out", _p), ("log_i", _p), ("log_f", _p), ("cap", _f)])
ScanArgs = _struct("ScanArgs", [(n, _i) for n in (
    "mode", "dtype", "fused", "bs", "heads", "kv_heads", "dim", "dim_pad", "vdim")] + [
    ("eps", _f), ("q", _p), ("k", _p), ("v", _p), ("g", _p), ("s0", _p), ("s1", _p), ("state", _p),
    ("state_slot_stride", _i64), ("num_slots", _i64), ("mstate", _p), ("scalars", _p),
    ("den", _p), ("cu_q", _p), ("start", _p),
    ("state_slot", _p), ("out", _p), ("raw_decay", Rows), ("a_log", _p), ("dt_bias", _p), ("gate", Rows), ("norm", _p),
    ("norm_head_stride", _i64), ("y", _p), ("ldy", _i64), ("skip", _p)])
ChunkScanArgs = _struct("ChunkScanArgs", [(n, _i) for n in ("m", "bs", "heads", "kv_heads", "dim", "dim_pad", "vdim", "max_q")] + [
    ("q", _p), ("k", _p), ("v", _p), ("ldq", _i64), ("ldk", _i64), ("ldv", _i64), ("ld_scalars", _i64), ("log_decay", _p), ("step", _p), ("skip", _p), ("state", _p), ("state_slot_stride", _i64),
    ("num_slots", _i64), ("cu_q", _p), ("start", _p), ("state_slot", _p), ("out", _p)])
MoeRouteArgs = _struct("MoeRouteArgs", [(n, _i) for n in ("m", "experts", "top", "groups", "keep")] + [
    ("logits", Rows), ("row_slot", _p), ("ids", _p), ("weights", _p)])
MoePlanArgs = _struct("MoePlanArgs", [(n, _i) for n in ("m", "top", "experts", "max_tiles")] + [
    ("ids", _p), ("slot", _p), ("row_token", _p), ("tile_expert", _p), ("num_tiles", _p)])

# name -> (restype, argtypes); mirrors include/mdb200.h one to one
SIGNATURES = {
    "mdb_strerror": (C.c_char_p, [_i]),
    "mdb_version": (_i, []),
    "mdb_set_option": (_i, [_i, _i]),
    "mdb_set_trace": (_i, [_p, _i64]),
    "mdb_get_option": (_i, [_i]),
    "mdb_last_device_status": (_i, [C.POINTER(C.c_uint), _i]),
    "mdb_kv_commit": (_i, [_p, _i64, _p, _i64, _p, _p, _p, _i, _i, _i64, _p]),
    "mdb_attn_paged_workspace_bytes": (_i64, [_i, _i, _i, _i]),
    "mdb_attn_block_paged": (_i, [_p, _p, _p, _p, _p, _i, _p, _i, _i, _i, _i, _i, _f, _i, _p, _i64, _p]),
    "mdb_attn_block_paged_noalloc_limit": (_i64, []),
    "mdb_attn_block_paged_noalloc": (_i, [_p, _p, _p, _p, _p, _i, _p, _i, _i, _i, _i, _i, _f, _i, _p]),
    "mdb_attn_staircase_varlen": (_i, [_p, _i64, _p, _i64, _p, _i64, _p, _i64, _p, _i, _i, _i64, _i, _i, _i, _p]),
    "mdb_gemm_bf16": (_i, [_p, _i64, _p, _p, _i64, _i, _i, _i, _p]),
    "mdb_gemm_pick_ksplit": (_i, [_i, _i, _i]),
    "mdb_gemm_splitk_workspace_bytes": (_i64, [_i, _i, _i]),
    "mdb_gemm_splitk_partials": (_i, [_p, _i64, _p, _p, _i, _i, _i, _i, _p]),
    "mdb_gemm_gateup_swiglu": (_i, [_p, _i64, _p, _p, _i64, _i, _i, _i, _p]),
    "mdb_silu_mul": (_i, [_p, _i64, _p, _i64, _i, _i, _p]),
    "mdb_add_rmsnorm": (_i, [_p, _p, _i, _p, _p, _f, _p, _p, _i, _i, _p]),
    "mdb_qknorm_rope_commit": (_i, [_p, _i64, _p, _i, _p, _p, _i, _p, _p, _f, _p, _p, _p, _p, _p, _p, _i64, _i, _i,
                                    _i, _p]),
    "mdb_gemm_qkv_rope_commit": (_i, [_p, _i64, _p, _i, _i, _p, _p, _i, _p, _p, _f, _p, _p, _p, _p, _p, _p, _i64, _i, _i,
                                      _p]),
    "mdb_gather_rows": (_i, [_p, _i64, _p, _p, _i, _i, _p]),
    "mdb_lmhead_workspace_bytes": (_i64, [_i, _i]),
    "mdb_lmhead_sample": (_i, [_p, _i64, _p, _i, _i, _i, _p, _i, _i, _p, _u32, _u32, _p, _p, _i64, _p, _p, _p]),
    "mdb_logits_sample": (_i, [_p, _i64, _i, _i, _p, _i, _i, _p, _u32, _u32, _p, _p, _i64, _p, _p, _p]),
    "mdb_gumbel_noise": (_i, [_p, _i, _i, _u32, _u32, _p]),
    "mdb_unmask_decide": (_i, [_p, _p, _p, _i, _i, _i64, _f, _i, _p, _p, _p, _p, _p]),
    "mdb_tp_alloc": (_i, [_i64, C.POINTER(C.c_void_p)]),
    "mdb_tp_free": (_i, [_p]),
    "mdb_tp_export": (_i, [_p, _p]),
    "mdb_tp_import": (_i, [_p, C.POINTER(C.c_void_p)]),
    "mdb_tp_release": (_i, [_p]),
    "mdb_gemm_splitk_partials_tp": (_i, [_p, _i64, _p, _p, _p, _i, _i, _i, _i, _p, _u32, _p, _p]),
    "mdb_tp_grid_size": (_i, [_i, _i, _i, _i]),
    "mdb_add_rmsnorm_tp": (_i, [_p, _p, _i, _p, _p, _f, _p, _p, _i, _i, _p, _i, _u32, _p, _p]),
    "mdb_lmhead_tp_workspace_bytes": (_i64, [_i, _i]),
    "mdb_lmhead_tp_slots": (_i, [_i, _i]),
    "mdb_gemm_bf16_tp": (_i, [_p, _i64, _p, _p, _p, _i64, _i, _i, _i, _p, _u32, _p, C.POINTER(C.c_int), _p]),
    "mdb_add_rmsnorm_tp_rows": (_i, [_p, _p, _p, _p, _f, _p, _p, _i, _i, _p, _i, _u32, _p, _p]),
    "mdb_lmhead_sample_tp": (_i, [_p, _i64, _p, _i, _i, _i, _p, _i, _i, _p, _u32, _u32, _p, _p, _p, _i64, _i, _i, _p,
                                  _p, _i, _u32, _p, _p, _p, _p]),
    "mdb_gemm": (_i, [C.POINTER(GemmArgs), _p]),
    "mdb_residual_norm": (_i, [C.POINTER(ResidualNormArgs), _p]),
    "mdb_rms_rows": (_i, [_i, C.POINTER(RmsSegment), _i, _i, _p]),
    "mdb_gated_norm": (_i, [C.POINTER(GatedNormArgs), _p]),
    "mdb_part_norm": (_i, [C.POINTER(PartNormArgs), _p]),
    "mdb_decay_prep": (_i, [C.POINTER(DecayPrepArgs), _p]),
    "mdb_rotary_commit": (_i, [C.POINTER(RotaryCommitArgs), _p]),
    "mdb_window_attn_workspace_bytes": (_i64, [_i, _i, _i, _i]),
    "mdb_window_attn": (_i, [C.POINTER(WindowAttnArgs), _p]),
    "mdb_scan_dim_pad": (_i, [_i]),
    "mdb_scan_blocks": (_i, [_i]),
    "mdb_scan_fusable": (_i, [_i, _i]),
    "mdb_delta_prep": (_i, [C.POINTER(DeltaPrepArgs), _p]),
    "mdb_channel_decay": (_i, [C.POINTER(DecayArgs), _p]),
    "mdb_mlstm_prep": (_i, [C.POINTER(MlstmPrepArgs), _p]),
    "mdb_scan": (_i, [C.POINTER(ScanArgs), _p]),
    "mdb_chunk_scan_supported": (_i, [_i, _i]),
    "mdb_chunk_scan": (_i, [C.POINTER(ChunkScanArgs), _p]),
    "mdb_moe_route": (_i, [C.POINTER(MoeRouteArgs), _p]),
    "mdb_moe_plan": (_i, [C.POINTER(MoePlanArgs), _p]),
    "mdb_moe_max_tiles": (_i, [_i, _i, _i]),
    "mdb_moe_gather": (_i, [_i, _p, _i64, _p, _i, _p, _p, _i, _p]),
    "mdb_latent_attn_workspace_bytes": (_i64, [_i, _i, _i, _i]),
    "mdb_latent_attn": (_i, [_i, _p, _p, _p, _p, _i, _p, _p, _i, _i, _i, _i, _f, _i, _p, _i64, _p]),
    "mdb_gather_latents": (_i, [_i, _p, _p, _i, _i, _p, _i, _i, _p, _i, _p]),
    "mdb_attn_causal_varlen": (_i, [_p, _i64, _p, _i64, _p, _i64, _p, _i64, _p, _p, _i, _i, _i64, _i64, _i, _i, _f, _p]),
    "mdb_pick_token": (_i, [_p, _i64, _i, _i, _p, _u32, _p, _p, _p, _p]),
}

_lib = None


class MdbError(RuntimeError):
    """A libmdb200 entry point returned a negative code."""


def lib():
    """The loaded library; raises if it has not been built."""
    global _lib
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise RuntimeError(
                f"{LIB_PATH} is missing: build it with `python mineru-diffusion_b200/build.py` "
                "(there is no CPU or torch fallback for these ops)")
        handle = C.CDLL(LIB_PATH)
        for name, (res, args) in SIGNATURES.items():
            fn = getattr(handle, name)
            fn.restype = res
            fn.argtypes = args
        _lib = handle
    return _lib


def check(rc: int, what: str):
    if rc != 0:
        msg = lib().mdb_strerror(rc).decode()
        raise MdbError(f"{what}: {msg} (code {rc})")


def device_status(clear: bool = True) -> int:
    out = C.c_uint(0)
    check(lib().mdb_last_device_status(C.byref(out), 1 if clear else 0), "mdb_last_device_status")
    return int(out.value)
