"""ctypes binding of ``libb200_decode.so`` (declarations in ``include/b200_decode.h``).

There is no fallback: if the library is missing the import of any op fails with a clear
error.  The library is built in-tree by ``megatron_mixtera_b200.build``.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import POINTER, c_char_p, c_float, c_int, c_int32, c_int64, c_size_t, c_void_p

from .build import LIB_PATH, TORCH_LIB_PATH

EXPORTED_SYMBOLS = (
    "b200_version",
    "b200_error_string",
    "b200_device_status",
    "b200_set_wait_limit_ns",
    "b200_copy_rows_h2d",
    "b200_gather_rows_bf16",
    "b200_add_norm_bf16",
    "b200_activation_bf16",
    "b200_set_gemm_split_policy",
    "b200_gemm_bf16_workspace_bytes",
    "b200_gemm_bf16",
    "b200_gemm_bf16_static_scratch_limit",
    "b200_gemm_bf16_static_scratch",
    "b200_mxfp8_scale_bytes",
    "b200_quantize_mxfp8",
    "b200_quantize_mxfp8_weight",
    "b200_fp8_weight_bytes",
    "b200_add_norm_mxfp8",
    "b200_activation_mxfp8",
    "b200_gemm_mxfp8_workspace_bytes",
    "b200_gemm_mxfp8",
    "b200_gemm_mxfp8_swiglu",
    "b200_quantize_fp8_weight_block128",
    "b200_quantize_fp8_rowblock",
    "b200_add_norm_fp8_rowblock",
    "b200_activation_fp8_rowblock",
    "b200_set_fp8_block_cta_pairs",
    "b200_gemm_fp8_block_workspace_bytes",
    "b200_gemm_fp8_block",
    "b200_gemm_bf16_swiglu_supported",
    "b200_gemm_bf16_swiglu",
    "b200_gemm_bf16_splitk_bytes",
    "b200_gemm_bf16_splitk",
    "b200_gemm_mxfp8_splitk_bytes",
    "b200_gemm_mxfp8_splitk",
    "b200_gemm_fp8_block_splitk_bytes",
    "b200_gemm_fp8_block_splitk",
    "b200_add_norm_splitk_bf16",
    "b200_add_norm_splitk_mxfp8",
    "b200_add_norm_splitk_fp8_rowblock",
    "b200_activation_splitk_bf16",
    "b200_activation_splitk_mxfp8",
    "b200_activation_splitk_fp8_rowblock",
    "b200_peer_buffer_create",
    "b200_peer_buffer_open",
    "b200_peer_buffer_close",
    "b200_peer_buffer_destroy",
    "b200_allreduce_add_norm_bf16",
    "b200_allreduce_add_norm_mxfp8",
    "b200_allreduce_add_norm_fp8_rowblock",
    "b200_allreduce2_add_norm",
    "b200_allreduce2_add_norm_splitk",
    "b200_paged_attention_workspace_bytes",
    "b200_rope_append",
    "b200_paged_attention",
    "b200_paged_prefill_attention",
    "b200_fp8_value_position",
    "b200_argmax_bf16",
    "b200_argmax_shard_bf16",
    "b200_argmax_merge",
    "b200_topk_probs_bf16",
    "b200_topp_probs_bf16",
    "b200_argmax_f32",
    "b200_linear_bf16",
    "b200_linear_simt",
    "b200_out_norm",
    "b200_latent_attention_workspace_bytes",
    "b200_latent_decode_blocks",
    "b200_latent_append",
    "b200_latent_attention",
    "b200_latent_prompt_supported",
    "b200_latent_gather",
    "b200_latent_prompt_attention",
    "b200_delta_decode",
    "b200_delta_lora",
    "b200_delta_scan",
    "b200_delta_finish",
    "b200_attention_simt",
    "b200_residual_norm",
    "b200_conv_silu",
    "b200_conv_qkv",
    "b200_token_shift",
    "b200_recurrence_decode",
    "b200_recurrence_scan",
    "b200_recurrence_finish",
    "b200_recurrence_lora",
    "b200_moe_route",
    "b200_moe_gather",
    "b200_moe_up",
    "b200_moe_down",
    "b200_recurrence_gates",
    "b200_rotate_append",
    "b200_stream_norm",
    "b200_swiglu",
    "b200_conv_add",
    "b200_gated_scan",
)


class AttentionArgs(ctypes.Structure):
    """Mirror of ``b200_attention_args``."""

    _fields_ = [
        ("qkv", c_void_p),
        ("k_cache", c_void_p),
        ("v_cache", c_void_p),
        ("block_table", c_void_p),
        ("kv_seq_lengths", c_void_p),
        ("row_of_token", c_void_p),
        ("token_to_pos_ids", c_void_p),
        ("token_to_pos_in_request", c_void_p),
        ("token_to_chunk_idx", c_void_p),
        ("token_to_local_pos", c_void_p),
        ("rope_cos", c_void_p),
        ("rope_sin", c_void_p),
        ("out", c_void_p),
        ("workspace", c_void_p),
        ("workspace_bytes", c_size_t),
        ("num_tokens", c_int32),
        ("num_q_heads", c_int32),
        ("num_kv_heads", c_int32),
        ("head_dim", c_int32),
        ("chunk_size", c_int32),
        ("num_chunks", c_int32),
        ("max_chunks_per_row", c_int32),
        ("num_splits", c_int32),
        ("fuse_rope_append", c_int32),
        ("softmax_scale", c_float),
        ("kv_cache_fp8", c_int32),
        ("k_scale", c_void_p),
        ("v_scale", c_void_p),
        ("qkv_partials", c_void_p),
        ("qkv_num_splits", c_int32),
        ("row_order", c_void_p),
        ("out_q", c_void_p),
        ("out_scales", c_void_p),
        ("out_q_mode", c_int32),
        ("out_m_pad", c_int32),
        ("separate", c_int32),
        ("value_dim", c_int32),
        ("window", c_int32),
        ("pool_row_elems", c_int64),
        ("q_ld", c_int64),
        ("out_ld", c_int64),
        ("distance_bias", c_void_p),
        ("sinks", c_void_p),
        ("gate", c_void_p),
        ("gate_ld", c_int64),
        ("out_scale", c_float),
        ("softcap", c_float),
        ("lambda_", c_float),
        ("diff_scale", c_float),
        ("eps", c_float),
        ("bias_len", c_int32),
        ("keep_first", c_int32),
        ("maps", c_int32),
        ("value_gates", c_int32),
    ]


class OutNormArgs(ctypes.Structure):
    """Mirror of ``b200_out_norm_args``."""

    _fields_ = [(n, c_void_p) for n in ("partials", "table", "ids", "rows_in", "row_index", "gamma", "hidden", "y")] + [
        ("table_rows", c_int64)] + [
        (n, c_int32) for n in ("num_splits", "rows", "source_rows", "width", "accumulate", "dtype")] + [("eps", c_float)]


class LatentArgs(ctypes.Structure):
    """Mirror of ``b200_latent_args``."""

    _fields_ = [(n, c_void_p) for n in (
        "proj", "norm_weight", "rope_cos", "rope_sin", "token_to_pos", "token_to_chunk_idx", "token_to_local_pos",
        "block_table", "kv_seq_lengths", "units", "pool", "q_full", "out", "workspace")] + [
        ("workspace_bytes", c_size_t), ("proj_ld", c_int64)] + [
        (n, c_int32) for n in (
            "dkv_offset", "gate_offset", "num_tokens", "heads", "dim", "rot_dim", "rot_dims", "kv_rank", "kv_pad", "row_width",
            "num_chunks", "chunk_size", "max_chunks_per_row", "max_positions", "window", "num_units", "unit_tokens",
            "num_splits", "dtype")] + [("scale", c_float), ("eps", c_float), ("q_stride", c_int32), ("q_rot_at", c_int32)] + [
        (n, c_void_p) for n in ("cu_tokens", "cu_keys", "key_start", "key_rows", "key_values")] + [
        (n, c_int32) for n in ("num_rows", "num_keys", "max_row_tokens", "vdim")] + [
        (n, c_void_p) for n in ("sinks", "q", "q_norm_weight", "q_latent_out")] + [
        ("q_ld", c_int64)] + [(n, c_int32) for n in ("q_rank", "q_latent_offset", "value_gates")] + [("key_end", c_void_p)]


class DeltaArgs(ctypes.Structure):
    """Mirror of ``b200_delta_args``."""

    _fields_ = [(n, c_void_p) for n in (
        "proj", "z", "w2", "decay_bias", "removal_bias", "norm_weight", "state", "state_in", "state_out", "cu_tokens", "o_f32",
        "lora", "out")] + [("proj_ld", c_int64), ("state_slots", c_int64)] + [
        (n, c_int32) for n in (
            "off_r", "off_k", "off_v", "off_g", "off_a", "off_w1", "rank", "heads", "dim", "num_tokens", "num_rows",
            "dtype")] + [(n, c_float) for n in ("decay_scale", "unit_eps", "eps")]


def _fields(*groups):
    return [(name, ctype) for ctype, names in groups for name in names.split()]


class ResidualNormArgs(ctypes.Structure):
    """Mirror of ``b200_residual_norm_args``."""

    _fields_ = _fields((c_void_p, "table ids partials branch expert_rows pairs offsets shared_rows shared_gate row_index hidden")) + [
        ("gamma", c_void_p * 2), ("y", c_void_p * 2)] + _fields(
        (c_int64, "table_rows expert_row_count"), (c_int32, "num_splits rows source_rows width top experts dtype"),
        (c_float, "table_scale eps gain out_scale"), (c_void_p, "pair_weight")) + [("filter", c_void_p * 2)] + _fields(
        (c_void_p, "state state_in state_out"), (c_int64, "state_slots"), (c_int32, "taps"))


class ConvArgs(ctypes.Structure):
    """Mirror of ``b200_conv_args``."""

    _fields_ = _fields(
        (c_void_p, "proj filter state state_in state_out cu_tokens row_of_token out q_norm k_norm k_pool v_pool chunk_idx local_pos "
                   "v_first_in v_first_out mix"),
        (c_int64, "proj_ld state_slots pool_row_elems"),
        (c_int32, "channels taps num_tokens num_rows heads kv_heads dim vdim chunk_size num_chunks dtype"), (c_float, "eps"),
        (c_void_p, "filter_2 out_2"))


class ShiftArgs(ctypes.Structure):
    """Mirror of ``b200_shift_args``."""

    _fields_ = _fields((c_void_p, "x mu state state_in state_out cu_tokens row_of_token out out_last"), (c_int64, "state_slots"),
                       (c_int32, "num_tokens num_rows width mixes dtype"))


class RecurrenceArgs(ctypes.Structure):
    """Mirror of ``b200_recurrence_args``."""

    _fields_ = _fields(
        (c_void_p, "proj conv z lora w2 decay_bias decay_rate bonus norm_weight conv_filter conv_state state state_in state_out cu_tokens "
                   "o_f32 out"),
        (c_int64, "proj_ld state_slots"),
        (c_int32, "kind off_r off_k off_v off_g off_a off_b rank heads kv_heads dim vdim taps num_tokens num_rows z_splits norm_per_head "
                  "dtype"), (c_float, "unit_eps eps"), (c_void_p, "top gates below"), (c_float, "gate_cap out_scale"),
        (c_int32, "z_ld"), (c_int64, "out_ld"))


class MoeArgs(ctypes.Structure):
    """Mirror of ``b200_moe_args``."""

    _fields_ = _fields(
        (c_void_p, "x router up down shared_up shared_down counts pairs pair_weight offsets tiles num_tiles shared_gate x_sorted row_scale "
                   "inter y shared_inter shared_y"),
        (c_int32, "num_tokens width experts top ff shared_ff router_splits router_ld tile_tokens max_tiles simt dtype"),
        (c_float, "limit shared_limit alpha"), (c_int32, "plain identity groups keep_groups"), (c_void_p, "correction"),
        (c_float, "weight_scale"), (c_int32, "relu2"))


class RotateAppendArgs(ctypes.Structure):
    """Mirror of ``b200_rotate_append_args``."""

    _fields_ = _fields(
        (c_void_p, "proj q_bias k_bias v_bias rope_cos rope_sin token_to_pos chunk_idx local_pos q_out k_pool v_pool"),
        (c_int64, "proj_ld pool_row_elems"),
        (c_int32, "off_q off_k off_v q_vecs k_vecs v_vecs dim vdim rot_dims halves rms num_tokens chunk_size num_chunks max_positions dtype"),
        (c_float, "eps"), (c_void_p, "v_first_in v_first_out mix"))


class StreamNormArgs(ctypes.Structure):
    """Mirror of ``b200_stream_norm_args``."""

    _fields_ = _fields(
        (c_void_p, "table ids partials branch_bias expert_rows pairs pair_weight offsets expert_input row_index hidden mix out in_ gamma beta y"),
        (c_int64, "table_rows expert_row_count"),
        (c_int32, "num_splits rows source_rows width streams top experts identity dtype"), (c_float, "table_scale eps"))


class SwigluArgs(ctypes.Structure):
    """Mirror of ``b200_swiglu_args``."""

    _fields_ = _fields((c_void_p, "in_ out"), (c_int64, "rows"), (c_int32, "width dtype"))


class GatedScanArgs(ctypes.Structure):
    """Mirror of ``b200_gated_scan_args``."""

    _fields_ = _fields((c_void_p, "proj partials z_bias u_bias state state_in state_out cu_tokens out"), (c_int64, "proj_ld out_ld state_slots"),
                       (c_int32, "off_z off_u off_g width num_tokens num_rows num_splits dtype"))


class TpComm(ctypes.Structure):
    """Mirror of ``b200_tp_comm``."""

    _fields_ = [
        ("world_size", c_int32),
        ("rank", c_int32),
        ("max_rows", c_int32),
        ("hidden", c_int32),
        ("data", c_void_p * 8),
        ("flags", c_void_p * 8),
        ("counters", c_void_p),
    ]


class TpExchange(ctypes.Structure):
    """Mirror of ``b200_tp_exchange``."""

    _fields_ = [
        ("world_size", c_int32),
        ("rank", c_int32),
        ("max_rows", c_int32),
        ("hidden", c_int32),
        ("m_pad", c_int32),
        ("in_", c_void_p * 8),
        ("hidden_out", c_void_p * 8),
        ("normed_out", c_void_p * 8),
        ("scales_out", c_void_p * 8),
        ("flags", c_void_p * 8),
        ("counters", c_void_p),
    ]


class B200Error(RuntimeError):
    """A C-ABI entry point returned a negative code."""

    def __init__(self, fn: str, code: int, text: str):
        super().__init__(f"{fn} failed: {text} ({code})")
        self.code = code


_lib = None


def load() -> ctypes.CDLL:
    """Load (once) and type the shared library; raises if it has not been built."""
    global _lib
    if _lib is not None:
        return _lib
    if not os.path.exists(LIB_PATH):
        raise ImportError(
            f"{LIB_PATH} is missing: build it with `python -m megatron_mixtera_b200.build` "
            "(there is no CPU or PyTorch fallback for the decode kernels)"
        )
    lib = ctypes.CDLL(LIB_PATH)
    lib.b200_version.restype = c_int
    lib.b200_error_string.restype = c_char_p
    lib.b200_error_string.argtypes = [c_int]
    lib.b200_device_status.argtypes = [c_int, POINTER(c_int)]
    lib.b200_copy_rows_h2d.argtypes = [c_void_p, c_size_t, c_void_p, c_size_t, c_size_t, c_size_t, c_void_p]
    lib.b200_gather_rows_bf16.argtypes = [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int64, c_int64, c_void_p,
                                          c_void_p, c_void_p]
    lib.b200_add_norm_bf16.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int,
                                       c_int, c_float, c_void_p]
    lib.b200_activation_bf16.argtypes = [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]
    lib.b200_set_gemm_split_policy.argtypes = [c_int, c_int, c_int]
    lib.b200_set_fp8_block_cta_pairs.argtypes = [c_int]
    lib.b200_gemm_bf16_workspace_bytes.restype = c_size_t
    lib.b200_gemm_bf16_workspace_bytes.argtypes = [c_int, c_int, c_int]
    lib.b200_gemm_bf16.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_void_p, c_int64, c_int, c_int, c_int,
                                   c_void_p, c_size_t, c_void_p]
    lib.b200_gemm_bf16_swiglu_supported.argtypes = [c_int, c_int, c_int]
    lib.b200_gemm_bf16_swiglu.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_int64, c_int, c_int, c_int, c_void_p]
    lib.b200_gemm_bf16_static_scratch_limit.restype = c_size_t
    lib.b200_gemm_bf16_static_scratch_limit.argtypes = []
    lib.b200_gemm_bf16_static_scratch.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_void_p, c_int64, c_int, c_int,
                                                  c_int, c_void_p]
    lib.b200_mxfp8_scale_bytes.restype = c_size_t
    lib.b200_mxfp8_scale_bytes.argtypes = [c_int, c_int]
    lib.b200_quantize_mxfp8.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_int, c_int, c_void_p]
    lib.b200_quantize_mxfp8_weight.argtypes = [c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p]
    lib.b200_fp8_weight_bytes.restype = c_size_t
    lib.b200_fp8_weight_bytes.argtypes = [c_int, c_int]
    lib.b200_add_norm_mxfp8.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                        c_int, c_int, c_float, c_void_p]
    lib.b200_activation_mxfp8.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]
    lib.b200_gemm_mxfp8_workspace_bytes.restype = c_size_t
    lib.b200_gemm_mxfp8_workspace_bytes.argtypes = [c_int, c_int, c_int]
    lib.b200_gemm_mxfp8.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int64, c_int, c_int,
                                    c_int, c_void_p, c_size_t, c_void_p]
    lib.b200_gemm_mxfp8_swiglu.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int64,
                                           c_int, c_int, c_int, c_void_p]
    lib.b200_activation_splitk_bf16.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]
    lib.b200_activation_splitk_mxfp8.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]
    lib.b200_activation_splitk_fp8_rowblock.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                                                        c_int, c_void_p]
    lib.b200_quantize_fp8_weight_block128.argtypes = [c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p]
    lib.b200_quantize_fp8_rowblock.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]
    lib.b200_add_norm_fp8_rowblock.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                               c_void_p, c_int, c_int, c_int, c_float, c_void_p]
    lib.b200_activation_fp8_rowblock.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                                 c_void_p]
    lib.b200_gemm_fp8_block_workspace_bytes.restype = c_size_t
    lib.b200_gemm_fp8_block_workspace_bytes.argtypes = [c_int, c_int, c_int]
    lib.b200_gemm_fp8_block.argtypes = [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int64, c_int,
                                        c_int, c_int, c_void_p, c_size_t, c_void_p]
    for name in ("b200_gemm_bf16_splitk_bytes", "b200_gemm_mxfp8_splitk_bytes", "b200_gemm_fp8_block_splitk_bytes"):
        getattr(lib, name).restype = c_size_t
        getattr(lib, name).argtypes = [c_int, c_int, c_int]
    lib.b200_gemm_bf16_splitk.argtypes = [c_void_p, c_int64, c_void_p, c_int, c_int, c_int, c_void_p, c_size_t,
                                          POINTER(c_int), c_void_p]
    lib.b200_gemm_mxfp8_splitk.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_size_t,
                                           POINTER(c_int), c_void_p]
    lib.b200_gemm_fp8_block_splitk.argtypes = [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p,
                                               c_size_t, POINTER(c_int), c_void_p]
    lib.b200_add_norm_splitk_bf16.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                              c_int, c_int, c_float, c_void_p]
    lib.b200_add_norm_splitk_mxfp8.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                               c_void_p, c_int, c_int, c_float, c_void_p]
    lib.b200_add_norm_splitk_fp8_rowblock.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                                      c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_void_p]
    lib.b200_peer_buffer_create.argtypes = [c_size_t, POINTER(c_void_p), ctypes.c_char_p]
    lib.b200_peer_buffer_open.argtypes = [ctypes.c_char_p, POINTER(c_void_p)]
    lib.b200_peer_buffer_close.argtypes = [c_void_p]
    lib.b200_peer_buffer_destroy.argtypes = [c_void_p]
    lib.b200_allreduce_add_norm_bf16.argtypes = [POINTER(TpComm), c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                                 c_void_p, c_int, c_int, c_float, c_void_p]
    lib.b200_allreduce_add_norm_mxfp8.argtypes = [POINTER(TpComm), c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                                  c_void_p, c_void_p, c_int, c_int, c_float, c_void_p]
    lib.b200_allreduce_add_norm_fp8_rowblock.argtypes = [POINTER(TpComm), c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                                                         c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_void_p]
    lib.b200_allreduce2_add_norm.argtypes = [POINTER(TpExchange), c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                                             c_float, c_void_p]
    lib.b200_allreduce2_add_norm_splitk.argtypes = [POINTER(TpExchange), c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                                                    c_int, c_int, c_int, c_float, c_void_p]
    lib.b200_set_wait_limit_ns.argtypes = [ctypes.c_uint64]
    lib.b200_paged_attention_workspace_bytes.restype = c_size_t
    lib.b200_paged_attention_workspace_bytes.argtypes = [c_int, c_int, c_int, c_int]
    lib.b200_rope_append.argtypes = [POINTER(AttentionArgs), c_void_p]
    lib.b200_paged_attention.argtypes = [POINTER(AttentionArgs), c_void_p]
    lib.b200_fp8_value_position.argtypes = [c_int]
    lib.b200_paged_prefill_attention.argtypes = [POINTER(AttentionArgs), c_void_p, c_int, c_void_p]
    lib.b200_argmax_bf16.argtypes = [c_void_p, c_int64, c_void_p, c_int, c_int, c_void_p]
    lib.b200_argmax_shard_bf16.argtypes = [c_void_p, c_int64, c_void_p, c_int, c_int, c_int64, c_void_p]
    lib.b200_argmax_merge.argtypes = [c_void_p, c_int, c_int, c_void_p, c_void_p]
    lib.b200_topk_probs_bf16.argtypes = [c_void_p, c_int64, c_void_p, c_int, c_int, c_int, c_float, c_void_p]
    lib.b200_topp_probs_bf16.argtypes = [c_void_p, c_int64, c_void_p, c_int, c_int, c_float, c_float, c_void_p]
    lib.b200_argmax_f32.argtypes = [c_void_p, c_int64, c_void_p, c_int, c_int, c_void_p]
    lib.b200_linear_bf16.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_int64, c_int, c_int, c_int, c_int, c_int, c_int,
                                     c_int64, c_void_p, c_size_t, c_void_p, c_int64, c_void_p]
    lib.b200_linear_simt.argtypes = [c_void_p, c_int64, c_void_p, c_void_p, c_int64, c_int, c_int, c_int, c_int, c_int, c_int,
                                     c_int64, c_int, c_int, c_void_p, c_int64, c_void_p]
    lib.b200_out_norm.argtypes = [POINTER(OutNormArgs), c_void_p]
    lib.b200_latent_attention_workspace_bytes.restype = c_size_t
    lib.b200_latent_attention_workspace_bytes.argtypes = [c_int, c_int, c_int, c_int]
    lib.b200_latent_decode_blocks.argtypes = [c_int, c_int, c_int, c_int]
    lib.b200_latent_prompt_supported.argtypes = [c_int, c_int, c_int, c_int]
    for name in ("b200_latent_append", "b200_latent_attention", "b200_latent_gather", "b200_latent_prompt_attention"):
        getattr(lib, name).argtypes = [POINTER(LatentArgs), c_void_p]
    for name in ("b200_delta_decode", "b200_delta_lora", "b200_delta_scan", "b200_delta_finish"):
        getattr(lib, name).argtypes = [POINTER(DeltaArgs), c_void_p]
    lib.b200_attention_simt.argtypes = [POINTER(AttentionArgs), c_int, c_void_p]
    lib.b200_residual_norm.argtypes = [POINTER(ResidualNormArgs), c_void_p]
    for name in ("b200_conv_silu", "b200_conv_add", "b200_conv_qkv"):
        getattr(lib, name).argtypes = [POINTER(ConvArgs), c_void_p]
    lib.b200_token_shift.argtypes = [POINTER(ShiftArgs), c_void_p]
    for name in ("b200_recurrence_decode", "b200_recurrence_scan", "b200_recurrence_finish", "b200_recurrence_lora",
                 "b200_recurrence_gates"):
        getattr(lib, name).argtypes = [POINTER(RecurrenceArgs), c_void_p]
    for name in ("b200_moe_route", "b200_moe_gather", "b200_moe_up", "b200_moe_down"):
        getattr(lib, name).argtypes = [POINTER(MoeArgs), c_void_p]
    lib.b200_rotate_append.argtypes = [POINTER(RotateAppendArgs), c_void_p]
    lib.b200_stream_norm.argtypes = [POINTER(StreamNormArgs), c_void_p]
    lib.b200_swiglu.argtypes = [POINTER(SwigluArgs), c_void_p]
    lib.b200_gated_scan.argtypes = [POINTER(GatedScanArgs), c_void_p]
    for name in EXPORTED_SYMBOLS:
        fn = getattr(lib, name)
        if fn.restype is c_int or name.startswith("b200_") and fn.restype not in (c_char_p, c_size_t):
            fn.restype = c_int
    _lib = lib
    return lib


_torch_ops = None


def load_torch_ops():
    """Register (once) the torch custom ops of ``libb200_decode_torch.so`` and return ``torch.ops.b200_decode``.

    The front links ``libb200_decode.so``; loading the C-ABI library first with its full path makes the dynamic
    linker reuse that copy.  Raises if either library has not been built: there is no fallback."""
    global _torch_ops
    if _torch_ops is not None:
        return _torch_ops
    load()
    if not os.path.exists(TORCH_LIB_PATH):
        raise ImportError(
            f"{TORCH_LIB_PATH} is missing: build it with `python -m megatron_mixtera_b200.build` "
            "(the decode operators have no CPU or PyTorch fallback)"
        )
    import torch

    torch.ops.load_library(TORCH_LIB_PATH)
    _torch_ops = torch.ops.b200_decode
    return _torch_ops


TORCH_OPS = (
    "gather_rows", "add_norm", "activation", "quantize", "gemm", "gemm_splitk", "gemm_bf16_swiglu", "gemm_mxfp8_swiglu",
    "attention", "argmax", "argmax_shard", "argmax_merge", "filtered_probs", "allreduce_add_norm", "linear", "hybrid",
)


def check(fn_name: str, code: int) -> None:
    if code != 0:
        raise B200Error(fn_name, code, load().b200_error_string(code).decode())
