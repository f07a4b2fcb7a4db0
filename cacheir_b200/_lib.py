"""ctypes binding of libcacheir_b200.so (the C ABI declared in include/cacheir_b200.h) and of the libraries of the
ragged families: libcacheir_b200_ragged.so, _hybrid.so, _recurrence.so, _experts.so, _talking.so and _delta.so (headers of the
same names).

There is no fallback: if the shared library is missing the import of any
compute entry point raises, telling the user to build it.
"""
from __future__ import annotations

import ctypes
from ctypes import c_char_p, c_float, c_int, c_longlong, c_size_t, c_void_p
from pathlib import Path

LIB_PATH = Path(__file__).resolve().parent / "lib" / "libcacheir_b200.so"
GROUP_PATHS = {name: LIB_PATH.with_name(f"libcacheir_b200_{name}.so") for name in ("ragged", "hybrid", "recurrence", "experts", "talking", "delta")}

# name -> (restype, argtypes); mirrors include/cacheir_b200.h one to one
SIGNATURES: dict[str, tuple[object, list[object]]] = {
    "cacheir_b200_version": (c_int, []),
    "cacheir_b200_build_info": (c_char_p, []),
    "cacheir_b200_error_string": (c_char_p, [c_int]),
    "cacheir_b200_paged_attention_workspace_bytes": (c_size_t, [c_int, c_int, c_int, c_int]),
    "cacheir_b200_paged_attention_auto_splits": (c_int, [c_int] * 6),
    "cacheir_b200_paged_attention_decode_batch": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,  # q k v page_table seq_lens out
         c_int, c_int, c_int, c_int, c_int, c_int, c_int,              # batch heads kv_heads max_pages page D dtype
         c_longlong, c_longlong, c_float, c_int,                       # q_stride out_stride scale num_splits
         c_void_p, c_size_t, c_void_p]),                               # workspace bytes stream
    "cacheir_b200_paged_attention_decode_batch_ex": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
         c_int, c_int, c_int, c_int, c_int, c_int, c_int,
         c_longlong, c_longlong, c_float, c_int,
         c_void_p, c_size_t, c_int, c_int, c_void_p, c_void_p]),      # workspace bytes num_slots kv_dtype kv_scales stream
    "cacheir_b200_paged_attention_decode_batch_quantize": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
         c_int, c_int, c_int, c_int, c_int, c_int, c_int,
         c_longlong, c_float, c_int, c_void_p, c_size_t, c_void_p]),  # q_stride scale num_slots gemm_workspace bytes stream
    "cacheir_b200_paged_attention_quantize_supported": (c_int, [c_int, c_int, c_int, c_int, c_int, c_int, c_int]),
    "cacheir_b200_paged_attention_noalloc_max_workspace_bytes": (c_size_t, []),
    "cacheir_b200_paged_attention_decode_batch_noalloc": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
         c_int, c_int, c_int, c_int, c_int, c_int, c_int,
         c_longlong, c_longlong, c_float, c_int, c_void_p]),
    "cacheir_b200_qgemv": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,  # x packed scales zero_points residual y
         c_int, c_int, c_int, c_int, c_int, c_int, c_int,              # M N K bits group x_dtype scale_dtype
         c_longlong, c_int, c_void_p]),                                # x_stride epilogue stream
    "cacheir_b200_qgemv_workspace_bytes": (c_size_t, [c_int, c_int]),
    "cacheir_b200_qgemv_ex": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
         c_int, c_int, c_int, c_int, c_int, c_int, c_int,
         c_longlong, c_int, c_int, c_void_p, c_size_t, c_void_p]),
    "cacheir_b200_rmsnorm_qgemv": (
        c_int,
        [c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,   # x norm_w eps packed scales zero residual y
         c_int, c_int, c_int, c_int, c_int, c_longlong, c_int, c_int, c_void_p, c_size_t, c_void_p]),
    "cacheir_b200_qgemv_plan": (c_int, [c_int] * 8),
    "cacheir_b200_rmsnorm_qkv_rope_append": (
        c_int,
        [c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_longlong, c_int,
         c_int, c_int, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
         c_void_p, c_void_p, c_void_p, c_size_t, c_void_p]),
    "cacheir_b200_qkv_rope_append": (
        c_int,
        [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_longlong, c_int,  # x..qkv M N K scale_dtype stride layout
         c_int, c_int, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,             # q_dim k_dim hd theta table n pos table maxp page
         c_void_p, c_void_p, c_void_p, c_size_t, c_void_p]),                                             # k v ws bytes stream
    "cacheir_b200_rope_table": (c_int, [c_void_p, c_int, c_int, c_float, c_void_p]),
    "cacheir_b200_quantize_activations": (c_int, [c_void_p, c_int, c_int, c_longlong, c_int, c_void_p, c_size_t, c_void_p]),
    "cacheir_b200_rms_norm_quantize": (
        c_int, [c_void_p] * 5 + [c_int, c_int, c_float, c_int, c_void_p, c_size_t, c_void_p]),
    "cacheir_b200_pack_tiled_bytes": (c_size_t, [c_int, c_int, c_int]),
    "cacheir_b200_pack_relayout": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
    "cacheir_b200_pack_unrelayout": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
    "cacheir_b200_peer_alloc": (c_int, [c_size_t, c_void_p, c_void_p]),
    "cacheir_b200_peer_open": (c_int, [c_void_p, c_void_p]),
    "cacheir_b200_peer_close": (c_int, [c_void_p]),
    "cacheir_b200_peer_free": (c_int, [c_void_p]),
    "cacheir_b200_peer_all_reduce": (c_int, [c_void_p, c_void_p, c_void_p, c_size_t, c_int, c_int, c_int, c_void_p, c_void_p]),
    "cacheir_b200_peer_all_reduce_two_step": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_size_t, c_int, c_int, c_int, c_void_p,
                                                      c_void_p]),
    "cacheir_b200_peer_all_reduce_ll": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_size_t, c_int, c_int, c_int, c_void_p,
                                                c_void_p]),
    "cacheir_b200_peer_all_gather": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_size_t, c_int, c_int, c_int, c_void_p, c_void_p]),
    "cacheir_b200_device_status": (c_int, [c_int]),
    "cacheir_b200_pack_rows": (c_int, [c_void_p] * 5 + [c_int, c_int, c_int, c_void_p]),
    "cacheir_b200_dequantize_rows": (c_int, [c_void_p] * 4 + [c_int, c_int, c_int, c_int, c_void_p]),
    "cacheir_b200_rms_norm": (c_int, [c_void_p] * 5 + [c_int, c_int, c_float, c_int, c_void_p]),
    "cacheir_b200_rope_inplace": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_int, c_longlong, c_void_p]),
    "cacheir_b200_rope_append": (c_int, [c_void_p] * 5 + [c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int, c_longlong, c_void_p]),
    "cacheir_b200_kv_append": (
        c_int, [c_void_p] * 6 + [c_int, c_int, c_int, c_int, c_int, c_int, c_longlong, c_longlong, c_void_p]),
    "cacheir_b200_kv_append_q8": (
        c_int, [c_void_p] * 7 + [c_int, c_int, c_int, c_int, c_int, c_int, c_longlong, c_longlong, c_void_p]),
    "cacheir_b200_silu_mul": (c_int, [c_void_p, c_void_p, c_void_p, c_size_t, c_int, c_void_p]),
    "cacheir_b200_add": (c_int, [c_void_p, c_void_p, c_void_p, c_size_t, c_int, c_void_p]),
    "cacheir_b200_embedding_gather": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
    "cacheir_b200_argmax_rows": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "cacheir_b200_advance_positions": (c_int, [c_void_p, c_void_p, c_int, c_void_p]),
}


class DenseArgs(ctypes.Structure):
    """cacheir_b200_dense_args"""

    _fields_ = [("x", c_void_p), ("w", c_void_p), ("y", c_void_p),
                ("T", c_int), ("N", c_int), ("K", c_int), ("batch", c_int),
                ("w_batch_rows", c_int), ("x_batch_cols", c_int), ("y_batch_cols", c_int), ("epilogue", c_int),
                ("w_stride", c_longlong), ("x_stride", c_longlong), ("y_stride", c_longlong),
                ("act_cols", c_int), ("next_mode", c_int), ("vocab", c_int), ("table_col", c_int),
                ("gate", c_void_p), ("gate_stride", c_longlong), ("residual", c_void_p), ("norm_w", c_void_p), ("norm_b", c_void_p),
                ("next_w", c_void_p), ("next_b", c_void_p), ("next_out", c_void_p), ("norm_alpha", c_float), ("next_alpha", c_float),
                ("ids", c_void_p), ("table", c_void_p), ("table_stride", c_longlong),
                ("bias", c_void_p), ("limit", c_float), ("tail_cols", c_int), ("tail", c_void_p), ("tail_stride", c_longlong)]


class LatentArgs(ctypes.Structure):
    """cacheir_b200_latent_args"""

    _fields_ = [("positions", c_void_p), ("row_seg", c_void_p), ("cu_rows", c_void_p), ("page_table", c_void_p),
                ("rows", c_int), ("segments", c_int), ("max_pages", c_int), ("page_size", c_int), ("num_slots", c_int),
                ("heads", c_int), ("dim", c_int), ("rot_dim", c_int), ("vdim", c_int), ("kv_rank", c_int), ("window", c_int),
                ("scale", c_float), ("pool", c_void_p), ("dtype", c_int), ("decode", c_int)]


class RecurrenceArgs(ctypes.Structure):
    """cacheir_b200_recurrence_args"""

    _fields_ = [("positions", c_void_p), ("cu_rows", c_void_p), ("slots", c_void_p), ("rows", c_int), ("segments", c_int),
                ("heads", c_int), ("dim", c_int), ("vdim", c_int), ("q", c_void_p), ("k", c_void_p), ("v", c_void_p),
                ("stride", c_longlong), ("decay_pow", c_void_p), ("state", c_void_p), ("num_slots", c_int), ("out", c_void_p),
                ("dtype", c_int), ("slot_stride", c_longlong), ("log_decay", c_void_p), ("log_take", c_void_p),
                ("normaliser", c_void_p), ("q_scale", c_float), ("key_heads", c_int), ("skip", c_void_p)]


class ConvArgs(ctypes.Structure):
    """cacheir_b200_conv_args"""

    _fields_ = [("positions", c_void_p), ("cu_rows", c_void_p), ("slots", c_void_p),
                ("rows", c_int), ("segments", c_int), ("channels", c_int), ("taps", c_int), ("x", c_void_p), ("stride", c_longlong),
                ("w", c_void_p), ("bias", c_void_p), ("state", c_void_p), ("slot_stride", c_longlong), ("num_slots", c_int), ("dtype", c_int),
                ("out", c_void_p), ("out_stride", c_longlong)]


class DeltaArgs(ctypes.Structure):
    """cacheir_b200_delta_args"""

    _fields_ = [("positions", c_void_p), ("cu_rows", c_void_p), ("slots", c_void_p),
                ("rows", c_int), ("segments", c_int), ("heads", c_int), ("key_heads", c_int), ("dim", c_int), ("vdim", c_int),
                ("q", c_void_p), ("k", c_void_p), ("v", c_void_p), ("stride", c_longlong), ("z", c_void_p), ("z_stride", c_longlong),
                ("bias", c_void_p), ("log_rate", c_void_p), ("state", c_void_p), ("slot_stride", c_longlong), ("num_slots", c_int),
                ("dtype", c_int), ("out", c_void_p)]


class TalkingArgs(ctypes.Structure):
    """cacheir_b200_talking_args"""

    _fields_ = [("positions", c_void_p), ("row_seg", c_void_p), ("cu_rows", c_void_p), ("page_table", c_void_p),
                ("rows", c_int), ("segments", c_int), ("max_pages", c_int), ("page_size", c_int), ("num_slots", c_int),
                ("heads", c_int), ("kv_heads", c_int), ("dim", c_int), ("vdim", c_int), ("window", c_int), ("scale", c_float),
                ("talk", c_void_p), ("keys", c_void_p), ("values", c_void_p), ("dtype", c_int), ("decode", c_int)]


class TiedArgs(ctypes.Structure):
    """cacheir_b200_tied_args"""

    _fields_ = [("positions", c_void_p), ("row_seg", c_void_p), ("cu_rows", c_void_p), ("page_table", c_void_p),
                ("rows", c_int), ("segments", c_int), ("max_pages", c_int), ("page_size", c_int), ("num_slots", c_int),
                ("heads", c_int), ("kv_heads", c_int), ("dim", c_int), ("width", c_int), ("key_from", c_int), ("window", c_int),
                ("keep_first", c_int), ("scale", c_float), ("cap", c_float), ("reach", c_float), ("pool", c_void_p), ("inv_rms", c_void_p), ("sink", c_void_p),
                ("dtype", c_int), ("decode", c_int)]


class RouteRule(ctypes.Structure):
    """cacheir_b200_route_rule"""

    _fields_ = [("softmax", c_int), ("identity", c_int), ("groups", c_int), ("keep", c_int), ("correction", c_void_p), ("scale", c_float)]


_NEXT = [c_int, c_void_p, c_void_p, c_float, c_void_p]      # next_mode next_w next_b next_alpha next_out
# group -> signatures; each mirrors include/cacheir_b200_<group>.h one to one
GROUP_SIGNATURES: dict[str, dict[str, tuple[object, list[object]]]] = {
    "ragged": {
        "cacheir_b200_dense_supported": (c_int, [c_int, c_longlong, c_longlong, c_int, c_int]),
        "cacheir_b200_dense_gemm": (c_int, [c_void_p, c_void_p]),
        "cacheir_b200_dense_simple": (c_int, [c_void_p] * 3 + [c_int] * 7 + [c_longlong] * 3 + [c_void_p, c_int, c_int, c_void_p]),
        "cacheir_b200_scaled_embedding": (c_int, [c_void_p] * 3 + [c_int, c_int, c_int, c_float, c_int] + _NEXT + [c_int, c_void_p]),
        "cacheir_b200_dyt_rows": (c_int, [c_void_p] * 4 + [c_float, c_void_p, c_int, c_int, c_int, c_void_p]),
        "cacheir_b200_rms_rows": (c_int, [c_void_p] * 3 + [c_float, c_void_p, c_int, c_int, c_int, c_void_p]),
        "cacheir_b200_residual_dyt": (c_int, [c_void_p] * 4 + [c_float, c_int, c_int] + _NEXT + [c_int, c_void_p]),
        "cacheir_b200_layer_norm_rows": (c_int, [c_void_p] * 3 + [c_float, c_void_p, c_int, c_int, c_int, c_void_p]),
        "cacheir_b200_join_embedding": (c_int, [c_void_p] * 4 + [c_int] * 4 + [c_void_p]),
        "cacheir_b200_residual_add": (c_int, [c_void_p] * 3 + [c_int, c_int] + _NEXT + [c_int, c_void_p]),
        "cacheir_b200_residual_rms_pair": (c_int, [c_void_p] * 5 + [c_float, c_float, c_int, c_int] + _NEXT + [c_int, c_void_p]),
        "cacheir_b200_residual_rms": (c_int, [c_void_p] * 3 + [c_float, c_int, c_int] + _NEXT + [c_int, c_void_p]),
        "cacheir_b200_gated_rms": (c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_float, c_void_p, c_int, c_int, c_int, c_void_p]),
        "cacheir_b200_glu_pairs": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_int, c_void_p]),
        "cacheir_b200_gelu_embed": (c_int, [c_void_p] * 3 + [c_longlong, c_int, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
        "cacheir_b200_silu_cols": (c_int, [c_void_p, c_int, c_longlong, c_int, c_int, c_void_p]),
        "cacheir_b200_relu2_cols": (c_int, [c_void_p, c_int, c_longlong, c_int, c_int, c_void_p]),
        "cacheir_b200_gated_parts_rms": (c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_int, c_int, c_float, c_void_p, c_int, c_int, c_int,
                                                 c_int, c_void_p]),
        "cacheir_b200_ragged_device_status": (c_int, [c_int]),
    },
    "hybrid": {
        "cacheir_b200_latent_prepare": (
            c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_float, c_void_p, c_longlong, c_void_p, c_longlong, c_int, c_void_p,
                    c_int, c_int, c_void_p]),
        "cacheir_b200_latent_attention_simple": (
            c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_void_p]),
        "cacheir_b200_latent_attention_supported": (c_int, [c_int] * 4),
        "cacheir_b200_latent_attention_splits": (c_int, [c_int] * 5),
        "cacheir_b200_latent_attention": (c_int, [c_void_p] * 4 + [c_int, c_void_p]),
        "cacheir_b200_hybrid_device_status": (c_int, [c_int]),
    },
    "recurrence": {
        "cacheir_b200_recurrence_simple": (c_int, [c_void_p, c_void_p]),
        "cacheir_b200_recurrence_step": (c_int, [c_void_p, c_void_p]),
        "cacheir_b200_recurrence_chunked_supported": (c_int, [c_int] * 3),
        "cacheir_b200_recurrence_workspace_bytes": (c_size_t, [c_int] * 5),
        "cacheir_b200_recurrence_chunked": (c_int, [c_void_p, c_void_p, c_size_t, c_void_p]),
        "cacheir_b200_memory_gates": (c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_float] + [c_void_p] * 4),
        "cacheir_b200_memory_norm": (c_int, [c_void_p] * 4 + [c_longlong, c_void_p, c_float, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
        "cacheir_b200_memory_step": (
            c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_float, c_void_p, c_longlong, c_void_p, c_float, c_void_p]),
        "cacheir_b200_state_space_gates": (c_int, [c_void_p, c_void_p, c_longlong] + [c_void_p] * 5),
        "cacheir_b200_state_space_step": (c_int, [c_void_p, c_void_p, c_longlong] + [c_void_p] * 3),
        "cacheir_b200_recurrence_device_status": (c_int, [c_int]),
    },
    "talking": {
        "cacheir_b200_talking_prepare": (
            c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_longlong, c_void_p, c_longlong, c_int, c_void_p, c_int, c_float, c_int, c_void_p,
                    c_void_p]),
        "cacheir_b200_talking_simple": (c_int, [c_void_p] * 4),
        "cacheir_b200_talking_step_supported": (c_int, [c_int] * 6),
        "cacheir_b200_talking_step_splits": (c_int, [c_int] * 8),
        "cacheir_b200_talking_step": (c_int, [c_void_p] * 3 + [c_int, c_void_p]),
        "cacheir_b200_talking_prompt_supported": (c_int, [c_int] * 6),
        "cacheir_b200_talking_prompt": (c_int, [c_void_p] * 4),
        "cacheir_b200_talking_device_status": (c_int, [c_int]),
    },
    "delta": {
        "cacheir_b200_short_conv": (c_int, [c_void_p, c_void_p]),
        "cacheir_b200_delta_simple": (c_int, [c_void_p, c_void_p]),
        "cacheir_b200_delta_step": (c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_float, c_void_p]),
        "cacheir_b200_delta_chunked_supported": (c_int, [c_int] * 3),
        "cacheir_b200_delta_workspace_bytes": (c_size_t, [c_int] * 3),
        "cacheir_b200_delta_chunked": (c_int, [c_void_p, c_void_p, c_size_t, c_void_p]),
        "cacheir_b200_delta_device_status": (c_int, [c_int]),
    },
    "experts": {
        "cacheir_b200_tied_prepare": (
            c_int, [c_void_p, c_void_p, c_longlong, c_void_p, c_longlong, c_void_p, c_longlong, c_int, c_int, c_void_p, c_void_p, c_float,
                    c_void_p, c_int, c_void_p, c_void_p]),
        "cacheir_b200_tied_attention_simple": (c_int, [c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_void_p]),
        "cacheir_b200_tied_prompt_supported": (c_int, [c_int] * 7),
        "cacheir_b200_tied_attention_prompt": (c_int, [c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_void_p]),
        "cacheir_b200_tied_step_supported": (c_int, [c_int] * 7),
        "cacheir_b200_tied_step_splits": (c_int, [c_int] * 7),
        "cacheir_b200_tied_attention_step": (c_int, [c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_int, c_void_p]),
        "cacheir_b200_route": (c_int, [c_void_p, c_longlong, c_void_p, c_int, c_int, c_int] + [c_void_p] * 9 + [c_int, c_void_p]),
        "cacheir_b200_grouped_all_rows": (c_int, []),
        "cacheir_b200_grouped_gemm": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p]),
        "cacheir_b200_grouped_simple": (c_int, [c_void_p] * 5 + [c_int] * 4 + [c_longlong] * 3 + [c_int, c_void_p]),
        "cacheir_b200_combine_residual_rms": (
            c_int, [c_void_p] * 4 + [c_int, c_void_p, c_void_p, c_float, c_int, c_int, c_int, c_void_p, c_int, c_void_p]),
        "cacheir_b200_combine_residual": (
            c_int, [c_void_p] * 4 + [c_int, c_void_p, c_void_p, c_void_p, c_longlong, c_int, c_int] + _NEXT + [c_int, c_void_p]),
        "cacheir_b200_experts_device_status": (c_int, [c_int]),
    },
}
# entry points of glue.cu and misc.cu, which the core and the ragged library carry
SHARED_NAMES = ("cacheir_b200_version", "cacheir_b200_error_string", "cacheir_b200_argmax_rows", "cacheir_b200_advance_positions")

_LIB: ctypes.CDLL | None = None
_GROUPS: dict[str, ctypes.CDLL] = {}


class CacheIRB200Error(RuntimeError):
    """A C-ABI call returned a non-zero status."""


def _open(path: Path, table: dict[str, tuple[object, list[object]]], how: str) -> ctypes.CDLL:
    if not path.exists():
        raise CacheIRB200Error(f"{path} is missing: build the CUDA library first (python -m cacheir_b200.build{how}). "
                               "cacheir_b200 has no CPU or PyTorch fallback.")
    lib = ctypes.CDLL(str(path))
    for name, (restype, argtypes) in table.items():
        fn = getattr(lib, name)  # AttributeError here means header and library disagree
        fn.restype = restype
        fn.argtypes = argtypes
    return lib


def load() -> ctypes.CDLL:
    """Load the core library once and attach the prototypes. Raises if it is not built."""
    global _LIB
    if _LIB is None:
        _LIB = _open(LIB_PATH, SIGNATURES, "")
    return _LIB


def load_group(name: str) -> ctypes.CDLL:
    """A library of the ragged families, loaded once. Raises if it is not built."""
    if name not in _GROUPS:
        table = dict(GROUP_SIGNATURES[name])
        if name == "ragged":
            table.update({shared: SIGNATURES[shared] for shared in SHARED_NAMES})
        _GROUPS[name] = _open(GROUP_PATHS[name], table, f" --group {name}")
    return _GROUPS[name]


def load_shared() -> ctypes.CDLL:
    """A library that has the entry points of SHARED_NAMES: the one in use, else whichever is built."""
    if _LIB is not None:
        return _LIB
    if "ragged" in _GROUPS or (GROUP_PATHS["ragged"].exists() and not LIB_PATH.exists()):
        return load_group("ragged")
    return load()


def group_device_status(reset: bool = True) -> int:
    """First bounded wait that gave up in any loaded library of the ragged families (0: none)."""
    found = [int(getattr(lib, f"cacheir_b200_{name}_device_status")(int(reset))) for name, lib in _GROUPS.items()]
    return next((status for status in found if status != 0), 0)


def check(code: int, what: str) -> None:
    if code != 0:
        text = load_shared().cacheir_b200_error_string(int(code)).decode("utf-8", "replace")
        raise CacheIRB200Error(f"{what} failed with status {code}: {text}")
