"""ctypes binding of libminivllm_b200.so, the C-ABI library declared in
include/minivllm_b200.h.

The library is the only compute path of this package: if it has not been built
(`python -m minivllm_b200.csrc.build`) importing an operator raises, there is
no PyTorch or CPU fallback.
"""
import ctypes
import os

import torch

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "csrc", "libminivllm_b200.so")

MV_F16, MV_BF16, MV_F32 = 0, 1, 2

_c_i64 = ctypes.c_int64
_c_int = ctypes.c_int
_c_ptr = ctypes.c_void_p
_c_f32 = ctypes.c_float

# name -> (restype, argtypes); must list every symbol of include/minivllm_b200.h
SIGNATURES = {
    "mv_last_error_string": (ctypes.c_char_p, []),
    "mv_abi_version": (_c_int, []),
    "mv_store_kvcache": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr,
                                  _c_i64, _c_i64, _c_int, _c_int, _c_int, _c_ptr]),
    "mv_paged_decode_workspace_bytes": (_c_i64, [_c_int, _c_int, _c_int, _c_int, _c_int, _c_int]),
    "mv_paged_decode": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_int,
                                 _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_i64, _c_f32,
                                 _c_ptr, _c_i64, _c_int, _c_ptr]),
    "mv_paged_decode_static_capacity": (_c_i64, []),
    "mv_paged_decode_static": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_int,
                                        _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_i64, _c_f32,
                                        _c_int, _c_ptr]),
    "mv_prefill_varlen": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_i64, _c_i64, _c_ptr, _c_int, _c_i64,
                                   _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_int, _c_ptr]),
    "mv_prefill_paged": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int,
                                  _c_i64, _c_int, _c_i64, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_int, _c_ptr]),
    "mv_build_decode_meta": (_c_int, [_c_ptr, _c_ptr, _c_int, _c_ptr, _c_i64, _c_int, _c_int, _c_ptr, _c_ptr,
                                      _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr]),
    "mv_build_prefill_meta": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_int, _c_i64, _c_ptr, _c_i64, _c_int, _c_int,
                                       _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr]),
    "mv_update_block_tables": (_c_int, [_c_ptr, _c_int, _c_ptr, _c_i64, _c_int, _c_int, _c_ptr]),
    "mv_qk_norm_rope_store": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_ptr, _c_ptr, _c_f32,
                                       _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_i64, _c_int,
                                       _c_int, _c_int, _c_int, _c_ptr]),
    "mv_argmax_rows": (_c_int, [_c_ptr, _c_i64, _c_i64, _c_i64, _c_i64, _c_ptr, _c_ptr, _c_int, _c_ptr]),
    "mv_argmax_decode": (_c_int, [_c_ptr, _c_int, _c_i64, _c_ptr, _c_ptr]),
    "mv_sample_rows": (_c_int, [_c_ptr, _c_i64, _c_i64, _c_i64, _c_i64, _c_ptr, ctypes.c_uint64, _c_ptr, _c_ptr, _c_ptr,
                                _c_int, _c_ptr]),
    "mv_philox4x32_10": (_c_int, [ctypes.c_uint64, ctypes.c_uint64, ctypes.c_uint32, ctypes.c_uint32, _c_ptr]),
    "mv_comm_handle_bytes": (_c_i64, []),
    "mv_comm_create": (_c_int, [_c_int, _c_int, _c_i64, _c_int, ctypes.POINTER(_c_ptr), _c_ptr]),
    "mv_comm_connect": (_c_int, [_c_ptr, _c_ptr]),
    "mv_comm_create_emulated": (_c_int, [_c_int, _c_i64, _c_int, ctypes.POINTER(_c_ptr)]),
    "mv_comm_destroy": (_c_int, [_c_ptr]),
    "mv_comm_reset": (_c_int, [_c_ptr]),
    "mv_comm_set_max_blocks": (_c_int, [_c_ptr, _c_int]),
    "mv_comm_input": (_c_ptr, [_c_ptr, _c_int]),
    "mv_comm_output": (_c_ptr, [_c_ptr, _c_int]),
    "mv_allreduce_residual_rmsnorm": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_f32, _c_int, _c_int, _c_ptr,
                                               _c_int, _c_ptr]),
    "mv_allreduce_residual_rmsnorm_staged": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_f32, _c_int, _c_int, _c_ptr,
                                               _c_int, _c_ptr]),
    "mv_add_rmsnorm": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_i64, _c_ptr, _c_f32, _c_i64, _c_int,
                                _c_int, _c_ptr]),
    "mv_silu_mul": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_i64, _c_int, _c_int, _c_ptr]),
    "mv_embed_norm": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_f32,
        _c_int, _c_ptr]),
    "mv_gated_residual_norm": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr,
        _c_f32, _c_i64, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_moe_residual_norm": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_ptr, _c_i64, _c_ptr,
        _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_f32, _c_i64, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_pair_residual_norm": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr,
        _c_f32, _c_i64, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_head_norm_gate": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_int, _c_int,
        _c_f32, _c_i64, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_gated_group_norm": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_int, _c_int, _c_f32,
        _c_int, _c_ptr]),
    "mv_gate_mul": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_i64, _c_int, _c_ptr, _c_i64, _c_int, _c_f32, _c_i64, _c_int, _c_int,
        _c_ptr]),
    "mv_latent_prep": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr,
        _c_ptr, _c_ptr, _c_i64, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_latent_attention_rows": (_c_int, [_c_ptr, _c_i64, _c_i64, _c_ptr, _c_i64, _c_i64, _c_ptr, _c_i64, _c_i64, _c_ptr, _c_ptr, _c_i64,
        _c_int, _c_int, _c_i64, _c_ptr, _c_int, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_int, _c_f32, _c_int,
        _c_ptr]),
    "mv_conv_silu": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_int, _c_int, _c_ptr, _c_int, _c_i64,
        _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_ptr]),
    "mv_conv_add": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_int, _c_int, _c_ptr, _c_int, _c_i64,
        _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_ptr]),
    "mv_conv_state_update": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_ptr, _c_int, _c_ptr, _c_ptr,
        _c_int, _c_int, _c_ptr]),
    "mv_ssm_scan": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_ptr, _c_ptr,
        _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_ptr]),
    "mv_moe_route": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_int,
        _c_f32, _c_ptr]),
    "mv_moe_sort_workspace_bytes": (_c_i64, [_c_i64, _c_int, _c_int]),
    "mv_moe_sort": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_ptr, _c_i64, _c_ptr]),
    "mv_gather_rows": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_int, _c_int, _c_ptr]),
    "mv_grouped_rows": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_i64, _c_int, _c_int, _c_int, _c_f32, _c_int,
        _c_ptr]),
    "mv_grouped_gemm": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_i64, _c_int, _c_int, _c_int, _c_f32, _c_ptr,
        _c_ptr]),
    "mv_latent_decode_workspace_bytes": (_c_i64, [_c_int, _c_int, _c_int, _c_int]),
    "mv_latent_decode": (_c_int, [_c_ptr, _c_i64, _c_i64, _c_ptr, _c_i64, _c_i64, _c_ptr, _c_i64, _c_i64, _c_ptr,
        _c_ptr, _c_i64, _c_int, _c_int, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_f32,
        _c_ptr, _c_i64, _c_ptr, _c_ptr]),
    "mv_latent_gather": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_i64, _c_ptr, _c_i64, _c_int, _c_int, _c_i64,
        _c_int, _c_int, _c_ptr]),
    "mv_latent_prefill": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64,
        _c_ptr, _c_ptr, _c_int, _c_i64, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_ptr, _c_ptr]),
    "mv_ssm_chunk_takes": (_c_int, [_c_int, _c_int]),
    "mv_ssm_chunk_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr,
        _c_int, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_ptr]),
    "mv_ssm_step": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_int, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr,
        _c_ptr, _c_int, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_ptr]),
    "mv_kv_norm_store": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_i64,
        _c_int, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_window_attention_rows": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_i64,
        _c_ptr, _c_int, _c_ptr, _c_ptr, _c_i64, _c_int, _c_ptr, _c_ptr, _c_i64, _c_i64, _c_int, _c_int, _c_int,
        _c_int, _c_i64, _c_f32, _c_int, _c_ptr]),
    "mv_window_decode_workspace_bytes": (_c_i64, [_c_int, _c_int, _c_int, _c_int, _c_int, _c_i64]),
    "mv_window_decode": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_i64, _c_ptr,
        _c_ptr, _c_i64, _c_int, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_int, _c_i64, _c_f32,
        _c_ptr, _c_i64, _c_ptr]),
    "mv_window_prefill_distances": (_c_int, [_c_int, _c_int]),
    "mv_window_prefill": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr,
        _c_int, _c_i64, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_i64, _c_f32, _c_ptr, _c_i64, _c_int, _c_ptr,
        _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr]),
    "mv_gla_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_f32, _c_ptr, _c_int, _c_ptr,
        _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_i64, _c_ptr, _c_f32, _c_int, _c_ptr]),
    "mv_delta_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int,
        _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_int, _c_ptr, _c_ptr, _c_i64,
        _c_ptr, _c_f32, _c_int, _c_ptr]),
    "mv_gla_chunk_workspace_bytes": (_c_i64, [_c_i64, _c_int, _c_int, _c_int, _c_int]),
    "mv_gla_chunk_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_f32, _c_ptr, _c_int,
        _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_i64, _c_ptr]),
    "mv_delta_chunk_workspace_bytes": (_c_i64, [_c_i64, _c_int, _c_int, _c_int, _c_int]),
    "mv_delta_chunk_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int,
        _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_i64, _c_ptr]),
    "mv_qkv_rope_store": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int,
        _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_i64, _c_int, _c_int, _c_int, _c_int,
        _c_int, _c_f32, _c_int, _c_ptr]),
        "mv_mlstm_gates": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_f32, _c_ptr, _c_int, _c_ptr, _c_ptr,
        _c_ptr, _c_int, _c_int, _c_int, _c_ptr]),
        "mv_mlstm_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_int,
        _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
        "mv_mlstm_chunk_workspace_bytes": (_c_i64, [_c_i64, _c_int, _c_int, _c_int, _c_int]),
        "mv_mlstm_chunk_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr,
        _c_int, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_i64,
        _c_ptr]),
        "mv_mlstm_step": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_int, _c_ptr,
        _c_ptr, _c_f32, _c_int, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_f32,
        _c_ptr, _c_i64, _c_ptr, _c_f32, _c_int, _c_ptr]),
    "mv_stream_step": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr,
        _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_i64, _c_i64, _c_int, _c_int,
        _c_f32, _c_int, _c_ptr]),
    "mv_talk_decode_workspace_bytes": (_c_i64, [_c_int, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_i64]),
    "mv_talk_decode": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_i64,
        _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_f32, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_f32, _c_ptr,
        _c_i64, _c_ptr]),
    "mv_talk_prefill_takes": (_c_int, [_c_int, _c_int, _c_f32]),
    "mv_talk_prefill": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_int,
        _c_i64, _c_i64, _c_ptr, _c_ptr, _c_f32, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr, _c_ptr]),
    "mv_talk_attention_rows": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_i64,
        _c_ptr, _c_int, _c_ptr, _c_ptr, _c_ptr, _c_f32, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_int,
        _c_ptr]),
    "mv_head_mix": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_int, _c_ptr, _c_f32, _c_i64, _c_int, _c_int, _c_int, _c_int,
        _c_ptr]),
    "mv_diff_decode_workspace_bytes": (_c_i64, [_c_int, _c_int, _c_int, _c_int, _c_int, _c_i64]),
    "mv_diff_decode": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_i64, _c_ptr,
        _c_i64, _c_ptr, _c_i64, _c_f32, _c_f32, _c_f32, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_ptr,
        _c_i64, _c_ptr]),
    "mv_diff_prefill_takes": (_c_int, [_c_int, _c_int]),
    "mv_diff_prefill": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_int,
        _c_i64, _c_i64, _c_i64, _c_ptr, _c_i64, _c_f32, _c_f32, _c_f32, _c_int, _c_int, _c_int, _c_int, _c_f32,
        _c_ptr, _c_ptr]),
    "mv_diff_attention_rows": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_i64, _c_int, _c_int, _c_i64,
        _c_ptr, _c_int, _c_ptr, _c_i64, _c_i64, _c_int, _c_int, _c_int, _c_int, _c_f32, _c_int, _c_ptr]),
    "mv_diff_norm_gate": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_i64, _c_f32, _c_f32, _c_f32, _c_i64, _c_int, _c_int,
        _c_int, _c_ptr]),
    "mv_time_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr,
        _c_int, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_ptr, _c_i64, _c_ptr, _c_f32, _c_f32,
        _c_int, _c_ptr]),
    "mv_time_chunk_scan": (_c_int, [_c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_i64, _c_ptr, _c_ptr,
        _c_ptr, _c_int, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_int, _c_int, _c_int, _c_ptr, _c_i64, _c_ptr]),
    "mv_tanh_step": (_c_int, [_c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr, _c_ptr, _c_ptr, _c_i64, _c_ptr,
        _c_ptr, _c_int, _c_f32, _c_ptr, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_ptr, _c_ptr, _c_ptr, _c_int, _c_ptr,
        _c_int, _c_i64, _c_int, _c_int, _c_ptr]),
    "mv_xielu": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_f32, _c_f32, _c_i64, _c_int, _c_int, _c_ptr]),
    "mv_tanh_rows": (_c_int, [_c_ptr, _c_ptr, _c_i64, _c_i64, _c_int, _c_int, _c_ptr]),
}

_lib = None
_lib_path = LIB_PATH


def use_library(path):
    """Selects the library to load: one that holds the kernels of a single model family (csrc/build.py)."""
    global _lib, _lib_path
    if path != _lib_path:
        _lib, _lib_path = None, path


def lib():
    """Loads the shared library once; raises if it is missing."""
    global _lib
    if _lib is None:
        if not os.path.exists(_lib_path):
            raise RuntimeError(
                f"{_lib_path} is missing: build it with `python -m minivllm_b200.csrc.build` "
                "(this package has no fallback path)")
        handle = ctypes.CDLL(_lib_path)
        for name, (restype, argtypes) in SIGNATURES.items():
            if _lib_path != LIB_PATH and not hasattr(handle, name):
                continue             # another family's kernel
            fn = getattr(handle, name)
            fn.restype = restype
            fn.argtypes = argtypes
        _lib = handle
    return _lib


def check(status, exc=RuntimeError):
    """Turns a non-zero mv_status into a Python exception carrying the library's message."""
    if status != 0:
        msg = lib().mv_last_error_string().decode()
        # shape / dtype / null problems are argument errors, as in the reference's asserts
        if status in (1, 2, 3, 5, 7):
            raise ValueError(f"minivllm_b200 status {status}: {msg}")
        raise exc(f"minivllm_b200 status {status}: {msg}")


def dtype_code(dt):
    if dt == torch.float16:
        return MV_F16
    if dt == torch.bfloat16:
        return MV_BF16
    raise ValueError(f"minivllm_b200 kernels take float16 or bfloat16 tensors, got {dt}")


def layer_dtype_code(dt):
    """Element type of the operators that run in bf16 or in 32-bit."""
    if dt == torch.bfloat16:
        return MV_BF16
    if dt == torch.float32:
        return MV_F32
    raise ValueError(f"this operator takes bfloat16 or float32 tensors, got {dt}")


def logits_dtype_code(dt):
    return MV_F32 if dt == torch.float32 else dtype_code(dt)


def stream_ptr():
    return torch.cuda.current_stream().cuda_stream


def require_cuda(*tensors):
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise RuntimeError("minivllm_b200 operators run on CUDA tensors only (no CPU path)")
