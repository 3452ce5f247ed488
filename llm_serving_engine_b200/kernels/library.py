"""Loads the compiled CUDA libraries and declares their C entry points.

Every CUDA source is a library of its own, built and loaded when one of its entry points is first used; a model
names the sources of its parts when it is built (:func:`require`), so that they compile side by side and those of other
models not at all.  There is no fallback: if a library cannot be built or loaded, or a launch reports an error, an
exception is raised.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import c_float, c_int, c_longlong, c_uint, c_void_p

from ..csrc import build

_lib = None

_SIGNATURES = {
    "lse_moe_route_groups": [c_void_p, c_int, c_longlong, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
                             c_void_p, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int, c_void_p],
    "lse_head_norm_pair_rope_kv_write": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_void_p, c_void_p,
                                         c_float, c_void_p, c_void_p, c_void_p, c_float, c_int, c_void_p, c_void_p,
                                         c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                         c_void_p, c_void_p, c_void_p, c_void_p, c_void_p],
    "lse_gate_heads": [c_void_p, c_void_p, c_longlong, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_latent_front": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int, c_int, c_int, c_void_p,
                         c_float, c_int, c_int, c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int,
                         c_void_p, c_int, c_int, c_int, c_void_p, c_int, c_int, c_void_p],
    "lse_layer_norm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_void_p, c_float, c_int,
                       c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_void_p],
    "lse_embedding_hidden": [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_float,
                             c_void_p],
    "lse_embedding": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_embedding_copies": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p],
    "lse_streams_update_rmsnorm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_float, c_void_p, c_void_p,
                                   c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_float, c_int,
                                   c_int, c_void_p],
    "lse_gated_act_mul": [c_void_p, c_int, c_int, c_longlong, c_void_p, c_int, c_int, c_int, c_int, c_void_p],
    "lse_linear_attention_scan": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int, c_void_p,
                                  c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
                                  c_int, c_void_p, c_int, c_void_p],
    "lse_gated_rmsnorm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_void_p, c_int,
                          c_int, c_int, c_float, c_void_p, c_void_p],
    "lse_latent_prepare": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_void_p, c_void_p, c_int,
                           c_int, c_void_p, c_int, c_int, c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_int,
                           c_int, c_int, c_void_p, c_float, c_int, c_int, c_int, c_void_p],
    "lse_latent_query": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int, c_int, c_int, c_void_p,
                         c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p],
    "lse_latent_attention_chunk": [],
    "lse_latent_attention": [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
                             c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int, c_void_p, c_int,
                             c_void_p],
    "lse_latent_attention_merge": [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                   c_int, c_int, c_int, c_void_p],
    "lse_latent_attention_mma_supported": [c_int, c_int],
    "lse_latent_attention_mma": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int,
                                 c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_void_p, c_int, c_int,
                                 c_void_p],
    "lse_head_gemm": [c_void_p, c_int, c_longlong, c_longlong, c_void_p, c_int, c_longlong, c_longlong, c_longlong,
                      c_void_p, c_int, c_longlong, c_longlong, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p],
    "lse_add_rmsnorm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_int, c_void_p, c_int,
                        c_int, c_float, c_int, c_int, c_void_p],
    "lse_rope_kv_write": [c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                          c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_longlong, c_int, c_void_p],
    "lse_silu_mul": [c_void_p, c_int, c_int, c_longlong, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_gemm_bf16_skinny": [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p],
    "lse_gemm_bf16_skinny_pad": [c_int],
    "lse_gemm_bf16_skinny_splits": [c_int, c_int],
    "lse_gemm_bf16_skinny_test_hooks": [c_uint, c_int],
    "lse_gemm_bf16_skinny_status": [],
    "lse_gemm_bf16_skinny_status_async": [c_void_p, c_void_p],
    "lse_gemm_bf16_skinny_status_reset": [],
    "lse_attention_tc_status_async": [c_void_p, c_void_p],
    "lse_attention_tc_status_reset": [],
    "lse_gemm_f32_nt": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_longlong,
                        c_longlong, c_longlong, c_int, c_longlong, c_void_p],
    "lse_gemm_f32_ranges": [c_int],
    "lse_gemm_f32_stack_ok": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_longlong],
    "lse_paged_attention_generic": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                    c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_float,
                                    c_int, c_int, c_int, c_void_p, c_int, c_void_p],
    "lse_attention_generic_chunk": [],
    "lse_paged_attention_decode": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                   c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int,
                                   c_void_p, c_void_p, c_void_p],
    "lse_paged_attention_prefill": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                    c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int, c_void_p],
    "lse_attention_mma_supported": [c_int, c_int, c_int],
    "lse_paged_attention_prefill_tc": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                       c_int, c_int, c_longlong, c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_void_p,
                                       c_void_p, c_longlong, c_void_p],
    "lse_attention_tc_scratch_floats": [],
    "lse_attention_tc_supported": [c_int, c_int, c_int, c_int],
    "lse_attention_tc_status": [],
    "lse_set_pdl": [c_int],
    "lse_embedding_positions": [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_int,
                                c_int, c_int, c_int, c_void_p],
    "lse_scaled_add_rmsnorm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_float, c_void_p,
                               c_void_p, c_int, c_int, c_int, c_float, c_void_p],
    "lse_head_norm_kv_write": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_void_p, c_void_p, c_float,
                               c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                               c_int, c_void_p],
    "lse_softcap": [c_void_p, c_longlong, c_float, c_void_p],
    "lse_moe_route": [c_void_p, c_int, c_longlong, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int,
                      c_int, c_int, c_int, c_void_p],
    "lse_moe_gated_act": [c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                          c_int, c_float, c_float, c_void_p, c_void_p],
    "lse_moe_group_rows": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_moe_gather_rows": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_moe_combine": [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                        c_int, c_int, c_void_p],
    "lse_attention_scored_chunk": [],
    "lse_attention_scored": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p, c_int, c_void_p, c_void_p,
                             c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float,
                             c_int, c_int, c_void_p, c_int, c_void_p],
    "lse_attention_scored_merge": [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                   c_int, c_int, c_void_p],
    "lse_attention_scored_mma_supported": [c_int, c_int, c_int, c_int],
    "lse_attention_scored_mma": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_int,
                                 c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float,
                                 c_int, c_void_p, c_int, c_void_p],
    "lse_head_mix_gate": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_void_p,
                          c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p],
    "lse_head_mix_gate_stages": [c_int, c_int, c_int],
    "lse_attention_scored_tc": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
                                c_longlong, c_int, c_int, c_int, c_int, c_float, c_void_p, c_void_p, c_void_p, c_int,
                                c_void_p, c_void_p, c_longlong, c_void_p, c_void_p],
    "lse_embedding_scaled": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_float, c_void_p],
    "lse_tanh_norm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                      c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_gated_linear_attention_scan": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int, c_void_p,
                                        c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                                        c_int, c_int, c_int, c_void_p, c_int, c_void_p],
    "lse_mlstm_gates": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_void_p, c_void_p, c_float,
                        c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_mlstm_readout": [c_void_p, c_void_p, c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_void_p,
                          c_int, c_int, c_int, c_int, c_float, c_void_p, c_void_p],
    "lse_short_conv_act": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                           c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p],
    "lse_short_conv_state": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_void_p, c_void_p, c_int,
                             c_int, c_int, c_int, c_void_p],
    "lse_conv_qk_norm_rope": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_void_p, c_void_p, c_void_p,
                              c_void_p, c_float, c_void_p, c_float, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                              c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int,
                              c_int, c_int, c_int, c_int, c_int, c_void_p],
    "lse_head_gate_scale": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_longlong, c_int, c_int, c_int, c_float,
                            c_void_p, c_void_p],
    "lse_ssm_step_sizes": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_void_p, c_void_p, c_int, c_int,
                           c_int, c_void_p],
    "lse_selective_scan": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p,
                           c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                           c_void_p, c_void_p, c_int, c_longlong, c_float, c_int, c_int, c_int, c_int, c_int, c_void_p,
                           c_void_p, c_int, c_void_p],
    "lse_moe_route_biased": [c_void_p, c_int, c_longlong, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                             c_int, c_int, c_int, c_int, c_void_p, c_int, c_void_p],
    "lse_moe_gated_act_kind": [c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                               c_int, c_int, c_float, c_float, c_void_p, c_int, c_void_p],
    "lse_gated_act_mul_limit": [c_void_p, c_int, c_int, c_longlong, c_void_p, c_int, c_int, c_int, c_int, c_float, c_void_p],
    "lse_head_norm_rope_kv_write": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_void_p, c_void_p, c_float,
                                    c_void_p, c_void_p, c_void_p, c_float, c_int, c_void_p, c_void_p, c_void_p, c_int,
                                    c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_int, c_void_p],
    "lse_conv_norm_supported": [c_int, c_int],
    "lse_conv_norm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_float, c_void_p, c_float, c_void_p,
                      c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int,
                      c_int, c_void_p],
    "lse_delta_norm_rmsnorm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_float, c_void_p, c_float,
                               c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_void_p],
    "lse_residual_settle": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_token_gate": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_longlong, c_int, c_void_p, c_int, c_void_p,
                       c_int, c_int, c_int, c_int, c_void_p],
    "lse_embedding_add": [c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_void_p],
    "lse_delta_prepare": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                          c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                          c_int, c_int, c_float, c_int, c_int, c_int, c_void_p],
    "lse_delta_scan": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_longlong, c_longlong, c_void_p, c_void_p,
                       c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p],
    "lse_delta_chunk_rows": [],
    "lse_delta_chunk_floats": [c_int, c_int],
    "lse_delta_chunk_scan": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_longlong, c_longlong, c_void_p, c_void_p,
                             c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                             c_int, c_void_p],
    "lse_attention_scored_windowed": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p, c_int, c_void_p,
                                      c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
                                      c_int, c_float, c_int, c_int, c_void_p, c_int, c_int, c_int, c_float, c_void_p,
                                      c_void_p, c_void_p],
    "lse_gated_linear_attention_scan_shared": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int,
                                               c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int,
                                               c_int, c_int, c_int, c_int, c_int, c_void_p, c_int, c_int, c_int, c_void_p],
    "lse_vector_decay_attention_scan": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int, c_void_p,
                                        c_float, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                        c_int, c_void_p, c_int, c_void_p, c_void_p],
    "lse_ssd_gates": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                      c_int, c_int, c_void_p],
    "lse_sigmoid_power": [c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_float, c_void_p, c_int, c_int,
                          c_void_p],
    "lse_gated_group_rmsnorm": [c_void_p, c_void_p, c_int, c_int, c_longlong, c_longlong, c_int, c_void_p, c_longlong,
                                c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_longlong, c_int, c_int, c_int,
                                c_float, c_float, c_int, c_int, c_void_p, c_void_p],
    "lse_attention_scored_mma_windowed": [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p,
                                          c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                          c_float, c_int, c_void_p, c_int, c_int, c_int, c_float, c_void_p, c_void_p, c_void_p],
    "lse_attention_scored_merge_windowed": [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                                            c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p],
    "lse_attention_sigmoid_tc": [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
                                 c_longlong, c_int, c_int, c_int, c_int, c_float, c_void_p, c_float, c_void_p, c_void_p,
                                 c_longlong, c_void_p],
    "lse_argmax": [c_void_p, c_longlong, c_int, c_int, c_void_p, c_void_p],
    "lse_sample": [c_void_p, c_longlong, c_int, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                   c_void_p, c_void_p, c_void_p],
}


class KernelError(RuntimeError):
    """A kernel launcher refused its arguments or CUDA reported an error."""


class KernelLibrary:
    """The C entry points of all kernel libraries as attributes; a source's library is built (if it is not) and
    loaded at the first use of one of its entry points."""

    def __init__(self) -> None:
        # LSE_TRACE=1: the tuning variant; LSE_CHECK=1: the checked variant (indices compared with their ranges)
        self._trace = os.environ.get("LSE_TRACE", "0") == "1"
        self._check = os.environ.get("LSE_CHECK", "0") == "1" and not self._trace
        self._source_of = {name: path.stem for path in build.sources() for name in build.exported_names(path)}
        self._loaded: dict[str, ctypes.CDLL] = {}

    @property
    def checked(self) -> bool:
        return self._check

    def check_readers(self) -> list[tuple[str, str]]:
        """(entry point, source) of every reader of a checked variant's records."""
        return sorted((name, source) for name, source in self._source_of.items() if name.startswith("lse_check_"))

    def source_loaded(self, source: str) -> bool:
        return source in self._loaded

    def require(self, sources) -> None:
        """Build (side by side) and load the libraries of these sources."""
        missing = [name for name in sources if name not in self._loaded]
        if not missing:
            return
        for name, path in build.library_paths(missing, trace=self._trace, check=self._check).items():
            self._loaded[name] = ctypes.CDLL(str(path))

    def __getattr__(self, name: str):
        source = self.__dict__.get("_source_of", {}).get(name)
        if source is None:
            raise AttributeError(f"no CUDA source defines {name!r}")
        self.require([source])
        function = getattr(self._loaded[source], name)
        if name in _SIGNATURES:
            function.argtypes = _SIGNATURES[name]
        function.restype = c_int
        setattr(self, name, function)
        return function


def load() -> KernelLibrary:
    """The kernel libraries' entry points (each library is built and loaded at its first use)."""
    global _lib
    if _lib is None:
        lib = KernelLibrary()
        if os.environ.get("LSE_PDL", "1") == "0":   # programmatic dependent launch off (for comparisons)
            lib.lse_set_pdl(0)
        _lib = lib
    return _lib


def require(sources) -> None:
    """Build and load the libraries of these CUDA sources now, side by side."""
    load().require(sorted(set(sources)))


def register_signatures(signatures: dict) -> None:
    """Declare further entry points (used by kernel files added later)."""
    _SIGNATURES.update(signatures)
    for name in signatures:
        if _lib is not None:
            _lib.__dict__.pop(name, None)


CHECK_KINDS = {1: "token id", 2: "cache slot", 3: "block-table entry", 4: "segment number", 5: "row index"}


def check_report(reset: bool = True) -> list[str]:
    """What the checked variant of the library (``LSE_CHECK=1``) has recorded: one line per source file whose
    kernels met an index outside its range (empty: none).  Synchronises the device.  Raises when the loaded
    library is not the checked variant."""
    lib = load()
    found = []
    if not lib.checked:
        raise KernelError("the loaded kernel library is not the checked variant (set LSE_CHECK=1 before the first use)")
    for name, source in lib.check_readers():
        if not lib.source_loaded(source):       # none of its kernels has run
            continue
        reader = getattr(lib, name)
        reader.argtypes = [c_void_p, c_int]
        reader.restype = c_int
        words = (c_int * 4)()
        if reader(words, int(reset)) != 0:
            raise KernelError(f"{name}: the check words could not be read")
        if words[0]:
            found.append(f"{name[len('lse_check_'):]}: {CHECK_KINDS.get(words[0], words[0])} {words[1]} outside [{words[2]}, {words[3]})")
    return found


_launch_count = 0


def launches() -> int:
    """How many kernels of this library have been launched by this process."""
    return _launch_count


def check(code: int, name: str) -> None:
    global _launch_count
    _launch_count += 1
    if code == 0:
        return
    if code == -1:
        raise KernelError(f"{name}: unsupported or inconsistent arguments")
    if code == -2:
        raise KernelError(f"{name}: size beyond what this kernel was built for")
    raise KernelError(f"{name}: CUDA error {code}")
