"""ctypes binding of liblogismos_kernels.so (the C ABI declared in include/*.h)."""
from __future__ import annotations

import ctypes as C
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
_SO = os.path.join(_HERE, "liblogismos_kernels.so")

vp, i32, i64, u32, u64, f32, sz = C.c_void_p, C.c_int32, C.c_int64, C.c_uint32, C.c_uint64, C.c_float, C.c_size_t


class LogismosError(RuntimeError):
    """A launcher or runtime call returned a non-zero status (kernels::Error::Launch in the
    reference, crates/kernels/src/error.rs:30-41): carries the raw code and its classified kind."""

    def __init__(self, op: str, code: int, kind: str = "", message: str = ""):
        self.op, self.code, self.kind = op, code, kind
        super().__init__(f"{op}: {kind or 'error'} (code {code}) {message}".strip())


class NoGpuBuild(LogismosError):
    """The CUDA library is absent (Error::NoGpuBuild, crates/kernels/src/error.rs:58-64)."""


def library_path() -> str:
    return _SO


class _LStella(C.Structure):
    pass


def _declare(l, partial=False):
    sig = {
        # runtime shim
        "lg_device_count": [C.POINTER(i32)],
        "lg_device_set_current": [i32],
        "lg_device_props_get": [i32, vp],
        "lg_device_mem_info": [i32, C.POINTER(C.c_uint64), C.POINTER(C.c_uint64)],
        "lg_device_synchronize": [i32],
        "lg_malloc": [i32, sz, C.POINTER(vp)],
        "lg_free": [i32, vp],
        "lg_memset": [i32, vp, i32, sz],
        "lg_memcpy_h2d": [i32, vp, vp, sz],
        "lg_memcpy_d2h": [i32, vp, vp, sz],
        "lg_memcpy_h2d_async": [i32, vp, vp, sz, vp],
        "lg_stream_create": [i32, C.POINTER(vp)],
        "lg_stream_synchronize": [i32, vp],
        "lg_stream_destroy": [i32, vp],
        "lg_event_create": [i32, C.POINTER(vp)],
        "lg_event_record": [i32, vp, vp],
        "lg_event_synchronize": [i32, vp],
        "lg_event_elapsed_ms": [vp, vp, C.POINTER(f32)],
        "lg_event_destroy": [i32, vp],
        "lg_error_kind_from_raw": [u32],
        # reference launchers
        "logismos_launch_matmul_naive_fp16": [vp, vp, vp, i32, i32, i32, vp],
        "logismos_launch_matmul_wmma_fp16": [vp, vp, vp, i32, i32, i32, vp],
        "logismos_launch_rms_norm_fp16": [vp, vp, vp, i32, i32, f32, vp],
        "logismos_launch_softmax_fp16": [vp, vp, i32, i32, vp],
        "logismos_launch_rope_fp16": [vp, vp, i32, i32, i32, i32, vp],
        # encoder path
        "logismos_launch_embed_lookup_bf16": [vp, vp, vp, i32, i32, i32, vp],
        "logismos_launch_rms_norm_f32": [vp, vp, vp, i32, i32, f32, i32, vp],
        "logismos_launch_linear_t_bf16": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_linear_t_naive_bf16": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, vp],
        "logismos_launch_rope_halves_bf16": [vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_swiglu_bf16": [vp, vp, i32, i32, vp],
        "logismos_launch_varlen_attention_bf16": [vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, i32, vp],
        "logismos_launch_varlen_attention_tc_bf16": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_rope_varlen_attention_tc_bf16": [vp, vp, vp, vp, i32, i32, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_paged_prefix_attention_tc_bf16": [vp, i32, vp, vp, vp, vp, vp, i32, i32, vp, vp, i32, i32, i32, i32, i32, i32,
                                                           i32, i32, vp, vp],
        "logismos_launch_paged_prefix_attention_turbo3_bf16": [vp, i32, vp, vp, vp, vp, vp, i32, i32, vp, vp, i32, i32, i32, i32, i32, i32,
                                                               i32, i32, vp, vp],
        "logismos_launch_pool_head_f32": [vp, vp, vp, vp, vp, vp, i32, i32, i32, vp],
        # decode path
        "logismos_launch_gemv_int4_g32_bf16": [vp, vp, vp, vp, i32, i32, i32, vp],
        "logismos_launch_gemv_int4_g32_f32": [vp, vp, vp, vp, i32, i32, i32, vp],
        "logismos_launch_skinny_int4_g32_bf16": [vp, vp, vp, vp, i32, i32, i32, vp, vp, vp],
        "logismos_skinny_int4_route": [i32, i32, i32],
        "logismos_launch_dequant_int4_g32_bf16": [vp, vp, vp, i32, i32, vp],
        "logismos_launch_qlinear_int4_g32_acc_f32": [vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_qlinear_int4_g32_acc_f32_static": [vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_qlinear_finish_bf16": [vp, vp, vp, i32, i32, i32, i32, i32, vp],
        "logismos_launch_paged_attention_decode_bf16": [vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32,
                                                        i32, i32, i32, i32, i32, vp],
        "logismos_launch_paged_attention_decode_noalloc_bf16": [vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32,
                                                                i32, i32, i32, i32, i32, vp],
        "logismos_launch_paged_kv_store_bf16": [vp, vp, i32, vp, vp, vp, i32, i32, i64, vp, vp],
        "logismos_launch_paged_kv_gather_bf16": [vp, vp, vp, i32, i32, i32, i32, vp, vp, vp, vp],
        "logismos_launch_paged_kv_store_turbo3": [vp, vp, i32, vp, vp, vp, i32, i32, i64, vp, vp],
        "logismos_launch_paged_kv_gather_turbo3": [vp, vp, vp, i32, i32, i32, i32, vp, vp, vp, vp],
        "logismos_launch_gather_rows_f32": [vp, vp, vp, i32, i32, i32, vp, vp],
        "logismos_launch_gdn_decode_step": [vp, vp, vp, vp, vp, vp, vp, i32, i32, f32, vp],
        "logismos_launch_gdn_prefill": [vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, f32, i32, vp],
        "logismos_launch_gdn_decode_from_acc": [vp, vp, i32, vp, vp, vp, vp, vp, vp, i32, i32, f32, vp],
        "logismos_launch_gdn_chunked": [vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, f32, vp, i32, vp],
        "logismos_launch_gdn_prepare": [vp, vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, vp],
        "logismos_launch_gated_mul_bf16": [vp, i32, vp, i32, i32, i32, i32, vp],
        "logismos_launch_greedy_argmax": [vp, i32, vp, i32, i32, vp],
        "logismos_launch_temperature_f32": [vp, i32, i32, f32, vp],
        "logismos_launch_top_k_f32": [vp, i32, i32, i32, vp],
        "logismos_launch_top_p_f32": [vp, i32, i32, f32, vp],
        "logismos_launch_min_p_f32": [vp, i32, i32, f32, vp],
        "logismos_launch_repetition_penalty_f32": [vp, i32, i32, vp, vp, i32, f32, vp],
        "logismos_launch_multinomial_f32": [vp, i32, i32, vp, vp, vp],
        # model
        "logismos_launch_quantize_int4_g32": [vp, vp, vp, i32, i32, vp],
        "lg_safetensors_open": [C.c_char_p, C.POINTER(vp)],
        "lg_safetensors_get": [vp, C.c_char_p, vp],
        "lg_stella_load": [i32, C.c_char_p, vp, C.POINTER(vp)],
        "lg_decoder_load": [i32, C.c_char_p, vp, C.POINTER(vp)],
        "lg_stella_create": [i32, vp, vp, C.POINTER(vp)],
        "lg_stella_encode_ids_batch": [vp, vp, vp, i32, i32, i32, vp],
        "lg_stella_forward_device": [vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
        "lg_stella_last_hidden": [vp, i32, vp],
        "lg_decoder_create": [i32, vp, vp, C.POINTER(vp)],
        "lg_decoder_step": [vp, vp, vp, vp, i32, vp, vp],
        "lg_decoder_replay_device": [vp, vp],
        "lg_decoder_last_hidden": [vp, i32, vp],
        "lg_decoder_last_logits": [vp, i32, vp],
        "logismos_launch_add_f32": [vp, vp, i64, vp],
        "logismos_launch_gdn_finish": [vp, i32, vp, vp, vp, i32, vp, vp, i32, i32, vp],
        "lg_hybrid_set_allreduce": [vp, vp, vp],
        "lg_hybrid_set_reduce_add": [vp, vp, vp],
        "lg_tp_comm_alloc": [i32, i32, u64, C.POINTER(vp), vp],
        "lg_tp_comm_open": [i32, vp, i32, i32, u64, vp, C.POINTER(vp)],
        "lg_tp_reduce_add_f32": [vp, vp, vp, u64, vp, vp],
        "lg_hybrid_create": [i32, vp, vp, C.POINTER(vp)],
        "lg_hybrid_step": [vp, vp, vp, vp, i32, vp, vp, vp],
        "lg_hybrid_replay_device": [vp, vp],
        "lg_hybrid_last_hidden": [vp, i32, vp],
        "lg_hybrid_last_logits": [vp, i32, vp],
        # latent-attention decoder
        "logismos_launch_linear_t_act_bf16": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, f32, f32, f32, vp, vp],
        "logismos_launch_linear_small_bf16": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i64, i64, i64, i32, f32, f32, f32, vp],
        "logismos_launch_linear_f32": [vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i64, i64, i64, i32, f32, f32, f32, vp],
        "logismos_launch_varlen_attention_kv_tc_bf16": [vp, i32, vp, vp, vp, vp, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, f32, vp, i32, vp, vp],
        "logismos_launch_depth_mix_f32": [vp, i64, i32, vp, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, f32, vp, vp],
        "logismos_launch_norm_conv": [vp, vp, vp, vp, vp, vp, vp, i32, vp, vp, vp, vp, vp, vp, i32, i32, i32, vp],
        "logismos_launch_depth_mix_conv_decode": [vp, i64, i32, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp, vp, vp, i32, i32, i32, f32, i32, vp],
        "logismos_launch_latent_norm_store": [vp, i32, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, f32, i64, i32, i32, vp, vp, vp],
        "logismos_launch_latent_gather_bf16": [vp, vp, i32, i32, vp, vp, vp, i32, i32, i32, i32, vp, vp],
        "logismos_launch_latent_decode_bf16": [vp, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, vp, i32, vp, i32, i32, vp, vp],
        "logismos_launch_latent_attention_f32": [vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, f32, vp, i32, vp, vp],
        "lg_latent_create": [i32, vp, vp, C.POINTER(vp)],
        "lg_latent_load": [i32, C.c_char_p, vp, C.POINTER(vp)],
        "lg_latent_step": [vp, vp, vp, vp, i32, vp, vp, vp, i32, vp],
        "lg_latent_replay_device": [vp, vp],
        "lg_latent_last_logits": [vp, i32, vp],
        "lg_latent_snapshot": [vp, i32, i32, vp],
        # state-space / parallel decoder
        "logismos_launch_linear_groups_tc_bf16": [vp, vp, vp, i32, i32, i32, i32, i32, vp, vp, vp],
        "logismos_launch_linear_groups_small_bf16": [vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_linear_small_tanh_norm": [vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, vp],
        "logismos_launch_linear_groups_finish": [vp, vp, i32, i32, i32, i32, vp, vp],
        "logismos_launch_linear_groups_f32": [vp, vp, vp, i32, i32, i32, i32, i32, vp, vp],
        "logismos_launch_post_norm": [vp, i32, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, f32, vp, vp],
        "logismos_launch_post_norm_shift_decode": [vp, i32, vp, vp, vp, vp, i32, vp, i32, vp, vp, vp, vp, i32, i32, i32, f32, vp],
        "logismos_launch_token_shift": [vp, vp, i32, vp, i32, vp, vp, vp, vp, vp, vp, i32, i32, vp],
        "logismos_launch_time_mix_step": [vp, i32, i32, vp],
        "logismos_launch_ssd_step": [vp, i32, i32, vp],
        "logismos_launch_time_mix_chunked_bf16": [vp, i32, vp],
        "logismos_launch_ssd_conv": [vp, vp, i32, i32, i32, i32, vp],
        "logismos_launch_ssd_chunked_bf16": [vp, i32, vp],
        "logismos_launch_gated_group_norm": [vp, i32, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, vp],
        "logismos_launch_ssd_segmented_bf16": [vp, i32, i32, vp, i32, vp],
        "logismos_launch_norm_gate": [vp, i32, vp, i32, vp, vp, i32, i32, i32, i32, i32, i32, f32, vp],
        "logismos_launch_head_norm_store": [vp, i32, vp, vp],
        "logismos_launch_pool_blocks": [vp, i32, vp, vp],
        "logismos_launch_attention_difference": [vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, f32, f32, f32, vp],
        "logismos_launch_gated_residual": [vp, vp, vp],
        "logismos_launch_differential_prefix_bf16": [vp, i32, vp, vp, vp, vp, vp, i32, i32, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32, vp, i32, f32, f32, f32, vp, vp],
        "logismos_launch_differential_decode_bf16": [vp, i32, vp, vp, vp, vp, vp, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32, vp, i32, f32, f32, f32, vp, vp],
        "logismos_launch_unit_qk_store": [vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, f32, f32, f32, i64, i32, vp, vp],
        "logismos_launch_bias_attention_decode_bf16": [vp, i32, vp, vp, vp, vp, vp, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32, vp, vp, vp],
        "logismos_launch_bias_attention_prefix_bf16": [vp, i32, vp, vp, vp, vp, vp, i32, i32, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32,
                                                       vp, vp, vp],
        "logismos_launch_bias_attention_f32": [vp, i32, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, vp, vp, vp],
        # norms without statistics, rotary positions, windows, mixtures of experts
        "logismos_launch_tanh_norm": [vp, i32, vp, vp, i32, vp, vp, vp, vp, i32, i32, i32, vp, vp],
        "logismos_launch_qk_norm_rotary_store": [vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, vp, vp, f32, vp, i32, i64, i32, vp, vp],
        "logismos_launch_rotary_heads": [vp, i32, vp, i32, i32, i32, i32, vp, i32, i32, vp],
        "logismos_launch_window_attention_decode_bf16": [vp, i32, vp, vp, vp, vp, vp, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32, vp, vp, vp],
        "logismos_launch_window_attention_prefix_bf16": [vp, i32, vp, vp, vp, vp, vp, i32, i32, vp, i32, vp, i32, i32, i32, i32, i32, i32, i32, i32,
                                                         vp, vp, vp],
        "logismos_launch_window_attention_f32": [vp, i32, vp, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, vp, vp, vp],
        "logismos_launch_moe_route": [vp, i32, vp],
        "logismos_launch_moe_place": [vp, vp, vp, i32, i32, vp],
        "logismos_launch_linear_experts_small_bf16": [vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, i32, f32, f32, f32, vp],
        "logismos_launch_linear_experts_f32": [vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, f32, f32, vp],
        "logismos_launch_linear_experts_tc_bf16": [vp, i32, vp, i32, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32, f32, f32, vp, vp],
        "lg_mixer_create": [i32, vp, vp, C.POINTER(vp)],
        "lg_mixer_load": [i32, C.c_char_p, vp, C.POINTER(vp)],
        "lg_mixer_step": [vp, vp, vp, vp, i32, vp, vp, vp, i32, vp],
        "lg_mixer_replay_device": [vp, vp],
        "lg_mixer_last_logits": [vp, i32, vp],
        "lg_mixer_snapshot": [vp, i32, i32, vp],
    }
    # everything that does not return a status
    other = {
        "lg_error_kind_name": ([u32], C.c_char_p),
        "lg_error_string": ([u32], C.c_char_p),
        "lg_last_error": ([], C.c_char_p),
        "logismos_paged_decode_scratch_bytes": ([i32, i32, i32], sz),
        "logismos_varlen_attention_tc_scratch_bytes": ([i32, i32, i32, i32], sz),
        "logismos_paged_prefix_attention_scratch_bytes": ([i32, i32, i32, i32], sz),
        "logismos_turbo3_row_bytes": ([i32], sz),
        "logismos_build_packing": ([vp, vp, i32, vp, i32, i32, i32, vp, vp, vp, vp], i64),
        "logismos_build_decode_chunks": ([vp, i32, i32, vp], i32),
        "logismos_pick_decode_chunk": ([vp, i32, i32, i32], i32),
        "lg_tp_comm_region_bytes": ([i32, u64], sz),
        "lg_tp_comm_destroy": ([vp, i32], None),
        "logismos_set_deterministic": ([i32], None),
        "logismos_get_deterministic": ([], i32),
        "logismos_skinny_int4_route": ([i32, i32, i32], i32),
        "logismos_gdn_chunked_scratch_bytes": ([i32, i32, i32], sz),
        "logismos_set_dependent_launch": ([i32], None),
        "logismos_get_dependent_launch": ([], i32),
        "lg_safetensors_close": ([vp], None),
        "lg_safetensors_len": ([vp], i32),
        "lg_safetensors_name": ([vp, i32], C.c_char_p),
        "lg_safetensors_data_region_start": ([vp], u64),
        "lg_stella_destroy": ([vp], None),
        "lg_decoder_destroy": ([vp], None),
        "lg_hybrid_destroy": ([vp], None),
        "lg_stella_supported_dims": ([vp, C.POINTER(i32), i32], i32),
        "lg_decoder_launches_last_step": ([vp], i32),
        "lg_decoder_device_status": ([vp], i32),
        "lg_hybrid_launches_last_step": ([vp], i32),
        "lg_hybrid_device_status": ([vp], i32),
        "lg_stella_default_dim": ([vp], i32),
        "lg_stella_max_tokens": ([vp], i32),
        "lg_stella_launches_per_forward": ([vp], i32),
        "lg_stella_device_status": ([vp], i32),
        "lg_latent_launches_last_step": ([vp], i32),
        "lg_latent_device_status": ([vp], i32),
        "lg_latent_destroy": ([vp], None),
        "lg_latent_logits_device": ([vp], vp),
        "logismos_time_mix_has_chunked": ([i32, i32], i32),
        "logismos_ssd_has_chunked": ([i32, i32], i32),
        "logismos_ssd_segments": ([i32, i32, i32, i32], i32),
        "logismos_ssd_scratch_bytes": ([i32, i32, i32, i32], sz),
        "lg_mixer_launches_last_step": ([vp], i32),
        "lg_mixer_device_status": ([vp], i32),
        "lg_mixer_destroy": ([vp], None),
        "lg_mixer_logits_device": ([vp], vp),
        "logismos_window_context": ([i32, i32, i32], i32),
        "logismos_differential_has_prompts": ([i32], i32),
        "logismos_window_view_context": ([vp, i32], i32),
        "logismos_window_view_keys": ([vp, i32, i32], i32),
        "logismos_window_keys": ([i32, i32, i32, i32], i32),
        "logismos_moe_streams": ([i32] * 7, i32),
        "logismos_moe_max_tiles": ([i32, i32, i32, i32], i32),
        "logismos_latent_gather_rows": ([i32, i32], i32),
        "logismos_pick_latent_chunk": ([vp, i32, i32], i32),
        "logismos_latent_max_chunks": ([i32], i32),
        "logismos_latent_decode_scratch_bytes": ([i32, i32, i32], sz),
    }
    for name, (args, res) in {**{n: (a, u32) for n, a in sig.items()}, **other}.items():
        fn = getattr(l, name, None)
        if fn is None:
            if partial:
                continue  # a build of one model family: the other families' entry points are not in it
            raise AttributeError(f"{_SO} lacks {name}: rebuild it with `python -m logismos_b200.build`")
        fn.argtypes = args
        fn.restype = res
    return l


class _Lazy:
    """Loads the shared library on first use; a missing library is an error, never a fallback."""

    def __init__(self):
        self._l, self._path = None, _SO

    def use(self, path: str):
        """Load this file instead of the whole library: a build of one model family (build.ensure)."""
        if self._l is not None and path != self._path:
            raise LogismosError("load", 0, "", f"{self._path} is loaded already")
        self._path = path

    def _load(self):
        if self._l is None:
            _SO = self._path
            if not os.path.exists(_SO):
                raise NoGpuBuild("load", 0, "NoGpuBuild",
                                 f"{_SO} is missing: build it with `python -m logismos_b200.build` "
                                 "(there is no CPU fallback)")
            self._l = _declare(C.CDLL(_SO), partial=_SO != library_path())
        return self._l

    def __getattr__(self, name):
        return getattr(self._load(), name)


lib = _Lazy()


def check(code: int, op: str):
    """Raise LogismosError for a non-zero launcher / runtime status."""
    if code:
        kind = lib.lg_error_kind_name(lib.lg_error_kind_from_raw(code)).decode()
        raise LogismosError(op, int(code), kind, lib.lg_error_string(code).decode())
