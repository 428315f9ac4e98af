"""Loads the CUDA kernel library and declares its C entry points.

There is no fallback: if the library cannot be built or loaded, or no CUDA
device is present, importing an op raises.
"""

from __future__ import annotations

import ctypes
import os
from collections import Counter
from ctypes import c_float, c_int, c_int64, c_void_p

import torch

from ..build import ensure_kernels


class KernelError(RuntimeError):
    """A kernel refused its arguments or the launch failed."""


_lib: ctypes.CDLL | None = None

P, I, L, F = c_void_p, c_int, c_int64, c_float

# name -> argument types (every entry point returns an int status, 0 = ok)
_SIGNATURES: dict[str, list] = {
    # (ids, table, table_dtype, out_f32, T, H, V, stream)
    "psb_embedding": [P, P, I, P, I, I, I, P],
    # (h, delta, delta_dtype, weight, rows, x, x_dtype, n_rows, H, eps, update_h, delta_scale, delta_shift, stream)
    "psb_add_rmsnorm": [P, P, I, P, P, P, I, I, I, F, I, P, P, P],
    # (a, a_dtype, w, w_dtype, c, c_dtype, M, N, K, lda, ldw, ldc, accumulate, stream)
    "psb_gemm_nt": [P, I, P, I, P, I, I, I, I, L, L, L, I, P],
    # (qkv, dtype, positions, token_item, cos, sin, table, table_width, kv, kv_dtype, q_out,
    #  T, hq, hkv, D, page_size, num_pages, max_positions, rotate, write_kv, paired, rotary_dim, interleaved, stream)
    "psb_rope_append": [P, I, P, P, P, P, P, I, P, I, P, I, I, I, I, I, I, I, I, I, I, I, I, P],
    # (h_in, pending, gain, h_out, W, M, K, eps, sms, positions, token_item, table, table_width, cos, sin, kv, q_out,
    #  hq, hkv, D, page_size, num_pages, max_positions, stream)
    "psb_gemm_stream_norm_rope": [P, P, P, P, P, I, I, F, I, P, P, P, I, P, P, P, P, I, I, I, I, I, I, P],
    # (q, dtype, kv, kv_dtype, table, table_width, positions, token_item, out, T, hq, hkv, D, page_size, window,
    #  scale, sink, stream)
    "psb_attention_generic": [P, I, P, I, P, I, P, P, P, I, I, I, I, I, I, F, P, P],
    # (gate_up, dtype, out, T, I, activation, stream)
    "psb_silu_mul": [P, I, P, I, I, I, P],
    # (h, delta, delta_dtype, total, stream)
    "psb_residual_add": [P, P, I, L, P],
    # (q, kv, table, table_width, item_start, kv_len, out, num_items, num_tiles, hq, hkv, D, page_size, window, scale,
    #  skip_single, sink, stream)
    "psb_attention_prefill_bf16": [P, P, P, I, P, P, P, I, I, I, I, I, I, I, F, I, P, P],
    # (D) -> rows per CTA
    "psb_attention_prefill_rows_per_cta": [I],
    # (D, page_size) -> 1 if the tcgen05 prefill attention takes them
    "psb_attention_prefill_tcgen05_supported": [I, I],
    # () -> rows per CTA
    "psb_attention_prefill_tcgen05_rows_per_cta": [],
    # (q, kv, table, table_width, item_start, kv_len, out, num_items, num_pairs, T, hq, hkv, D, page_size, num_pages,
    #  window, scale, skip_single, rows_per_cta, kv_splits, part_o, part_ml, token_item, sink, stream)
    "psb_attention_prefill_tcgen05": [P, P, P, I, P, P, P, I, I, I, I, I, I, I, L, I, F, I, I, I, P, P, P, P, P],
    # () -> 0 while no bounded wait of the tcgen05 attention kernel has ever run out
    "psb_attention_tcgen05_status": [],
    # (q, kv, table, table_width, item_start, kv_len, out, part_o, part_ml, num_items, hq, hkv, D, page_size, window,
    #  scale, chunk, max_splits, all_single, sink, stream)
    "psb_attention_decode_bf16": [P, P, P, I, P, P, P, P, P, I, I, I, I, I, I, F, I, I, I, P, P],
    # (hq, hkv, D, page_size) -> 1 if the TMA-fed decode attention takes the shape
    "psb_attention_decode_tma_supported": [I, I, I, I],
    # (q, kv, table, table_width, item_start, kv_len, out, part_o, part_ml, num_items, hq, hkv, D, page_size, num_pages,
    #  window, scale, chunk, max_splits, all_single, sink, stream)
    "psb_attention_decode_tma_bf16": [P, P, P, I, P, P, P, P, P, I, I, I, I, I, L, I, F, I, I, I, P, P],
    "psb_attention_decode_tma_status": [],
    # (part_o, part_ml, item_start, kv_len, out, num_items, hq, D, window, chunk, max_splits, all_single, sink, stream)
    "psb_attention_decode_merge_bf16": [P, P, P, P, P, I, I, I, I, I, I, I, P, P],
    # (x, W, y, out_dtype, M, N, K, sms, stream)
    "psb_gemm_stream": [P, P, P, I, I, I, I, I, P],
    # (x, W, act, M, I, K, sms, activation, stream)
    "psb_gemm_stream_gated": [P, P, P, I, I, I, I, I, P],
    # (M, K) -> 1 if the norm-fused streaming product takes the shape
    "psb_gemm_stream_norm_supported": [I, I],
    # (h_in, pending, gain, rows, h_out, W, y, out_dtype, M, N, K, eps, sms, stream)
    "psb_gemm_stream_norm": [P, P, P, P, P, P, P, I, I, I, I, F, I, P],
    # (h_in, pending, gain, h_out, W, act, M, I, K, eps, sms, activation, stream)
    "psb_gemm_stream_norm_gated": [P, P, P, P, P, P, I, I, I, F, I, I, P],
    # (a, w, c, M, N, K, sms, stream)
    "psb_gemm_tcgen05": [P, P, P, I, I, I, I, P],
    # (a, w, act, M, I, K, sms, activation, stream)
    "psb_gemm_tcgen05_gated": [P, P, P, I, I, I, I, I, P],
    # (a, w, act, M, I, K, sms, limit, alpha, offset, stream)
    "psb_gemm_tcgen05_gated_clipped": [P, P, P, I, I, I, I, F, F, F, P],
    # (x, W, act, M, I, K, sms, limit, alpha, offset, stream)
    "psb_gemm_stream_gated_clipped": [P, P, P, I, I, I, I, F, F, F, P],
    # (h_in, pending, gain, h_out, W, act, M, I, K, eps, sms, limit, alpha, offset, stream)
    "psb_gemm_stream_norm_gated_clipped": [P, P, P, P, P, P, I, I, I, F, I, F, F, F, P],
    "psb_gemm_tcgen05_tile_width": [I],
    # (M, N_out, kind, D, sms) -> output tiles at the width the kernel would choose
    "psb_gemm_tcgen05_tiles": [I, I, I, I, I],
    "psb_gemm_tcgen05_rope": [P, P, I, I, I, P, P, P, I, P, P, P, P, I, I, I, I, I, I, P],
    # () -> 0 while no bounded wait of the tcgen05 kernel has ever run out
    "psb_tcgen05_status": [],
    # the product for a few dozen rows (up to 64): (a, w, c, M, N, K, stream)
    "psb_gemm_fewrows": [P, P, P, I, I, I, P],
    # (a, w, act, M, I, K, activation, stream)
    "psb_gemm_fewrows_gated": [P, P, P, I, I, I, I, P],
    # (a, w, M, K, positions, token_item, table, table_width, cos, sin, kv, q_out, hq, hkv, D, page_size, num_pages, max_positions, stream)
    "psb_gemm_fewrows_rope": [P, P, I, I, P, P, P, I, P, P, P, P, I, I, I, I, I, I, P],
    # behind a norm: (..., ssq_in, ssq_parts, eps, stream)
    "psb_gemm_fewrows_scaled": [P, P, P, I, I, I, P, I, F, P],
    "psb_gemm_fewrows_gated_scaled": [P, P, P, I, I, I, I, P, I, F, P],
    "psb_gemm_fewrows_rope_scaled": [P, P, I, I, P, P, P, I, P, P, P, P, I, I, I, I, I, I, P, I, F, P],
    # in front of a norm: (a, w, stream float32 in/out, gain, gained bf16 out, ssq_out, M, N, K, stream)
    "psb_gemm_fewrows_add_norm": [P, P, P, P, P, P, I, I, I, P],
    "psb_gemm_fewrows_splits": [I],
    "psb_gemm_fewrows_status": [],
    # (logits, temperature, seed, position, out, scratch, S, V, stream)
    "psb_sample": [P, P, P, P, P, P, I, I, P],
    # (logits, records, row_slot, record_words, out, scratch, S, V, stream)
    "psb_sample_slots": [P, P, P, I, P, P, I, I, P],
    # (resident, pairs, n, limit, stream)
    "psb_scatter_words": [P, P, I, I, P],
    # (records, record_words, kv_len, slots, rows, row_width, out, width, num_items, num_slots, stream)
    "psb_step_prepare": [P, I, P, P, P, I, P, I, I, I, P],
    # (limit, who, out int32[3], stream)
    "psb_selftest_bounded_wait": [I, I, P, P],
    # (bytes, void** out) / (pointer)
    "psb_pool_alloc": [L, ctypes.POINTER(c_void_p)],
    "psb_pool_free": [P],
    # (S, V) -> bytes of scratch psb_sample wants
    "psb_sample_scratch_bytes": [I, I],
    # (a, a_dtype, w, w_dtype, c, c_dtype, M, N, K, lda, ldw, ldc, batch, batch_a, batch_w, batch_c, stream)
    "psb_gemm_nt_batched": [P, I, P, I, P, I, I, I, I, L, L, L, I, L, L, L, P],
    # (ids, positions, token_item, item_start, slots, last_token, table, pair_table, table_dtype, out_f32, copy, copy_dtype,
    #  T, items, H, V, buckets, mul_prev, mul_cur, num_slots, stream)
    "psb_hashed_embedding": [P, P, P, P, P, P, P, P, I, P, P, I, I, I, I, I, I, L, L, I, P],
    # (h, y, y_dtype, g, g_dtype, bias, gain, copy, copy_dtype, rows, H, eps, mult, stream)
    "psb_gated_norm_add": [P, P, I, P, I, P, P, P, I, I, I, F, F, P],
    # (x, dtype, out, total, cols, ldo, code, params, stream)
    "psb_unary_act": [P, I, P, L, L, L, I, P, P],
    # (x, x_dtype, gate_f32, out, out_dtype, total, stream)
    "psb_gate_mul": [P, I, P, P, I, L, P],
    # (proj, dtype, positions, token_item, table, table_width, cos, sin, gain_q, gain_kv, cq_out, gate_out, cache, cache_dtype,
    #  T, q_rank, rank, rot, rot_dims, heads, page_size, num_pages, max_positions, eps, stream)
    "psb_latent_prepare": [P, I, P, P, P, I, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, F, L, P],
    # (q, dtype, positions, cos, sin, q_lat, T, heads, plain, rot, rot_dims, rank, max_positions, stream)
    "psb_latent_query_rotate": [P, I, P, P, P, P, I, I, I, I, I, I, I, L, P],
    # (q_lat, cache, cache_dtype, table, table_width, positions, token_item, gate, out, out_dtype, T, heads, rank, rot,
    #  page_size, num_pages, window, scale, heads_per_block, splits, partial, stream)
    "psb_latent_attention": [P, P, I, P, I, P, P, P, P, I, I, I, I, I, I, I, I, F, I, I, P, P, P],
    # (cache_dtype, rank, rot) -> 1 if the kernel that reads rows side by side takes the case
    "psb_latent_attention_rows_supported": [I, I, I],
    "psb_latent_attention_max_rank": [],
    # (cache, dtype, table, table_width, positions, token_item, band, values2, t0, n, KP, D, rank, page_size, num_pages, window, stream)
    "psb_latent_band_gather": [P, I, P, I, P, P, P, P, I, I, I, I, I, I, I, I, P],
    # (x float32, hi, lo, total, stream)
    "psb_split_pairs": [P, P, P, L, P],
    # (scores, positions, weights [rows, 2 KP], t0, n, heads, KP, window, scale, stream)
    "psb_latent_band_softmax": [P, P, P, I, I, I, I, I, F, P, P],
    # (o, gate, out, out_dtype, rank, total, stream)
    "psb_latent_band_finish": [P, P, P, I, I, L, P],
    # (proj, dtype, bias_x, conv_w, conv_b, state, positions, token_item, item_start, slots, u_out, T, W, K, num_slots, stream)
    "psb_causal_conv": [P, I, P, P, P, P, P, P, P, P, P, I, I, I, I, P],
    # (proj, u, dtype, gates, bias_y, bias_x, bias_r, bias_i, lam, state, item_start, slots, carry, out, items, T, W, K, blocks,
    #  num_slots, chunk, decay, stream)
    "psb_recurrence_scan": [P, P, I, P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, P],
    "psb_recurrence_max_taps": [],
    # (ids, positions, table, pos_table, table_dtype, out_f32, T, H, V, P, scale, stream)
    "psb_embedding_pos": [P, P, P, P, I, P, I, I, I, I, F, P],
    # (h, y, y_dtype, gain_post, gain_pre, rows, x, x_dtype, n_rows, H, eps_post, eps_pre, stream)
    "psb_norm_add_norm": [P, P, I, P, P, P, P, I, I, I, F, F, P],
    # (qkv, dtype, positions, token_item, table, table_width, kv, kv_dtype, q_out, T, hq, hkv, dim, vdim, page_size, num_pages, stream)
    "psb_attention_biased_append": [P, I, P, P, P, I, P, I, P, I, I, I, I, I, I, I, P],
    # (q, dtype, kv, kv_dtype, table, table_width, positions, token_item, bias, sink, out, T, hq, hkv, dim, vdim, page_size,
    #  window, chunk, reach, scale, item_start, skip_from, stream)
    "psb_attention_biased": [P, I, P, I, P, I, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, P, I, I, P, I, P, L, L, F, F, P],
    # (q, kv, table, table_width, positions, token_item, bias, sink, out, T, hq, hkv, dim, vdim, page_size, window, chunk, reach, scale,
    #  keep_first, partial, splits, gate, ldg, ldo, out_scale, softcap, stream)
    "psb_attention_rows_single": [P, P, P, I, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, I, P, L, L, F, F, P],
    "psb_attention_rows_single_supported": [I, I, I, I],
    "psb_attention_biased_tile_tokens": [],
    "psb_attention_biased_tile_supported": [I, I, I, I],
    # (q, kv, table, table_width, positions, item_start, items, T, min_tokens, bias, sink, out, hq, hkv, dim, vdim,
    #  page_size, window, chunk, reach, scale, stream)
    "psb_attention_biased_tiles": [P, P, P, I, P, P, I, I, I, P, P, P, I, I, I, I, I, I, I, I, F, I, P, L, L, F, F, P],
    "psb_attention_biased_mma_supported": [I, I, I, I],
    "psb_attention_biased_mma": [P, P, P, I, P, P, I, I, I, P, P, P, I, I, I, I, I, I, I, I, F, I, P, L, L, F, F, P],
    "psb_delta_max_taps": [],
    # (proj, dtype, ld, beta_at, ba, decay, taps, a_log, dt_bias, state, positions, token_item, item_start, slots, qkv_out, bd_out, T,
    #  G, H, dim, vdim, K, num_slots, slot_floats, stream)
    "psb_delta_prepare": [P, I, L, I, P, P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, L, P],
    # (qkv, bd, decay, proj, dtype, ld, state, item_start, slots, o_out, items, G, H, dim, vdim, K, num_slots, slot_floats, lanes, stream)
    "psb_channel_delta_rule": [P, P, P, P, I, L, P, P, P, P, I, I, I, I, I, I, I, L, I, P],
    # (qkv, bd, proj, dtype, state, item_start, slots, o_out, items, G, H, dim, vdim, K, num_slots, slot_floats, lanes, stream)
    "psb_delta_rule": [P, P, P, I, P, P, P, P, I, I, I, I, I, I, I, L, I, P],
    # (dim, vdim) -> float32 numbers of a chunk's record, 0 if the chunked form does not take the sizes
    "psb_channel_delta_record": [I, I],
    # (qkv, bd, decay, proj, dtype, ld, state, item_start, slots, records, o_out, items, chunks, G, H, dim, vdim, K, num_slots,
    #  slot_floats, stream)
    "psb_channel_delta_chunks": [P, P, P, P, I, L, P, P, P, P, P, I, I, I, I, I, I, I, I, L, P],
    # (o, proj, dtype, gain, out, T, G, H, dim, vdim, eps, stream)
    "psb_delta_finish": [P, P, I, P, P, I, I, I, I, I, F, P],
    # (z, ldz, correction, chosen, weight, T, E, top, groups, keep, scale, stream)
    "psb_moe_route": [P, I, P, P, P, I, I, I, I, I, F, I, I, I, P],
    # (chosen, offsets, row_pair, pair_row, tile_expert, pairs, E, pad, rows_room, weight, row_weight, stream)
    "psb_moe_group": [P, P, P, P, P, I, I, I, I, P, P, P],
    # (x, row_pair, out, rows, K, top, stream)
    "psb_moe_gather": [P, P, P, I, I, I, P],
    # (a, w, c, M, N, K, experts, tile_expert, relu2, sms, stream)
    "psb_gemm_tcgen05_grouped": [P, P, P, I, I, I, I, P, I, I, P],
    # (a, w, act, M, I, K, experts, tile_expert, limit, alpha, offset, sms, stream)
    "psb_gemm_tcgen05_grouped_gated_clipped": [P, P, P, I, I, I, I, P, F, F, F, I, P],
    # (a, w, act, M, I, K, experts, tile_expert, row_weight, sms, stream)
    "psb_gemm_tcgen05_grouped_gated_silu": [P, P, P, I, I, I, I, P, P, I, P],
    # (a, a_dtype, w, w_dtype, c, c_dtype, offsets, row_pair, pairs, E, N, K, top, gather, act, glu, limit, alpha, offset, row_weight, stream)
    "psb_moe_gemm": [P, I, P, I, P, I, P, P, I, I, I, I, I, I, I, I, F, F, F, P, P],
    # (y, y_dtype, pair_row, weight, shared, shared_dtype, gate, ldg, out, out_dtype, T, H, top, stream)
    "psb_moe_combine": [P, I, P, P, P, I, P, I, P, I, I, I, I, P],
    # (x, dtype, mix, state, stride, positions, token_item, item_start, slots, y, T, W, num_slots, stream)
    "psb_token_shift": [P, I, P, P, L, P, P, P, P, P, I, I, I, P],
    # (h, delta, delta_dtype, gain, eps, mix, state, stride, positions, token_item, slots, y, y_dtype, T, W, num_slots, stream)
    "psb_add_rmsnorm_shift": [P, P, I, P, F, P, P, L, P, P, P, P, I, I, I, I, P],
    # (a, b, dtype, gain_a, gain_b, out_f32, T, W, eps, weight, stream)
    "psb_normed_pair_sum": [P, P, I, P, P, P, I, I, F, F, P],
    # (proj, ld, dtype, positions, token_item, table, table_width, cos, sin, head_factor, kv, kv_dtype, q_out, T, hq, hkv, dim, vdim,
    #  page_size, num_pages, max_positions, rotary_dim, interleaved, eps, values_are_keys, split_planes, stream)
    "psb_attention_prepare": [P, L, I, P, P, P, I, P, P, P, P, I, P, I, I, I, I, I, I, I, I, I, I, F, I, I, P, I, P],
    # (proj, ld, dtype, bias_z, bias_x, state, stride, item_start, slots, carry, start, out, items, T, W, num_slots, chunk,
    #  two_pass, stream)
    "psb_min_gru": [P, L, I, P, P, P, L, P, P, P, P, P, I, I, I, I, I, I, P],
    # (h, mixed, a, b, gain_a, gain_b, eps_pair, weight, fed, dtype, gain, eps, rows, x, ldx, n_rows, W, update, stream)
    "psb_stream_sum": [P, P, P, P, P, P, F, F, P, I, P, F, P, P, L, I, I, I, P],
    # (a, a_dtype, lda, w, w_dtype, bias, rates, per_rate, constant, code, out, T, C, r, stream)
    "psb_low_rank": [P, I, L, P, I, P, P, I, F, I, P, I, I, I, P],
    # (proj, dtype, ld, alpha, state, slot_floats, item_start, slots, local_b, local_a, o, items, chunks, H, dim, vdim, num_slots,
    #  chunk, scale, stream)
    "psb_linear_attention": [P, I, L, P, P, L, P, P, P, P, P, I, I, I, I, I, I, I, F, P],
    # (o, gate, gate_dtype, ldg, gate_act, gain, head_gains, out, out_dtype, ldo, T, H, vdim, eps, stream)
    "psb_normed_readout": [P, P, I, L, I, P, I, P, I, L, I, I, I, F, P],
    # (h, pending, dtype, gain1, shift1, gain2, shift2, rows, x1, x2, n_rows, W, eps, update, stream)
    "psb_add_layer_norm": [P, P, I, P, P, P, P, P, P, P, I, I, F, I, P],
    # (proj, ld, dtype, positions, token_item, table, table_width, cos, sin, bias, gain_q, gain_k, first, ld_first, first_bias, share,
    #  kv, kv_dtype, q_out, T, hq, hkv, dim, vdim, page_size, num_pages, max_positions, rotary_dim, interleaved, eps, split_planes, stream)
    "psb_attention_prepare_heads": [P, L, I, P, P, P, I, P, P, P, P, P, P, L, P, P, P, I, P, I, I, I, I, I, I, I, I, I, I, F, I, P],
    # (proj, dtype, ld, bias_i, bias_f, gain, state, slot_floats, item_start, slots, out, ldo, o32, scratch, items, chunks, H, dim, vdim,
    #  nb, num_slots, cap, eps, scale, stream)
    "psb_matrix_memory": [P, I, L, P, P, P, P, L, P, P, P, L, P, P, I, I, I, I, I, I, I, F, F, F, P],
    "psb_matrix_memory_chunks_supported": [I, I],
    # (a, w, c, M, N, K, ldc, sms, activation, stream)
    "psb_gemm_tcgen05_unary": [P, P, P, I, I, I, I, I, I, P],
    # (x, W, y, M, N, K, ldy, sms, activation, stream)
    "psb_gemm_stream_unary": [P, P, P, I, I, I, I, I, I, P],
    # (a, w, c, M, N, K, ldc, activation, stream)
    "psb_gemm_fewrows_unary": [P, P, P, I, I, I, I, I, P],
    # (proj, ld, dtype, positions, token_item, table, table_width, bias, gain, kv, kv_dtype, q_out, T, hq, hkv, dim, vdim, page_size,
    #  num_pages, eps, split_planes, stream)
    "psb_attention_prepare_normed": [P, L, I, P, P, P, I, P, P, P, I, P, I, I, I, I, I, I, I, F, I, P],
    # (z, dtype, out, act, rows, W, eps, stream)
    "psb_poly_norm": [P, I, P, P, I, I, F, P],
    # (x, total, cap, stream)
    "psb_soft_cap": [P, L, F, P],
    # (gate_up, dtype, out, T, I, limit, alpha, offset, stream)
    "psb_clipped_glu": [P, I, P, I, I, F, F, F, P],
}


def lib() -> ctypes.CDLL:
    global _lib
    if _lib is None:
        path = ensure_kernels()
        handle = ctypes.CDLL(str(path))
        for name, argtypes in _SIGNATURES.items():
            fn = getattr(handle, name)
            fn.argtypes = argtypes
            fn.restype = c_int
        handle.psb_sample_scratch_bytes.restype = ctypes.c_longlong
        handle.psb_last_error.restype = ctypes.c_char_p
        handle.psb_last_error.argtypes = []
        handle.psb_set_pdl.argtypes = [c_int]
        handle.psb_set_pdl.restype = None
        handle.psb_get_pdl.argtypes = []
        handle.psb_get_pdl.restype = c_int
        if os.environ.get("PSB200_PDL", "1") == "0":  # plain stream order between kernels (for comparisons)
            handle.psb_set_pdl(0)
        _lib = handle
    return _lib


def set_pdl(on: bool) -> None:
    """Whether kernels are launched so that each may overlap its start with the end of its predecessor
    (programmatic dependent launch).  Graphs captured earlier keep the mode they were captured with."""
    lib().psb_set_pdl(1 if on else 0)


def pdl_enabled() -> bool:
    return bool(lib().psb_get_pdl())


_pinned_stream: int | None = None


def stream_handle() -> int:
    """The raw handle of the stream kernels are launched on: torch's current stream, looked up on every call unless a
    step has pinned it (``pinned_stream``): the lookup costs more host time than the launch it serves."""
    if _pinned_stream is not None:
        return _pinned_stream
    return torch.cuda.current_stream().cuda_stream


class pinned_stream:
    """Within the block, ``stream_handle()`` is torch's current stream as it was at entry.  For code that launches many
    kernels on one stream and does not switch streams itself (a step of the engine, the capture of one)."""

    def __enter__(self):
        global _pinned_stream
        self._before = _pinned_stream
        _pinned_stream = torch.cuda.current_stream().cuda_stream
        return self

    def __exit__(self, *exc):
        global _pinned_stream
        _pinned_stream = self._before


def tcgen05_status() -> int:
    """0 unless a bounded wait inside a tcgen05 kernel ever gave up (then its results are void). Synchronises.

    The product's code sits in the low byte, prefill attention's in the next, the TMA-fed decode attention's in the
    third, the few-row product's in the fourth."""
    return (int(lib().psb_tcgen05_status()) | (int(lib().psb_attention_tcgen05_status()) << 8)
            | (int(lib().psb_attention_decode_tma_status()) << 16) | (int(lib().psb_gemm_fewrows_status()) << 24))


def declare(name: str, argtypes: list) -> None:
    """Adds an entry point (used by kernels that arrive in later files)."""
    _SIGNATURES[name] = argtypes
    if _lib is not None:
        fn = getattr(_lib, name)
        fn.argtypes = argtypes
        fn.restype = c_int


launches = 0  # kernels of this library launched so far (benchmarks report the difference over a timed region)
launch_counts: Counter = Counter()  # the same by entry point ("attention_decode", "gemm_tcgen05", ...)


def check(status: int, what: str) -> None:
    global launches
    launches += 1
    launch_counts[what] += 1
    if status != 0:
        detail = lib().psb_last_error().decode(errors="replace")
        raise KernelError(f"{what}: {detail} (status {status})")


_parked: list[tuple[int, torch.device]] = []  # pool memory waiting to be freed (see DevicePool.free)


def _free_parked() -> None:
    if _lib is None or not _parked:
        return
    try:
        if torch.cuda.is_current_stream_capturing():
            return
    except Exception:  # noqa: BLE001  (interpreter shutdown)
        return
    while _parked:
        ptr, device = _parked.pop()
        with torch.cuda.device(device):
            _lib.psb_pool_free(c_void_p(ptr))


class DevicePool:
    """Device memory for cache pages, allocated and freed by the kernel library itself (not by torch's caching
    allocator): the address never moves and the bytes are given back the moment the owner goes.  ``tensor`` views
    the memory without copying; the views must not outlive the pool."""

    def __init__(self, nbytes: int, device: torch.device) -> None:
        self.nbytes, self.device = int(nbytes), torch.device(device)
        self.ptr = 0
        _free_parked()
        with torch.cuda.device(self.device):
            out = c_void_p()
            status = lib().psb_pool_alloc(self.nbytes, ctypes.byref(out))
            if status != 0:
                raise KernelError("pool: " + lib().psb_last_error().decode(errors="replace"))
            self.ptr = int(out.value)

    def tensor(self, shape: tuple, dtype: torch.dtype) -> torch.Tensor:
        typestr = {torch.bfloat16: "<u2", torch.float32: "<f4", torch.float16: "<f2"}[dtype]
        count = 1
        for n in shape:
            count *= int(n)
        if count * torch.empty((), dtype=dtype).element_size() > self.nbytes:
            raise KernelError(f"pool of {self.nbytes} bytes cannot hold a {dtype} tensor of shape {tuple(shape)}")

        class _Span:  # what torch needs to wrap foreign device memory; it keeps the pool alive while a view of it lives
            owner = self
            __cuda_array_interface__ = {"shape": tuple(int(n) for n in shape), "typestr": typestr, "data": (self.ptr, False),
                                        "version": 2, "strides": None}
        raw = torch.as_tensor(_Span(), device=self.device)
        return raw.view(dtype) if raw.dtype != dtype else raw

    def free(self) -> None:
        """Gives the memory back.  Freeing device memory waits for the device, which a stream capture in progress does
        not survive; a pool that dies during one (the collector may run its finaliser at any moment) is parked and
        freed by the next pool that is made or freed outside a capture."""
        if self.ptr:
            _parked.append((self.ptr, self.device))
            self.ptr = 0
        _free_parked()

    def __del__(self) -> None:
        try:
            self.free()
        except Exception:  # noqa: BLE001  (interpreter shutdown)
            pass
