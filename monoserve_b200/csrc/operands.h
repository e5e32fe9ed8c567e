// Operand blocks of model tiles: the wire format between the Python program
// builders and the device tiles.  Field names, types and order are the ABI of
// the reference (csrc/fabric/model_types.h:50-235), because its Python side
// packs these blocks by the offsets the native library reports
// (monoserve/fabric/args.py:11-31).  Each block is declared once, as an
// X-macro list, from which both the C struct and the layout table are built.
#pragma once
#include <cstddef>
#include <cstdint>

namespace mf {

#define MF_GEMM_ARGS(U64, U32, F32) \
  U64(out) U64(pair_token) U64(pair_weight) U64(residual) U64(bias) \
  U32(ld_out) U32(ld_res) U32(k_tiles) U32(epi) U32(bm) U32(n_limit) U32(up_offset) U32(w_fp8)

#define MF_ATTN_ARGS(U64, U32, F32) \
  U64(q_map) U64(k_map) U64(v_map) U64(out) U64(ws_o) U64(ws_m) U64(ws_l) U64(block_table) U64(req_info) \
  F32(scale_log2) U32(bt_stride) U32(hq) U32(hkv) U32(group) U32(chunk_blocks) U32(max_chunks) \
  U32(page_size) U64(q_map_small)

/* acc_parts / acc_rows are not in the reference: with acc_parts > 1 the add-norm tile's `acc` is that many
 * fp32 slabs of acc_rows rows (the partial sums of a K-split GEMM, one slab per K range), added in slab order
 * and left as they are; otherwise it is one accumulator, zeroed once read. */
#define MF_NORM_ARGS(U64, U32, F32) \
  U64(x) U64(x2) U64(acc) U64(w) U64(out) U64(embed) U64(tokens) U64(gather) U64(out2) U64(step) \
  U32(H) U32(ld) F32(eps) U32(acc_parts) U32(acc_rows)

#define MF_STEP_ARGS(U64, U32, F32) \
  U64(row_req) U64(last_token) U64(seq_len) U64(block_table) U64(tok_pos) U64(tok_slot) U64(req_info) \
  U32(bt_stride) U32(page_size)

/* qkv_parts / qkv_rows are not in the reference: with qkv_parts > 1 `qkv` is that many fp32 slabs of qkv_rows
 * rows (the partial sums of a K-split projection, one slab per K range, the first with the bias); the tile adds
 * them in slab order and rounds the sum to bf16, which is the value a one-range projection would have stored. */
#define MF_QK_ARGS(U64, U32, F32) \
  U64(qkv) U64(q_out) U64(k_cache) U64(v_cache) U64(q_norm) U64(k_norm) U64(tok_pos) U64(tok_slot) \
  U64(cos_sin) U32(ld_qkv) U32(hq) U32(hkv) U32(rot_dim) F32(theta) F32(eps) U32(max_pos) U32(qkv_parts) \
  U32(qkv_rows)

#define MF_ROUTER_ARGS(U64, U32, F32) \
  U64(logits) U64(topk_ids) U64(topk_w) U64(counts) U64(bias) U32(E) U32(K) U32(scoring) U32(renorm) \
  F32(scale) U32(reserved0) U64(chunk_counts) U64(pair_rank)

#define MF_EXPAND_ARGS(U64, U32, F32) \
  U64(counts) U64(starts) U64(fill) U64(table) U64(w13_maps) U64(w2_maps) U64(xp_maps) U64(h_maps) \
  U64(w13_args) U64(w2_args) U64(hist) U64(w13_asym_args) U64(w2_asym_args) U64(red_args) \
  U64(w13_scale) U64(w2_scale) U32(E) U32(H) U32(I) U32(host_region) U32(w13_stage0) U32(w2_stage0) \
  U32(red_stage0) U32(dyn_first) U32(dyn_cap) U32(lane) U32(join_stage) U32(chunks) U64(chunk_counts) \
  U64(chunk_prefix) U64(staging) U32(fetch_stage0) U32(permute_rows) U64(permute_args)

/* ExpandArgs::permute_args / permute_rows are not in the reference: when set, the expand tile itself runs the
 * permute of rows [0, permute_rows) once its prefixes are written (the batch is small and a stage costs more than
 * the copy), and the program has no permute stage. */
/* Not in the reference: the staged form of a host-resident expert with many rows.  Its weights are
 * copied once into an HBM staging stack (slot = expert id) by fetch tiles, and its GEMM tiles read
 * that copy, so the expert crosses the host link once however many row blocks it has. */
#define MF_STAGING_ARGS(U64, U32, F32) \
  U64(w13_src) U64(w13_dst) U64(w13_bytes) U64(w2_src) U64(w2_dst) U64(w2_bytes) U32(chunk_bytes) U32(min_rows)

#define MF_REDUCE_ARGS(U64, U32, F32) U64(ws) U64(out) U32(I) U32(ld_ws) U32(ld_out)

#define MF_PERMUTE_ARGS(U64, U32, F32) \
  U64(topk_ids) U64(topk_w) U64(starts) U64(fill) U64(pair_token) U64(pair_weight) U64(src) U64(dst) \
  U32(K) U32(H) U64(pair_rank) U64(chunk_prefix) U64(pair_pos) U32(E)

#define MF_SAMPLE_ARGS(U64, U32, F32) \
  U64(logits) U64(temperature) U64(last_token) U64(steps) U64(host_tokens) U64(host_steps) U64(seed) \
  U32(V) U32(ring)

#define MF_ATTN_PLAN_ARGS(U64, U32, F32) \
  U64(attn) U64(req_info) U32(rows) U32(hkv) U32(chunk_keys) U32(stage_attn) U32(stage_comb) \
  U32(dyn_first) U32(dyn_cap) U32(workers) U32(reserved0) U64(row_req)

/* Not in the reference: the deterministic router projection and the deterministic
 * un-permute + weighted combine as fabric tiles. */
#define MF_LOGITS_ARGS(U64, U32, F32) U64(x) U64(wr) U64(logits) U32(T) U32(H) U32(E)

#define MF_COMBINE_ARGS(U64, U32, F32) \
  U64(y) U64(pair_pos) U64(topk_w) U64(x2) U64(x) U64(w) U64(out) U32(K) U32(H) F32(eps) U32(reserved0) \
  U64(shared)

/* Operand blocks of the layer-list decoders (hyper-connected residual streams, selective scan, matrix memory,
 * latent attention; fabric_layer_tiles.cuh).  None of them is in the reference.  Activations are bf16, or fp32
 * where a block's `f32` is set; `ld_*` are row strides in elements.
 *
 * StreamArgs: the residual streams xs fp32 [rows][streams][W].  hc_mix [from][to] and hc_out [to] belong to the
 * sublayer that has just produced y (y_parts fp32 slabs of y_rows rows; 0 parts: no update), hc_in to the one
 * that follows, w is the norm's multiplier (fp32).  embed set: the streams start as copies of the token's row.
 * split > 0: h16's row also receives what bf16 rounding leaves of the row, in two further bf16 parts `split` and
 * 2 split columns on (the three add up to the fp32 row). */
#define MF_STREAM_ARGS(U64, U32, F32) \
  U64(xs) U64(y) U64(hc_out) U64(hc_mix) U64(hc_in) U64(w) U64(h16) U64(h32) U64(gather) U64(out16) U64(out32) \
  U64(embed) U64(tokens) U64(step) U64(sum_out) U32(W) U32(streams) U32(ld_h16) U32(ld_h32) U32(ld_out) \
  U32(y_parts) U32(y_rows) F32(eps) U32(split)

/* out fp32 = x (fp32, or bf16 with f32 = 0) times w^T (bf16 rows), fp32 products and sums. */
#define MF_PRODUCT_ARGS(U64, U32, F32) \
  U64(x) U64(w) U64(out) U32(ld_x) U32(ld_w) U32(ld_out) U32(K) U32(N) U32(f32)

/* silu: the activation of the gate is silu, else gelu (tanh form). */
#define MF_GATED_ARGS(U64, U32, F32) U64(in) U64(out) U32(ff) U32(ld_in) U32(ld_out) U32(silu)

/* Adds `parts` fp32 slabs of part_rows rows; out32 receives every column, out16 the first c16 rounded to bf16. */
#define MF_SUM_ARGS(U64, U32, F32) \
  U64(in) U64(out32) U64(out16) U32(cols) U32(parts) U32(part_rows) U32(ld_in) U32(ld_32) U32(ld_16) U32(c16)

/* Causal convolution per channel over a request's rows, then silu; tail fp32 [slot][taps - 1][channels] holds the
 * inputs before the portion (read here; advanced by the scan tile, or with `advance` set by the tile of the request's
 * first rows, the only one that reads it).  bias may be 0. */
#define MF_CONV_ARGS(U64, U32, F32) \
  U64(x) U64(tail) U64(w) U64(bias) U64(out) U64(tok_pos) U32(ld_x) U32(ld_out) U32(channels) U32(taps) U32(f32) U32(advance)

#define MF_SCAN_ARGS(U64, U32, F32) \
  U64(x) U64(z) U64(dt) U64(dt_bias) U64(b) U64(c) U64(A) U64(D) U64(state) U64(tail) U64(x_in) U64(y) \
  U64(tok_pos) U32(ld_x) U32(ld_z) U32(ld_dt) U32(ld_bc) U32(ld_y) U32(channels) U32(n) U32(taps) U32(f32)

/* gates fp32 [rows][ld_gates]: raw input gates of the heads, then forget gates, as gate_parts slabs of
 * gate_rows rows to be added; gate_bias fp32 [2 heads].
 * state fp32 [slot][head][e + 1][d] (column e: the normaliser), m fp32 [slot][head][column
 * block]; out fp32 [rows][heads][e, the denominator, padding to a multiple of four]. */
#define MF_MEMORY_ARGS(U64, U32, F32) \
  U64(q) U64(k) U64(v) U64(gates) U64(gate_bias) U64(state) U64(m) U64(out) U64(tok_pos) U32(ld_qkv) U32(ld_gates) \
  U32(gate_parts) U32(gate_rows) U32(heads) U32(d) U32(e) U32(f32) F32(q_scale) F32(cap)

/* An item of o is e values, with `divide` set their denominator, and padding to a multiple of four.  w: head h's
 * multipliers at h * w_head; the gate g enters through silu, or else through sigmoid. */
#define MF_HEAD_NORM_ARGS(U64, U32, F32) \
  U64(o) U64(g) U64(w) U64(out) U32(heads) U32(e) U32(ld_g) U32(ld_out) U32(f32) F32(eps) U32(divide) U32(w_head) U32(silu)

/* qc fp32 [rows][heads * (d + r) | kv_rank | r]: queries, latent, shared rotated key part.  q_un [head][rows_max][ld_un]
 * unrotated query parts; q_all [head][rows_max][ld_q] = kv_rank absorbed columns (written by a product) then r rotated
 * ones; cache [page slots][ld_cache]; rows (optional) [rows][ld_rows]: a copy of the cached rows in token order. */
#define MF_LATENT_ARGS(U64, U32, F32) \
  U64(qc) U64(c_norm) U64(q_un) U64(q_all) U64(cache) U64(rows) U64(tok_pos) U64(tok_slot) U64(cos_sin) U32(ld_qc) U32(heads) \
  U32(d) U32(r) U32(kv_rank) U32(ld_un) U32(ld_q) U32(rows_max) U32(ld_cache) U32(ld_rows) U32(max_pos) U32(f32) F32(eps)

/* ws_o fp32 [(row * heads + head) * parts + part][kv_rank], ws_ml float2 of the same rows.  For the tensor-core tile:
 * q_map dims (kv_rank + r, rows_max, heads), box (64, tokens, group); kv_map dims (64, 8, chunks, page slots / 8), box
 * (64, 8, chunks, page / 8); buffers: key tiles of 128 in shared memory. */
#define MF_LATENT_ATTN_ARGS(U64, U32, F32) \
  U64(q) U64(cache) U64(block_table) U64(out) U64(ws_o) U64(ws_ml) U64(tok_pos) U64(q_map) U64(kv_map) U32(ld_q) \
  U32(heads) U32(kv_rank) U32(r) U32(ld_cache) U32(page) U32(bt_stride) U32(rows_max) U32(ld_out) U32(f32) F32(scale) \
  U32(tokens) U32(group) U32(buffers)

/* Whole prompts: q_map dims (d, heads * rows_max) and qr_map (r, heads * rows_max), kv_map (heads * (d + e), rows): keys
 * then values of every head, kr_map (r, rows); boxes (64, 128).  out bf16 [rows][ld_out], head h at column h e. */
#define MF_LATENT_DIRECT_ARGS(U64, U32, F32) \
  U64(q_map) U64(qr_map) U64(kv_map) U64(kr_map) U64(out) U32(d) U32(r) U32(e) U32(heads) U32(rows_max) U32(ld_out) \
  U32(buffers) F32(scale)

/* The plain residual x fp32 [rows][W] with a norm on both sides of a sublayer: x += post_w norm(y), then the next
 * sublayer's input w norm(x) in h16 / h32 (and, for rows with gather >= 0, in out16 / out32).  y is the sum of y0_parts
 * fp32 slabs of y_rows rows at y0; with y1_parts > 0 it is branch_scale * (w0 norm(y0) + w1 norm(y1)).  embed set: x starts
 * as embed[token] * embed_scale + pos[position] instead (pos optional, max_pos rows). */
#define MF_RESIDUAL_ARGS(U64, U32, F32) \
  U64(x) U64(y0) U64(y1) U64(w0) U64(w1) U64(post_w) U64(w) U64(h16) U64(h32) U64(gather) U64(out16) U64(out32) U64(embed) \
  U64(pos) U64(tokens) U64(tok_pos) U64(step) U64(sum_out) U32(W) U32(ld_h16) U32(ld_h32) U32(ld_out) U32(y0_parts) \
  U32(y1_parts) U32(y_rows) U32(max_pos) F32(eps) F32(embed_scale) F32(branch_scale)

/* z fp32 [rows][ld] in place: expm1(-coef[channel] * softplus(z + bias[channel])) for n channels, the distance to one of a
 * gated memory's decays; bias, coef fp32 [n].  (bf16 models have it as the projection's epilogue.) */
#define MF_DECAY_ARGS(U64, U32, F32) U64(z) U64(bias) U64(coef) U32(ld) U32(n)

/* Gated memory: per head S <- diag(1 + decay) S + k u^T, o = S^T q, state fp32 [slot][head][e][d padded to 4].
 * beta = 0: u = v; else the delta rule u = sigmoid(beta) (v - S^T k) on the decayed S.  unit: keys and queries are
 * divided by sqrt(sum of squares + 1e-6).  q is multiplied by q_scale; value head h reads key head h / group.  q, k, v,
 * beta: activations; decay fp32 [rows][heads * d]; out fp32 [rows][heads][e padded to 4]. */
#define MF_GATED_MEMORY_ARGS(U64, U32, F32) \
  U64(q) U64(k) U64(v) U64(beta) U64(decay) U64(state) U64(out) U64(tok_pos) U32(ld_qkv) U32(ld_beta) U32(ld_decay) \
  U32(heads) U32(group) U32(d) U32(e) U32(f32) U32(unit) F32(q_scale)

/* Grouped-query attention around the paged cache.  q, k, v: activations of a row; q_out [rows][heads][ld_q], caches
 * [page slots][kv_heads][ld_k or ld_v], columns past d (e) are written as zero.  Queries and keys are divided by their
 * root mean square and multiplied by q_norm / k_norm (fp32 [d]; 0: left as they are). */
#define MF_QKV_ARGS(U64, U32, F32) \
  U64(q) U64(k) U64(v) U64(q_norm) U64(k_norm) U64(q_out) U64(k_cache) U64(v_cache) U64(tok_slot) U32(ld_x) U32(heads) \
  U32(kv_heads) U32(d) U32(e) U32(ld_q) U32(ld_k) U32(ld_v) U32(f32) F32(eps)

/* The simple form of the attention itself, for sizes and precisions the tensor-core tiles do not take; out
 * [rows][heads][ld_out]. */
#define MF_GROUPED_ATTN_ARGS(U64, U32, F32) \
  U64(q) U64(k_cache) U64(v_cache) U64(block_table) U64(out) U64(tok_pos) U32(heads) U32(kv_heads) U32(d) U32(e) U32(ld_q) \
  U32(ld_k) U32(ld_v) U32(ld_out) U32(page) U32(bt_stride) U32(f32) F32(scale)

/* out [rows][ld_out], head h at column h e = in [rows][heads][ld_in] (e columns) times sigmoid(g [rows][ld_g]). */
#define MF_HEAD_GATE_ARGS(U64, U32, F32) \
  U64(in) U64(g) U64(out) U32(heads) U32(e) U32(ld_in) U32(ld_g) U32(ld_out) U32(f32)

#define MF_FIELD_U64(name) unsigned long long name;
#define MF_FIELD_U32(name) uint32_t name;
#define MF_FIELD_F32(name) float name;

#define MF_DECLARE(Name, LIST, SIZE)                                   \
  struct alignas(64) Name {                                            \
    LIST(MF_FIELD_U64, MF_FIELD_U32, MF_FIELD_F32)                     \
  };                                                                   \
  static_assert(sizeof(Name) == SIZE, #Name " has the wrong size");

MF_DECLARE(GemmArgs, MF_GEMM_ARGS, 128)
MF_DECLARE(AttnArgs, MF_ATTN_ARGS, 128)
MF_DECLARE(NormArgs, MF_NORM_ARGS, 128)
MF_DECLARE(StepArgs, MF_STEP_ARGS, 64)
MF_DECLARE(QkArgs, MF_QK_ARGS, 128)
MF_DECLARE(RouterArgs, MF_ROUTER_ARGS, 128)
MF_DECLARE(ExpandArgs, MF_EXPAND_ARGS, 256)
MF_DECLARE(StagingArgs, MF_STAGING_ARGS, 64)
MF_DECLARE(ReduceArgs, MF_REDUCE_ARGS, 64)
MF_DECLARE(PermuteArgs, MF_PERMUTE_ARGS, 128)
MF_DECLARE(SampleArgs, MF_SAMPLE_ARGS, 64)
MF_DECLARE(AttnPlanArgs, MF_ATTN_PLAN_ARGS, 64)
MF_DECLARE(LogitsArgs, MF_LOGITS_ARGS, 64)
MF_DECLARE(CombineArgs, MF_COMBINE_ARGS, 128)
MF_DECLARE(StreamArgs, MF_STREAM_ARGS, 192)
MF_DECLARE(ProductArgs, MF_PRODUCT_ARGS, 64)
MF_DECLARE(GatedArgs, MF_GATED_ARGS, 64)
MF_DECLARE(SumArgs, MF_SUM_ARGS, 64)
MF_DECLARE(ConvArgs, MF_CONV_ARGS, 128)
MF_DECLARE(ScanArgs, MF_SCAN_ARGS, 192)
MF_DECLARE(MemoryArgs, MF_MEMORY_ARGS, 128)
MF_DECLARE(HeadNormArgs, MF_HEAD_NORM_ARGS, 128)
MF_DECLARE(LatentArgs, MF_LATENT_ARGS, 128)
MF_DECLARE(LatentAttnArgs, MF_LATENT_ATTN_ARGS, 128)
MF_DECLARE(LatentDirectArgs, MF_LATENT_DIRECT_ARGS, 128)
MF_DECLARE(ResidualArgs, MF_RESIDUAL_ARGS, 192)
MF_DECLARE(DecayArgs, MF_DECAY_ARGS, 64)
MF_DECLARE(GatedMemoryArgs, MF_GATED_MEMORY_ARGS, 128)
MF_DECLARE(QkvArgs, MF_QKV_ARGS, 128)
MF_DECLARE(GroupedAttnArgs, MF_GROUPED_ATTN_ARGS, 128)
MF_DECLARE(HeadGateArgs, MF_HEAD_GATE_ARGS, 64)

}  // namespace mf
