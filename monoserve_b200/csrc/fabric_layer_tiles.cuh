// Tiles of the layer-list decoders inside the persistent fabric kernel: hyper-connected residual streams or a plain
// residual with their norms, short causal convolution, selective scan, matrix memory, gated memories (linear attention
// and delta rule), latent attention over a paged cache of latents, what surrounds grouped-query attention, and 32-bit
// matrix products.  Kinds in fabric_types.h, operand blocks in operands.h.  What the recurrences,
// norms, scores and residual sums compute is 32-bit throughout; activations between tiles are bf16, or fp32 when a
// block's f32 is set.
//
// The tiles are compiled in translation units of their own (fabric_layer_*.cu) and called from the worker's exec warps
// through run_layer_tile: their registers and stack are then their own affair, not the kernel's.
//
// Recurrent state lives in slot-indexed buffers.  A tile that starts at position 0 of its sequence takes the state
// as zero, so a slot needs no clearing when another request takes it over; one tile owns a piece of a slot's state
// (a channel block, a column block of a head) for a whole portion of the prompt.
#pragma once
#include <cuda_bf16.h>

#include <type_traits>

#include "fabric_types.h"
#include "operands.h"

namespace mf {
namespace fab {

constexpr int kExecThreads = 128;
// Scratch ints of the tile the exec warps are running (the kernel's static shared memory).
constexpr int kLayerScratchInts = 1120;
constexpr int kMaxStreams = 8;
constexpr int kMaxTaps = 8;

// What the worker lends a tile.
struct LayerCtx {
  int* scratch;              // kLayerScratchInts ints of shared memory
  uint8_t* ring;             // the operand ring (shared memory, 1024-byte aligned), for wide tiles only
  uint32_t tmem_base;        // all of the worker's TMEM, for wide tiles only
  volatile int* abort_flag;
};

// Runs tile kinds kTileProduct32 .. kTileHeadGate: false for a kind or size these tiles do not take, or when a bounded
// wait gave up.  All exec threads call it with the same tile.
__device__ bool run_layer_tile(const TileDesc& t, int tid, const LayerCtx& ctx);
// Wide tiles: their exec warps use the operand ring as scratch memory, and TMEM.
__device__ __forceinline__ bool tile_is_wide(uint32_t kind) {
  return kind == kTileMemory || kind == kTileScan || kind == kTileGatedMemory || kind == kTileGatedStep || kind == kTileLatentMma || kind == kTileLatentDirect;
}

__device__ void tile_streams(const TileDesc& t, int tid, int* scratch);
__device__ void tile_product32(const TileDesc& t, int tid, int* scratch);
__device__ void tile_gated_act(const TileDesc& t, int tid);
__device__ void tile_sum_slabs(const TileDesc& t, int tid);
__device__ void tile_conv(const TileDesc& t, int tid);
__device__ bool tile_scan(const TileDesc& t, int tid, uint8_t* ring);
__device__ bool tile_memory_step(const TileDesc& t, int tid);
__device__ void tile_scan_step(const TileDesc& t, int tid);
__device__ bool tile_memory(const TileDesc& t, int tid, uint8_t* ring);
__device__ void tile_head_norm(const TileDesc& t, int tid);
__device__ void tile_latent_kv(const TileDesc& t, int tid);
__device__ bool tile_latent_attn(const TileDesc& t, int tid);
__device__ bool tile_latent_mma(const TileDesc& t, int tid, const LayerCtx& ctx);
__device__ bool tile_latent_direct(const TileDesc& t, int tid, const LayerCtx& ctx);
__device__ void tile_latent_merge(const TileDesc& t, int tid);
__device__ void tile_residual(const TileDesc& t, int tid, int* scratch);
__device__ void tile_decay(const TileDesc& t, int tid);
__device__ bool tile_gated_memory(const TileDesc& t, int tid, uint8_t* ring);
__device__ bool tile_gated_step(const TileDesc& t, int tid, const LayerCtx& ctx);
__device__ void tile_qkv(const TileDesc& t, int tid);
__device__ bool tile_grouped_attn(const TileDesc& t, int tid);
__device__ void tile_head_gate(const TileDesc& t, int tid);

__device__ __forceinline__ void exec_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kExecThreads) : "memory"); }

template <class T>
__device__ __forceinline__ void load_block(T& dst, unsigned long long addr) {
  static_assert(sizeof(T) % 16 == 0, "operand blocks are multiples of 16 bytes");
  const uint4* src = reinterpret_cast<const uint4*>(addr);
  uint4* d = reinterpret_cast<uint4*>(&dst);
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T) / 16); ++i) d[i] = __ldcg(src + i);
}

// Decode bookkeeping of row r (one warp; lane 0 writes): position = the request's length (clamped to the block
// table), length + 1, the cache slot of the new key, req_info row {row, position, 1, position + 1}.  Returns the
// request's last token.
__device__ __forceinline__ int step_row(const StepArgs& St, int page, int r, int lane) {
  const int slot = reinterpret_cast<const int*>(St.row_req)[r];
  if (lane == 0) {
    int* seq_len = reinterpret_cast<int*>(St.seq_len);
    const int pos = min(seq_len[slot], static_cast<int>(St.bt_stride) * page - 1);
    seq_len[slot] = pos + 1;
    reinterpret_cast<int*>(St.tok_pos)[r] = pos;
    const int pg = reinterpret_cast<const int*>(St.block_table)[static_cast<size_t>(slot) * St.bt_stride + pos / page];
    reinterpret_cast<int*>(St.tok_slot)[r] = pg * page + pos % page;
    int4* info = reinterpret_cast<int4*>(St.req_info);
    info[r] = make_int4(r, pos, 1, pos + 1);
  }
  return reinterpret_cast<const int*>(St.last_token)[slot];
}

__device__ __forceinline__ float act_ld(unsigned long long base, size_t i, bool f32) {
  return f32 ? reinterpret_cast<const float*>(base)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(base)[i]);
}
__device__ __forceinline__ void act_st(unsigned long long base, size_t i, bool f32, float v) {
  if (f32) reinterpret_cast<float*>(base)[i] = v;
  else reinterpret_cast<__nv_bfloat16*>(base)[i] = __float2bfloat16(v);
}
__device__ __forceinline__ const float* f32p(unsigned long long base) { return reinterpret_cast<const float*>(base); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float sigmoid32(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <int V>
__device__ __forceinline__ void ld_vec(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  } else {
    v[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void st_vec(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}

}  // namespace fab
}  // namespace mf
