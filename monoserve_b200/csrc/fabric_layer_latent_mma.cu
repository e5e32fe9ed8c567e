// Latent attention on the tensor cores: the bf16 form of the tile in fabric_layer_latent.cu (fabric_layer_tiles.cuh).
//
// Keys are the MMA's M dimension and (head, token) pairs its N dimension, so one cached latent row serves every head
// of the tile and a decode step with sixteen heads wastes nothing:
//   S^T [128 keys][N]          = K [128][latent | rotated part] . Q^T      (A K-major)
//   O^T [latent dims, 128 at a time][N] += V^T [dims][128 keys] . P^T      (A MN-major: the same tile, read as V)
// A key tile comes through one TMA box per page in groups of eight keys: [group][64-element chunk][8 keys][128 bytes],
// 128-byte swizzle, which serves both as K (rows = keys) and as V^T (rows = latent columns).
//
// The tile is wide: it runs on the exec warps alone, with the operand ring as its shared memory and the worker's TMEM
// (nothing else of the worker is in flight meanwhile).  Thread = key: a thread turns its key's N scores into P^T; the
// row maxima move only when a score exceeds the reference by more than kSlack (in the exp2 domain), so the reductions
// over keys are rare, and the sums stay in registers to the end.  S of the next key tile is issued right behind O of this
// one.  Every wait is bounded; the threads agree on going on once per key tile.
#include "fabric_layer_tiles.cuh"
#include "ptx.cuh"
#include "wide_tile.cuh"

namespace mf {
namespace fab {

constexpr int kKeyTile = 128;

// N columns: (head of the group) * tokens + token.
template <int N>
__device__ __noinline__ bool latent_mma(const TileDesc& t, int tid, const LayerCtx& ctx) {
  LatentAttnArgs A;
  load_block(A, t.a[0]);
  __builtin_assume(__isShared(ctx.ring));
  __builtin_assume(__isShared(ctx.scratch));
  const int warp = tid >> 5, lane = tid & 31, quad = (warp + 1) & 3;   // exec warps are warps 1 .. 4 of the CTA
  const int row0 = static_cast<int>(t.i0), n_tok = static_cast<int>(t.i1 & 0xffffu), h0 = static_cast<int>(t.i1 >> 16);
  const int part = static_cast<int>(t.i2), parts = static_cast<int>(t.i3);
  const int H = static_cast<int>(A.heads), kvr = static_cast<int>(A.kv_rank), page = static_cast<int>(A.page);
  const int box_tok = static_cast<int>(A.tokens), hg = static_cast<int>(A.group), n_h = min(hg, H - h0);
  const int chunks = (kvr + static_cast<int>(A.r) + 63) / 64, blocks = (kvr + 127) / 128;
  const int pos0 = reinterpret_cast<const int*>(A.tok_pos)[row0];
  const int keys = pos0 + n_tok;
  const int per = (keys + parts - 1) / parts;
  const int k_lo = min(part * per, keys), k_hi = min(k_lo + per, keys);

  uint64_t* const bar = reinterpret_cast<uint64_t*>(ctx.scratch);   // q, k[2], s, o
  uint64_t *const bar_q = bar, *const bar_k = bar + 1, *const bar_s = bar + 3, *const bar_o = bar + 4;
  float* const s_m = reinterpret_cast<float*>(ctx.scratch) + 16;    // [64] reference of each column
  float* const s_a = s_m + 64;                                      // [64] factor of the last move, later 1 / sum
  float* const s_red = s_a + 64;                                    // [4][64]
  const uint32_t group_bytes = chunks * 1024u, tile_bytes = (kKeyTile / 8) * group_bytes;
  const uint32_t q_bytes = chunks * N * 128u, p_bytes = N * 256u;
  uint8_t* const sQ = ctx.ring;
  uint8_t* const sP = ctx.ring + q_bytes;
  uint8_t* const sK = sP + ((p_bytes + 1023u) & ~1023u);
  const int nbuf = A.buffers > 1 ? 2 : 1;
  const uint32_t tmem_s = ctx.tmem_base, tmem_o = ctx.tmem_base + 64;
  const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;

  if (tid == 0) {
    for (int i = 0; i < 5; ++i) mbar_init(bar + i, 1);
    fence_barrier_init();
  }
  if (tid < N) s_m[tid] = -1e30f;
  exec_sync();

  const int* bt = reinterpret_cast<const int*>(A.block_table) + static_cast<size_t>(t.a[1] & 0xffffffffull) * A.bt_stride;
  const int last_page = (max(k_hi, 1) - 1) / page, per_tile = kKeyTile / page;
  const int first_key = k_lo / page * page;   // key tiles start at a page
  const int tiles = k_hi > k_lo ? (k_hi - first_key + kKeyTile - 1) / kKeyTile : 0;
  auto page_of = [&](int j) {   // this lane's page of key tile j; pages past the visible range repeat the last visible one
    return lane < per_tile ? bt[min(first_key / page + j * per_tile + lane, last_page)] : 0;
  };
  int pg_next = 0;
  auto load_keys = [&](int j) {   // warp 0, in the order of the tiles; the tile behind it is brought to L2
    const int s = j % nbuf, pg = j == 0 ? page_of(0) : pg_next;
    if (lane == 0) {
      if (j == 0) fence_proxy_async_all();
      mbar_arrive_expect_tx(bar_k + s, tile_bytes);
    }
    __syncwarp();
    if (lane < per_tile) tma_box_4d(sK + s * tile_bytes + lane * (page / 8) * group_bytes, A.kv_map, bar_k + s, 0, 0, 0, pg * (page / 8));
    if (j + 1 < tiles) {
      pg_next = page_of(j + 1);
      if (lane < per_tile) tma_prefetch_4d(A.kv_map, 0, 0, 0, pg_next * (page / 8));
    }
  };
  // The MMAs are issued by warp 0 in step, one elected lane issuing: descriptors are then warp-uniform values that only
  // their start addresses tell apart (all of them below 2^18, so plain additions of address / 16).
  const bool leader = warp == 0 && elect_one();
  const uint64_t desc_q = sw128_desc(smem_u32(sQ), 0, 1024), desc_p = sw128_desc(smem_u32(sP), 0, 1024);
  auto issue_s = [&](int j) {   // S^T of key tile j
    uint64_t k = sw128_desc(smem_u32(sK + (j % nbuf) * tile_bytes), 0, group_bytes), q = desc_q;
    const uint32_t idesc = umma_idesc_bf16(128, N);
    tc_fence_after_sync();
#pragma unroll 1
    for (int c = 0; c < chunks; ++c, k += 1024 >> 4, q += (N * 128) >> 4) {
      if (leader) {
#pragma unroll
        for (int i = 0; i < 4; ++i) umma_bf16(tmem_s, k + 2 * i, q + 2 * i, idesc, (c | i) != 0);
      }
    }
    if (leader) umma_commit(bar_s);
    __syncwarp();
  };
  auto issue_o = [&](int j) {   // O^T += V^T P^T of key tile j
    uint64_t v = sw128_desc(smem_u32(sK + (j % nbuf) * tile_bytes), 1024, group_bytes);
    const uint32_t idesc = umma_idesc_bf16(128, N) | (1u << 15), step = group_bytes >> 3;   // A is MN-major; 16 keys on
    tc_fence_after_sync();
#pragma unroll 1
    for (int b = 0; b < blocks; ++b, v += 2048 >> 4) {
      if (leader) {
        uint64_t vi = v;
#pragma unroll
        for (int i = 0; i < kKeyTile / 16; ++i, vi += step)
          umma_bf16(tmem_o + b * N, vi, desc_p + (i >> 2) * ((N * 128) >> 4) + (i & 3) * 2, idesc, (j | i) != 0);
      }
    }
    if (leader) umma_commit(bar_o);
    __syncwarp();
  };
  auto wait = [&](uint64_t* b, int phase) { return mbar_wait_bounded(b, phase & 1, ctx.abort_flag, kWideWaitNs); };

  bool ok = true;
  if (warp == 0 && tiles > 0) {
    if (lane == 0) {
      fence_proxy_async_all();
      mbar_arrive_expect_tx(bar_q, static_cast<uint32_t>(chunks) * 128u * box_tok * hg);
      for (int c = 0; c < chunks; ++c) tma_box_3d(sQ + c * (N * 128u), A.q_map, bar_q, c * 64, row0, h0);
    }
    __syncwarp();
    load_keys(0);
    if (nbuf > 1 && tiles > 1) load_keys(1);
  }
  if (warp == 0 && tiles > 0) {
    ok = __all_sync(0xffffffffu, wait(bar_q, 0) && wait(bar_k, 0));
    if (ok) issue_s(0);
  }
  const float scale = A.scale * 1.4426950408889634f;
  float l[N];
#pragma unroll
  for (int c = 0; c < N; ++c) l[c] = 0.f;
  const int n_col = box_tok * hg;
  const int my_key = quad * 32 + lane;
  for (int j = 0; j < tiles; ++j) {
    ok = ok && mbar_wait_bounded(bar_s, j & 1, ctx.abort_flag, kWideWaitNs) &&
         (j == 0 || mbar_wait_bounded(bar_o, (j - 1) & 1, ctx.abort_flag, kWideWaitNs));
    if (!exec_and(ok)) {
      ok = false;
      break;
    }
    tc_fence_after_sync();
    float v[N];
#pragma unroll
    for (int c0 = 0; c0 < N; c0 += 16) {
      __syncwarp();
      tmem_ld_32x16(tmem_s + lane_off + c0, *reinterpret_cast<uint32_t(*)[16]>(&v[c0]));
    }
    tmem_ld_wait();
    const int key = first_key + j * kKeyTile + my_key;
    // token t of a column sees the key when pos0 + t >= key; keys outside [k_lo, k_hi) belong to another part
    const int t_min = (key < k_lo || key >= k_hi) ? 0x7fffffff : key - pos0;
    bool move = false;
    {
      int tok = 0;
#pragma unroll
      for (int c = 0; c < N; ++c) {
        const bool see = c < n_col && tok >= t_min;
        v[c] = see ? v[c] * scale : -INFINITY;
        move |= v[c] > s_m[c] + kSlack;
        if (++tok == box_tok) tok = 0;
      }
    }
    if (!exec_and(!move)) {   // some column's reference moves: reduce over the tile's keys, rescale O
#pragma unroll
      for (int c = 0; c < N; ++c) {
        float m = v[c];
#pragma unroll
        for (int o = 16; o; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        if (lane == 0) s_red[warp * 64 + c] = m;
      }
      exec_sync();
      if (tid < N) {
        const float old = s_m[tid];
        const float m = fmaxf(fmaxf(s_red[tid], s_red[64 + tid]), fmaxf(s_red[128 + tid], s_red[192 + tid]));
        const float now = m > old + kSlack ? m : old;
        s_m[tid] = now;
        s_a[tid] = ex2(old - now);
      }
      exec_sync();
#pragma unroll
      for (int c = 0; c < N; ++c) l[c] *= s_a[c];
      if (j > 0)   // O of the tiles before is complete: S of this tile was issued behind it
        for (int b = 0; b < blocks; ++b)
#pragma unroll
          for (int c0 = 0; c0 < N; c0 += 16) {
            uint32_t o[16];
            __syncwarp();
            tmem_ld_32x16(tmem_o + lane_off + b * N + c0, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_a[c0 + i]);
            tmem_st_32x16(tmem_o + lane_off + b * N + c0, o);
          }
      tmem_st_done();
    }
    // P^T as bf16: row = column of S^T, 64 keys per 128-byte row, 128-byte swizzle
    uint8_t* const p_half = sP + (my_key >> 6) * (N * 128);
    const int k6 = my_key & 63;
#pragma unroll
    for (int c = 0; c < N; ++c) {
      const __nv_bfloat16 p = __float2bfloat16(ex2(v[c] - s_m[c]));
      l[c] += __bfloat162float(p);
      *reinterpret_cast<__nv_bfloat16*>(p_half + c * 128 + ((((k6 >> 3) ^ (c & 7)) << 4) | ((k6 & 7) << 1))) = p;
    }
    tc_fence_before_sync();
    fence_proxy_async_smem();
    exec_sync();
    if (warp == 0) {
      issue_o(j);
      if (nbuf > 1 && j + 1 < tiles) {
        ok = __all_sync(0xffffffffu, wait(bar_k + ((j + 1) & 1), (j + 1) >> 1));
        if (ok) issue_s(j + 1);
      }
      if (j + nbuf < tiles) {   // the key tile's buffer goes to the loads of tile j + nbuf when O has read it
        ok = __all_sync(0xffffffffu, ok && wait(bar_o, j));
        if (ok) load_keys(j + nbuf);
        if (nbuf == 1 && ok) {
          ok = __all_sync(0xffffffffu, wait(bar_k, j + 1));
          if (ok) issue_s(j + 1);
        }
      }
    }
  }
  if (ok && tiles > 0) ok = mbar_wait_bounded(bar_o, (tiles - 1) & 1, ctx.abort_flag, kWideWaitNs);
  ok = exec_and(ok);
  tc_fence_after_sync();
  if (ok) {
#pragma unroll
    for (int c = 0; c < N; ++c) {
      const float s = warp_sum(l[c]);
      if (lane == 0) s_red[warp * 64 + c] = s;
    }
    exec_sync();
    if (tid < N) {
      const float s = s_red[tid] + s_red[64 + tid] + s_red[128 + tid] + s_red[192 + tid];
      s_a[tid] = parts == 1 ? 1.f / s : s;
    }
    exec_sync();
    if (parts > 1 && tid < n_tok * n_h) {
      const int h = tid / n_tok, tok = tid - h * n_tok, c = h * box_tok + tok;
      const size_t w = (static_cast<size_t>(row0 + tok) * H + h0 + h) * parts + part;
      reinterpret_cast<float2*>(A.ws_ml)[w] = tiles ? make_float2(s_m[c] * 0.6931471805599453f, s_a[c]) : make_float2(-INFINITY, 0.f);
    }
    for (int b = 0; b < blocks; ++b) {
      const int dim = b * 128 + quad * 32 + lane;
#pragma unroll
      for (int c0 = 0; c0 < N; c0 += 16) {
        uint32_t o[16];
        __syncwarp();
        if (tiles > 0) {
          tmem_ld_32x16(tmem_o + lane_off + b * N + c0, o);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = 0u;
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int c = c0 + i, h = box_tok == 1 ? c : c / box_tok, tok = c - h * box_tok;
          if (h >= n_h || tok >= n_tok || dim >= kvr) continue;
          const float x = __uint_as_float(o[i]);
          if (parts == 1) {
            reinterpret_cast<__nv_bfloat16*>(A.out)[(static_cast<size_t>(h0 + h) * A.rows_max + row0 + tok) * A.ld_out + dim] =
                __float2bfloat16(x * s_a[c]);
          } else {
            reinterpret_cast<float*>(A.ws_o)[((static_cast<size_t>(row0 + tok) * H + h0 + h) * parts + part) * kvr + dim] = x;
          }
        }
      }
    }
  }
  tc_fence_before_sync();
  exec_sync();
  if (tid == 0)
    for (int i = 0; i < 5; ++i) mbar_inval(bar + i);
  return ok;
}

__device__ bool tile_latent_mma(const TileDesc& t, int tid, const LayerCtx& ctx) {
  const LatentAttnArgs* p = reinterpret_cast<const LatentAttnArgs*>(t.a[0]);
  const uint32_t n = __ldcg(&p->tokens) * __ldcg(&p->group);
  if (n <= 16) return latent_mma<16>(t, tid, ctx);
  if (n <= 32) return latent_mma<32>(t, tid, ctx);
  if (n <= 64) return latent_mma<64>(t, tid, ctx);
  return false;
}

}  // namespace fab
}  // namespace mf
