// Latent attention of whole prompts on the tensor cores (fabric_layer_tiles.cuh): keys and values are first mapped out of
// the latents for every head (one GEMM over the prompt's own rows), which needs fewer FLOPs per (query, key) pair than
// the absorbed form of fabric_layer_latent_mma.cu and a seventh of its operand traffic.
//
//   S [128 queries][128 keys] = Q_un K_un^T + Q_rot K_rot^T      (K_rot shared by the heads)
//   O [128 queries][values]  += P V
// A wide tile on the exec warps alone: thread = query row; S is double-buffered in TMEM and S of the next key tile is
// issued before this one's exponentials; K is double-buffered in shared memory where that fits.  Operand tiles are 128
// rows x 64 columns of bf16 (16 KB), 128-byte swizzle.  Every wait is bounded.
#include "fabric_layer_tiles.cuh"
#include "ptx.cuh"
#include "wide_tile.cuh"

namespace mf {
namespace fab {

constexpr uint32_t kOperandTile = 16384;

__device__ __noinline__ bool latent_direct(const TileDesc& t, int tid, const LayerCtx& ctx) {
  LatentDirectArgs A;
  load_block(A, t.a[0]);
  __builtin_assume(__isShared(ctx.ring));
  __builtin_assume(__isShared(ctx.scratch));
  const int warp = tid >> 5, lane = tid & 31, quad = (warp + 1) & 3;   // exec warps are warps 1 .. 4 of the CTA
  const int row0 = static_cast<int>(t.i0), n = static_cast<int>(t.i1), q0 = static_cast<int>(t.i2), h = static_cast<int>(t.i3);
  const int d = static_cast<int>(A.d), e = static_cast<int>(A.e), H = static_cast<int>(A.heads);
  const int nd = (d + 63) / 64, nr = (static_cast<int>(A.r) + 63) / 64, ne = (e + 63) / 64, nq = nd + nr;
  const int tiles = (min(n, q0 + 128) + 127) / 128;
  const int nbuf = A.buffers > 1 ? 2 : 1;
  uint64_t* const bar = reinterpret_cast<uint64_t*>(ctx.scratch);
  uint64_t *const bar_q = bar, *const bar_k = bar + 1, *const bar_v = bar + 3, *const bar_s = bar + 4, *const bar_o = bar + 6;
  uint8_t* const sQ = ctx.ring;
  uint8_t* const sK = sQ + nq * kOperandTile;
  uint8_t* const sV = sK + nbuf * nq * kOperandTile;
  uint8_t* const sP = sV + ne * kOperandTile;
  const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
  const uint32_t tmem_s = ctx.tmem_base, tmem_o = ctx.tmem_base + 256;
  const int ncol = (e + 15) & ~15;

  if (tid == 0) {
    for (int i = 0; i < 7; ++i) mbar_init(bar + i, 1);
    fence_barrier_init();
  }
  exec_sync();
  // one thread issues the loads, the MMAs and their commits
  auto load_k = [&](int j) {
    uint8_t* dst = sK + (j % nbuf) * nq * kOperandTile;
    uint64_t* b = bar_k + j % nbuf;
    mbar_arrive_expect_tx(b, nq * kOperandTile);
    for (int c = 0; c < nd; ++c) tma_box_2d(dst + c * kOperandTile, A.kv_map, b, h * d + c * 64, row0 + j * 128);
    for (int c = 0; c < nr; ++c) tma_box_2d(dst + (nd + c) * kOperandTile, A.kr_map, b, c * 64, row0 + j * 128);
  };
  auto load_v = [&](int j) {
    mbar_arrive_expect_tx(bar_v, ne * kOperandTile);
    for (int c = 0; c < ne; ++c) tma_box_2d(sV + c * kOperandTile, A.kv_map, bar_v, H * d + h * e + c * 64, row0 + j * 128);
  };
  auto wait = [&](uint64_t* b, int phase) { return mbar_wait_bounded(b, phase & 1, ctx.abort_flag, kWideWaitNs); };
  auto issue_s = [&](int j) {
    tc_fence_after_sync();
    const uint32_t q = smem_u32(sQ), k = smem_u32(sK + (j % nbuf) * nq * kOperandTile), idesc = umma_idesc_bf16(128, 128);
    for (int c = 0; c < nq; ++c)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        umma_bf16(tmem_s + (j & 1) * 128, sw128_desc(q + c * kOperandTile + i * 32u, 0, 1024),
                  sw128_desc(k + c * kOperandTile + i * 32u, 0, 1024), idesc, (c | i) != 0);
    umma_commit(bar_s + (j & 1));
  };
  bool ok = true;
  if (tid == 0) {
    fence_proxy_async_all();
    mbar_arrive_expect_tx(bar_q, nq * kOperandTile);
    const int y = h * static_cast<int>(A.rows_max) + row0 + q0;
    for (int c = 0; c < nd; ++c) tma_box_2d(sQ + c * kOperandTile, A.q_map, bar_q, c * 64, y);
    for (int c = 0; c < nr; ++c) tma_box_2d(sQ + (nd + c) * kOperandTile, A.qr_map, bar_q, c * 64, y);
    load_k(0);
    load_v(0);
    if (nbuf > 1 && tiles > 1) load_k(1);
    ok = wait(bar_q, 0) && wait(bar_k, 0);
    if (ok) issue_s(0);
  }
  const float scale = A.scale * 1.4426950408889634f;
  const int row = quad * 32 + lane;         // query of the block = TMEM lane
  const int q_pos = q0 + row;
  float m = -1e30f, l = 0.f;
  for (int j = 0; j < tiles; ++j) {
    if (tid == 0 && nbuf > 1 && ok && j + 1 < tiles) {
      ok = wait(bar_k + ((j + 1) & 1), (j + 1) >> 1);
      if (ok) issue_s(j + 1);
    }
    ok = ok && wait(bar_s + (j & 1), j >> 1) && (j == 0 || wait(bar_o, j - 1));
    if (!exec_and(ok)) {
      ok = false;
      break;
    }
    tc_fence_after_sync();
    if (tid == 0) {   // K of this tile has been read, V of the tile before too
      if (j > 0) load_v(j);
      if (j + nbuf < tiles) load_k(j + nbuf);
      if (nbuf == 1 && j + 1 < tiles) {
        ok = wait(bar_k, j + 1);
        if (ok) issue_s(j + 1);
      }
    }
    __syncwarp();
    const int lim = min(min(n, q_pos + 1) - j * 128, 128);   // keys [0, lim) of the tile count
    float v[128];
#pragma unroll
    for (int c0 = 0; c0 < 128; c0 += 32) {
      __syncwarp();
      tmem_ld_32x32(tmem_s + (j & 1) * 128 + lane_off + c0, *reinterpret_cast<uint32_t(*)[32]>(&v[c0]));
    }
    tmem_ld_wait();
    float mx = -1e30f;
    if (lim >= 128) {
#pragma unroll
      for (int i = 0; i < 128; ++i) mx = fmaxf(mx, v[i]);
    } else {
#pragma unroll
      for (int i = 0; i < 128; ++i)
        if (i < lim) mx = fmaxf(mx, v[i]);
    }
    mx = mx > -1e30f ? mx * scale : -1e30f;
    // the reference moves only when the maximum has outgrown it by more than kSlack (P stays within 2^kSlack)
    mx = mx > m + kSlack ? mx : m;
    if (j > 0 && __any_sync(0xffffffffu, mx > m)) {   // O of the tiles before is complete
      const float f = ex2(m - mx);
      for (int c0 = 0; c0 < ncol; c0 += 16) {
        uint32_t o[16];
        __syncwarp();
        tmem_ld_32x16(tmem_o + lane_off + c0, o);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
        tmem_st_32x16(tmem_o + lane_off + c0, o);
      }
      tmem_st_done();
      l *= f;
    }
    m = mx;
    float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
    for (int c0 = 0; c0 < 128; c0 += 8) {
      uint32_t pk[4];
#pragma unroll
      for (int i = 0; i < 8; i += 2) {
        const float p0 = c0 + i < lim ? ex2(fmaf(v[c0 + i], scale, -m)) : 0.f;
        const float p1 = c0 + i + 1 < lim ? ex2(fmaf(v[c0 + i + 1], scale, -m)) : 0.f;
        const __nv_bfloat162 b = __floats2bfloat162_rn(p0, p1);
        pk[i >> 1] = *reinterpret_cast<const uint32_t*>(&b);
        sum0 += __uint_as_float(pk[i >> 1] << 16);
        sum1 += __uint_as_float(pk[i >> 1] & 0xffff0000u);
      }
      *reinterpret_cast<uint4*>(sP + (c0 >> 6) * kOperandTile + row * 128 + ((((c0 & 63) >> 3) ^ (row & 7)) << 4)) =
          make_uint4(pk[0], pk[1], pk[2], pk[3]);
    }
    l += sum0 + sum1;
    tc_fence_before_sync();
    fence_proxy_async_smem();
    exec_sync();
    if (tid == 0 && ok) {
      ok = wait(bar_v, j);
      if (ok) {
        tc_fence_after_sync();
        const uint32_t p = smem_u32(sP), vv = smem_u32(sV), idesc = umma_idesc_bf16(128, ncol) | (1u << 16);   // B is MN-major
#pragma unroll
        for (int i = 0; i < 8; ++i)
          umma_bf16(tmem_o, sw128_desc(p + (i >> 2) * kOperandTile + (i & 3) * 32u, 0, 1024),
                    sw128_desc(vv + i * 2048u, kOperandTile, 1024), idesc, (j | i) != 0);
        umma_commit(bar_o);
      }
    }
  }
  ok = ok && wait(bar_o, tiles - 1);
  ok = exec_and(ok);
  tc_fence_after_sync();
  if (ok) {
    const float inv = l > 0.f ? 1.f / l : 0.f;
    __nv_bfloat16* const out = reinterpret_cast<__nv_bfloat16*>(A.out) + static_cast<size_t>(row0 + q_pos) * A.ld_out + h * e;
    for (int c0 = 0; c0 < e; c0 += 8) {   // e is a multiple of 8; sixteen columns are read, eight may lie past it
      if ((c0 & 15) != 0) continue;
      uint32_t o[16];
      __syncwarp();
      tmem_ld_32x16(tmem_o + lane_off + c0, o);
      tmem_ld_wait();
      __syncwarp();
      if (q_pos < n) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          if (c0 + 8 * k >= e) continue;
          __nv_bfloat162 b[4];
#pragma unroll
          for (int i = 0; i < 4; ++i)
            b[i] = __floats2bfloat162_rn(__uint_as_float(o[8 * k + 2 * i]) * inv, __uint_as_float(o[8 * k + 2 * i + 1]) * inv);
          *reinterpret_cast<uint4*>(out + c0 + 8 * k) = *reinterpret_cast<const uint4*>(b);
        }
      }
    }
  }
  tc_fence_before_sync();
  exec_sync();
  if (tid == 0)
    for (int i = 0; i < 7; ++i) mbar_inval(bar + i);
  return ok;
}

__device__ bool tile_latent_direct(const TileDesc& t, int tid, const LayerCtx& ctx) { return latent_direct(t, tid, ctx); }

}  // namespace fab
}  // namespace mf
