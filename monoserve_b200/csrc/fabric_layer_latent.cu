// Latent attention of the layer-list decoders (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ latent attention
// Kind 59, LatentArgs: items [i0, i0 + i1), item = row * (heads + 1) + j, one warp each.  j < heads: the head's query
// parts, the rotated one rotated; j == heads: the latent, normed, and the shared rotated key part into the cache.
// Interleaved pairs (2 i, 2 i + 1); cos_sin fp32 [max_pos][r / 2][2].
__device__ void tile_latent_kv(const TileDesc& t, int tid) {
  LatentArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31;
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), r = static_cast<int>(A.r), kvr = static_cast<int>(A.kv_rank);
  for (uint32_t it = t.i0 + warp; it < t.i0 + t.i1; it += kExecThreads / 32) {
    const int row = static_cast<int>(it / (H + 1)), j = static_cast<int>(it % (H + 1));
    const float* src = f32p(A.qc) + static_cast<size_t>(row) * A.ld_qc;
    const int pos = min(reinterpret_cast<const int*>(A.tok_pos)[row], static_cast<int>(A.max_pos) - 1);
    const float2* cs = reinterpret_cast<const float2*>(A.cos_sin) + static_cast<size_t>(pos) * (r / 2);
    const float* rot;
    unsigned long long dst;
    size_t at;
    if (j < H) {
      src += j * (d + r);
      const size_t un = (static_cast<size_t>(j) * A.rows_max + row) * A.ld_un;
      for (int c = lane; c < d; c += 32) act_st(A.q_un, un + c, A.f32, src[c]);
      rot = src + d;
      dst = A.q_all;
      at = (static_cast<size_t>(j) * A.rows_max + row) * A.ld_q + kvr;
    } else {
      src += H * (d + r);
      dst = A.cache;
      at = static_cast<size_t>(reinterpret_cast<const int*>(A.tok_slot)[row]) * A.ld_cache;
      float ss = 0.f;
      for (int c = lane; c < kvr; c += 32) ss = fmaf(src[c], src[c], ss);
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(kvr) + A.eps);
      for (int c = lane; c < kvr; c += 32) act_st(dst, at + c, A.f32, src[c] * inv * f32p(A.c_norm)[c]);
      rot = src + kvr;
      at += kvr;
    }
    for (int i = lane; i < r / 2; i += 32) {
      const float u = rot[2 * i], v = rot[2 * i + 1];
      const float2 q = cs[i];
      act_st(dst, at + 2 * i, A.f32, u * q.x - v * q.y);
      act_st(dst, at + 2 * i + 1, A.f32, v * q.x + u * q.y);
    }
  }
}

// Kind 60, LatentAttnArgs: row i0, heads i1 & 0xffff .. (i1 >> 16 of them), part i2 of i3 equal key ranges, slot a[1].
// One warp per head: the absorbed query (kv_rank latent columns, r rotated ones) against every cached row it sees, the
// weighted sum of the latents as the output.  i3 = 1 writes `out`; otherwise the unnormalised sum with (max, sum).
template <int NR, bool F32>
__device__ __noinline__ void latent_attn_warps(const TileDesc& t, int tid) {
  LatentAttnArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31;
  const int row = static_cast<int>(t.i0), H = static_cast<int>(A.heads), kvr = static_cast<int>(A.kv_rank);
  const int dims = kvr + static_cast<int>(A.r), page = static_cast<int>(A.page);
  const int keys = reinterpret_cast<const int*>(A.tok_pos)[row] + 1;
  const int parts = static_cast<int>(t.i3), part = static_cast<int>(t.i2);
  const int per = (keys + parts - 1) / parts;
  const int k_lo = min(part * per, keys), k_hi = min(k_lo + per, keys);
  const int* bt = reinterpret_cast<const int*>(A.block_table) + static_cast<size_t>(t.a[1]) * A.bt_stride;
  const int h0 = static_cast<int>(t.i1 & 0xffffu), nh = static_cast<int>(t.i1 >> 16);
  for (int h = h0 + warp; h < h0 + nh; h += kExecThreads / 32) {
    float q[NR], acc[NR];
    const size_t q0 = (static_cast<size_t>(h) * A.rows_max + row) * A.ld_q;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      q[i] = i * 32 + lane < dims ? act_ld(A.q, q0 + i * 32 + lane, F32) * A.scale : 0.f;
      acc[i] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    for (int k0 = k_lo; k0 < k_hi; k0 += 2) {
      float kv[2][NR], s[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int k = min(k0 + u, k_hi - 1);
        const size_t at = (static_cast<size_t>(bt[k / page]) * page + k % page) * A.ld_cache;
        s[u] = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) kv[u][i] = i * 32 + lane < dims ? act_ld(A.cache, at + i * 32 + lane, F32) : 0.f;
      }
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int i = 0; i < NR; ++i) s[u] = fmaf(q[i], kv[u][i], s[u]);
#pragma unroll
      for (int u = 0; u < 2; ++u) s[u] = warp_sum(s[u]);
      if (k0 + 1 >= k_hi) s[1] = -INFINITY;
      const float mx = fmaxf(m, fmaxf(s[0], s[1]));
      const float f = expf(m - mx), p0 = expf(s[0] - mx), p1 = expf(s[1] - mx);
      m = mx;
      l = fmaf(l, f, p0 + p1);
#pragma unroll
      for (int i = 0; i < NR; ++i) acc[i] = fmaf(acc[i], f, fmaf(p0, kv[0][i], p1 * kv[1][i]));
    }
    if (parts == 1) {
      const float inv = 1.f / l;
      const size_t o0 = (static_cast<size_t>(h) * A.rows_max + row) * A.ld_out;
#pragma unroll
      for (int i = 0; i < NR; ++i)
        if (i * 32 + lane < kvr) act_st(A.out, o0 + i * 32 + lane, F32, acc[i] * inv);
    } else {
      const size_t w = (static_cast<size_t>(row) * H + h) * parts + part;
      float* o = reinterpret_cast<float*>(A.ws_o) + w * kvr;
#pragma unroll
      for (int i = 0; i < NR; ++i)
        if (i * 32 + lane < kvr) o[i * 32 + lane] = acc[i];
      if (lane == 0) reinterpret_cast<float2*>(A.ws_ml)[w] = make_float2(m, l);   // no keys: (-inf, 0)
    }
  }
}

__device__ bool tile_latent_attn(const TileDesc& t, int tid) {
  const LatentAttnArgs* p = reinterpret_cast<const LatentAttnArgs*>(t.a[0]);
  const uint32_t nr = (__ldcg(&p->kv_rank) + __ldcg(&p->r) + 31) / 32;
  const bool f32 = __ldcg(&p->f32) != 0;
#define MF_LATENT(N)                            \
  if (nr <= N) {                                \
    if (f32) latent_attn_warps<N, true>(t, tid); \
    else latent_attn_warps<N, false>(t, tid);   \
    return true;                                \
  }
  MF_LATENT(4)
  MF_LATENT(9)
  MF_LATENT(18)
  MF_LATENT(36)
#undef MF_LATENT
  return false;
}

// Kind 61, LatentAttnArgs: items [i0, i0 + i1), item = row * heads + head, i2 parts; parts added in order.
__device__ void tile_latent_merge(const TileDesc& t, int tid) {
  LatentAttnArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, kvr = static_cast<int>(A.kv_rank), parts = static_cast<int>(t.i2);
  for (uint32_t it = t.i0 + warp; it < t.i0 + t.i1; it += kExecThreads / 32) {
    const int row = static_cast<int>(it / A.heads), h = static_cast<int>(it % A.heads);
    const float2* ml = reinterpret_cast<const float2*>(A.ws_ml) + static_cast<size_t>(it) * parts;
    float M = -INFINITY, L = 0.f;
    for (int q = 0; q < parts; ++q) M = fmaxf(M, ml[q].x);
    for (int q = 0; q < parts; ++q) L += ml[q].y * expf(ml[q].x - M);
    const float inv = 1.f / L;
    const size_t o0 = (static_cast<size_t>(h) * A.rows_max + row) * A.ld_out;
    for (int c = lane; c < kvr; c += 32) {
      float acc = 0.f;
      for (int q = 0; q < parts; ++q)
        acc = fmaf(f32p(A.ws_o)[(static_cast<size_t>(it) * parts + q) * kvr + c], expf(ml[q].x - M), acc);
      act_st(A.out, o0 + c, A.f32, acc * inv);
    }
  }
}

}  // namespace fab
}  // namespace mf
