// Latent attention of the layer-list decoders (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ latent attention
// Kind 59, LatentArgs: rows [i0, i0 + i1), one warp each: every head's query parts, the rotated one rotated; the latent,
// normed, and the shared rotated key part into the cache.  Interleaved pairs (2 i, 2 i + 1); cos_sin fp32
// [max_pos][r / 2][2].  V elements at a time (4 where the sizes allow it, else a pair), eight loads in flight.
template <int V>
__device__ __forceinline__ void act_st_vec(unsigned long long base, size_t i, bool f32, const float (&v)[V]) {
  if constexpr (V == 4) {
    if (f32) {
      *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + i) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
      const __nv_bfloat162 q[2] = {__floats2bfloat162_rn(v[0], v[1]), __floats2bfloat162_rn(v[2], v[3])};
      *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(base) + i) = *reinterpret_cast<const uint2*>(q);
    }
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) act_st(base, i + j, f32, v[j]);
  }
}
template <int V>
__device__ __forceinline__ void rotate_vec(float (&v)[V], const float2* cs, int pair) {
#pragma unroll
  for (int j = 0; j < V; j += 2) {
    const float2 q = cs[pair + j / 2];
    const float a = v[j], b = v[j + 1];
    v[j] = a * q.x - b * q.y;
    v[j + 1] = b * q.x + a * q.y;
  }
}

template <int V>
__device__ __noinline__ void latent_kv_rows(const TileDesc& t, int tid) {
  LatentArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31;
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), r = static_cast<int>(A.r), kvr = static_cast<int>(A.kv_rank);
  const bool f32 = A.f32 != 0;
  for (uint32_t row = t.i0 + warp; row < t.i0 + t.i1; row += kExecThreads / 32) {
    const float* src = f32p(A.qc) + static_cast<size_t>(row) * A.ld_qc;
    const int pos = min(reinterpret_cast<const int*>(A.tok_pos)[row], static_cast<int>(A.max_pos) - 1);
    const float2* cs = reinterpret_cast<const float2*>(A.cos_sin) + static_cast<size_t>(pos) * (r / 2);
    // queries: pieces of V (pairs of d's odd last element and the first rotated one cannot occur with V == 1)
    const int per = d + r, n = H * per / V;
    for (int i0 = lane; i0 < n; i0 += 32 * 8) {
      float v[8][V];
#pragma unroll
      for (int u = 0; u < 8; ++u)
        if (i0 + 32 * u < n) ld_vec<V>(src + (i0 + 32 * u) * V, v[u]);
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int at = (i0 + 32 * u) * V;
        if (i0 + 32 * u >= n) break;
        const int h = at / per, c = at - h * per;
        if (c < d) {
          act_st_vec<V>(A.q_un, (static_cast<size_t>(h) * A.rows_max + row) * A.ld_un + c, f32, v[u]);
        } else {
          if constexpr (V > 1) {
            rotate_vec<V>(v[u], cs, (c - d) / 2);
          } else {   // one element: its partner is the neighbour in memory
            const int k = c - d;
            const float2 q = cs[k / 2];
            const float other = src[at + ((k & 1) ? -1 : 1)];
            v[u][0] = (k & 1) ? v[u][0] * q.x + other * q.y : v[u][0] * q.x - other * q.y;
          }
          act_st_vec<V>(A.q_all, (static_cast<size_t>(h) * A.rows_max + row) * A.ld_q + kvr + c - d, f32, v[u]);
        }
      }
    }
    // latent and shared rotated part
    src += H * per;
    const size_t at = static_cast<size_t>(reinterpret_cast<const int*>(A.tok_slot)[row]) * A.ld_cache;
    const size_t copy = static_cast<size_t>(row) * A.ld_rows;
    auto put = [&](int c, const float (&v)[V]) {
      act_st_vec<V>(A.cache, at + c, f32, v);
      if (A.rows) act_st_vec<V>(A.rows, copy + c, f32, v);
    };
    float ss = 0.f;
    for (int c = lane * V; c < kvr; c += 32 * V) {
      float v[V];
      ld_vec<V>(src + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) ss = fmaf(v[j], v[j], ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(kvr) + A.eps);
    for (int c = lane * V; c < kvr; c += 32 * V) {
      float v[V], w[V];
      ld_vec<V>(src + c, v);
      ld_vec<V>(f32p(A.c_norm) + c, w);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = v[j] * inv * w[j];
      put(c, v);
    }
    for (int c = lane * V; c < r; c += 32 * V) {
      float v[V];
      ld_vec<V>(src + kvr + c, v);
      if constexpr (V > 1) {
        rotate_vec<V>(v, cs, c / 2);
      } else {
        const float2 q = cs[c / 2];
        const float other = src[kvr + c + ((c & 1) ? -1 : 1)];
        v[0] = (c & 1) ? v[0] * q.x + other * q.y : v[0] * q.x - other * q.y;
      }
      put(kvr + c, v);
    }
  }
}

__device__ void tile_latent_kv(const TileDesc& t, int tid) {
  const LatentArgs* p = reinterpret_cast<const LatentArgs*>(t.a[0]);
  if (((__ldcg(&p->d) | __ldcg(&p->r) | __ldcg(&p->kv_rank)) & 3) == 0) latent_kv_rows<4>(t, tid);
  else latent_kv_rows<1>(t, tid);
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

// Kind 61, LatentAttnArgs: items [i0, i0 + i1), item = row * heads + head, i2 parts (at most 32); parts added in order.
template <int V>
__device__ __noinline__ void latent_merge_items(const TileDesc& t, int tid) {
  LatentAttnArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, kvr = static_cast<int>(A.kv_rank), parts = static_cast<int>(t.i2);
  for (uint32_t it = t.i0 + warp; it < t.i0 + t.i1; it += kExecThreads / 32) {
    const int row = static_cast<int>(it / A.heads), h = static_cast<int>(it % A.heads);
    const float2* ml = reinterpret_cast<const float2*>(A.ws_ml) + static_cast<size_t>(it) * parts;
    const float2 mine = lane < parts ? ml[lane] : make_float2(-INFINITY, 0.f);
    float M = mine.x;
#pragma unroll
    for (int o = 16; o; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    const float w = expf(mine.x - M);
    const float scale = w / warp_sum(mine.y * w);   // this lane's part in the merged row
    const size_t o0 = (static_cast<size_t>(h) * A.rows_max + row) * A.ld_out;
    const float* src = f32p(A.ws_o) + static_cast<size_t>(it) * parts * kvr;
    for (int c0 = 0; c0 < kvr; c0 += 32 * V) {
      const int c = c0 + lane * V;
      float acc[V] = {};
      for (int q0 = 0; q0 < parts; q0 += 8) {
        float v[8][V];
#pragma unroll
        for (int q = 0; q < 8; ++q)
          if (c < kvr && q0 + q < parts) ld_vec<V>(src + static_cast<size_t>(q0 + q) * kvr + c, v[q]);
#pragma unroll
        for (int q = 0; q < 8; ++q) {
          const float s = __shfl_sync(0xffffffffu, scale, (q0 + q) & 31);
          if (c < kvr && q0 + q < parts)
#pragma unroll
            for (int j = 0; j < V; ++j) acc[j] = fmaf(v[q][j], s, acc[j]);
        }
      }
      if (c < kvr) act_st_vec<V>(A.out, o0 + c, A.f32 != 0, acc);
    }
  }
}

__device__ void tile_latent_merge(const TileDesc& t, int tid) {
  if ((__ldcg(&reinterpret_cast<const LatentAttnArgs*>(t.a[0])->kv_rank) & 3) == 0) latent_merge_items<4>(t, tid);
  else latent_merge_items<1>(t, tid);
}

}  // namespace fab
}  // namespace mf
