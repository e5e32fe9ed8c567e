// What surrounds grouped-query attention in the layer-list decoders, and its simple form (fabric_layer_tiles.cuh).  The
// fast form is the paged attention of fabric_seq_tiles.cuh / attention_core.cuh on heads padded to 128 columns.
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// Kind 70, QkvArgs: items [i0, i0 + i1), item = row * (heads + 2 kv_heads) + query heads, then key heads, then value
// heads.  Eight columns per lane (V = 8: 16-byte pieces of bf16), as many items side by side in a warp as fit.
template <int V>
__device__ __noinline__ void qkv_items(const TileDesc& t, int tid) {
  QkvArgs A;
  load_block(A, t.a[0]);
  const int H = static_cast<int>(A.heads), G = static_cast<int>(A.kv_heads), per = H + 2 * G;
  const int d = static_cast<int>(A.d), e = static_cast<int>(A.e);
  const bool f32 = A.f32 != 0;
  const int widest = static_cast<int>(max(max(A.ld_q, A.ld_k), A.ld_v));
  int lanes = 1;   // of an item
  while (lanes < 32 && lanes * V < widest) lanes <<= 1;
  const int at_once = kExecThreads / lanes, mine = tid / lanes, l = tid & (lanes - 1);
  for (uint32_t it0 = t.i0; it0 < t.i0 + t.i1; it0 += at_once) {   // uniform: every lane takes part in the sums
    const bool ok = it0 + mine < t.i0 + t.i1;
    const uint32_t it = ok ? it0 + mine : t.i0 + t.i1 - 1;
    const uint32_t row = it / per;
    const int k = static_cast<int>(it % per);
    const bool is_q = k < H, is_v = k >= H + G;
    const int n = is_v ? e : d, head = is_q ? k : is_v ? k - H - G : k - H;
    const unsigned long long src = is_q ? A.q : is_v ? A.v : A.k, wn = is_q ? A.q_norm : is_v ? 0ull : A.k_norm;
    const int ld = static_cast<int>(is_q ? A.ld_q : is_v ? A.ld_v : A.ld_k);
    const size_t s0 = static_cast<size_t>(row) * A.ld_x + static_cast<size_t>(head) * n;
    const size_t place = is_q ? row : static_cast<size_t>(reinterpret_cast<const int*>(A.tok_slot)[row]);
    const unsigned long long dst = is_q ? A.q_out : is_v ? A.v_cache : A.k_cache;
    const size_t d0 = (place * (is_q ? H : G) + head) * ld;
    auto load = [&](int c, float (&v)[V]) {
      if constexpr (V == 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(src) + s0 + c);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(h[i]);
          v[2 * i] = f.x;
          v[2 * i + 1] = f.y;
        }
      } else {
        v[0] = act_ld(src, s0 + c, f32);
      }
    };
    float first[V];   // most heads are one piece per lane
    float ss = 0.f;
    for (int c = l * V; c < n; c += lanes * V) {
      float v[V];
      load(c, v);
      if (c == l * V)
#pragma unroll
        for (int j = 0; j < V; ++j) first[j] = v[j];
#pragma unroll
      for (int j = 0; j < V; ++j) ss = fmaf(v[j], v[j], ss);
    }
    for (int o = lanes >> 1; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!ok) continue;
    const float inv = wn ? 1.f / sqrtf(ss / static_cast<float>(n) + A.eps) : 1.f;
    for (int c = l * V; c < ld; c += lanes * V) {
      float v[V];
      if (c < n) {
        if (c == l * V) {
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = first[j];
        } else {
          load(c, v);
        }
        if (wn)
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = v[j] * inv * f32p(wn)[c + j];
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = 0.f;
      }
      if constexpr (V == 8) {
        __nv_bfloat162 h[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(dst) + d0 + c) = *reinterpret_cast<const uint4*>(h);
      } else {
        act_st(dst, d0 + c, f32, v[0]);
      }
    }
  }
}

// The same for heads that are one 16-byte piece per lane at most: four rounds of items in flight.
__device__ __noinline__ void qkv_narrow(const TileDesc& t, int tid) {
  constexpr int U = 4;
  QkvArgs A;
  load_block(A, t.a[0]);
  const int H = static_cast<int>(A.heads), G = static_cast<int>(A.kv_heads), per = H + 2 * G;
  const int widest = static_cast<int>(max(max(A.ld_q, A.ld_k), A.ld_v));
  int lanes = 1;   // of an item
  while (lanes * 8 < widest) lanes <<= 1;
  const int at_once = kExecThreads / lanes, mine = tid / lanes, c = (tid & (lanes - 1)) * 8;
  const uint32_t end = t.i0 + t.i1;
  for (uint32_t it0 = t.i0 + mine; it0 - mine < end; it0 += U * at_once) {
    uint4 raw[U];
    __nv_bfloat16* to[U];
    const float* w[U];
    int n[U];
    float ss[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t it = min(it0 + u * at_once, end - 1), row = it / per;
      const int k = static_cast<int>(it - row * per);
      const bool is_q = k < H, is_v = k >= H + G;
      const int head = is_q ? k : is_v ? k - H - G : k - H;
      n[u] = static_cast<int>(is_v ? A.e : A.d);
      w[u] = is_v ? nullptr : f32p(is_q ? A.q_norm : A.k_norm);
      const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(is_q ? A.q : is_v ? A.v : A.k) + static_cast<size_t>(row) * A.ld_x + static_cast<size_t>(head) * n[u];
      raw[u] = c < n[u] ? *reinterpret_cast<const uint4*>(src + c) : make_uint4(0, 0, 0, 0);
      const int ld = static_cast<int>(is_q ? A.ld_q : is_v ? A.ld_v : A.ld_k);
      const size_t place = is_q ? row : static_cast<size_t>(reinterpret_cast<const int*>(A.tok_slot)[row]);
      to[u] = it0 + u * at_once < end && c < ld
                  ? reinterpret_cast<__nv_bfloat16*>(is_q ? A.q_out : is_v ? A.v_cache : A.k_cache) + (place * (is_q ? H : G) + head) * ld + c
                  : nullptr;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw[u]);
      ss[u] = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        ss[u] = fmaf(f.x, f.x, fmaf(f.y, f.y, ss[u]));
      }
    }
    for (int o = lanes >> 1; o; o >>= 1)
#pragma unroll
      for (int u = 0; u < U; ++u) ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (!to[u]) continue;
      if (w[u] && c < n[u]) {
        const float inv = 1.f / sqrtf(ss[u] / static_cast<float>(n[u]) + A.eps);
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw[u]);
        float wv[8];
        ld_vec<4>(w[u] + c, *reinterpret_cast<float(*)[4]>(wv));
        ld_vec<4>(w[u] + c + 4, *reinterpret_cast<float(*)[4]>(wv + 4));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(h[i]);
          h[i] = __floats2bfloat162_rn(f.x * inv * wv[2 * i], f.y * inv * wv[2 * i + 1]);
        }
      }
      *reinterpret_cast<uint4*>(to[u]) = raw[u];
    }
  }
}

__device__ void tile_qkv(const TileDesc& t, int tid) {
  const QkvArgs* p = reinterpret_cast<const QkvArgs*>(t.a[0]);
  const uint32_t cols = __ldcg(&p->d) | __ldcg(&p->e) | __ldcg(&p->ld_q) | __ldcg(&p->ld_k) | __ldcg(&p->ld_v) | __ldcg(&p->ld_x);
  const unsigned long long at = __ldcg(&p->q) | __ldcg(&p->k) | __ldcg(&p->v);
  const bool pieces = !__ldcg(&p->f32) && (cols & 7) == 0 && (at & 15) == 0;
  if (pieces && max(max(__ldcg(&p->ld_q), __ldcg(&p->ld_k)), __ldcg(&p->ld_v)) <= 256) qkv_narrow(t, tid);
  else if (pieces) qkv_items<8>(t, tid);
  else qkv_items<1>(t, tid);
}

// Kind 71, GroupedAttnArgs: row i0, query heads i1 & 0xffff .. (i1 >> 16 of them), slot a[1]; one warp per head, all keys
// of the row in order, four at a time.  32-bit scores, weights and sums.
template <int NR, bool F32>
__device__ __noinline__ void grouped_attn_warps(const TileDesc& t, int tid) {
  GroupedAttnArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, d = static_cast<int>(A.d), e = static_cast<int>(A.e);
  const int row = static_cast<int>(t.i0), page = static_cast<int>(A.page), G = static_cast<int>(A.kv_heads);
  const int keys = reinterpret_cast<const int*>(A.tok_pos)[row] + 1, group = static_cast<int>(A.heads) / G;
  const int* bt = reinterpret_cast<const int*>(A.block_table) + static_cast<size_t>(t.a[1]) * A.bt_stride;
  const int h0 = static_cast<int>(t.i1 & 0xffffu), nh = static_cast<int>(t.i1 >> 16);
  for (int h = h0 + warp; h < h0 + nh; h += kExecThreads / 32) {
    const int kh = h / group;
    float q[NR], acc[NR];
    const size_t q0 = (static_cast<size_t>(row) * A.heads + h) * A.ld_q;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      q[i] = i * 32 + lane < d ? act_ld(A.q, q0 + i * 32 + lane, F32) * A.scale : 0.f;
      acc[i] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    constexpr int KU = NR <= 4 ? 4 : 2;
    for (int k0 = 0; k0 < keys; k0 += KU) {
      float v[KU][NR], s[KU];
#pragma unroll
      for (int u = 0; u < KU; ++u) {
        const int k = min(k0 + u, keys - 1);
        const size_t at = (static_cast<size_t>(bt[k / page]) * page + k % page) * G + kh;
        float kv[NR];
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          kv[i] = i * 32 + lane < d ? act_ld(A.k_cache, at * A.ld_k + i * 32 + lane, F32) : 0.f;
          v[u][i] = i * 32 + lane < e ? act_ld(A.v_cache, at * A.ld_v + i * 32 + lane, F32) : 0.f;
        }
        s[u] = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) s[u] = fmaf(q[i], kv[i], s[u]);
      }
#pragma unroll
      for (int u = 0; u < KU; ++u) s[u] = warp_sum(s[u]);
      float mx = m;
#pragma unroll
      for (int u = 0; u < KU; ++u) {
        if (k0 + u >= keys) s[u] = -INFINITY;
        mx = fmaxf(mx, s[u]);
      }
      const float f = expf(m - mx);
      m = mx;
      l *= f;
#pragma unroll
      for (int i = 0; i < NR; ++i) acc[i] *= f;
#pragma unroll
      for (int u = 0; u < KU; ++u) {
        const float p = expf(s[u] - mx);
        l += p;
#pragma unroll
        for (int i = 0; i < NR; ++i) acc[i] = fmaf(p, v[u][i], acc[i]);
      }
    }
    const float inv = 1.f / l;
    const size_t o0 = (static_cast<size_t>(row) * A.heads + h) * A.ld_out;
#pragma unroll
    for (int i = 0; i < NR; ++i)
      if (i * 32 + lane < e) act_st(A.out, o0 + i * 32 + lane, F32, acc[i] * inv);
  }
}

__device__ bool tile_grouped_attn(const TileDesc& t, int tid) {
  const GroupedAttnArgs* p = reinterpret_cast<const GroupedAttnArgs*>(t.a[0]);
  const uint32_t nr = (max(__ldcg(&p->d), __ldcg(&p->e)) + 31) / 32;
  const bool f32 = __ldcg(&p->f32) != 0;
#define MF_GROUPED(N)                             \
  if (nr <= N) {                                  \
    if (f32) grouped_attn_warps<N, true>(t, tid); \
    else grouped_attn_warps<N, false>(t, tid);    \
    return true;                                  \
  }
  MF_GROUPED(2)
  MF_GROUPED(4)
  MF_GROUPED(8)
  MF_GROUPED(16)
#undef MF_GROUPED
  return false;
}

// Kind 72, HeadGateArgs: rows [i0, i0 + i1), one warp each.
template <int V>
__device__ __noinline__ void head_gate_rows(const TileDesc& t, int tid) {
  HeadGateArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, H = static_cast<int>(A.heads), e = static_cast<int>(A.e), n = H * e;
  const bool f32 = A.f32 != 0;
  for (uint32_t row = t.i0 + warp; row < t.i0 + t.i1; row += kExecThreads / 32)
#pragma unroll 4
    for (int c = lane * V; c < n; c += 32 * V) {
      const int h = c / e;
      const float z = act_ld(A.g, static_cast<size_t>(row) * A.ld_g + h, f32);
      const float g = f32 ? sigmoid32(z) : __fdividef(1.f, 1.f + __expf(-z));
      const size_t src = (static_cast<size_t>(row) * H + h) * A.ld_in + c - h * e, dst = static_cast<size_t>(row) * A.ld_out + c;
      if constexpr (V == 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(A.in) + src);
        const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&raw);
        __nv_bfloat162 o[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(x[i]);
          o[i] = __floats2bfloat162_rn(f.x * g, f.y * g);
        }
        *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(A.out) + dst) = *reinterpret_cast<const uint4*>(o);
      } else {
        act_st(A.out, dst, f32, act_ld(A.in, src, f32) * g);
      }
    }
}

__device__ void tile_head_gate(const TileDesc& t, int tid) {
  const HeadGateArgs* p = reinterpret_cast<const HeadGateArgs*>(t.a[0]);
  if (!__ldcg(&p->f32) && (__ldcg(&p->in) & 15) == 0 && ((__ldcg(&p->e) | __ldcg(&p->ld_in) | __ldcg(&p->ld_out)) & 7) == 0) head_gate_rows<8>(t, tid);
  else head_gate_rows<1>(t, tid);
}

}  // namespace fab
}  // namespace mf
