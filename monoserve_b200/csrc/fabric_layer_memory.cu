// The matrix memory of the layer-list decoders (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"
#include "wide_tile.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ matrix memory
// Packed fp32 pairs (each half rounded like the scalar instruction).
__device__ __forceinline__ unsigned long long pk2(float a, float b) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpk2(unsigned long long v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// Kind 57, MemoryArgs: rows [i0, i0 + i1) of one request; i2 = head | column block << 16 (32 of the e + 1 columns of
// the augmented memory, whose column e accumulates k alone: the normaliser); slot i3.  A wide tile: keys, queries and
// values come `tokens` rows at a time through double-buffered asynchronous copies into the operand ring.  A warp holds
// eight columns, a lane four-row groups 4 lane + 128 i of each, in registers for the whole portion.  Each lane prepares
// one token's gates, with F the running sum of the log forget gates.
constexpr int kMemColumns = 32;

template <bool F32>
__device__ __forceinline__ float4 ld_four(const void* p) {
  if constexpr (F32) return *reinterpret_cast<const float4*>(p);
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}

// Log gate of a head from its raw projection: cap tanh(z / cap), the forget gate through log sigmoid.
__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// The raw gate at `p`: the sum of a K-split product's slabs.
__device__ __forceinline__ float raw_gate(const MemoryArgs& A, const float* p) {
  float v = *p;
  for (uint32_t q = 1; q < A.gate_parts; ++q) v += p[static_cast<size_t>(q) * A.gate_rows * A.ld_gates];
  return v;
}

// R values per lane (R <= 32, a power of two) summed over the warp: lane l ends with the sum of value l / (32 / R).
template <int R>
__device__ __forceinline__ float warp_sum_each(float (&r)[R], int lane) {
#pragma unroll
  for (int half = R / 2, bit = 16; half >= 1; half >>= 1, bit >>= 1) {
    const bool hi = lane & bit;
#pragma unroll
    for (int c = 0; c < half; ++c) {
      const float give = hi ? r[c] : r[c + half], have = hi ? r[c + half] : r[c];
      r[c] = have + __shfl_xor_sync(0xffffffffu, give, bit);
    }
  }
#pragma unroll
  for (int bit = 16 / R; bit >= 1; bit >>= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], bit);
  return r[0];
}

template <int ND, bool F32>
__device__ __noinline__ void memory_rows(const TileDesc& t, int tid, uint8_t* ring) {
  using T = typename std::conditional<F32, float, __nv_bfloat16>::type;
  constexpr int kPer16 = 16 / static_cast<int>(sizeof(T));
  constexpr int kTokens = (ND == 4 && F32) ? 16 : 32, kGroup = ND == 4 ? 2 : 4;
  MemoryArgs A;
  load_block(A, t.a[0]);
  __builtin_assume(__isShared(ring));
  const int row0 = static_cast<int>(t.i0), rows = static_cast<int>(t.i1), slot = static_cast<int>(t.i3);
  const int head = static_cast<int>(t.i2 & 0xffffu), col0 = static_cast<int>(t.i2 >> 16) * kMemColumns;
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e);
  const int dp = (d + 3) & ~3, ds = (d + 7) & ~7, oe = (e + 4) & ~3, warp = tid >> 5, lane = tid & 31;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  T* const buf = reinterpret_cast<T*>(ring);
  const int buf_elems = kTokens * (2 * ds + kMemColumns);   // k, q, v
  const int c_lo = col0 + warp * 8;                          // this warp's first column
  const bool edge = c_lo + 8 > e;
  const int n_v = min(kMemColumns, e - col0);                // columns of v in this block (at most 0: only the normaliser)
  float* const state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * H + head) * (e + 1) * dp;
  unsigned long long S[8][ND][2];
#pragma unroll
  for (int c = 0; c < 8; ++c)
#pragma unroll
    for (int i = 0; i < ND; ++i) {
      const int at = i * 128 + lane * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && at < dp && c_lo + c <= e) v = *reinterpret_cast<const float4*>(state + static_cast<size_t>(c_lo + c) * dp + at);
      S[c][i][0] = pk2(v.x, v.y);
      S[c][i][1] = pk2(v.z, v.w);
    }
  // every column block computes the same m and keeps a copy of its own
  float* const m_state = reinterpret_cast<float*>(A.m) +
                         (static_cast<size_t>(slot) * H + head) * ((e + kMemColumns) / kMemColumns) + (t.i2 >> 16);
  float m0 = fresh ? 0.f : *m_state;
  const float *gates = f32p(A.gates), bi = f32p(A.gate_bias)[head], bf = f32p(A.gate_bias)[H + head];
  const T *gk = reinterpret_cast<const T*>(A.k) + head * d, *gq = reinterpret_cast<const T*>(A.q) + head * d;
  const T* gv = reinterpret_cast<const T*>(A.v) + head * e + col0;
  const bool kq16 = d % kPer16 == 0 && ((A.k | A.q) & 15) == 0;
  const bool v16 = e % kPer16 == 0 && n_v > 0 && n_v % kPer16 == 0 && (A.v & 15) == 0;
  if (d & 3) {   // the padding of keys and queries stays zero
    for (int i = tid; i < 2 * buf_elems; i += kExecThreads) buf[i] = static_cast<T>(0.f);
    exec_sync();
  }
  auto stage = [&](int base, T* b) {
    const int nt = min(kTokens, rows - base);
    for (int tok = warp; tok < nt; tok += kExecThreads / 32) {
      const size_t at = static_cast<size_t>(row0 + base + tok) * A.ld_qkv;
      T *k = b + tok * ds, *q = b + (kTokens + tok) * ds, *v = b + 2 * kTokens * ds + tok * kMemColumns;
      if (kq16) {
        for (int p = lane; p < d / kPer16; p += 32) {
          cp16(k + p * kPer16, gk + at + p * kPer16);
          cp16(q + p * kPer16, gq + at + p * kPer16);
        }
      } else {
        for (int p = lane; p < d; p += 32) {
          k[p] = gk[at + p];
          q[p] = gq[at + p];
        }
      }
      if (v16) {
        if (lane < n_v / kPer16) cp16(v + lane * kPer16, gv + at + lane * kPer16);
      } else if (lane < n_v) {
        v[lane] = gv[at + lane];
      }
    }
    cp_commit();
  };
  auto load_gates = [&](int base, float& gi, float& gf) {   // one token per lane
    const int nt = min(kTokens, rows - base);
    const size_t at = static_cast<size_t>(row0 + base + min(lane, nt - 1)) * A.ld_gates + head;
    gi = lane < nt ? capped(raw_gate(A, gates + at) + bi, A.cap) : -INFINITY;
    gf = lane < nt ? log_sigmoid(capped(raw_gate(A, gates + at + H) + bf, A.cap)) : 0.f;
  };
  stage(0, buf);
  float gi, gf;
  load_gates(0, gi, gf);
  for (int base = 0, s = 0; base < rows; base += kTokens, s ^= 1) {
    const int nt = min(kTokens, rows - base);
    float gi_next = 0.f, gf_next = 0.f;
    if (base + kTokens < rows) {
      stage(base + kTokens, buf + (s ^ 1) * buf_elems);
      load_gates(base + kTokens, gi_next, gf_next);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    float F = gf;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, F, o);
      if (lane >= o) F += v;
    }
    // M_t = max(m_0, max_{s <= t} (i_s - F_s)): m_t = F_t + M_t, so f_t + m_(t-1) - m_t is M_(t-1) - M_t, which is
    // exactly zero while the maximum decays, and i_t - m_t is (i_t - F_t) - M_t
    const float rel = gi - F;
    float M = rel;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) M = fmaxf(M, v);
    }
    M = fmaxf(m0, M);
    const float M_up = __shfl_up_sync(0xffffffffu, M, 1), m = F + M;
    const float keep = expf((lane == 0 ? m0 : M_up) - M), add = expf(rel - M), floor_ = expf(-m);
    m0 = __shfl_sync(0xffffffffu, m, nt - 1);
    exec_sync();
    const T* const sk = buf + s * buf_elems;
    const T* const sq = sk + kTokens * ds;
    const T* const sv = sq + kTokens * ds + warp * 8;
#pragma unroll 1
    for (int t0 = 0; t0 < nt; t0 += kGroup) {   // the read-outs of kGroup tokens are summed over the warp together
      float r[8 * kGroup];                       // [token][column]
#pragma unroll
      for (int u = 0; u < kGroup; ++u) {
        const int tok = min(t0 + u, nt - 1);
        float kp = __shfl_sync(0xffffffffu, keep, tok), ad = __shfl_sync(0xffffffffu, add, tok);
        if (t0 + u >= nt) {                      // a token past the end keeps the state and adds nothing
          kp = 1.f;
          ad = 0.f;
        }
        const unsigned long long kp2 = pk2(kp, kp);
        const float4 va = ld_four<F32>(sv + tok * kMemColumns), vb = ld_four<F32>(sv + tok * kMemColumns + 4);
        float v[8] = {va.x, va.y, va.z, va.w, vb.x, vb.y, vb.z, vb.w};
        if (edge) {                              // this warp's columns reach past the values: the normaliser's v is 1
#pragma unroll
          for (int c = 0; c < 8; ++c) v[c] = c_lo + c < e ? v[c] : (c_lo + c == e ? 1.f : 0.f);
        }
        unsigned long long kk[ND][2], qq[ND][2];
#pragma unroll
        for (int i = 0; i < ND; ++i) {
          const int at = i * 128 + lane * 4;
          float4 k4 = make_float4(0.f, 0.f, 0.f, 0.f), q4 = k4;
          if (at < dp) {
            k4 = ld_four<F32>(sk + tok * ds + at);
            q4 = ld_four<F32>(sq + tok * ds + at);
          }
          kk[i][0] = mul2(pk2(ad, ad), pk2(k4.x, k4.y));
          kk[i][1] = mul2(pk2(ad, ad), pk2(k4.z, k4.w));
          qq[i][0] = pk2(q4.x, q4.y);
          qq[i][1] = pk2(q4.z, q4.w);
        }
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          unsigned long long acc = 0ull;
          const unsigned long long v2 = pk2(v[c], v[c]);
#pragma unroll
          for (int i = 0; i < ND; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              S[c][i][j] = fma2(v2, kk[i][j], mul2(kp2, S[c][i][j]));
              acc = fma2(S[c][i][j], qq[i][j], acc);
            }
          const float2 f = unpk2(acc);
          r[u * 8 + c] = f.x + f.y;
        }
      }
      const float read = warp_sum_each<8 * kGroup>(r, lane) * A.q_scale;
      constexpr int kStep = 4 / kGroup;          // lanes per sum
      const int tok = t0 + lane / (8 * kStep), c = c_lo + (lane / kStep) % 8;
      const float fl = __shfl_sync(0xffffffffu, floor_, tok & 31);
      if (lane % kStep == 0 && tok < nt && c <= e)
        reinterpret_cast<float*>(A.out)[(static_cast<size_t>(row0 + base + tok) * H + head) * oe + c] =
            c < e ? read : fmaxf(fabsf(read), fl) + 1e-6f;
    }
    gi = gi_next;
    gf = gf_next;
    exec_sync();
  }
#pragma unroll
  for (int c = 0; c < 8; ++c)
#pragma unroll
    for (int i = 0; i < ND; ++i) {
      const int at = i * 128 + lane * 4;
      if (at < dp && c_lo + c <= e) {
        const float2 a = unpk2(S[c][i][0]), b = unpk2(S[c][i][1]);
        *reinterpret_cast<float4*>(state + static_cast<size_t>(c_lo + c) * dp + at) = make_float4(a.x, a.y, b.x, b.y);
      }
    }
  if (tid == 0) *m_state = m0;
}

// Kind 56, MemoryArgs: one token.  Row i0, i2 = head | first column block << 16, i1 column blocks, slot i3.  The state
// streams through registers, the next block's loads issued before this one's arithmetic.
template <int ND, bool F32>
__device__ __noinline__ void memory_step(const TileDesc& t, int tid) {
  using T = typename std::conditional<F32, float, __nv_bfloat16>::type;
  MemoryArgs A;
  load_block(A, t.a[0]);
  const int row = static_cast<int>(t.i0), slot = static_cast<int>(t.i3), n_blocks = static_cast<int>(t.i1);
  const int head = static_cast<int>(t.i2 & 0xffffu), block0 = static_cast<int>(t.i2 >> 16);
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e);
  const int dp = (d + 3) & ~3, oe = (e + 4) & ~3, warp = tid >> 5, lane = tid & 31;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row] == 0;
  const size_t at_row = static_cast<size_t>(row) * A.ld_qkv;
  const T *gk = reinterpret_cast<const T*>(A.k) + at_row + head * d, *gq = reinterpret_cast<const T*>(A.q) + at_row + head * d;
  const T* gv = reinterpret_cast<const T*>(A.v) + at_row + head * e;
  float* const m_state = reinterpret_cast<float*>(A.m) + (static_cast<size_t>(slot) * H + head) * ((e + kMemColumns) / kMemColumns);
  float* const state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * H + head) * (e + 1) * dp;
  const float* gates = f32p(A.gates) + static_cast<size_t>(row) * A.ld_gates;
  auto value = [](const T& v) -> float {
    if constexpr (F32) return v;
    else return __bfloat162float(v);
  };
  float4 st[2][8][ND];
  float v8[2][8];
  auto fetch = [&](int b, float4 (&S)[8][ND], float (&v)[8]) {
    const int c_lo = b * kMemColumns + warp * 8;
#pragma unroll
    for (int c = 0; c < 8; ++c) {
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        const int at = i * 128 + lane * 4;
        S[c][i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && at < dp && c_lo + c <= e) S[c][i] = __ldcs(reinterpret_cast<const float4*>(state + static_cast<size_t>(c_lo + c) * dp + at));
      }
      v[c] = c_lo + c < e ? value(gv[c_lo + c]) : (c_lo + c == e ? 1.f : 0.f);
    }
  };
  fetch(block0, st[0], v8[0]);
  const float m_old = fresh ? 0.f : m_state[block0];
  float k[ND][4], q[ND][4];
#pragma unroll
  for (int i = 0; i < ND; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int at = i * 128 + lane * 4 + j;
      k[i][j] = at < d ? value(gk[at]) : 0.f;
      q[i][j] = at < d ? value(gq[at]) * A.q_scale : 0.f;
    }
  const float gi = capped(raw_gate(A, gates + head) + f32p(A.gate_bias)[head], A.cap);
  const float gf = log_sigmoid(capped(raw_gate(A, gates + H + head) + f32p(A.gate_bias)[H + head], A.cap));
  const float m = fmaxf(gf + m_old, gi);
  const float keep = expf(gf + m_old - m), add = expf(gi - m), floor_ = expf(-m);
  exec_sync();   // every thread has read the old maximum
  auto run = [&](int b, float4 (&S)[8][ND], const float (&v)[8]) {
    const int c_lo = b * kMemColumns + warp * 8;
    float r[8];
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      const float av = add * v[c];
      r[c] = 0.f;
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        float4 s = S[c][i];
        s.x = fmaf(av, k[i][0], keep * s.x);
        s.y = fmaf(av, k[i][1], keep * s.y);
        s.z = fmaf(av, k[i][2], keep * s.z);
        s.w = fmaf(av, k[i][3], keep * s.w);
        r[c] = fmaf(s.x, q[i][0], fmaf(s.y, q[i][1], fmaf(s.z, q[i][2], fmaf(s.w, q[i][3], r[c]))));
        const int at = i * 128 + lane * 4;
        if (at < dp && c_lo + c <= e) __stcs(reinterpret_cast<float4*>(state + static_cast<size_t>(c_lo + c) * dp + at), s);
      }
    }
    const float read = warp_sum_each<8>(r, lane);
    const int c = c_lo + (lane >> 2);
    if ((lane & 3) == 0 && c <= e)
      reinterpret_cast<float*>(A.out)[(static_cast<size_t>(row) * H + head) * oe + c] =
          c < e ? read : fmaxf(fabsf(read), floor_) + 1e-6f;
  };
  for (int b = block0; b < block0 + n_blocks; b += 2) {
    if (b + 1 < block0 + n_blocks) fetch(b + 1, st[1], v8[1]);
    run(b, st[0], v8[0]);
    if (b + 1 < block0 + n_blocks) {
      if (b + 2 < block0 + n_blocks) fetch(b + 2, st[0], v8[0]);
      run(b + 1, st[1], v8[1]);
    }
  }
  if (tid < n_blocks) m_state[block0 + tid] = m;
}

__device__ bool tile_memory_step(const TileDesc& t, int tid) {
  const MemoryArgs* p = reinterpret_cast<const MemoryArgs*>(t.a[0]);
  const uint32_t d = __ldcg(&p->d);
  const bool f32 = __ldcg(&p->f32) != 0;
  if (t.i1 > static_cast<uint32_t>(kExecThreads)) return false;
#define MF_STEP(N)                         \
  if (d <= 128 * N) {                      \
    if (f32) memory_step<N, true>(t, tid); \
    else memory_step<N, false>(t, tid);    \
    return true;                           \
  }
  MF_STEP(1)
  MF_STEP(2)
  MF_STEP(4)
#undef MF_STEP
  return false;
}

__device__ bool tile_memory(const TileDesc& t, int tid, uint8_t* ring) {
  const MemoryArgs* p = reinterpret_cast<const MemoryArgs*>(t.a[0]);
  const uint32_t d = __ldcg(&p->d);
  const bool f32 = __ldcg(&p->f32) != 0;
#define MF_MEMORY(N)                             \
  if (d <= 128 * N) {                            \
    if (f32) memory_rows<N, true>(t, tid, ring); \
    else memory_rows<N, false>(t, tid, ring);    \
    return true;                                 \
  }
  MF_MEMORY(1)
  MF_MEMORY(2)
  MF_MEMORY(4)
#undef MF_MEMORY
  return false;
}

// Kind 58, HeadNormArgs: items [i0, i0 + i1), item = row * heads + head, one warp each: the head's read-out over its
// denominator (if it has one), over its root mean square, times the norm weight and sigmoid(g) or silu(g).
template <int V>
__device__ __noinline__ void head_norm_items(const TileDesc& t, int tid) {
  constexpr int NV = 8;   // V-element pieces per lane kept in registers
  HeadNormArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, e = static_cast<int>(A.e), oe = (e + (A.divide ? 4 : 3)) & ~3;
  const bool f32 = A.f32 != 0, silu = A.silu != 0;
  for (uint32_t it = t.i0 + warp; it < t.i0 + t.i1; it += kExecThreads / 32) {
    const uint32_t row = it / A.heads, head = it % A.heads;
    const float* o = f32p(A.o) + static_cast<size_t>(it) * oe;
    const size_t g0 = static_cast<size_t>(row) * A.ld_g + head * e, o0 = static_cast<size_t>(row) * A.ld_out + head * e;
    const float* w = f32p(A.w) + head * A.w_head;
    const float inv_den = A.divide ? 1.f / o[e] : 1.f;
    auto gate = [&](int c, float (&g)[V]) {
      if constexpr (V == 4) {
        if (!f32) {
          const uint2 u = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(A.g) + g0 + c);
          const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
          const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
          g[0] = a.x; g[1] = a.y; g[2] = b.x; g[3] = b.y;
          return;
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) g[j] = act_ld(A.g, g0 + c + j, f32);
    };
    auto put = [&](int c, const float (&v)[V], const float (&g)[V], const float (&ww)[V], float inv) {
      float x[V];
#pragma unroll
      for (int j = 0; j < V; ++j)
        x[j] = v[j] * inv_den * inv * ww[j] * (f32 ? sigmoid32(g[j]) : __fdividef(1.f, 1.f + __expf(-g[j]))) * (silu ? g[j] : 1.f);
      if constexpr (V == 4) {
        if (!f32) {
          const __nv_bfloat162 q[2] = {__floats2bfloat162_rn(x[0], x[1]), __floats2bfloat162_rn(x[2], x[3])};
          *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(A.out) + o0 + c) = *reinterpret_cast<const uint2*>(q);
          return;
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) act_st(A.out, o0 + c + j, f32, x[j]);
    };
    float ss = 0.f;
    if (e <= 32 * V * NV) {
      float v[NV][V], g[NV][V], ww[NV][V];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * 32 + lane) * V;
        if (c < e) {
          ld_vec<V>(o + c, v[i]);
          gate(c, g[i]);
          ld_vec<V>(w + c, ww[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if ((i * 32 + lane) * V < e)
#pragma unroll
          for (int j = 0; j < V; ++j) ss = fmaf(v[i][j] * inv_den, v[i][j] * inv_den, ss);
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(e) + A.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * 32 + lane) * V;
        if (c < e) put(c, v[i], g[i], ww[i], inv);
      }
    } else {
      for (int c = lane * V; c < e; c += 32 * V) {
        float v[V];
        ld_vec<V>(o + c, v);
#pragma unroll
        for (int j = 0; j < V; ++j) ss = fmaf(v[j] * inv_den, v[j] * inv_den, ss);
      }
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(e) + A.eps);
      for (int c = lane * V; c < e; c += 32 * V) {
        float v[V], g[V], ww[V];
        ld_vec<V>(o + c, v);
        gate(c, g);
        ld_vec<V>(w + c, ww);
        put(c, v, g, ww, inv);
      }
    }
  }
}

// Heads of at most 128 columns, bf16: four items of a warp in flight.
__device__ __noinline__ void head_norm_narrow(const TileDesc& t, int tid) {
  constexpr int U = 4;
  HeadNormArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, e = static_cast<int>(A.e), oe = (e + (A.divide ? 4 : 3)) & ~3, c = lane * 4;
  const bool in = c < e;
  const uint32_t end = t.i0 + t.i1;
  for (uint32_t it0 = t.i0 + warp * U; it0 < end; it0 += U * (kExecThreads / 32)) {
    float v[U][4], w[U][4], den[U], ss[U];
    uint2 g[U];
    size_t to[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t it = min(it0 + u, end - 1), row = it / A.heads, head = it - row * A.heads;
      const float* o = f32p(A.o) + static_cast<size_t>(it) * oe;
      to[u] = static_cast<size_t>(row) * A.ld_out + head * e + c;
#pragma unroll
      for (int j = 0; j < 4; ++j) v[u][j] = 0.f;
      if (in) {
        ld_vec<4>(o + c, v[u]);
        ld_vec<4>(f32p(A.w) + head * A.w_head + c, w[u]);
        g[u] = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(A.g) + static_cast<size_t>(row) * A.ld_g + head * e + c);
      }
      den[u] = A.divide ? o[e] : 1.f;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const float inv_den = 1.f / den[u];
      ss[u] = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        v[u][j] *= inv_den;
        ss[u] = fmaf(v[u][j], v[u][j], ss[u]);
      }
    }
#pragma unroll
    for (int o = 16; o; o >>= 1)
#pragma unroll
      for (int u = 0; u < U; ++u) ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (!in || it0 + u >= end) continue;
      const float inv = 1.f / sqrtf(ss[u] / static_cast<float>(e) + A.eps);
      const float2 ga = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&g[u].x));
      const float2 gb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&g[u].y));
      const float gate[4] = {ga.x, ga.y, gb.x, gb.y};
      float x[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j] = v[u][j] * inv * w[u][j] * __fdividef(A.silu ? gate[j] : 1.f, 1.f + __expf(-gate[j]));
      const __nv_bfloat162 q[2] = {__floats2bfloat162_rn(x[0], x[1]), __floats2bfloat162_rn(x[2], x[3])};
      *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(A.out) + to[u]) = *reinterpret_cast<const uint2*>(q);
    }
  }
}

__device__ void tile_head_norm(const TileDesc& t, int tid) {
  const HeadNormArgs* p = reinterpret_cast<const HeadNormArgs*>(t.a[0]);
  if (!__ldcg(&p->f32) && __ldcg(&p->e) <= 128 && (__ldcg(&p->e) & 3) == 0 && (__ldcg(&p->g) & 7) == 0) head_norm_narrow(t, tid);
  else if ((__ldcg(&p->e) & 3) == 0 && (__ldcg(&p->g) & 7) == 0) head_norm_items<4>(t, tid);
  else head_norm_items<1>(t, tid);
}

}  // namespace fab
}  // namespace mf
