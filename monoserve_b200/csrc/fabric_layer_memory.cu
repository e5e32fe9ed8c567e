// The matrix memory of the layer-list decoders (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ matrix memory
// Kind 56, MemGateArgs: rows [i0, i0 + i1), outputs [i2, i2 + i3) of the 2 heads (input gates, then forget gates).
// A warp takes one output and four rows at a time.
__device__ void tile_mem_gates(const TileDesc& t, int tid) {
  MemGateArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, K = static_cast<int>(A.K), H = static_cast<int>(A.heads);
  for (int o = static_cast<int>(t.i2) + warp; o < static_cast<int>(t.i2 + t.i3); o += kExecThreads / 32) {
    const bool forget = o >= H;
    const int h = forget ? o - H : o;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(forget ? A.wf : A.wi) + static_cast<size_t>(h) * K;
    const float bias = f32p(forget ? A.bf : A.bi)[h];
    for (uint32_t r = t.i0; r < t.i0 + t.i1; r += 4) {
      const float* x[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = f32p(A.h) + static_cast<size_t>(min(r + i, t.i0 + t.i1 - 1)) * A.ld_h;
      float acc[4] = {};
      if ((K & 3) == 0 && (A.ld_h & 3) == 0) {
#pragma unroll 4
        for (int k = 4 * lane; k < K; k += 128) {
          const uint2 raw = __ldg(reinterpret_cast<const uint2*>(w + k));
          const float2 wa = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
          const float2 wb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float4 v = *reinterpret_cast<const float4*>(x[i] + k);
            acc[i] = fmaf(v.x, wa.x, fmaf(v.y, wa.y, fmaf(v.z, wb.x, fmaf(v.w, wb.y, acc[i]))));
          }
        }
      } else {
        for (int k = lane; k < K; k += 32) {
          const float wv = __bfloat162float(w[k]);
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[i] = fmaf(x[i][k], wv, acc[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i] = warp_sum(acc[i]);
      if (lane < 4 && r + lane < t.i0 + t.i1) {
        const float z = (lane == 0 ? acc[0] : lane == 1 ? acc[1] : lane == 2 ? acc[2] : acc[3]) + bias;
        const float g = A.cap * tanhf(z / A.cap);
        reinterpret_cast<float*>(A.out)[static_cast<size_t>(r + lane) * 2 * H + o] =
            forget ? fminf(g, 0.f) - log1pf(expf(-fabsf(g))) : g;
      }
    }
  }
}

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
// the augmented memory, whose column e accumulates k alone: the normaliser); slot i3.  A wide tile: `ring` is the
// worker's operand ring.  A warp holds eight columns, a lane four-row groups 4 lane + 128 i of each, in registers for
// the whole portion.  32 tokens at a time: keys and scaled queries as fp32 in shared memory, and each lane prepares
// one token's gates, with F the running sum of the log forget gates.
constexpr int kMemTokens = 32, kMemColumns = 32;

template <int ND>
__device__ __noinline__ void memory_rows(const TileDesc& t, int tid, uint8_t* ring) {
  MemoryArgs A;
  load_block(A, t.a[0]);
  const int row0 = static_cast<int>(t.i0), rows = static_cast<int>(t.i1), slot = static_cast<int>(t.i3);
  const int head = static_cast<int>(t.i2 & 0xffffu), col0 = static_cast<int>(t.i2 >> 16) * kMemColumns;
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e);
  const int dp = (d + 3) & ~3, warp = tid >> 5, lane = tid & 31;
  const bool f32 = A.f32 != 0;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  __builtin_assume(__isShared(ring));
  float* const sk = reinterpret_cast<float*>(ring);      // [32][dp]
  float* const sq = sk + kMemTokens * dp;                // [32][dp]
  float* const sv = sq + kMemTokens * dp;                // [32][32]
  const int c_lo = col0 + warp * 8;                      // this warp's first column
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
  const float* gates = f32p(A.gates);
  for (int base = 0; base < rows; base += kMemTokens) {
    const int nt = min(kMemTokens, rows - base);
    exec_sync();
    for (int i = tid; i < nt * dp; i += kExecThreads) {
      const int tok = i / dp, k = i - tok * dp;
      const size_t at = static_cast<size_t>(row0 + base + tok) * A.ld_qkv + head * d + k;
      sk[i] = k < d ? act_ld(A.k, at, f32) : 0.f;
      sq[i] = k < d ? act_ld(A.q, at, f32) * A.q_scale : 0.f;
    }
    for (int i = tid; i < nt * kMemColumns; i += kExecThreads) {
      const int tok = i / kMemColumns, c = col0 + (i & (kMemColumns - 1));
      sv[i] = c < e ? act_ld(A.v, static_cast<size_t>(row0 + base + tok) * A.ld_qkv + head * e + c, f32) : (c == e ? 1.f : 0.f);
    }
    // gates of this chunk, one token per lane
    const size_t gat = static_cast<size_t>(row0 + base + min(lane, nt - 1)) * 2 * H + head;
    const float gi = lane < nt ? gates[gat] : -INFINITY, gf = lane < nt ? gates[gat + H] : 0.f;
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
    for (int tok = 0; tok < nt; ++tok) {
      const float kp = __shfl_sync(0xffffffffu, keep, tok), ad = __shfl_sync(0xffffffffu, add, tok);
      const unsigned long long kp2 = pk2(kp, kp);
      unsigned long long acc[8];
#pragma unroll
      for (int c = 0; c < 8; ++c) acc[c] = 0ull;
      const float4 va = *reinterpret_cast<const float4*>(sv + tok * kMemColumns + warp * 8);
      const float4 vb = *reinterpret_cast<const float4*>(sv + tok * kMemColumns + warp * 8 + 4);
      const float v[8] = {va.x, va.y, va.z, va.w, vb.x, vb.y, vb.z, vb.w};
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        const int at = i * 128 + lane * 4;
        if (ND == 1 && at >= dp) continue;
        float4 k4 = make_float4(0.f, 0.f, 0.f, 0.f), q4 = k4;
        if (at < dp) {
          k4 = *reinterpret_cast<const float4*>(sk + tok * dp + at);
          q4 = *reinterpret_cast<const float4*>(sq + tok * dp + at);
        }
        const unsigned long long k0 = pk2(k4.x, k4.y), k1 = pk2(k4.z, k4.w), q0 = pk2(q4.x, q4.y), q1 = pk2(q4.z, q4.w);
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const float av = ad * v[c];
          const unsigned long long av2 = pk2(av, av);
          S[c][i][0] = fma2(av2, k0, mul2(kp2, S[c][i][0]));
          S[c][i][1] = fma2(av2, k1, mul2(kp2, S[c][i][1]));
          acc[c] = fma2(S[c][i][0], q0, acc[c]);
          acc[c] = fma2(S[c][i][1], q1, acc[c]);
        }
      }
      float s[8];
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const float2 f = unpk2(acc[c]);
        s[c] = f.x + f.y;
      }
      // the eight columns' sums over the warp; lane ends with column (lane >> 2) & 7 bit-reversed through the halves
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const bool hi = lane & 16;
        const float give = hi ? s[c] : s[c + 4], have = hi ? s[c + 4] : s[c];
        s[c] = have + __shfl_xor_sync(0xffffffffu, give, 16);
      }
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const bool hi = lane & 8;
        const float give = hi ? s[c] : s[c + 2], have = hi ? s[c + 2] : s[c];
        s[c] = have + __shfl_xor_sync(0xffffffffu, give, 8);
      }
      {
        const bool hi = lane & 4;
        const float give = hi ? s[0] : s[1], have = hi ? s[1] : s[0];
        s[0] = have + __shfl_xor_sync(0xffffffffu, give, 4);
      }
      s[0] += __shfl_xor_sync(0xffffffffu, s[0], 2);
      s[0] += __shfl_xor_sync(0xffffffffu, s[0], 1);
      const float fl = __shfl_sync(0xffffffffu, floor_, tok);
      const int c = c_lo + ((lane >> 4) & 1) * 4 + ((lane >> 3) & 1) * 2 + ((lane >> 2) & 1);
      if ((lane & 3) == 0 && c <= e)
        reinterpret_cast<float*>(A.out)[(static_cast<size_t>(row0 + base + tok) * H + head) * (e + 1) + c] =
            c < e ? s[0] : fmaxf(fabsf(s[0]), fl) + 1e-6f;
    }
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

__device__ bool tile_memory(const TileDesc& t, int tid, uint8_t* ring) {
  const uint32_t d = __ldcg(&reinterpret_cast<const MemoryArgs*>(t.a[0])->d);
  if (d <= 128) memory_rows<1>(t, tid, ring);
  else if (d <= 256) memory_rows<2>(t, tid, ring);
  else if (d <= 512) memory_rows<4>(t, tid, ring);
  else return false;
  return true;
}

// Kind 58, HeadNormArgs: items [i0, i0 + i1), item = row * heads + head, one warp each: the head's output over its
// denominator, over its root mean square, times the norm weight and sigmoid(g).
__device__ void tile_head_norm(const TileDesc& t, int tid) {
  HeadNormArgs A;
  load_block(A, t.a[0]);
  const int warp = tid >> 5, lane = tid & 31, e = static_cast<int>(A.e);
  for (uint32_t it = t.i0 + warp; it < t.i0 + t.i1; it += kExecThreads / 32) {
    const uint32_t row = it / A.heads, head = it % A.heads;
    const float* o = f32p(A.o) + static_cast<size_t>(it) * (e + 1);
    const float inv_den = 1.f / o[e];
    float ss = 0.f;
    for (int c = lane; c < e; c += 32) {
      const float v = o[c] * inv_den;
      ss = fmaf(v, v, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(e) + A.eps);
    const size_t g0 = static_cast<size_t>(row) * A.ld_g + head * e, o0 = static_cast<size_t>(row) * A.ld_out + head * e;
    for (int c = lane; c < e; c += 32) {
      const float g = act_ld(A.g, g0 + c, A.f32);
      act_st(A.out, o0 + c, A.f32, o[c] * inv_den * inv * f32p(A.w)[head * e + c] * sigmoid32(g));
    }
  }
}

}  // namespace fab
}  // namespace mf
