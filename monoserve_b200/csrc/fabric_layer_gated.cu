// Gated memories of the layer-list decoders (fabric_layer_tiles.cuh): gated linear attention and the gated delta rule, both
// with a decay per key channel,
//   S <- diag(a) S;  u = v, or beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// and the decays themselves.  All of it is 32-bit arithmetic on the tensors' values.
#include "fabric_layer_tiles.cuh"
#include "wide_tile.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ decays
// Kind 67, DecayArgs: rows [i0, i0 + i1), at most 32, channels [i2, i2 + i3), at most 128: a thread per channel.
__device__ void tile_decay(const TileDesc& t, int tid, int* scratch) {
  constexpr int KC = 32, kRows = 32;
  static_assert(kRows * KC <= kLayerScratchInts, "decay scratch");
  float* const sx = reinterpret_cast<float*>(scratch);   // [row][KC]
  DecayArgs A;
  load_block(A, t.a[0]);
  const int rows = static_cast<int>(t.i1), R = static_cast<int>(A.r);
  const bool ok = tid < static_cast<int>(t.i3);
  const int ch = static_cast<int>(t.i2) + (ok ? tid : 0);
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(A.w) + static_cast<size_t>(ch) * A.ld_w;
  float acc[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) acc[r] = 0.f;
  for (int k0 = 0; k0 < R; k0 += KC) {
    for (int i = tid; i < kRows * KC; i += kExecThreads) {
      const int r = i / KC, k = k0 + i % KC;
      sx[i] = r < rows && k < R ? act_ld(A.x, static_cast<size_t>(t.i0 + r) * A.ld_x + k, A.f32 != 0) : 0.f;
    }
    exec_sync();
    // rows of w are padded with zeros to whole 64-column steps
#pragma unroll 1
    for (int k = 0; k < KC && k0 + k < R; k += 8) {
      const uint4 raw = *reinterpret_cast<const uint4*>(w + k0 + k);
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
      float wv[8];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        wv[2 * i] = f.x;
        wv[2 * i + 1] = f.y;
      }
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        if (r >= rows) break;
        const float4 a = *reinterpret_cast<const float4*>(sx + r * KC + k), b = *reinterpret_cast<const float4*>(sx + r * KC + k + 4);
        acc[r] += fmaf(a.x, wv[0], fmaf(a.y, wv[1], fmaf(a.z, wv[2], a.w * wv[3]))) +
                  fmaf(b.x, wv[4], fmaf(b.y, wv[5], fmaf(b.z, wv[6], b.w * wv[7])));
      }
    }
    exec_sync();
  }
  if (!ok) return;
  const float bias = f32p(A.bias)[ch], coef = f32p(A.coef)[ch / static_cast<int>(A.d)];
  float* out = reinterpret_cast<float*>(A.out) + static_cast<size_t>(t.i0) * A.ld_out + ch;
#pragma unroll
  for (int r = 0; r < kRows; ++r)
    if (r < rows) out[static_cast<size_t>(r) * A.ld_out] = expm1f(-coef * softplus32(A.sign * (acc[r] + bias)));
}

// ------------------------------------------------------------------ packed fp32 pairs (each half rounded like the scalar)
using Pair = unsigned long long;
__device__ __forceinline__ Pair pair(float a, float b) {
  Pair r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpair(Pair v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ Pair fma_pair(Pair a, Pair b, Pair c) {
  Pair r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ void ld_pairs(const float* p, Pair& a, Pair& b) {
  const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(p);
  a = q.x;
  b = q.y;
}

// NV values per lane summed over groups of LB lanes: lane l of a group ends with values [l NV / LB, ..), max(1, NV / LB) of
// them, at the front of v.
template <int NV, int LB>
__device__ __forceinline__ void group_sum(float (&v)[NV], int lane) {
  int n = NV;
#pragma unroll
  for (int bit = LB / 2; bit >= 1; bit >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool hi = lane & bit;
#pragma unroll
      for (int c = 0; c < n; ++c) {
        const float give = hi ? v[c] : v[c + n], have = hi ? v[c + n] : v[c];
        v[c] = have + __shfl_xor_sync(0xffffffffu, give, bit);
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], bit);
    }
  }
}

constexpr float kUnitFloor = 1e-6f;

// ------------------------------------------------------------------ a request's rows
// Kind 68, GatedMemoryArgs: rows [i0, i0 + i1) of one request; i2 = head | column block << 16, slot i3, a[1] columns of a
// block (32 C).  A wide tile: inputs come kTokens rows at a time through double-buffered asynchronous copies into the ring.
//
// Four tokens are one step.  With c_i the product of their decays up to token i, s_j that of the decays behind token j, and
// d_ij that of the decays after j up to i (all per key channel), S the state in front of the four:
//   p_i = S^T (c_i k_i) + sum_{j < i} u_j (k_i d_ij k_j)       u_i = beta_i (v_i - p_i)
//   o_i = S^T (c_i q_i) + sum_{j <= i} u_j (q_i d_ij k_j)      S <- c_3 S + sum_j (s_j k_j) u_j^T
// so the state is read once and written once per step, and the dot products between keys and queries are numbers of the
// step.  A pass over the chunk in front prepares c k, c q, s k and those numbers; no decay is ever divided by.  c_3 enters
// as S + S (c_3 - 1), with c_3 - 1 composed from the decays' distances to one, so that rounding a factor just below one
// does not add up over a long memory.
//
// A warp holds 8 C columns, 32 C in the tile: lane = 4 * (column group) + g, with rows 4 (g + 4 i) .. + 3 of its C columns
// in registers for the whole portion.  Lane g ends with the read-out of token g of the step.
constexpr int kStep = 4;
constexpr int kCoefs = 36;   // of a step: [0] d_ij products with queries (rows of four), [16] key scales, [20] betas,
                             // [24] products between keys (1,0) (2,0) (2,1) (3,0) (3,1) (3,2), [32] query scales

template <int R, int C, bool DELTA>
__device__ __noinline__ void gated_rows(const TileDesc& t, int tid, uint8_t* ring) {
  constexpr int DP = 4 * R;                                    // key channels, padded
  constexpr int kTokens = R <= 32 ? 32 : R == 64 ? 16 : 8, kSteps = kTokens / kStep;
  constexpr int CB = 32 * C, I4 = R / 4;
  constexpr int LB = R < 32 ? R : 32, NV = DELTA ? 32 : 16;    // lanes that prepare a step, sums of a step
  struct Shared {
    float kh[DELTA ? kTokens : 1][DP], qh[kTokens][DP], kt[kTokens][DP], em[kSteps][DP];
    float coef[kSteps][kCoefs], sums[kSteps][32], beta[32], v[kTokens][CB];
    float decay[2][kTokens][DP];
  };
  static_assert(sizeof(Shared) + 2 * kTokens * (2 * DP + CB) * 4 <= 216 * 1024, "the operand ring");
  static_assert(sizeof(Shared) % 16 == 0, "raw inputs start on 16 bytes");
  __builtin_assume(__isShared(ring));
  Shared& sh = *reinterpret_cast<Shared*>(ring);
  GatedMemoryArgs A;
  load_block(A, t.a[0]);
  const int row0 = static_cast<int>(t.i0), rows = static_cast<int>(t.i1), slot = static_cast<int>(t.i3);
  const int head = static_cast<int>(t.i2 & 0xffffu), col0 = static_cast<int>(t.i2 >> 16) * CB;
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e), kv = head / static_cast<int>(A.group);
  const int dp = (d + 3) & ~3, ds = (d + 7) & ~7, oe = (e + 3) & ~3, n_v = min(CB, e - col0);
  const int warp = tid >> 5, lane = tid & 31, g = lane & 3;
  const bool f32 = A.f32 != 0, unit = A.unit != 0;
  const int es = f32 ? 4 : 2, per16 = 16 / es;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  // raw inputs: [2][k rows, q rows, v rows]
  uint8_t* const raw = ring + sizeof(Shared);
  const int raw_k = kTokens * ds * es, raw_bytes = 2 * raw_k + kTokens * CB * es;

  const int c_lo = (warp * 8 + (lane >> 2)) * C;               // this lane's first column of the block
  float* const state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * H + head) * e * dp;
  Pair S[C][I4][2];
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < I4; ++i) {
      const int at = 4 * (g + 4 * i);
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && at < dp && col0 + c_lo + c < e) v = *reinterpret_cast<const float4*>(state + static_cast<size_t>(col0 + c_lo + c) * dp + at);
      S[c][i][0] = pair(v.x, v.y);
      S[c][i][1] = pair(v.z, v.w);
    }

  const size_t k_at = static_cast<size_t>(kv) * d, v_at = static_cast<size_t>(head) * e + col0;
  const bool kq16 = (d % per16) == 0 && ((A.k | A.q) & 15) == 0;
  const bool v16 = (e % per16) == 0 && (n_v % per16) == 0 && (A.v & 15) == 0;
  const bool d16 = (d & 3) == 0;
  if (d & 7) {   // the padding of keys, queries and decays stays zero
    for (int i = tid; i < 2 * raw_bytes / 16; i += kExecThreads) reinterpret_cast<uint4*>(raw)[i] = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < 2 * kTokens * DP; i += kExecThreads) (&sh.decay[0][0][0])[i] = 0.f;
    exec_sync();
  }
  float beta_next = 0.f;
  auto copy_elem = [&](uint8_t* dst, unsigned long long src, size_t at) {
    if (f32) *reinterpret_cast<float*>(dst) = reinterpret_cast<const float*>(src)[at];
    else *reinterpret_cast<__nv_bfloat16*>(dst) = reinterpret_cast<const __nv_bfloat16*>(src)[at];
  };
  auto stage = [&](int base, int b) {
    const int nt = min(kTokens, rows - base);
    uint8_t *const rk = raw + b * raw_bytes, *const rq = rk + raw_k, *const rv = rq + raw_k;
    for (int tok = warp; tok < nt; tok += kExecThreads / 32) {
      const size_t row = static_cast<size_t>(row0 + base + tok), at = row * A.ld_qkv;
      const float* dec = f32p(A.decay) + row * A.ld_decay + static_cast<size_t>(head) * d;
      if (kq16) {
        for (int p = lane; p < d / per16; p += 32) {
          cp16(rk + (tok * ds + p * per16) * es, reinterpret_cast<const uint8_t*>(A.k) + (at + k_at + p * per16) * es);
          cp16(rq + (tok * ds + p * per16) * es, reinterpret_cast<const uint8_t*>(A.q) + (at + k_at + p * per16) * es);
        }
      } else {
        for (int p = lane; p < d; p += 32) {
          copy_elem(rk + (tok * ds + p) * es, A.k, at + k_at + p);
          copy_elem(rq + (tok * ds + p) * es, A.q, at + k_at + p);
        }
      }
      if (d16) {
        for (int p = lane; p < d / 4; p += 32) cp16(&sh.decay[b][tok][4 * p], dec + 4 * p);
      } else {
        for (int p = lane; p < d; p += 32) sh.decay[b][tok][p] = dec[p];
      }
      if (v16) {
        if (lane < n_v / per16) cp16(rv + (tok * CB + lane * per16) * es, reinterpret_cast<const uint8_t*>(A.v) + (at + v_at + lane * per16) * es);
      } else {
        for (int p = lane; p < n_v; p += 32) copy_elem(rv + (tok * CB + p) * es, A.v, at + v_at + p);
      }
    }
    cp_commit();
    if (DELTA && tid < nt) beta_next = act_ld(A.beta, static_cast<size_t>(row0 + base + tid) * A.ld_beta + head, f32);
  };
  auto load4 = [&](const uint8_t* p, float (&v)[4]) {
    if (f32) {
      ld_vec<4>(reinterpret_cast<const float*>(p), v);
    } else {
      const uint2 u = *reinterpret_cast<const uint2*>(p);
      v[0] = __uint_as_float(u.x << 16);
      v[1] = __uint_as_float(u.x & 0xffff0000u);
      v[2] = __uint_as_float(u.y << 16);
      v[3] = __uint_as_float(u.y & 0xffff0000u);
    }
  };
  stage(0, 0);
  for (int base = 0, b = 0; base < rows; base += kTokens, b ^= 1) {
    const int nt = min(kTokens, rows - base);
    cp_wait<0>();
    if (DELTA && tid < kTokens) sh.beta[tid] = tid < nt ? sigmoid32(beta_next) : 0.f;
    exec_sync();
    if (base + kTokens < rows) stage(base + kTokens, b ^ 1);
    // ---- prepare the chunk's steps: LB lanes to a step, four rows of each at a time
    const uint8_t *const rk = raw + b * raw_bytes, *const rq = rk + raw_k, *const rv = rq + raw_k;
    const int steps = (nt + kStep - 1) / kStep;
#pragma unroll 1
    for (int s0 = warp * (32 / LB); s0 < steps; s0 += (kExecThreads / 32) * (32 / LB)) {
      const int s = s0 + lane / LB, l = lane & (LB - 1);
      float sum[NV];
#pragma unroll
      for (int i = 0; i < NV; ++i) sum[i] = 0.f;
      if (s < steps) {
#pragma unroll 1
        for (int r = 4 * l; r < DP; r += 4 * LB) {
          float k[4][4], q[4][4], m[4][4];                     // [token][row]
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int tok = s * kStep + i;
            if (tok < nt && r < dp) {
              load4(rk + (tok * ds + r) * es, k[i]);
              load4(rq + (tok * ds + r) * es, q[i]);
              ld_vec<4>(&sh.decay[b][tok][r], m[i]);
            } else {
#pragma unroll
              for (int j = 0; j < 4; ++j) k[i][j] = q[i][j] = m[i][j] = 0.f;
            }
          }
          float kh[4][4], qh[4][4], kt[4][4], em[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float a1 = 1.f + m[1][j], a2 = 1.f + m[2][j], a3 = 1.f + m[3][j], a23 = a2 * a3;
            float c = 1.f + m[0][j], x = m[0][j];
            kh[0][j] = c * k[0][j];
            qh[0][j] = c * q[0][j];
#pragma unroll
            for (int i = 1; i < 4; ++i) {
              x += fmaf(x, m[i][j], m[i][j]);
              c *= 1.f + m[i][j];
              kh[i][j] = c * k[i][j];
              qh[i][j] = c * q[i][j];
            }
            em[j] = x;
            kt[3][j] = k[3][j];
            kt[2][j] = a3 * k[2][j];
            kt[1][j] = a23 * k[1][j];
            kt[0][j] = a1 * a23 * k[0][j];
            // keys as tokens 1, 2 and 3 find them
            const float k10 = a1 * k[0][j], k20 = a2 * k10, k21 = a2 * k[1][j];
#pragma unroll
            for (int i = 0; i < 4; ++i) sum[i * (i + 1) / 2 + i] = fmaf(q[i][j], k[i][j], sum[i * (i + 1) / 2 + i]);
            sum[1] = fmaf(q[1][j], k10, sum[1]);
            sum[3] = fmaf(q[2][j], k20, sum[3]);
            sum[4] = fmaf(q[2][j], k21, sum[4]);
            sum[6] = fmaf(q[3][j], kt[0][j], sum[6]);
            sum[7] = fmaf(q[3][j], kt[1][j], sum[7]);
            sum[8] = fmaf(q[3][j], kt[2][j], sum[8]);
            if constexpr (DELTA) {
              sum[10] = fmaf(k[1][j], k10, sum[10]);
              sum[11] = fmaf(k[2][j], k20, sum[11]);
              sum[12] = fmaf(k[2][j], k21, sum[12]);
              sum[13] = fmaf(k[3][j], kt[0][j], sum[13]);
              sum[14] = fmaf(k[3][j], kt[1][j], sum[14]);
              sum[15] = fmaf(k[3][j], kt[2][j], sum[15]);
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                sum[16 + i] = fmaf(k[i][j], k[i][j], sum[16 + i]);
                sum[20 + i] = fmaf(q[i][j], q[i][j], sum[20 + i]);
              }
            }
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if constexpr (DELTA) st_vec<4>(&sh.kh[s * kStep + i][r], kh[i]);
            st_vec<4>(&sh.qh[s * kStep + i][r], qh[i]);
            st_vec<4>(&sh.kt[s * kStep + i][r], kt[i]);
          }
          st_vec<4>(&sh.em[s][r], em);
        }
      }
      group_sum<NV, LB>(sum, lane);
      if (s < steps) {
        constexpr int kMine = NV > LB ? NV / LB : 1;
#pragma unroll
        for (int i = 0; i < kMine; ++i) sh.sums[s][l * NV / LB + i] = sum[i];
      }
      __syncwarp();
      if (s < steps) {
        const float* z = sh.sums[s];
        auto key_scale = [&](int i) { return DELTA && unit ? 1.f / sqrtf(z[16 + i] + kUnitFloor) : 1.f; };
        auto query_scale = [&](int i) { return A.q_scale * (DELTA && unit ? 1.f / sqrtf(z[20 + i] + kUnitFloor) : 1.f); };
        for (int x = l; x < kCoefs; x += LB) {
          float v = 0.f;
          if (x < 16) {
            const int i = x >> 2, j = x & 3;
            if (j <= i) v = query_scale(i) * key_scale(j) * z[i * (i + 1) / 2 + j];
          } else if (x < 20) {
            v = key_scale(x - 16);
          } else if (x < 24) {
            v = DELTA ? sh.beta[s * kStep + x - 20] : 0.f;
          } else if (x < 30) {
            const int i = x == 24 ? 1 : x < 27 ? 2 : 3, j = x - 24 - i * (i - 1) / 2;
            if (DELTA) v = key_scale(i) * key_scale(j) * z[x - 14];
          } else if (x >= 32) {
            v = query_scale(x - 32);
          }
          sh.coef[s][x] = v;
        }
      }
      __syncwarp();
    }
    for (int i = tid; i < kTokens * CB; i += kExecThreads) {
      const int tok = i / CB, c = i % CB;
      float v = 0.f;
      if (tok < nt && c < n_v) v = f32 ? reinterpret_cast<const float*>(rv)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(rv)[i]);
      sh.v[tok][c] = v;
    }
    exec_sync();
    // ---- the steps
#pragma unroll 1
    for (int s = 0; s < steps; ++s) {
      Pair P[DELTA ? 4 : 1][C], O[4][C];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int c = 0; c < C; ++c) {
          O[i][c] = 0ull;
          if constexpr (DELTA) P[i][c] = 0ull;
        }
#pragma unroll
      for (int i4 = 0; i4 < I4; ++i4) {
        const int at = 4 * (g + 4 * i4);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          Pair a, bb;
          ld_pairs(&sh.qh[s * kStep + i][at], a, bb);
#pragma unroll
          for (int c = 0; c < C; ++c) O[i][c] = fma_pair(S[c][i4][1], bb, fma_pair(S[c][i4][0], a, O[i][c]));
          if constexpr (DELTA) {
            ld_pairs(&sh.kh[s * kStep + i][at], a, bb);
#pragma unroll
            for (int c = 0; c < C; ++c) P[i][c] = fma_pair(S[c][i4][1], bb, fma_pair(S[c][i4][0], a, P[i][c]));
          }
        }
      }
      const float* z = sh.coef[s];
      float zk[4], mix[4];
      ld_vec<4>(z + 16, zk);
      ld_vec<4>(z + 4 * g, mix);
      const float zq = z[32 + g];
      Pair U[4][C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        float u[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) u[i] = sh.v[s * kStep + i][c_lo + c];
        if constexpr (DELTA) {
          float p[4], zb[4], kk[6];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float2 f = unpair(P[i][c]);
            p[i] = f.x + f.y;
          }
#pragma unroll
          for (int bit = 1; bit <= 2; bit <<= 1)
#pragma unroll
            for (int i = 0; i < 4; ++i) p[i] += __shfl_xor_sync(0xffffffffu, p[i], bit);
          ld_vec<4>(z + 20, zb);
#pragma unroll
          for (int i = 0; i < 6; ++i) kk[i] = z[24 + i];
          u[0] = zb[0] * (u[0] - zk[0] * p[0]);
          u[1] = zb[1] * (u[1] - fmaf(kk[0], u[0], zk[1] * p[1]));
          u[2] = zb[2] * (u[2] - fmaf(kk[2], u[1], fmaf(kk[1], u[0], zk[2] * p[2])));
          u[3] = zb[3] * (u[3] - fmaf(kk[5], u[2], fmaf(kk[4], u[1], fmaf(kk[3], u[0], zk[3] * p[3]))));
        }
        float o[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = unpair(O[i][c]);
          o[i] = f.x + f.y;
        }
        group_sum<4, 4>(o, lane);
        const float out = fmaf(mix[3], u[3], fmaf(mix[2], u[2], fmaf(mix[1], u[1], fmaf(mix[0], u[0], zq * o[0]))));
        const int tok = s * kStep + g;
        if (tok < nt && c_lo + c < n_v)
          reinterpret_cast<float*>(A.out)[(static_cast<size_t>(row0 + base + tok) * H + head) * oe + col0 + c_lo + c] = out;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float x = zk[i] * u[i];
          U[i][c] = pair(x, x);
        }
      }
#pragma unroll
      for (int i4 = 0; i4 < I4; ++i4) {
        const int at = 4 * (g + 4 * i4);
        Pair a, bb;
        ld_pairs(&sh.em[s][at], a, bb);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          S[c][i4][0] = fma_pair(S[c][i4][0], a, S[c][i4][0]);
          S[c][i4][1] = fma_pair(S[c][i4][1], bb, S[c][i4][1]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          ld_pairs(&sh.kt[s * kStep + i][at], a, bb);
#pragma unroll
          for (int c = 0; c < C; ++c) {
            S[c][i4][0] = fma_pair(a, U[i][c], S[c][i4][0]);
            S[c][i4][1] = fma_pair(bb, U[i][c], S[c][i4][1]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < I4; ++i) {
      const int at = 4 * (g + 4 * i);
      if (at < dp && col0 + c_lo + c < e) {
        const float2 a = unpair(S[c][i][0]), b = unpair(S[c][i][1]);
        *reinterpret_cast<float4*>(state + static_cast<size_t>(col0 + c_lo + c) * dp + at) = make_float4(a.x, a.y, b.x, b.y);
      }
    }
}

__device__ bool tile_gated_memory(const TileDesc& t, int tid, uint8_t* ring) {
  const GatedMemoryArgs* p = reinterpret_cast<const GatedMemoryArgs*>(t.a[0]);
  const uint32_t d = __ldcg(&p->d);
  const bool delta = __ldcg(&p->beta) != 0, two = t.a[1] == 64;
  if (t.a[1] != 32 && !two) return false;
#define MF_GATED(N, C)                                  \
  if (d <= 4 * N && two == (C == 2)) {                  \
    if (delta) gated_rows<N, C, true>(t, tid, ring);    \
    else gated_rows<N, C, false>(t, tid, ring);         \
    return true;                                        \
  }
  MF_GATED(8, 1)
  MF_GATED(8, 2)
  MF_GATED(16, 1)
  MF_GATED(16, 2)
  MF_GATED(32, 1)
  MF_GATED(32, 2)
  MF_GATED(64, 1)
  MF_GATED(128, 1)
#undef MF_GATED
  return false;
}

// ------------------------------------------------------------------ one token
// Kind 69, GatedMemoryArgs: row i0, i2 = head | first column block << 16, i1 column blocks, slot i3.  G lanes share a
// column (ND four-row groups of it each); a column block is 32 (32 / G) columns.  The state streams through registers, the
// next block's loads issued before this one's arithmetic; the read-out comes from the state in front of the token's write,
// S^T q + (k q) u, so one round of sums per column serves both products.
template <int G, int ND, bool DELTA>
__device__ __noinline__ void gated_step(const TileDesc& t, int tid) {
  constexpr int kSide = 32 / G, kBlock = 32 * kSide;           // columns side by side in a warp; of a block
  GatedMemoryArgs A;
  load_block(A, t.a[0]);
  const int row = static_cast<int>(t.i0), slot = static_cast<int>(t.i3), n_blocks = static_cast<int>(t.i1);
  const int head = static_cast<int>(t.i2 & 0xffffu), block0 = static_cast<int>(t.i2 >> 16);
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e), kv = head / static_cast<int>(A.group);
  const int dp = (d + 3) & ~3, oe = (e + 3) & ~3, warp = tid >> 5, lane = tid & 31, l = lane & (G - 1), side = lane / G;
  const bool f32 = A.f32 != 0, unit = A.unit != 0;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row] == 0;
  const size_t at_row = static_cast<size_t>(row) * A.ld_qkv;
  float* const state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * H + head) * e * dp;
  // column c of this lane's eight is c_lo + c * kSide; after the sums the lane owns column c_lo + own * kSide
  const int own = l * 8 / G;
  const bool writes = G == 8 || (l & (G / 8 - 1)) == 0;
  float4 st[2][8][ND];
  float v1[2];
  auto fetch = [&](int b, float4 (&S)[8][ND], float& v) {
    const int c_lo = b * kBlock + warp * 8 * kSide + side;
#pragma unroll
    for (int c = 0; c < 8; ++c)
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        const int at = 4 * (l + G * i), col = c_lo + c * kSide;
        S[c][i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && at < dp && col < e) S[c][i] = __ldcs(reinterpret_cast<const float4*>(state + static_cast<size_t>(col) * dp + at));
      }
    const int col = c_lo + own * kSide;
    v = col < e ? act_ld(A.v, at_row + static_cast<size_t>(head) * e + col, f32) : 0.f;
  };
  fetch(block0, st[0], v1[0]);
  float k[ND][4], q[ND][4], m[ND][4];
  float dots[4] = {0.f, 0.f, 0.f, 0.f};                        // k k, q q, k q
#pragma unroll
  for (int i = 0; i < ND; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int at = 4 * (l + G * i) + j;
      k[i][j] = at < d ? act_ld(A.k, at_row + static_cast<size_t>(kv) * d + at, f32) : 0.f;
      q[i][j] = at < d ? act_ld(A.q, at_row + static_cast<size_t>(kv) * d + at, f32) : 0.f;
      m[i][j] = at < d ? f32p(A.decay)[static_cast<size_t>(row) * A.ld_decay + static_cast<size_t>(head) * d + at] : 0.f;
      dots[0] = fmaf(k[i][j], k[i][j], dots[0]);
      dots[1] = fmaf(q[i][j], q[i][j], dots[1]);
      dots[2] = fmaf(k[i][j], q[i][j], dots[2]);
    }
#pragma unroll
  for (int bit = G / 2; bit >= 1; bit >>= 1)
#pragma unroll
    for (int i = 0; i < 3; ++i) dots[i] += __shfl_xor_sync(0xffffffffu, dots[i], bit);
  const float zk = unit ? 1.f / sqrtf(dots[0] + kUnitFloor) : 1.f;
  const float zq = A.q_scale * (unit ? 1.f / sqrtf(dots[1] + kUnitFloor) : 1.f), kq = dots[2] * zk * zq;
  const float beta = DELTA ? sigmoid32(act_ld(A.beta, static_cast<size_t>(row) * A.ld_beta + head, f32)) : 0.f;
  auto run = [&](int b, float4 (&S)[8][ND], float v) {
    const int c_lo = b * kBlock + warp * 8 * kSide + side;
    float o[8], p[8];
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      o[c] = p[c] = 0.f;
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        float4& s = S[c][i];
        s.x = fmaf(s.x, m[i][0], s.x);
        s.y = fmaf(s.y, m[i][1], s.y);
        s.z = fmaf(s.z, m[i][2], s.z);
        s.w = fmaf(s.w, m[i][3], s.w);
        o[c] = fmaf(s.x, q[i][0], fmaf(s.y, q[i][1], fmaf(s.z, q[i][2], fmaf(s.w, q[i][3], o[c]))));
        if constexpr (DELTA) p[c] = fmaf(s.x, k[i][0], fmaf(s.y, k[i][1], fmaf(s.z, k[i][2], fmaf(s.w, k[i][3], p[c]))));
      }
    }
    group_sum<8, G>(o, lane);
    float u = v;
    if constexpr (DELTA) {
      group_sum<8, G>(p, lane);
      u = beta * (v - zk * p[0]);
    }
    const int mine = c_lo + own * kSide;
    if (writes && mine < e) reinterpret_cast<float*>(A.out)[(static_cast<size_t>(row) * H + head) * oe + mine] = fmaf(kq, u, zq * o[0]);
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      const float x = zk * __shfl_sync(0xffffffffu, u, side * G + c * G / 8);
      const int col = c_lo + c * kSide;
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        float4 s = S[c][i];
        s.x = fmaf(k[i][0], x, s.x);
        s.y = fmaf(k[i][1], x, s.y);
        s.z = fmaf(k[i][2], x, s.z);
        s.w = fmaf(k[i][3], x, s.w);
        const int at = 4 * (l + G * i);
        if (at < dp && col < e) __stcs(reinterpret_cast<float4*>(state + static_cast<size_t>(col) * dp + at), s);
      }
    }
  };
  for (int b = block0; b < block0 + n_blocks; b += 2) {
    if (b + 1 < block0 + n_blocks) fetch(b + 1, st[1], v1[1]);
    run(b, st[0], v1[0]);
    if (b + 1 < block0 + n_blocks) {
      if (b + 2 < block0 + n_blocks) fetch(b + 2, st[0], v1[0]);
      run(b + 1, st[1], v1[1]);
    }
  }
}

__device__ bool tile_gated_step(const TileDesc& t, int tid) {
  const GatedMemoryArgs* p = reinterpret_cast<const GatedMemoryArgs*>(t.a[0]);
  const uint32_t d = __ldcg(&p->d);
  const bool delta = __ldcg(&p->beta) != 0;
#define MF_STEP(N, G, ND)                           \
  if (d <= N) {                                     \
    if (delta) gated_step<G, ND, true>(t, tid);     \
    else gated_step<G, ND, false>(t, tid);          \
    return true;                                    \
  }
  MF_STEP(32, 8, 1)
  MF_STEP(64, 16, 1)
  MF_STEP(128, 32, 1)
  MF_STEP(256, 32, 2)
  MF_STEP(512, 32, 4)
#undef MF_STEP
  return false;
}

}  // namespace fab
}  // namespace mf
