// Gated memories of the layer-list decoders (fabric_layer_tiles.cuh): gated linear attention and the gated delta rule, both
// with a decay per key channel,
//   S <- diag(a) S;  u = v, or beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// and the decays themselves.  All of it is 32-bit arithmetic on the tensors' values.
#include "fabric_layer_tiles.cuh"
#include "ptx.cuh"
#include "wide_tile.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ decays
// Kind 67, DecayArgs: rows [i0, i0 + i1).
__device__ void tile_decay(const TileDesc& t, int tid) {
  DecayArgs A;
  load_block(A, t.a[0]);
  for (uint32_t r = t.i0; r < t.i0 + t.i1; ++r) {
    float* z = reinterpret_cast<float*>(A.z) + static_cast<size_t>(r) * A.ld;
    for (uint32_t c = tid; c < A.n; c += kExecThreads) z[c] = expm1f(-f32p(A.coef)[c] * softplus32(z[c] + f32p(A.bias)[c]));
  }
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
__device__ __forceinline__ Pair add_pair(Pair a, Pair b) {
  Pair r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ Pair mul_pair(Pair a, Pair b) {
  Pair r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void ld_pairs(const float* p, Pair& a, Pair& b) {
  const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(p);
  a = q.x;
  b = q.y;
}

// NV values per lane summed over groups of LB lanes: lane l of a group ends with values [l NV / LB, ..), max(1, NV / LB) of
// them, at the front of v.
template <int N, int BIT, int NV>
__device__ __forceinline__ void group_sum_from(float (&v)[NV], int lane) {
  if constexpr (BIT >= 1) {
    if constexpr (N > 1) {
      const bool hi = lane & BIT;
#pragma unroll
      for (int c = 0; c < N / 2; ++c) {
        const float give = hi ? v[c] : v[c + N / 2], have = hi ? v[c + N / 2] : v[c];
        v[c] = have + __shfl_xor_sync(0xffffffffu, give, BIT);
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], BIT);
    }
    group_sum_from<(N > 1 ? N / 2 : 1), BIT / 2>(v, lane);
  }
}
template <int NV, int LB>
__device__ __forceinline__ void group_sum(float (&v)[NV], int lane) { group_sum_from<NV, LB / 2>(v, lane); }

constexpr float kUnitFloor = 1e-6f;

// ------------------------------------------------------------------ a request's rows
// Kind 68, GatedMemoryArgs: rows [i0, i0 + i1) of one request; i2 = head | column block << 16, slot i3, a[1] columns of a
// block.  A wide tile: inputs come kTokens rows at a time through double-buffered asynchronous copies into the ring.
//
// Four tokens are one step.  With c_i the product of their decays up to token i, s_j that of the decays behind token j, and
// d_ij that of the decays after j up to i (all per key channel), S the state in front of the four:
//   p_i = S^T (c_i k_i) + sum_{j < i} u_j (k_i d_ij k_j)       u_i = beta_i (v_i - p_i)
//   o_i = S^T (c_i q_i) + sum_{j <= i} u_j (q_i d_ij k_j)      S <- c_3 S + sum_j (s_j k_j) u_j^T
// so the state is read once and written once per step, and the dot products between keys and queries are numbers of the
// step.  A pass over the chunk in front prepares c k, c q, s k and those numbers; no decay is ever divided by.  c_3 enters
// as S + S (c_3 - 1), with c_3 - 1 composed from the decays' distances to one, so that rounding a factor just below one
// does not add up over a long memory.  Keys and queries stay as they come: their scales (unit norms, q_scale) go into the
// numbers.
//
// G lanes share C columns of the state, R rows each in groups of four, 4 (l + G i) .. + 3, in registers for the whole
// portion: 128 C / G columns in a tile.  A column's sums end in 4 G / (4 C) lanes of its group, which solve for its u, and
// hand them to the others through shared memory.
constexpr int kStep = 4;

// i = 1: 0; i = 2: 1, 2; i = 3: 3, 4, 5 (j < i), and with the diagonal 0; 1, 2; 3, 4, 5; 6 .. 9
__device__ __forceinline__ int below(int i, int j) { return i * (i - 1) / 2 + j; }
__device__ __forceinline__ int upto(int i, int j) { return i * (i + 1) / 2 + j; }

template <int G, int R, int C, bool DELTA, bool F32>
__device__ __noinline__ void gated_rows(const TileDesc& t, int tid, uint8_t* ring) {
  using T = typename std::conditional<F32, float, __nv_bfloat16>::type;
  constexpr int DP = G * R;                                    // key channels, padded
  constexpr int kTokens = DP <= 128 ? 32 : DP == 256 ? 16 : 8, kSteps = kTokens / kStep;
  constexpr int kSide = 32 / G, CB = 4 * kSide * C, I4 = R / 4;
  constexpr int LB = DP < 64 ? DP / 2 : 32, NV = DELTA ? 32 : 16;   // lanes that prepare a step, sums of a step
  constexpr int NS = 4 * C > G ? 4 * C / G : 1;                // sums of a step that a lane ends with
  constexpr int kPer16 = 16 / static_cast<int>(sizeof(T));
  struct Raw {
    T k[kTokens][DP], q[kTokens][DP], v[kTokens][CB];
    float decay[kTokens][DP];
  };
  struct Shared {
    Raw in[2];
    float kh[DELTA ? kTokens : 1][DP], qh[kTokens][DP], kt[kTokens][DP], em[kSteps][DP];
    float mix[kSteps][16], keys[kSteps][8], scale[kSteps][8], sums[kSteps][32], beta[2][32];
    float u[2][CB][4];
    GatedMemoryArgs args;                                      // read again for each chunk rather than kept in registers
  };
  static_assert(sizeof(Shared) <= 216 * 1024, "the operand ring");
  __builtin_assume(__isShared(ring));
  Shared& sh = *reinterpret_cast<Shared*>(ring);
  GatedMemoryArgs& A = sh.args;
  if (tid < static_cast<int>(sizeof(GatedMemoryArgs) / 16))
    reinterpret_cast<uint4*>(&A)[tid] = __ldcg(reinterpret_cast<const uint4*>(t.a[0]) + tid);
  exec_sync();
  const int row0 = static_cast<int>(t.i0), rows = static_cast<int>(t.i1), slot = static_cast<int>(t.i3);
  const int head = static_cast<int>(t.i2 & 0xffffu), col0 = static_cast<int>(t.i2 >> 16) * CB;
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e), kv = head / static_cast<int>(A.group);
  const int dp = (d + 3) & ~3, oe = (e + 3) & ~3, n_v = min(CB, e - col0);
  const int warp = tid >> 5, lane = tid & 31, l = lane & (G - 1);
  const bool unit = A.unit != 0;
  const float q_scale = A.q_scale;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  const int c_lo = (warp * kSide + lane / G) * C;              // this lane's first column of the block
  float* const state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * H + head) * e * dp + static_cast<size_t>(col0 + c_lo) * dp;
  Pair S[C][I4][2];
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < I4; ++i) {
      const int at = 4 * (l + G * i);
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && at < dp && c_lo + c < n_v) v = *reinterpret_cast<const float4*>(state + static_cast<size_t>(c) * dp + at);
      S[c][i][0] = pair(v.x, v.y);
      S[c][i][1] = pair(v.z, v.w);
    }

  const size_t k_at = static_cast<size_t>(kv) * d, v_at = static_cast<size_t>(head) * e + col0;
  const bool kq16 = (d % kPer16) == 0 && ((A.k | A.q) & 15) == 0, d16 = (d & 3) == 0;
  const bool v16 = (e % kPer16) == 0 && (n_v % kPer16) == 0 && (A.v & 15) == 0;
  if (d < DP)   // the padding of keys, queries and decays stays zero
    for (int i = tid; i < static_cast<int>(sizeof(sh.in) / 16); i += kExecThreads) reinterpret_cast<uint4*>(sh.in)[i] = make_uint4(0, 0, 0, 0);
  exec_sync();
  float beta_next = 0.f;
  // Rows of n elements, nt of them: 16-byte pieces (each thread keeps its place in a row), or single elements.  Rows past nt
  // that belong to its last step become zero.
  auto copy_rows = [&](auto* dst, const auto* src, size_t ld, auto width, int nt, int n, bool pieces) {
    using E = std::remove_reference_t<decltype(*dst)>;
    constexpr int N = decltype(width)::value, per = 16 / static_cast<int>(sizeof(E)), PP = N / per;
    constexpr int kPass = kExecThreads / PP < kTokens ? kExecThreads / PP : kTokens;
    const int tok0 = tid / PP, p = (tid % PP) * per, end = (nt + kStep - 1) & ~(kStep - 1);
    if (pieces && tok0 < kPass && p < n) {
      E* to = dst + tok0 * N + p;
      const E* from = src + tok0 * ld + p;
#pragma unroll
      for (int tok = 0; tok < kTokens; tok += kPass) {
        if (tok + tok0 < nt) cp16(to + tok * N, from + tok * ld);
        else if (tok + tok0 < end) *reinterpret_cast<uint4*>(to + tok * N) = make_uint4(0, 0, 0, 0);
      }
    }
    if (!pieces) {
#pragma unroll 1
      for (int tok = warp; tok < end; tok += kExecThreads / 32)
        for (int i = lane; i < n; i += 32) dst[tok * N + i] = tok < nt ? src[tok * ld + i] : static_cast<E>(0.f);
    }
  };
  using DPc = std::integral_constant<int, DP>;
  using CBc = std::integral_constant<int, CB>;
  auto stage = [&](int base, int b) {
    const int nt = min(kTokens, rows - base);
    Raw& in = sh.in[b];
    const size_t row = static_cast<size_t>(row0 + base), at = row * A.ld_qkv, ld = A.ld_qkv;
    copy_rows(&in.k[0][0], reinterpret_cast<const T*>(A.k) + at + k_at, ld, DPc(), nt, d, kq16);
    copy_rows(&in.q[0][0], reinterpret_cast<const T*>(A.q) + at + k_at, ld, DPc(), nt, d, kq16);
    copy_rows(&in.v[0][0], reinterpret_cast<const T*>(A.v) + at + v_at, ld, CBc(), nt, n_v, v16);
    copy_rows(&in.decay[0][0], f32p(A.decay) + row * A.ld_decay + static_cast<size_t>(head) * d, static_cast<size_t>(A.ld_decay), DPc(), nt, d, d16);
    cp_commit();
    if (DELTA && tid < nt) beta_next = act_ld(A.beta, (row + tid) * A.ld_beta + head, F32);
  };
  auto load2 = [&](const T* p) -> Pair {
    if constexpr (F32) return *reinterpret_cast<const Pair*>(p);
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    return pair(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
  };
  // the column and the tokens whose sums this lane ends with
  const int first = l * 4 * C / G, my_col = c_lo + first / 4, my_tok = first & 3;
  const bool owner = (l * 4 * C) % (4 * G) == 0;   // the first of the column's lanes
  const int col_lane = lane - l + (first / 4) * G / C;
  const size_t ld_out = static_cast<size_t>(H) * oe;
  float* out = reinterpret_cast<float*>(A.out) + static_cast<size_t>(row0 + my_tok) * ld_out + static_cast<size_t>(head) * oe + col0 + my_col;

  stage(0, 0);
  for (int base = 0, b = 0; base < rows; base += kTokens, b ^= 1) {
    const int nt = min(kTokens, rows - base);
    cp_wait<0>();
    if (DELTA && tid < kTokens) sh.beta[b][tid] = tid < nt ? sigmoid32(beta_next) : 0.f;
    exec_sync();
    if (base + kTokens < rows) stage(base + kTokens, b ^ 1);
    // ---- prepare the chunk's steps: LB lanes to a step, two rows of each at a time
    const Raw& in = sh.in[b];
    const int steps = (nt + kStep - 1) / kStep;
#pragma unroll 1
    for (int s0 = warp * (32 / LB); s0 < steps; s0 += (kExecThreads / 32) * (32 / LB)) {
      const int s = s0 + lane / LB, pl = lane & (LB - 1);
      Pair acc[24];   // products of queries and keys (10), of keys and keys (6), squares of keys, of queries
#pragma unroll
      for (int i = 0; i < 24; ++i) acc[i] = 0ull;
      if (s < steps) {
#pragma unroll 1
        for (int r = 2 * pl; r < DP; r += 2 * LB) {
          Pair k[4], q[4], m[4];                               // by token
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            k[i] = load2(&in.k[s * kStep + i][r]);
            q[i] = load2(&in.q[s * kStep + i][r]);
            m[i] = *reinterpret_cast<const Pair*>(&in.decay[s * kStep + i][r]);
          }
          auto put = [&](float* p, Pair v) { *reinterpret_cast<Pair*>(p + r) = v; };
          const Pair one = pair(1.f, 1.f), a1 = add_pair(m[1], one), a2 = add_pair(m[2], one), a3 = add_pair(m[3], one);
          Pair c = add_pair(m[0], one), x = m[0];
          if constexpr (DELTA) put(sh.kh[s * kStep], mul_pair(c, k[0]));
          put(sh.qh[s * kStep], mul_pair(c, q[0]));
#pragma unroll
          for (int i = 1; i < 4; ++i) {
            x = add_pair(x, fma_pair(x, m[i], m[i]));
            c = mul_pair(c, i == 1 ? a1 : i == 2 ? a2 : a3);
            if constexpr (DELTA) put(sh.kh[s * kStep + i], mul_pair(c, k[i]));
            put(sh.qh[s * kStep + i], mul_pair(c, q[i]));
          }
          put(sh.em[s], x);
          // keys as tokens 1, 2 and 3 find them; the last are also what the step leaves to the state
          const Pair k10 = mul_pair(a1, k[0]), k20 = mul_pair(a2, k10), k21 = mul_pair(a2, k[1]);
          const Pair kt[4] = {mul_pair(a3, k20), mul_pair(a3, k21), mul_pair(a3, k[2]), k[3]};
          acc[0] = fma_pair(q[0], k[0], acc[0]);
          acc[1] = fma_pair(q[1], k10, acc[1]);
          acc[2] = fma_pair(q[1], k[1], acc[2]);
          acc[3] = fma_pair(q[2], k20, acc[3]);
          acc[4] = fma_pair(q[2], k21, acc[4]);
          acc[5] = fma_pair(q[2], k[2], acc[5]);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            acc[6 + i] = fma_pair(q[3], kt[i], acc[6 + i]);
            put(sh.kt[s * kStep + i], kt[i]);
          }
          if constexpr (DELTA) {
            acc[10] = fma_pair(k[1], k10, acc[10]);
            acc[11] = fma_pair(k[2], k20, acc[11]);
            acc[12] = fma_pair(k[2], k21, acc[12]);
#pragma unroll
            for (int i = 0; i < 3; ++i) acc[13 + i] = fma_pair(k[3], kt[i], acc[13 + i]);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              acc[16 + i] = fma_pair(k[i], k[i], acc[16 + i]);
              acc[20 + i] = fma_pair(q[i], q[i], acc[20 + i]);
            }
          }
        }
      }
      float sum[NV];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const float2 f = unpair(i < 24 ? acc[i] : 0ull);
        sum[i] = f.x + f.y;
      }
      group_sum<NV, LB>(sum, lane);
      if (s < steps) {
#pragma unroll
        for (int i = 0; i < (NV > LB ? NV / LB : 1); ++i) sh.sums[s][pl * NV / LB + i] = sum[i];
      }
      __syncwarp();
      if (s < steps && pl < 8) {   // scales of the four keys, of the four queries
        float v = 1.f;
        if constexpr (DELTA) v = unit ? 1.f / sqrtf(sh.sums[s][16 + pl] + kUnitFloor) : 1.f;
        sh.scale[s][pl] = pl < 4 ? v : v * q_scale;
      }
      __syncwarp();
      if (s < steps) {
        const float *z = sh.sums[s], *zs = sh.scale[s];
        for (int x = pl; x < 16 + (DELTA ? 6 : 0); x += LB) {
          const int y = x - 16;
          const int i = x < 16 ? x >> 2 : y < 1 ? 1 : y < 3 ? 2 : 3, j = x < 16 ? x & 3 : y - below(i, 0);
          const float v = z[x < 16 ? min(upto(i, j), 9) : 10 + y] * zs[x < 16 ? 4 + i : i] * zs[j];
          if (x < 16) sh.mix[s][x] = j <= i ? v : 0.f;
          else sh.keys[s][y] = v;
        }
      }
      __syncwarp();
    }
    exec_sync();
    // ---- the steps
#pragma unroll 1
    for (int s = 0; s < steps; ++s) {
      float p[4 * C], o[4 * C];                                // [column][token]
      auto reads = [&](const float* rows4, float (&to)[4 * C]) {
        Pair acc[4][C];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int c = 0; c < C; ++c) acc[i][c] = 0ull;
        Pair x[2][4][2];   // loads run one group of rows ahead, and no further: more of them in flight would spill the state
        auto load = [&](int i4) {
#pragma unroll
          for (int i = 0; i < 4; ++i) ld_pairs(rows4 + i * DP + 4 * (l + G * i4), x[i4 & 1][i][0], x[i4 & 1][i][1]);
        };
        load(0);
#pragma unroll
        for (int i4 = 0; i4 < I4; ++i4) {
          asm volatile("" ::: "memory");
          if (i4 + 1 < I4) load(i4 + 1);
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
              for (int c = 0; c < C; ++c) acc[i][c] = fma_pair(S[c][i4][j], x[i4 & 1][i][j], acc[i][c]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int c = 0; c < C; ++c) {
            const float2 f = unpair(acc[i][c]);
            to[c * 4 + i] = f.x + f.y;
          }
        group_sum<4 * C, G>(to, lane);
      };
      // (the order of the passes is kept, so that only one has its sums in registers)
      if constexpr (DELTA) reads(sh.kh[s * kStep], p);
      asm volatile("" ::: "memory");
      reads(sh.qh[s * kStep], o);
      asm volatile("" ::: "memory");
      float u[4], zk[4];
      if constexpr (DELTA) ld_vec<4>(sh.scale[s], zk);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const T v = in.v[s * kStep + i][my_col];
        if constexpr (F32) u[i] = v;
        else u[i] = __bfloat162float(v);
      }
      if constexpr (DELTA) {
        float pp[4], zb[4], kk[4], kk4[2];
#pragma unroll
        for (int i = 0; i < 4; ++i) {   // the column's other lanes hold its other tokens
          if constexpr (NS == 4) pp[i] = p[i];
          else pp[i] = __shfl_sync(0xffffffffu, p[i % NS], col_lane + i * G / (4 * C));
        }
        ld_vec<4>(sh.beta[b] + s * kStep, zb);
        ld_vec<4>(sh.keys[s], kk);
        kk4[0] = sh.keys[s][4];
        kk4[1] = sh.keys[s][5];
        u[0] = zb[0] * (u[0] - zk[0] * pp[0]);
        u[1] = zb[1] * (u[1] - fmaf(kk[0], u[0], zk[1] * pp[1]));
        u[2] = zb[2] * (u[2] - fmaf(kk[2], u[1], fmaf(kk[1], u[0], zk[2] * pp[2])));
        u[3] = zb[3] * (u[3] - fmaf(kk4[1], u[2], fmaf(kk4[0], u[1], fmaf(kk[3], u[0], zk[3] * pp[3]))));
      }
      if constexpr (DELTA) {
        if (owner) *reinterpret_cast<float4*>(sh.u[s & 1][my_col]) = make_float4(zk[0] * u[0], zk[1] * u[1], zk[2] * u[2], zk[3] * u[3]);
      } else {
        if (owner) *reinterpret_cast<float4*>(sh.u[s & 1][my_col]) = make_float4(u[0], u[1], u[2], u[3]);
      }
#pragma unroll
      for (int n = 0; n < NS; ++n) {
        float mix[4];
        ld_vec<4>(sh.mix[s] + 4 * (my_tok + n), mix);
        const float y = fmaf(mix[3], u[3], fmaf(mix[2], u[2], fmaf(mix[1], u[1], fmaf(mix[0], u[0], sh.scale[s][4 + my_tok + n] * o[n]))));
        if (s * kStep + my_tok + n < nt && my_col < n_v) out[n * ld_out] = y;
      }
      out += kStep * ld_out;
      __syncwarp();
      Pair U[4][C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        float x[4];
        ld_vec<4>(sh.u[s & 1][c_lo + c], x);
#pragma unroll
        for (int i = 0; i < 4; ++i) U[i][c] = pair(x[i], x[i]);
      }
      Pair x[2][5][2];
      auto load = [&](int i4) {
        const int at = 4 * (l + G * i4);
        ld_pairs(&sh.em[s][at], x[i4 & 1][4][0], x[i4 & 1][4][1]);
#pragma unroll
        for (int i = 0; i < 4; ++i) ld_pairs(&sh.kt[s * kStep + i][at], x[i4 & 1][i][0], x[i4 & 1][i][1]);
      };
      load(0);
#pragma unroll
      for (int i4 = 0; i4 < I4; ++i4) {
        asm volatile("" ::: "memory");
        if (i4 + 1 < I4) load(i4 + 1);
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int c = 0; c < C; ++c) S[c][i4][j] = fma_pair(S[c][i4][j], x[i4 & 1][4][j], S[c][i4][j]);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int c = 0; c < C; ++c) S[c][i4][j] = fma_pair(x[i4 & 1][i][j], U[i][c], S[c][i4][j]);
      }
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < I4; ++i) {
      const int at = 4 * (l + G * i);
      if (at < dp && c_lo + c < n_v) {
        const float2 a = unpair(S[c][i][0]), b = unpair(S[c][i][1]);
        *reinterpret_cast<float4*>(state + static_cast<size_t>(c) * dp + at) = make_float4(a.x, a.y, b.x, b.y);
      }
    }
}

__device__ bool tile_gated_memory(const TileDesc& t, int tid, uint8_t* ring) {
  const GatedMemoryArgs* p = reinterpret_cast<const GatedMemoryArgs*>(t.a[0]);
  const uint32_t d = __ldcg(&p->d);
  const bool delta = __ldcg(&p->beta) != 0;
  const bool f32 = __ldcg(&p->f32) != 0;
  // a[1]: the columns of a block; 32-bit activations have the narrowest form only
#define MF_GATED(N, G, C, F32)                                                          \
  if (d <= N && t.a[1] == 128 * C / G && f32 == F32) {                                  \
    if (delta) gated_rows<G, (N) / (G), C, true, F32>(t, tid, ring);                    \
    else gated_rows<G, (N) / (G), C, false, F32>(t, tid, ring);                         \
    return true;                                                                        \
  }
  MF_GATED(32, 4, 2, false)
  MF_GATED(32, 4, 1, false)
  MF_GATED(32, 4, 1, true)
  MF_GATED(64, 8, 4, false)
  MF_GATED(64, 8, 2, false)
  MF_GATED(64, 8, 2, true)
  MF_GATED(128, 8, 4, false)
  MF_GATED(128, 8, 2, false)
  MF_GATED(128, 8, 2, true)
  MF_GATED(256, 8, 4, false)
  MF_GATED(256, 16, 4, false)
  MF_GATED(256, 16, 2, false)
  MF_GATED(256, 16, 2, true)
  MF_GATED(512, 32, 4, false)
  MF_GATED(512, 32, 4, true)
#undef MF_GATED
  return false;
}

// ------------------------------------------------------------------ one token
// Kind 69, GatedMemoryArgs: row i0, slot i3, i1 column blocks from block i2 on, counted through the heads (blocks of a head:
// its columns over kBlock, rounded up).  G lanes share a column (ND four-row groups of it each), NC columns a lane.  A wide
// tile: a warp's columns of a block are one piece of memory, which comes and goes by bulk copies through kDepth stages of
// its own in the ring.  The read-out comes from the state in front of the token's write, S^T q + (k q) u, so one round of
// sums per column serves both products.
template <int G, int ND, int NC, bool DELTA, bool F32>
__device__ __noinline__ bool gated_step(const TileDesc& t, int tid, const LayerCtx& ctx) {
  using T = typename std::conditional<F32, float, __nv_bfloat16>::type;
  constexpr int kSide = 32 / G, kWarp = NC * kSide, kBlock = 4 * kWarp;   // columns side by side in a warp; of a warp; of a block
  constexpr int kDepth = 6, kStageBytes = kWarp * G * ND * 16;
  static_assert(4 * kDepth * kStageBytes <= 216 * 1024 && kStageBytes % 128 == 0, "the operand ring");
  __builtin_assume(__isShared(ctx.ring));
  __builtin_assume(__isShared(ctx.scratch));
  struct Head {
    float k[ND][4], q[ND][4], m[ND][4], beta;
  };
  GatedMemoryArgs A;
  load_block(A, t.a[0]);
  const int row = static_cast<int>(t.i0), slot = static_cast<int>(t.i3), first = static_cast<int>(t.i2), last = first + static_cast<int>(t.i1);
  const int H = static_cast<int>(A.heads), d = static_cast<int>(A.d), e = static_cast<int>(A.e), group = static_cast<int>(A.group);
  const int dp = (d + 3) & ~3, oe = (e + 3) & ~3, warp = tid >> 5, lane = tid & 31, l = lane & (G - 1), side = lane / G;
  const int blocks = (e + kBlock - 1) / kBlock;
  const bool unit = A.unit != 0;
  const T* const k_row = reinterpret_cast<const T*>(A.k) + static_cast<size_t>(row) * A.ld_qkv;
  const T* const q_row = reinterpret_cast<const T*>(A.q) + static_cast<size_t>(row) * A.ld_qkv;
  const T* const v_row = reinterpret_cast<const T*>(A.v) + static_cast<size_t>(row) * A.ld_qkv;
  const float* const m_row = f32p(A.decay) + static_cast<size_t>(row) * A.ld_decay;
  const bool vec = (d & 3) == 0 && ((A.k | A.q) & (4 * sizeof(T) - 1)) == 0;
  float* const state = reinterpret_cast<float*>(A.state) + static_cast<size_t>(slot) * H * e * dp;
  // column c of this lane's NC is c_lo + c * kSide; after the sums the lane owns column c_lo + own * kSide
  const int own = l * NC / G;
  const bool writes = (l * NC) % G == 0;
  auto value = [](T v) -> float {
    if constexpr (F32) return v;
    else return __bfloat162float(v);
  };
  auto load4 = [&](const T* p, float (&v)[4]) {
    if constexpr (F32) {
      ld_vec<4>(p, v);
    } else {
      const uint2 u = *reinterpret_cast<const uint2*>(p);
      v[0] = __uint_as_float(u.x << 16);
      v[1] = __uint_as_float(u.x & 0xffff0000u);
      v[2] = __uint_as_float(u.y << 16);
      v[3] = __uint_as_float(u.y & 0xffff0000u);
    }
  };
  uint8_t* const stages = ctx.ring + warp * kDepth * kStageBytes;
  uint64_t* const bar = reinterpret_cast<uint64_t*>(ctx.scratch) + warp * kDepth;
  struct Place {
    int head, col, n;   // first column of this warp in the block, and how many it has
  };
  auto place = [&](int b) {
    Place x;
    x.head = b / blocks;
    x.col = (b - x.head * blocks) * kBlock + warp * kWarp;
    x.n = max(0, min(kWarp, e - x.col));
    return x;
  };
  auto state_at = [&](const Place& x) { return state + (static_cast<size_t>(x.head) * e + x.col) * dp; };
  auto fetch = [&](int i) {   // lane 0
    const Place x = place(first + i);
    if (x.n == 0) return;
    const uint32_t bytes = static_cast<uint32_t>(x.n * dp) * 4;
    mbar_arrive_expect_tx(bar + i % kDepth, bytes);
    bulk_in(stages + i % kDepth * kStageBytes, state_at(x), bytes, bar + i % kDepth);
  };
  auto fetch_v = [&](int b) {   // of the column this lane owns
    const Place x = place(min(b, last - 1));
    const int c = own * kSide + side;
    return c < x.n ? value(v_row[static_cast<size_t>(x.head) * e + x.col + c]) : 0.f;
  };
  auto fetch_head = [&](int head, Head& X) {
    const int kv = head / group;
#pragma unroll
    for (int i = 0; i < ND; ++i) {
      const int at = 4 * (l + G * i);
#pragma unroll
      for (int j = 0; j < 4; ++j) X.k[i][j] = X.q[i][j] = X.m[i][j] = 0.f;
      if (vec) {
        if (at < d) {
          load4(k_row + kv * d + at, X.k[i]);
          load4(q_row + kv * d + at, X.q[i]);
          ld_vec<4>(m_row + head * d + at, X.m[i]);
        }
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (at + j < d) {
            X.k[i][j] = value(k_row[kv * d + at + j]);
            X.q[i][j] = value(q_row[kv * d + at + j]);
            X.m[i][j] = m_row[head * d + at + j];
          }
      }
    }
    if constexpr (DELTA) X.beta = value(reinterpret_cast<const T*>(A.beta)[static_cast<size_t>(row) * A.ld_beta + head]);
  };
  fence_proxy_async_all();   // the state may have been written, and the ring used, by plain loads and stores
  if (lane < kDepth) mbar_init(bar + lane, 1);
  fence_barrier_init();
  exec_sync();
  const int n_blocks = last - first;
  if (lane == 0)
    for (int i = 0; i < min(n_blocks, kDepth - 1); ++i) fetch(i);
  Head next, X;
  fetch_head(first / blocks, next);
  float v0 = fetch_v(first), v1 = fetch_v(first + 1);
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row] == 0;
  int at_head = -1;
  float zk = 1.f, zq = 0.f, kq = 0.f, beta = 0.f;
  uint32_t phases = 0;   // a bit per stage: loads are counted only where the warp has columns
  bool ok = true;
#pragma unroll 1
  for (int it = 0; it < n_blocks; ++it) {
    const int s = it % kDepth;
    const Place at_block = place(first + it);
    const int head = at_block.head, n_cols = at_block.n;
    const float v = v0;
    v0 = v1;
    v1 = fetch_v(first + it + 2);
    if (head != at_head) {   // the next head's row, and the one after it on its way
      at_head = head;
      X = next;
      if (head < (last - 1) / blocks) fetch_head(head + 1, next);
      float dots[3] = {0.f, 0.f, 0.f};                         // k k, q q, k q
#pragma unroll
      for (int i = 0; i < ND; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          dots[0] = fmaf(X.k[i][j], X.k[i][j], dots[0]);
          dots[1] = fmaf(X.q[i][j], X.q[i][j], dots[1]);
          dots[2] = fmaf(X.k[i][j], X.q[i][j], dots[2]);
        }
#pragma unroll
      for (int bit = G / 2; bit >= 1; bit >>= 1)
#pragma unroll
        for (int i = 0; i < 3; ++i) dots[i] += __shfl_xor_sync(0xffffffffu, dots[i], bit);
      zk = unit ? 1.f / sqrtf(dots[0] + kUnitFloor) : 1.f;
      zq = A.q_scale * (unit ? 1.f / sqrtf(dots[1] + kUnitFloor) : 1.f);
      kq = dots[2] * zk * zq;
      if constexpr (DELTA) beta = sigmoid32(X.beta);
    }
    if (n_cols > 0) {
      ok = __all_sync(0xffffffffu, mbar_wait_bounded(bar + s, (phases >> s) & 1u, ctx.abort_flag, kWideWaitNs));
      if (!ok) {   // the loads behind this one end, or run out of their time, before the ring is left
        for (int j = it; j < min(n_blocks, it + kDepth - 1); ++j)
          for (int tries = 0; place(first + j).n > 0 && tries < 1 << 16 && !mbar_try_wait(bar + j % kDepth, (phases >> j % kDepth) & 1u); ++tries) {}
        break;
      }
      phases ^= 1u << s;
    }
    float* const S = reinterpret_cast<float*>(stages + s * kStageBytes) + side * dp;   // column c of this lane: c * kSide * dp on
    float4 reg[NC][ND];
    float o[NC], p[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      o[c] = p[c] = 0.f;
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        const int at = 4 * (l + G * i);
        float4& r = reg[c][i];
        r = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && at < dp && c * kSide + side < n_cols) r = *reinterpret_cast<const float4*>(S + c * kSide * dp + at);
        r.x = fmaf(r.x, X.m[i][0], r.x);
        r.y = fmaf(r.y, X.m[i][1], r.y);
        r.z = fmaf(r.z, X.m[i][2], r.z);
        r.w = fmaf(r.w, X.m[i][3], r.w);
        o[c] = fmaf(r.x, X.q[i][0], fmaf(r.y, X.q[i][1], fmaf(r.z, X.q[i][2], fmaf(r.w, X.q[i][3], o[c]))));
        if constexpr (DELTA) p[c] = fmaf(r.x, X.k[i][0], fmaf(r.y, X.k[i][1], fmaf(r.z, X.k[i][2], fmaf(r.w, X.k[i][3], p[c]))));
      }
    }
    group_sum<NC, G>(o, lane);
    float u = v;
    if constexpr (DELTA) {
      group_sum<NC, G>(p, lane);
      u = beta * (v - zk * p[0]);
    }
    if (writes && own * kSide + side < n_cols)
      reinterpret_cast<float*>(A.out)[(static_cast<size_t>(row) * H + head) * oe + at_block.col + own * kSide + side] = fmaf(kq, u, zq * o[0]);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const float x = zk * __shfl_sync(0xffffffffu, u, side * G + c * G / NC);
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        float4 r = reg[c][i];
        r.x = fmaf(X.k[i][0], x, r.x);
        r.y = fmaf(X.k[i][1], x, r.y);
        r.z = fmaf(X.k[i][2], x, r.z);
        r.w = fmaf(X.k[i][3], x, r.w);
        const int at = 4 * (l + G * i);
        if (at < dp && c * kSide + side < n_cols) *reinterpret_cast<float4*>(S + c * kSide * dp + at) = r;
      }
    }
    fence_proxy_async_smem();
    __syncwarp();
    if (lane == 0) {
      if (n_cols > 0) bulk_store(state_at(at_block), stages + s * kStageBytes, static_cast<uint32_t>(n_cols * dp) * 4);
      bulk_commit();
      if (it + kDepth - 1 < n_blocks) {   // into the stage of the block before, once its store has read it
        bulk_wait_read<1>();
        fetch(it + kDepth - 1);
      }
    }
    __syncwarp();
  }
  if (lane == 0) bulk_wait_all();
  ok = exec_and(ok);
  if (lane < kDepth) mbar_inval(bar + lane);
  return ok;
}

__device__ bool tile_gated_step(const TileDesc& t, int tid, const LayerCtx& ctx) {
  const GatedMemoryArgs* p = reinterpret_cast<const GatedMemoryArgs*>(t.a[0]);
  const uint32_t d = __ldcg(&p->d);
  const bool delta = __ldcg(&p->beta) != 0, f32 = __ldcg(&p->f32) != 0;
#define MF_STEP(N, G, ND, NC)                                             \
  if (d <= N) {                                                           \
    if (delta && f32) return gated_step<G, ND, NC, true, true>(t, tid, ctx);   \
    if (delta) return gated_step<G, ND, NC, true, false>(t, tid, ctx);         \
    if (f32) return gated_step<G, ND, NC, false, true>(t, tid, ctx);           \
    return gated_step<G, ND, NC, false, false>(t, tid, ctx);                   \
  }
  MF_STEP(32, 8, 1, 8)
  MF_STEP(64, 16, 1, 16)
  MF_STEP(128, 32, 1, 16)
  MF_STEP(256, 32, 2, 8)
  MF_STEP(512, 32, 4, 4)
#undef MF_STEP
  return false;
}

}  // namespace fab
}  // namespace mf
