// Short convolution and selective scan of the layer-list decoders (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"
#include "wide_tile.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ short convolution
// Kind 54, ConvArgs: i0 the request's first row, i1 first row of this tile, i2 rows | channels << 16, i3 slot,
// a[1] first channel, a[2] the request's rows (read with `advance`).  A thread walks down V channels with the last TAPS - 1 inputs in registers, eight rows' loads in
// flight.  V = 8: bf16 rows in 16-byte pieces.
template <bool F32, int V, int TAPS>
__device__ __noinline__ void conv_rows(const TileDesc& t, int tid) {
  ConvArgs A;
  load_block(A, t.a[0]);
  const int row0 = static_cast<int>(t.i0), r_lo = static_cast<int>(t.i1), r_hi = r_lo + static_cast<int>(t.i2 & 0xffffu);
  const int n_ch = static_cast<int>(t.i2 >> 16), ch0 = static_cast<int>(t.a[1]), taps = static_cast<int>(A.taps);
  const int C = static_cast<int>(A.channels);
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  float* tail = reinterpret_cast<float*>(A.tail) + static_cast<size_t>(t.i3) * (taps - 1) * C;
  using Raw = typename std::conditional<V == 8, uint4, float>::type;
  auto load = [&](int r, int c) -> Raw {   // row r >= row0
    const size_t at = static_cast<size_t>(r) * A.ld_x + c;
    if constexpr (V == 8) return *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(A.x) + at);
    else return act_ld(A.x, at, F32);
  };
  auto unpack = [&](const Raw& raw, float (&v)[V]) {
    if constexpr (V == 8) {
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
      }
    } else {
      v[0] = raw;
    }
  };
  for (int c = ch0 + tid * V; c < ch0 + n_ch; c += kExecThreads * V) {
    float w[TAPS][V], bias[V], win[TAPS][V];   // win: the inputs at rows r - TAPS + 1 .. r, newest last
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      const int tap = k - (TAPS - taps);
#pragma unroll
      for (int j = 0; j < V; ++j) w[k][j] = tap >= 0 ? f32p(A.w)[static_cast<size_t>(c + j) * taps + tap] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < V; ++j) bias[j] = A.bias ? f32p(A.bias)[c + j] : 0.f;
#pragma unroll
    for (int k = 1; k < TAPS; ++k) {
      const int r = r_lo - TAPS + k, place = r - row0 + taps - 1;   // place in the tail, for rows before the portion
      if (r >= row0) {
        unpack(load(r, c), win[k]);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) win[k][j] = (fresh || place < 0) ? 0.f : tail[static_cast<size_t>(place) * C + c + j];
      }
    }
    for (int r = r_lo; r < r_hi; r += 8) {
      Raw in[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) in[i] = load(min(r + i, r_hi - 1), c);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (r + i >= r_hi) break;
        float x[V], o[V];
        unpack(in[i], x);
#pragma unroll
        for (int j = 0; j < V; ++j) {
#pragma unroll
          for (int k = 0; k < TAPS - 1; ++k) win[k][j] = win[k + 1][j];
          win[TAPS - 1][j] = x[j];
          float acc = bias[j];
#pragma unroll
          for (int k = 0; k < TAPS; ++k) acc = fmaf(w[k][j], win[k][j], acc);
          o[j] = F32 ? acc / (1.f + expf(-acc)) : __fdividef(acc, 1.f + __expf(-acc));
        }
        const size_t at = static_cast<size_t>(r + i) * A.ld_out + c;
        if constexpr (V == 8) {
          __nv_bfloat162 h[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(o[2 * j], o[2 * j + 1]);
          *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(A.out) + at) = *reinterpret_cast<const uint4*>(h);
        } else {
          act_st(A.out, at, F32, o[0]);
        }
      }
    }
    if (A.advance && r_lo == row0) {   // the last taps - 1 inputs of [old tail, this portion]
      const int n = static_cast<int>(t.a[2]);
      for (int place = 0; place < taps - 1; ++place) {
        const int k = n + place;
        float in[V];
        if (k >= taps - 1) {
          unpack(load(row0 + k - (taps - 1), c), in);
        } else {
#pragma unroll
          for (int j = 0; j < V; ++j) in[j] = fresh ? 0.f : tail[static_cast<size_t>(k) * C + c + j];
        }
#pragma unroll
        for (int j = 0; j < V; ++j) tail[static_cast<size_t>(place) * C + c + j] = in[j];
      }
    }
  }
}

__device__ void tile_conv(const TileDesc& t, int tid) {
  const ConvArgs* p = reinterpret_cast<const ConvArgs*>(t.a[0]);
  const uint32_t taps = __ldcg(&p->taps);
  if (__ldcg(&p->f32)) conv_rows<true, 1, kMaxTaps>(t, tid);
  else if ((__ldcg(&p->channels) & 7) != 0) conv_rows<false, 1, kMaxTaps>(t, tid);
  else if (taps <= 4) conv_rows<false, 8, 4>(t, tid);
  else conv_rows<false, 8, kMaxTaps>(t, tid);
}

// ------------------------------------------------------------------ selective scan
// Kind 55, ScanArgs: rows [i0, i0 + i1) of one request, channels [i2, i2 + 32) (as many as there are), slot i3.  A wide
// tile: the inputs come 32 tokens at a time through double-buffered asynchronous copies into the operand ring.  Four
// lanes share a channel, each with NS of its states in registers.  Four tokens at a time: lane p prepares and finishes
// token p of the four (step size, output gate), so what a channel needs once per token is computed once; the four state
// updates of a token run in all lanes.  F32: the exact form.  It multiplies by e^x as S + S (e^x - 1), so that the
// rounding of a factor just below one does not add up over a long memory.
constexpr int kScanTokens = 32, kScanChannels = kExecThreads / 4;

template <int NS, bool F32>
__device__ __noinline__ void scan_rows(const TileDesc& t, int tid, uint8_t* ring) {
  using T = typename std::conditional<F32, float, __nv_bfloat16>::type;
  constexpr int NP = 4 * NS;                              // states, padded
  constexpr int kPer16 = 16 / static_cast<int>(sizeof(T));
  struct Chunk {
    float dt[kScanTokens][kScanChannels];
    float bc[kScanTokens][2 * NP];                        // B, then C
    T x[kScanTokens][kScanChannels];
    T z[kScanTokens][kScanChannels];
  };
  struct Shared {
    Chunk in[2];
    T y[kScanTokens][kScanChannels];
  };
  static_assert(sizeof(Shared) <= 216 * 1024, "the operand ring");
  __builtin_assume(__isShared(ring));
  Shared& sh = *reinterpret_cast<Shared*>(ring);
  ScanArgs A;
  load_block(A, t.a[0]);
  const int row0 = static_cast<int>(t.i0), rows = static_cast<int>(t.i1), slot = static_cast<int>(t.i3);
  const int ch0 = static_cast<int>(t.i2);
  const int n = static_cast<int>(A.n), C = static_cast<int>(A.channels), taps = static_cast<int>(A.taps);
  const int warp = tid >> 5, lane = tid & 31, p = tid & 3, my = tid >> 2;
  const int c = min(ch0 + my, C - 1);                     // a channel past the end repeats the last one
  const bool c_ok = ch0 + my < C;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  const int s0 = p * NS;
  float S[NS], a[NS];
  float* state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * C + c) * n;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool ok = s0 + i < n;
    S[i] = (ok && !fresh) ? state[s0 + i] : 0.f;
    a[i] = ok ? f32p(A.A)[static_cast<size_t>(c) * n + s0 + i] * (F32 ? 1.f : 1.4426950408889634f) : 0.f;
  }
  const float D = f32p(A.D)[c], dt_bias = f32p(A.dt_bias)[c];
  const bool z16 = (A.z & 15) == 0, bc16 = ((A.b | A.c) & 15) == 0 && (n & 3) == 0;
  // the padding of B and C, and their rows past the end of a short chunk, must be finite
  for (int i = tid; i < 2 * kScanTokens * 2 * NP; i += kExecThreads)
    (&sh.in[i / (kScanTokens * 2 * NP)].bc[0][0])[i % (kScanTokens * 2 * NP)] = 0.f;
  exec_sync();
  auto stage = [&](int base, Chunk& k) {
    const int nt = min(kScanTokens, rows - base);
    const T* x = reinterpret_cast<const T*>(A.x);
    const T* z = reinterpret_cast<const T*>(A.z);
    // rows of 32 channels: 8 pieces of dt, 32 / kPer16 of x and of z; rows are padded, so whole pieces may be read
    constexpr int kPieces = 8 + kScanChannels / kPer16;
    for (int i = tid; i < nt * kPieces; i += kExecThreads) {
      const int tok = i / kPieces, q = i - tok * kPieces;
      const size_t r = static_cast<size_t>(row0 + base + tok);
      if (q < 8) cp16(&k.dt[tok][4 * q], f32p(A.dt) + r * A.ld_dt + ch0 + 4 * q);
      else cp16(&k.x[tok][(q - 8) * kPer16], x + r * A.ld_x + ch0 + (q - 8) * kPer16);
    }
    if (z16) {
      constexpr int kZ = kScanChannels / kPer16;
      for (int i = tid; i < nt * kZ; i += kExecThreads)
        cp16(&k.z[i / kZ][(i % kZ) * kPer16], z + static_cast<size_t>(row0 + base + i / kZ) * A.ld_z + ch0 + (i % kZ) * kPer16);
    } else {
      for (int tok = warp; tok < nt; tok += kExecThreads / 32)
        k.z[tok][lane] = z[static_cast<size_t>(row0 + base + tok) * A.ld_z + min(ch0 + lane, C - 1)];
    }
    if (bc16) {
      const int np = n >> 2;
      for (int tok = warp; tok < nt; tok += kExecThreads / 32) {
        const size_t at = static_cast<size_t>(row0 + base + tok) * A.ld_bc;
        for (int q = lane; q < 2 * np; q += 32) {
          const bool second = q >= np;
          const int k4 = 4 * (second ? q - np : q);
          cp16(&k.bc[tok][(second ? NP : 0) + k4], f32p(second ? A.c : A.b) + at + k4);
        }
      }
    } else {
      for (int tok = warp; tok < nt; tok += kExecThreads / 32) {
        const size_t at = static_cast<size_t>(row0 + base + tok) * A.ld_bc;
        for (int q = lane; q < n; q += 32) {
          k.bc[tok][q] = f32p(A.b)[at + q];
          k.bc[tok][NP + q] = f32p(A.c)[at + q];
        }
      }
    }
    cp_commit();
  };
  auto value = [](const T& v) -> float {
    if constexpr (F32) return v;
    else return __bfloat162float(v);
  };
  stage(0, sh.in[0]);
  for (int base = 0, s = 0; base < rows; base += kScanTokens, s ^= 1) {
    const int nt = min(kScanTokens, rows - base);
    if (base + kScanTokens < rows) {
      stage(base + kScanTokens, sh.in[s ^ 1]);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    exec_sync();
    Chunk& k = sh.in[s];
    // Step sizes of the chunk, lane p those of tokens p, p + 4, ...; a token past the end gets step 0 and input 0, which
    // leaves the state as it is.  (Loops stay rolled: one warp per scheduler runs this, and a body beyond the instruction
    // cache costs more than it hides.)
#pragma unroll 2
    for (int mine = p; mine < kScanTokens; mine += 4) {
      const float u = k.dt[mine][my] + dt_bias;
      const float dt = F32 ? softplus32(u) : fmaxf(u, 0.f) + __logf(1.f + __expf(-fabsf(u)));
      k.dt[mine][my] = mine < nt ? dt : 0.f;
    }
    __syncwarp();
#pragma unroll 1
    for (int g = 0; g < nt; g += 4) {
      const int mine = g + p;
      const float x = value(k.x[mine][my]), z = value(k.z[mine][my]);
      float part[4];
#pragma unroll
      for (int i4 = 0; i4 < 4; ++i4) {
        const float dk = k.dt[g + i4][my];
        const float xk = g + i4 < nt ? dk * value(k.x[g + i4][my]) : 0.f;
        float B[NS], Cv[NS];
        const float *b = &k.bc[g + i4][s0], *cc = &k.bc[g + i4][NP + s0];
        if constexpr ((NS & 3) == 0) {
#pragma unroll
          for (int i = 0; i < NS; i += 4) {
            ld_vec<4>(b + i, *reinterpret_cast<float(*)[4]>(&B[i]));
            ld_vec<4>(cc + i, *reinterpret_cast<float(*)[4]>(&Cv[i]));
          }
        } else {
#pragma unroll
          for (int i = 0; i < NS; ++i) {
            B[i] = b[i];
            Cv[i] = cc[i];
          }
        }
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          if constexpr (F32) S[i] += fmaf(S[i], expm1f(dk * a[i]), xk * B[i]);
          else S[i] = fmaf(ex2(dk * a[i]), S[i], xk * B[i]);
          y = fmaf(S[i], Cv[i], y);
        }
        part[i4] = y;
      }
      // the four lanes' sums, lane p ending with token p's
      const bool odd = p & 1, hi = p & 2;
      const float t0 = (odd ? part[1] : part[0]) + __shfl_xor_sync(0xffffffffu, odd ? part[0] : part[1], 1);
      const float t1 = (odd ? part[3] : part[2]) + __shfl_xor_sync(0xffffffffu, odd ? part[2] : part[3], 1);
      const float out = (hi ? t1 : t0) + __shfl_xor_sync(0xffffffffu, hi ? t0 : t1, 2);
      if (mine < nt) {
        const float y = fmaf(D, x, out) * (F32 ? z / (1.f + expf(-z)) : __fdividef(z, 1.f + __expf(-z)));
        if constexpr (F32) sh.y[mine][my] = y;
        else sh.y[mine][my] = __float2bfloat16(y);
      }
    }
    exec_sync();
    // rows of y are padded to whole pieces
    constexpr int kY = kScanChannels / kPer16;
    for (int i = tid; i < nt * kY; i += kExecThreads)
      *reinterpret_cast<uint4*>(reinterpret_cast<T*>(A.y) + static_cast<size_t>(row0 + base + i / kY) * A.ld_y + ch0 + (i % kY) * kPer16) =
          *reinterpret_cast<const uint4*>(&sh.y[i / kY][(i % kY) * kPer16]);
  }
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (c_ok && s0 + i < n) state[s0 + i] = S[i];
  // the convolution's tail: the last taps - 1 inputs of [old tail, this portion]
  if (c_ok && p == 0) {
    float* tail = reinterpret_cast<float*>(A.tail) + static_cast<size_t>(slot) * (taps - 1) * C + c;
    for (int j = 0; j < taps - 1; ++j) {
      const int k = rows + j;
      tail[static_cast<size_t>(j) * C] =
          k >= taps - 1 ? act_ld(A.x_in, static_cast<size_t>(row0 + k - (taps - 1)) * A.ld_z + c, F32)
                        : (fresh ? 0.f : tail[static_cast<size_t>(k) * C]);
    }
  }
}

// Kind 65, ScanArgs: one token.  Row i0, channels [i2, i2 + i1), slot i3; a thread per channel, NS of its states at a
// time with their loads in flight together.
template <bool F32>
__device__ __noinline__ void scan_step(const TileDesc& t, int tid) {
  constexpr int NS = 16;
  ScanArgs A;
  load_block(A, t.a[0]);
  const int row = static_cast<int>(t.i0), slot = static_cast<int>(t.i3);
  const int n = static_cast<int>(A.n), C = static_cast<int>(A.channels), taps = static_cast<int>(A.taps);
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row] == 0;
  const float *gb = f32p(A.b) + static_cast<size_t>(row) * A.ld_bc, *gc = f32p(A.c) + static_cast<size_t>(row) * A.ld_bc;
  const bool vec = (n & 3) == 0 && ((A.b | A.c) & 15) == 0;
  auto ld4 = [&](const float* p, int i, float (&v)[4]) {
    if (vec) {
      ld_vec<4>(p + i, v);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = i + j < n ? p[i + j] : 0.f;
    }
  };
  for (int c = static_cast<int>(t.i2) + tid; c < static_cast<int>(t.i2 + t.i1); c += kExecThreads) {
    const size_t sc = (static_cast<size_t>(slot) * C + c) * n;
    float* state = reinterpret_cast<float*>(A.state) + sc;
    const float* a = f32p(A.A) + static_cast<size_t>(c) * n;
    const float u = f32p(A.dt)[static_cast<size_t>(row) * A.ld_dt + c] + f32p(A.dt_bias)[c];
    const float x = act_ld(A.x, static_cast<size_t>(row) * A.ld_x + c, F32), z = act_ld(A.z, static_cast<size_t>(row) * A.ld_z + c, F32);
    const float D = f32p(A.D)[c];
    float* tail = reinterpret_cast<float*>(A.tail) + static_cast<size_t>(slot) * (taps - 1) * C + c;
    float old[kMaxTaps];
#pragma unroll
    for (int j = 1; j < kMaxTaps; ++j)
      if (j < taps - 1) old[j] = fresh ? 0.f : tail[static_cast<size_t>(j) * C];
    const float newest = taps > 1 ? act_ld(A.x_in, static_cast<size_t>(row) * A.ld_z + c, F32) : 0.f;
    float dt = 0.f, y = 0.f;
    for (int s0 = 0; s0 < n; s0 += NS) {
      float S[NS / 4][4], av[NS / 4][4], B[NS / 4][4], Cv[NS / 4][4];
#pragma unroll
      for (int i = 0; i < NS / 4; ++i) {
        const int k = s0 + 4 * i;
        if (k >= n) break;
        if (!fresh) ld4(state, k, S[i]);
        else S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
        ld4(a, k, av[i]);
        ld4(gb, k, B[i]);
        ld4(gc, k, Cv[i]);
      }
      if (s0 == 0) dt = F32 ? softplus32(u) : fmaxf(u, 0.f) + __logf(1.f + __expf(-fabsf(u)));
#pragma unroll
      for (int i = 0; i < NS / 4; ++i) {
        const int k = s0 + 4 * i;
        if (k >= n) break;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if constexpr (F32) S[i][j] += fmaf(S[i][j], expm1f(dt * av[i][j]), dt * x * B[i][j]);
          else S[i][j] = fmaf(__expf(dt * av[i][j]), S[i][j], dt * x * B[i][j]);
          y = fmaf(S[i][j], Cv[i][j], y);
        }
        if (vec) {
          st_vec<4>(state + k, S[i]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (k + j < n) state[k + j] = S[i][j];
        }
      }
    }
    y = fmaf(D, x, y);
    act_st(A.y, static_cast<size_t>(row) * A.ld_y + c, F32, y * (F32 ? z / (1.f + expf(-z)) : __fdividef(z, 1.f + __expf(-z))));
#pragma unroll
    for (int j = 0; j < kMaxTaps - 1; ++j) {
      if (j < taps - 2) tail[static_cast<size_t>(j) * C] = old[j + 1];
      else if (j == taps - 2) tail[static_cast<size_t>(j) * C] = newest;
    }
  }
}

__device__ void tile_scan_step(const TileDesc& t, int tid) {
  if (__ldcg(&reinterpret_cast<const ScanArgs*>(t.a[0])->f32)) scan_step<true>(t, tid);
  else scan_step<false>(t, tid);
}

__device__ bool tile_scan(const TileDesc& t, int tid, uint8_t* ring) {
  const ScanArgs* p = reinterpret_cast<const ScanArgs*>(t.a[0]);
  const uint32_t ns = (__ldcg(&p->n) + 3) / 4;
  const bool f32 = __ldcg(&p->f32) != 0;
#define MF_SCAN(N)                             \
  if (ns <= N) {                               \
    if (f32) scan_rows<N, true>(t, tid, ring); \
    else scan_rows<N, false>(t, tid, ring);    \
    return true;                               \
  }
  MF_SCAN(1)
  MF_SCAN(2)
  MF_SCAN(4)
  MF_SCAN(6)
  MF_SCAN(8)
  MF_SCAN(16)
  MF_SCAN(32)
#undef MF_SCAN
  return false;
}

}  // namespace fab
}  // namespace mf
