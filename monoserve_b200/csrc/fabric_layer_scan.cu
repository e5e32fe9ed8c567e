// Short convolution and selective scan of the layer-list decoders (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ short convolution
// Kind 54, ConvArgs: i0 the request's first row, i1 first row of this tile, i2 rows | channels << 16, i3 slot,
// a[1] first channel.  A thread walks down one channel (two in bf16) with the last `taps` inputs in registers.
template <bool F32, int V>
__device__ __noinline__ void conv_rows(const TileDesc& t, int tid) {
  ConvArgs A;
  load_block(A, t.a[0]);
  const int row0 = static_cast<int>(t.i0), r_lo = static_cast<int>(t.i1), rows = static_cast<int>(t.i2 & 0xffffu);
  const int n_ch = static_cast<int>(t.i2 >> 16), ch0 = static_cast<int>(t.a[1]), taps = static_cast<int>(A.taps);
  const int C = static_cast<int>(A.channels);
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  const float* tail = f32p(A.tail) + static_cast<size_t>(t.i3) * (taps - 1) * C;
  auto load = [&](int r, int c, float (&v)[V]) {   // the input at row r of the portion, r < row0: before it
    if (r < row0) {
      const int k = r - row0 + taps - 1;   // place in the tail
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = (fresh || k < 0) ? 0.f : tail[static_cast<size_t>(k) * C + c + j];
    } else if constexpr (!F32 && V == 2) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(
          reinterpret_cast<const __nv_bfloat16*>(A.x) + static_cast<size_t>(r) * A.ld_x + c));
      v[0] = f.x; v[1] = f.y;
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = act_ld(A.x, static_cast<size_t>(r) * A.ld_x + c + j, F32);
    }
  };
  for (int c = ch0 + tid * V; c < ch0 + n_ch; c += kExecThreads * V) {
    float w[kMaxTaps][V], bias[V], win[kMaxTaps][V];   // win: the inputs at rows r - 7 .. r, newest last
#pragma unroll
    for (int k = 0; k < kMaxTaps; ++k) {
      const int tap = k - (kMaxTaps - taps);
#pragma unroll
      for (int j = 0; j < V; ++j) w[k][j] = tap >= 0 ? f32p(A.w)[static_cast<size_t>(c + j) * taps + tap] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < V; ++j) bias[j] = f32p(A.bias)[c + j];
#pragma unroll
    for (int k = 0; k < kMaxTaps - 1; ++k) {
      if (k >= kMaxTaps - taps) load(r_lo - (kMaxTaps - 1) + k, c, win[k + 1]);
      else
#pragma unroll
        for (int j = 0; j < V; ++j) win[k + 1][j] = 0.f;
    }
    for (int r = r_lo; r < r_lo + rows; r += 8) {
      float in[8][V];
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (r + i < r_lo + rows) load(r + i, c, in[i]);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (r + i >= r_lo + rows) break;
        float o[V];
#pragma unroll
        for (int j = 0; j < V; ++j) {
#pragma unroll
          for (int k = 0; k < kMaxTaps - 1; ++k) win[k][j] = win[k + 1][j];
          win[kMaxTaps - 1][j] = in[i][j];
          float acc = bias[j];
#pragma unroll
          for (int k = 0; k < kMaxTaps; ++k) acc = fmaf(w[k][j], win[k][j], acc);
          o[j] = acc / (1.f + expf(-acc));
        }
        const size_t at = static_cast<size_t>(r + i) * A.ld_out + c;
        if constexpr (!F32 && V == 2)
          *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(A.out) + at) = __floats2bfloat162_rn(o[0], o[1]);
        else
#pragma unroll
          for (int j = 0; j < V; ++j) act_st(A.out, at + j, F32, o[j]);
      }
    }
  }
}

__device__ void tile_conv(const TileDesc& t, int tid) {
  const ConvArgs* p = reinterpret_cast<const ConvArgs*>(t.a[0]);
  const uint32_t f32 = __ldcg(&p->f32), C = __ldcg(&p->channels);
  if (f32) conv_rows<true, 1>(t, tid);
  else if ((C & 1) == 0) conv_rows<false, 2>(t, tid);
  else conv_rows<false, 1>(t, tid);
}

// ------------------------------------------------------------------ selective scan
// Kind 55, ScanArgs: rows [i0, i0 + i1) of one request, channels [i2, i2 + 32) (as many as there are), slot i3.
// Four lanes share a channel, each with NS of its states.  Four tokens at a time: lane p loads, prepares and
// finishes token p of the four (step size, input, output gate), so what a channel needs once per token is computed
// once; the four state updates of a token run in all lanes.  The loads of the next four tokens are issued before
// the current four are computed.
// F32: the exact form.  It multiplies by e^x as S + S (e^x - 1), so that the rounding of a factor just below one does
// not add up over a long memory.
template <int NS, bool F32>
__device__ __noinline__ void scan_rows(const TileDesc& t, int tid) {
  ScanArgs A;
  load_block(A, t.a[0]);
  const int row0 = static_cast<int>(t.i0), rows = static_cast<int>(t.i1), slot = static_cast<int>(t.i3);
  const int n = static_cast<int>(A.n), C = static_cast<int>(A.channels), taps = static_cast<int>(A.taps);
  const int p = tid & 3, lane = tid & 31, quad = lane & ~3;
  const int c = min(static_cast<int>(t.i2) + (tid >> 2), C - 1);   // a channel past the end repeats the last one
  const bool c_ok = static_cast<int>(t.i2) + (tid >> 2) < C;
  const bool fresh = reinterpret_cast<const int*>(A.tok_pos)[row0] == 0;
  const int s0 = p * NS;
  float S[NS], a[NS];
  float* state = reinterpret_cast<float*>(A.state) + (static_cast<size_t>(slot) * C + c) * n;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool ok = s0 + i < n;
    S[i] = (ok && !fresh) ? state[s0 + i] : 0.f;
    a[i] = ok ? f32p(A.A)[static_cast<size_t>(c) * n + s0 + i] : 0.f;
  }
  const float D = f32p(A.D)[c], dt_bias = f32p(A.dt_bias)[c];
  struct Four {
    float dt, x, z;
    float B[4][NS], Cc[4][NS];
  };
  const bool vec = (NS & 3) == 0 && n == 4 * NS && (A.ld_bc & 3) == 0 && ((A.b | A.c) & 15) == 0;
  auto fetch = [&](int r, Four& f) {
    const int mine = min(r + p, row0 + rows - 1);   // rows past the end repeat the last one and are not used
    f.dt = f32p(A.dt)[static_cast<size_t>(mine) * A.ld_dt + c];
    f.x = act_ld(A.x, static_cast<size_t>(mine) * A.ld_x + c, F32);
    f.z = act_ld(A.z, static_cast<size_t>(mine) * A.ld_z + c, F32);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const size_t at = static_cast<size_t>(min(r + k, row0 + rows - 1)) * A.ld_bc + s0;
      const float *b = f32p(A.b) + at, *cc = f32p(A.c) + at;
      if (vec) {
        if constexpr ((NS & 3) == 0) {
#pragma unroll
          for (int i = 0; i < NS; i += 4) {
            ld_vec<4>(b + i, *reinterpret_cast<float(*)[4]>(&f.B[k][i]));
            ld_vec<4>(cc + i, *reinterpret_cast<float(*)[4]>(&f.Cc[k][i]));
          }
        }
      } else {
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          f.B[k][i] = s0 + i < n ? b[i] : 0.f;
          f.Cc[k][i] = s0 + i < n ? cc[i] : 0.f;
        }
      }
    }
  };
  auto run = [&](int r, const Four& f) {
    const float dt = softplus32(f.dt + dt_bias), dtx = dt * f.x;
    float mine = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (r + k < row0 + rows) {
        const float dk = __shfl_sync(0xffffffffu, dt, quad + k), xk = __shfl_sync(0xffffffffu, dtx, quad + k);
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          if constexpr (F32) S[i] += fmaf(S[i], expm1f(dk * a[i]), xk * f.B[k][i]);
          else S[i] = fmaf(expf(dk * a[i]), S[i], xk * f.B[k][i]);
          y = fmaf(S[i], f.Cc[k][i], y);
        }
        y += __shfl_xor_sync(0xffffffffu, y, 1);
        y += __shfl_xor_sync(0xffffffffu, y, 2);
        if (k == p) mine = y;
      }
    }
    if (c_ok && r + p < row0 + rows) {
      const float y = fmaf(D, f.x, mine);
      act_st(A.y, static_cast<size_t>(r + p) * A.ld_y + c, F32, y * (f.z / (1.f + expf(-f.z))));
    }
  };
  if constexpr (NS <= 8) {
    Four f0, f1;
    fetch(row0, f0);
    for (int r = row0; r < row0 + rows; r += 8) {
      if (r + 4 < row0 + rows) fetch(r + 4, f1);
      run(r, f0);
      if (r + 4 < row0 + rows) {
        if (r + 8 < row0 + rows) fetch(r + 8, f0);
        run(r + 4, f1);
      }
    }
  } else {
    Four f0;
    for (int r = row0; r < row0 + rows; r += 4) {
      fetch(r, f0);
      run(r, f0);
    }
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

__device__ bool tile_scan(const TileDesc& t, int tid) {
  const ScanArgs* p = reinterpret_cast<const ScanArgs*>(t.a[0]);
  const uint32_t ns = (__ldcg(&p->n) + 3) / 4;
  const bool f32 = __ldcg(&p->f32) != 0;
#define MF_SCAN(N)                       \
  if (ns <= N) {                         \
    if (f32) scan_rows<N, true>(t, tid); \
    else scan_rows<N, false>(t, tid);    \
    return true;                         \
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
