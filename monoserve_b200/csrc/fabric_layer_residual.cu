// The plain residual of the layer-list decoders, normed before and after each sublayer (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// Kind 66, ResidualArgs: rows [i0, i0 + i1), the four exec warps on one row.  Up to 8 V 128 columns stay in registers
// (kReg); wider rows are read again in each pass, x holding what the pass before has made of them.
constexpr int kResidualPieces = 8;

// Sums of two values over the exec threads; `slot` alternates, so that one barrier is enough.
__device__ __forceinline__ void block_sum2(float& a, float& b, float* red, int tid) {
  a = warp_sum(a);
  b = warp_sum(b);
  if ((tid & 31) == 0) {
    red[tid >> 5] = a;
    red[4 + (tid >> 5)] = b;
  }
  exec_sync();
  a = red[0] + red[1] + red[2] + red[3];
  b = red[4] + red[5] + red[6] + red[7];
}

// Column piece c of a sublayer's output: its K-range slabs added in order.
template <int V>
__device__ __forceinline__ void slab_sum(unsigned long long base, uint32_t parts, size_t slab, size_t at, float (&y)[V]) {
  const float* p = f32p(base) + at;
  ld_vec<V>(p, y);
  for (uint32_t q0 = 1; q0 < parts; q0 += 4) {   // four slabs' loads are issued before the first is used
    float b[4][V];
#pragma unroll
    for (uint32_t i = 0; i < 4; ++i) ld_vec<V>(p + min(q0 + i, parts - 1) * slab, b[i]);
#pragma unroll
    for (uint32_t i = 0; i < 4; ++i)
      if (q0 + i < parts)
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] += b[i][j];
  }
}

template <int V, bool kReg>
__device__ __noinline__ void residual_rows(const TileDesc& t, int tid, int* scratch) {
  constexpr int NU = kReg ? kResidualPieces : 1;
  ResidualArgs A;
  load_block(A, t.a[0]);
  StepArgs St{};
  if (A.step) load_block(St, A.step);
  const int page = St.page_size ? static_cast<int>(St.page_size) : 64;
  const int W = static_cast<int>(A.W), n = W / V;
  const size_t slab = static_cast<size_t>(A.y_rows) * W;
  float* const red = reinterpret_cast<float*>(scratch);   // three reductions of a row, eight floats each
  for (uint32_t r = t.i0; r < t.i0 + t.i1; ++r) {
    float* const xr = reinterpret_cast<float*>(A.x) + static_cast<size_t>(r) * W;
    float* const sum_out = A.sum_out ? reinterpret_cast<float*>(A.sum_out) + static_cast<size_t>(r) * W : nullptr;
    int token = 0, pos = 0;
    if (A.embed) {
      if (A.step) {
        const int slot = reinterpret_cast<const int*>(St.row_req)[r];
        pos = min(reinterpret_cast<const int*>(St.seq_len)[slot], static_cast<int>(St.bt_stride) * page - 1);
        token = reinterpret_cast<const int*>(St.last_token)[slot];
        exec_sync();   // every thread has the position: the row's bookkeeping may advance it
        if (tid == 0) step_row(St, page, static_cast<int>(r), 0);
      } else {
        pos = reinterpret_cast<const int*>(A.tok_pos)[r];
        token = reinterpret_cast<const int*>(A.tokens)[r];
      }
      pos = min(pos, static_cast<int>(A.max_pos) - 1);
    }
    float x[NU][V], y[NU][V], z[NU][V];
    float s0 = 0.f, s1 = 0.f;
    auto each = [&](auto&& f) {   // f(register piece, column piece)
      if constexpr (kReg) {
#pragma unroll
        for (int i = 0; i < NU; ++i)
          if (tid + i * kExecThreads < n) f(i, tid + i * kExecThreads);
      } else {
        for (int c = tid; c < n; c += kExecThreads) f(0, c);
      }
    };
    auto load_y = [&](int i, int c) {
      if (A.y0_parts) slab_sum<V>(A.y0, A.y0_parts, slab, static_cast<size_t>(r) * W + c * V, y[i]);
      if (A.y1_parts) slab_sum<V>(A.y1, A.y1_parts, slab, static_cast<size_t>(r) * W + c * V, z[i]);
    };
    float inv0 = 1.f, inv1 = 1.f;
    auto branches = [&](int i, int c) {   // y = branch_scale (w0 norm(y0) + w1 norm(y1))
      float a[V], b[V];
      ld_vec<V>(f32p(A.w0) + c * V, a);
      ld_vec<V>(f32p(A.w1) + c * V, b);
#pragma unroll
      for (int j = 0; j < V; ++j) y[i][j] = A.branch_scale * (y[i][j] * inv0 * a[j] + z[i][j] * inv1 * b[j]);
    };
    auto rms = [&](float ss) { return 1.f / sqrtf(ss / static_cast<float>(W) + A.eps); };
    if (A.embed) {
      each([&](int i, int c) {
        const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(A.embed) + static_cast<size_t>(token) * W + c * V;
        const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(A.pos) + static_cast<size_t>(pos) * W + c * V;
#pragma unroll
        for (int j = 0; j < V; ++j)
          x[i][j] = __bfloat162float(e[j]) * A.embed_scale + (A.pos ? __bfloat162float(p[j]) : 0.f);
        st_vec<V>(xr + c * V, x[i]);
        if (sum_out) st_vec<V>(sum_out + c * V, x[i]);
#pragma unroll
        for (int j = 0; j < V; ++j) s0 = fmaf(x[i][j], x[i][j], s0);
      });
    } else {
      each([&](int i, int c) {
        if constexpr (kReg) ld_vec<V>(xr + c * V, x[i]);
        load_y(i, c);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          s0 = fmaf(y[i][j], y[i][j], s0);
          if (A.y1_parts) s1 = fmaf(z[i][j], z[i][j], s1);
        }
      });
      block_sum2(s0, s1, red, tid);
      if (A.y1_parts) {
        inv0 = rms(s0);
        inv1 = rms(s1);
        s0 = s1 = 0.f;
        each([&](int i, int c) {
          if constexpr (!kReg) load_y(i, c);
          branches(i, c);
#pragma unroll
          for (int j = 0; j < V; ++j) s0 = fmaf(y[i][j], y[i][j], s0);
        });
        block_sum2(s0, s1, red + 8, tid);
      }
      const float inv = rms(s0);
      s0 = s1 = 0.f;
      each([&](int i, int c) {
        if constexpr (!kReg) {
          ld_vec<V>(xr + c * V, x[i]);
          load_y(i, c);
          if (A.y1_parts) branches(i, c);
        }
        float w[V];
        ld_vec<V>(f32p(A.post_w) + c * V, w);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          x[i][j] += y[i][j] * inv * w[j];
          s0 = fmaf(x[i][j], x[i][j], s0);
        }
        st_vec<V>(xr + c * V, x[i]);
        if (sum_out) st_vec<V>(sum_out + c * V, x[i]);
      });
    }
    block_sum2(s0, s1, red + 16, tid);
    const float inv = rms(s0);
    const int g = A.gather ? reinterpret_cast<const int*>(A.gather)[r] : -1;
    each([&](int i, int c) {
      if constexpr (!kReg) ld_vec<V>(xr + c * V, x[i]);   // this thread's own columns
      float h[V];
      ld_vec<V>(f32p(A.w) + c * V, h);
#pragma unroll
      for (int j = 0; j < V; ++j) h[j] = x[i][j] * inv * h[j];
      auto st16 = [&](unsigned long long base, size_t at) {
        __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(base) + at;
        if constexpr (V == 4) {
          const __nv_bfloat162 q[2] = {__floats2bfloat162_rn(h[0], h[1]), __floats2bfloat162_rn(h[2], h[3])};
          *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(q);
        } else {
          o[0] = __float2bfloat16(h[0]);
        }
      };
      if (A.h32) st_vec<V>(reinterpret_cast<float*>(A.h32) + static_cast<size_t>(r) * A.ld_h32 + c * V, h);
      if (A.h16) st16(A.h16, static_cast<size_t>(r) * A.ld_h16 + c * V);
      if (g >= 0 && A.out32) st_vec<V>(reinterpret_cast<float*>(A.out32) + static_cast<size_t>(g) * A.ld_out + c * V, h);
      if (g >= 0 && A.out16) st16(A.out16, static_cast<size_t>(g) * A.ld_out + c * V);
    });
  }
}

__device__ void tile_residual(const TileDesc& t, int tid, int* scratch) {
  const uint32_t W = __ldcg(&reinterpret_cast<const ResidualArgs*>(t.a[0])->W);
  if ((W & 3) == 0 && W <= kResidualPieces * 4 * kExecThreads) residual_rows<4, true>(t, tid, scratch);
  else if ((W & 3) == 0) residual_rows<4, false>(t, tid, scratch);
  else residual_rows<1, false>(t, tid, scratch);
}

}  // namespace fab
}  // namespace mf
