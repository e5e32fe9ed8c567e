// The plain residual of the layer-list decoders, normed before and after each sublayer (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// Kind 66, ResidualArgs: rows [i0, i0 + i1), the four exec warps on one row.

// Sums of two values over the exec threads.  Successive reductions of a row use scratch of their own, so that one barrier
// each is enough.
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

__device__ __forceinline__ float over_rms(float ss, const ResidualArgs& A) { return 1.f / sqrtf(ss / static_cast<float>(A.W) + A.eps); }

// Columns c .. c + V of the next sublayer's input.
template <int V>
__device__ __forceinline__ void put_input(const ResidualArgs& A, uint32_t r, int g, int c, const float (&h)[V]) {
  auto st16 = [&](unsigned long long base, size_t at) {
    __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(base) + at;
    if constexpr (V == 4) {
      const __nv_bfloat162 q[2] = {__floats2bfloat162_rn(h[0], h[1]), __floats2bfloat162_rn(h[2], h[3])};
      *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(q);
    } else {
      o[0] = __float2bfloat16(h[0]);
    }
  };
  if (A.h16) st16(A.h16, static_cast<size_t>(r) * A.ld_h16 + c);
  if (A.h32) st_vec<V>(reinterpret_cast<float*>(A.h32) + static_cast<size_t>(r) * A.ld_h32 + c, h);
  if (g >= 0 && A.out16) st16(A.out16, static_cast<size_t>(g) * A.ld_out + c);
  if (g >= 0 && A.out32) st_vec<V>(reinterpret_cast<float*>(A.out32) + static_cast<size_t>(g) * A.ld_out + c, h);
}

// Any width, and the embedding: a row is read again in each pass, x holding what the pass before has made of it (a thread
// keeps to its own columns).
template <int V>
__device__ __noinline__ void residual_rows(const TileDesc& t, int tid, int* scratch) {
  ResidualArgs A;
  load_block(A, t.a[0]);
  StepArgs St{};
  if (A.step) load_block(St, A.step);
  const int page = St.page_size ? static_cast<int>(St.page_size) : 64;
  const int W = static_cast<int>(A.W);
  const size_t slab = static_cast<size_t>(A.y_rows) * W;
  float* const red = reinterpret_cast<float*>(scratch);   // three reductions of a row, eight floats each
  for (uint32_t r = t.i0; r < t.i0 + t.i1; ++r) {
    float* const xr = reinterpret_cast<float*>(A.x) + static_cast<size_t>(r) * W;
    float* const sum_out = A.sum_out ? reinterpret_cast<float*>(A.sum_out) + static_cast<size_t>(r) * W : nullptr;
    float s0 = 0.f, s1 = 0.f;
    float x[V], y[V], z[V];
    if (A.embed) {
      int token, pos;
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
      const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(A.embed) + static_cast<size_t>(token) * W;
      const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(A.pos) + static_cast<size_t>(pos) * W;
#pragma unroll 4
      for (int c = tid * V; c < W; c += kExecThreads * V) {
#pragma unroll
        for (int j = 0; j < V; ++j) {
          x[j] = __bfloat162float(e[c + j]) * A.embed_scale + (A.pos ? __bfloat162float(p[c + j]) : 0.f);
          s0 = fmaf(x[j], x[j], s0);
        }
        st_vec<V>(xr + c, x);
        if (sum_out) st_vec<V>(sum_out + c, x);
      }
    } else {
      float inv0 = 1.f, inv1 = 1.f;
      auto load_y = [&](int c) {
        slab_sum<V>(A.y0, A.y0_parts, slab, static_cast<size_t>(r) * W + c, y);
        if (A.y1_parts) slab_sum<V>(A.y1, A.y1_parts, slab, static_cast<size_t>(r) * W + c, z);
      };
      auto branches = [&](int c) {   // y = branch_scale (w0 norm(y0) + w1 norm(y1))
        float a[V], b[V];
        ld_vec<V>(f32p(A.w0) + c, a);
        ld_vec<V>(f32p(A.w1) + c, b);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] = A.branch_scale * (y[j] * inv0 * a[j] + z[j] * inv1 * b[j]);
      };
      for (int c = tid * V; c < W; c += kExecThreads * V) {
        load_y(c);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          s0 = fmaf(y[j], y[j], s0);
          if (A.y1_parts) s1 = fmaf(z[j], z[j], s1);
        }
      }
      block_sum2(s0, s1, red, tid);
      if (A.y1_parts) {
        inv0 = over_rms(s0, A);
        inv1 = over_rms(s1, A);
        s0 = s1 = 0.f;
        for (int c = tid * V; c < W; c += kExecThreads * V) {
          load_y(c);
          branches(c);
#pragma unroll
          for (int j = 0; j < V; ++j) s0 = fmaf(y[j], y[j], s0);
        }
        block_sum2(s0, s1, red + 8, tid);
      }
      const float inv = over_rms(s0, A);
      s0 = s1 = 0.f;
      for (int c = tid * V; c < W; c += kExecThreads * V) {
        float w[V];
        ld_vec<V>(xr + c, x);
        load_y(c);
        if (A.y1_parts) branches(c);
        ld_vec<V>(f32p(A.post_w) + c, w);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          x[j] += y[j] * inv * w[j];
          s0 = fmaf(x[j], x[j], s0);
        }
        st_vec<V>(xr + c, x);
        if (sum_out) st_vec<V>(sum_out + c, x);
      }
    }
    block_sum2(s0, s1, red + 16, tid);
    const float inv = over_rms(s0, A);
    const int g = A.gather ? reinterpret_cast<const int*>(A.gather)[r] : -1;
#pragma unroll 4
    for (int c = tid * V; c < W; c += kExecThreads * V) {
      float h[V];
      ld_vec<V>(xr + c, x);
      ld_vec<V>(f32p(A.w) + c, h);
#pragma unroll
      for (int j = 0; j < V; ++j) h[j] = x[j] * inv * h[j];
      put_input<V>(A, r, g, c, h);
    }
  }
}

// Rows of at most 512 NU columns, kept in registers; the next row's loads are issued before this one's arithmetic.
template <int NU, bool kTwo>
__device__ __noinline__ void residual_rows_ahead(const TileDesc& t, int tid, int* scratch) {
  ResidualArgs A;
  load_block(A, t.a[0]);
  const int W = static_cast<int>(A.W);
  const size_t slab = static_cast<size_t>(A.y_rows) * W;
  float* const red = reinterpret_cast<float*>(scratch);
  float x[NU][4], y[NU][4], z[kTwo ? NU : 1][4];           // this row
  float nx[NU][4], ny[NU][4], nz[kTwo ? NU : 1][4];        // the next
  int g = -1;
  auto each = [&](auto&& f) {   // f(register piece, first column)
#pragma unroll
    for (int i = 0; i < NU; ++i)
      if ((tid + i * kExecThreads) * 4 < W) f(i, (tid + i * kExecThreads) * 4);
  };
  auto load = [&](uint32_t r) {
    each([&](int i, int c) {
      const size_t at = static_cast<size_t>(r) * W + c;
      ld_vec<4>(f32p(A.x) + at, nx[i]);
      slab_sum<4>(A.y0, A.y0_parts, slab, at, ny[i]);
      if constexpr (kTwo) slab_sum<4>(A.y1, A.y1_parts, slab, at, nz[i]);
    });
  };
  load(t.i0);
  for (uint32_t r = t.i0; r < t.i0 + t.i1; ++r) {
#pragma unroll
    for (int i = 0; i < NU; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        x[i][j] = nx[i][j];
        y[i][j] = ny[i][j];
        if constexpr (kTwo) z[i][j] = nz[i][j];
      }
    if (A.gather) g = reinterpret_cast<const int*>(A.gather)[r];
    float s0 = 0.f, s1 = 0.f;
    each([&](int i, int) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s0 = fmaf(y[i][j], y[i][j], s0);
        if constexpr (kTwo) s1 = fmaf(z[i][j], z[i][j], s1);
      }
    });
    if (r + 1 < t.i0 + t.i1) load(r + 1);
    block_sum2(s0, s1, red, tid);
    if constexpr (kTwo) {
      const float inv0 = over_rms(s0, A), inv1 = over_rms(s1, A);
      s0 = s1 = 0.f;
      each([&](int i, int c) {
        float a[4], b[4];
        ld_vec<4>(f32p(A.w0) + c, a);
        ld_vec<4>(f32p(A.w1) + c, b);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          y[i][j] = A.branch_scale * (y[i][j] * inv0 * a[j] + z[i][j] * inv1 * b[j]);
          s0 = fmaf(y[i][j], y[i][j], s0);
        }
      });
      block_sum2(s0, s1, red + 8, tid);
    }
    const float inv = over_rms(s0, A);
    s0 = s1 = 0.f;
    each([&](int i, int c) {
      float w[4];
      ld_vec<4>(f32p(A.post_w) + c, w);
      const size_t at = static_cast<size_t>(r) * W + c;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        x[i][j] += y[i][j] * inv * w[j];
        s0 = fmaf(x[i][j], x[i][j], s0);
      }
      st_vec<4>(reinterpret_cast<float*>(A.x) + at, x[i]);
      if (A.sum_out) st_vec<4>(reinterpret_cast<float*>(A.sum_out) + at, x[i]);
    });
    block_sum2(s0, s1, red + 16, tid);
    const float inv_x = over_rms(s0, A);
    each([&](int i, int c) {
      float h[4];
      ld_vec<4>(f32p(A.w) + c, h);
#pragma unroll
      for (int j = 0; j < 4; ++j) h[j] = x[i][j] * inv_x * h[j];
      put_input<4>(A, r, g, c, h);
    });
  }
}

__device__ void tile_residual(const TileDesc& t, int tid, int* scratch) {
  const ResidualArgs* p = reinterpret_cast<const ResidualArgs*>(t.a[0]);
  const uint32_t W = __ldcg(&p->W);
  const bool two = __ldcg(&p->y1_parts) != 0;
  if (__ldcg(&p->embed) == 0 && (W & 3) == 0 && W <= 2048) {
    if (two) residual_rows_ahead<4, true>(t, tid, scratch);
    else residual_rows_ahead<4, false>(t, tid, scratch);
  } else if (__ldcg(&p->embed) == 0 && (W & 3) == 0 && W <= 4096) {
    if (two) residual_rows_ahead<8, true>(t, tid, scratch);
    else residual_rows_ahead<8, false>(t, tid, scratch);
  } else if ((W & 3) == 0) {
    residual_rows<4>(t, tid, scratch);
  } else {
    residual_rows<1>(t, tid, scratch);
  }
}

}  // namespace fab
}  // namespace mf
