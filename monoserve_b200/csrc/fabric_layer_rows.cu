// Row-wise tiles of the layer-list decoders and their 32-bit products (fabric_layer_tiles.cuh).
#include "fabric_layer_tiles.cuh"

namespace mf {
namespace fab {

// ------------------------------------------------------------------ 32-bit product
// Kind 51, ProductArgs: rows [i0, i0 + i1) x columns [i2, i2 + i3), at most 32 x 32; a[1], a[2], a[3]: byte offsets
// of this tile's x, w and out (a product per head).  Two rows and four columns per thread.
__device__ void tile_product32(const TileDesc& t, int tid, int* scratch) {
  constexpr int KC = 16, LD = KC + 1;
  float* const sx = reinterpret_cast<float*>(scratch);   // [32][LD]
  float* const sw = sx + 32 * LD;                               // [32][LD]
  static_assert(2 * 32 * LD <= kLayerScratchInts, "product scratch");
  ProductArgs A;
  load_block(A, t.a[0]);
  const unsigned long long x = A.x + t.a[1], w = A.w + t.a[2];
  float* out = reinterpret_cast<float*>(A.out + t.a[3]);
  const int rows = static_cast<int>(t.i1), cols = static_cast<int>(t.i3), K = static_cast<int>(A.K);
  const int lr = tid >> 2, lk = (tid & 3) * 4;   // the loader's row and first column
  const int r = (tid >> 3) * 2, c = (tid & 7) * 4;
  float acc[2][4] = {};
  for (int k0 = 0; k0 < K; k0 += KC) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      sx[lr * LD + lk + i] = (lr < rows && k < K) ? act_ld(x, static_cast<size_t>(t.i0 + lr) * A.ld_x + k, A.f32) : 0.f;
      sw[lr * LD + lk + i] = (lr < cols && k < K) ? act_ld(w, static_cast<size_t>(t.i2 + lr) * A.ld_w + k, false) : 0.f;
    }
    exec_sync();
    float part[2][4] = {};   // sums of KC products are added up, not single products: the rounding of a long sum stays small
#pragma unroll
    for (int k = 0; k < KC; ++k) {
      const float x0 = sx[r * LD + k], x1 = sx[(r + 1) * LD + k];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float wv = sw[(c + j) * LD + k];
        part[0][j] = fmaf(x0, wv, part[0][j]);
        part[1][j] = fmaf(x1, wv, part[1][j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      acc[0][j] += part[0][j];
      acc[1][j] += part[1][j];
    }
    exec_sync();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (r + i < rows && c + j < cols) out[static_cast<size_t>(t.i0 + r + i) * A.ld_out + t.i2 + c + j] = acc[i][j];
}

// Kind 52, GatedArgs: rows [i0, i0 + i1) of fp32 [gate | up] -> gelu_tanh(gate) * up or silu(gate) * up, fp32.
__device__ void tile_gated_act(const TileDesc& t, int tid) {
  GatedArgs A;
  load_block(A, t.a[0]);
  for (uint32_t r = t.i0; r < t.i0 + t.i1; ++r) {
    const float* in = f32p(A.in) + static_cast<size_t>(r) * A.ld_in;
    float* out = reinterpret_cast<float*>(A.out) + static_cast<size_t>(r) * A.ld_out;
    for (uint32_t f = tid; f < A.ff; f += kExecThreads) {
      const float g = in[f];
      const float a = A.silu ? g * sigmoid32(g) : 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
      out[f] = a * in[A.ff + f];
    }
  }
}

// Kind 62, SumArgs: rows [i0, i0 + i1), V columns at a time.
template <int V>
__device__ __noinline__ void sum_rows(const TileDesc& t, int tid) {
  SumArgs A;
  load_block(A, t.a[0]);
  const size_t slab = static_cast<size_t>(A.part_rows) * A.ld_in;
  const uint32_t per = A.cols / V, n = t.i1 * per;
  for (uint32_t i = tid; i < n; i += kExecThreads) {
    const uint32_t r = t.i0 + i / per, c = (i % per) * V;
    const float* in = f32p(A.in) + static_cast<size_t>(r) * A.ld_in + c;
    float v[V];
    ld_vec<V>(in, v);
    for (uint32_t q0 = 1; q0 < A.parts; q0 += 4) {
      float b[4][V];
#pragma unroll
      for (uint32_t q = 0; q < 4; ++q) ld_vec<V>(in + min(q0 + q, A.parts - 1) * slab, b[q]);
#pragma unroll
      for (uint32_t q = 0; q < 4; ++q)
        if (q0 + q < A.parts)
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] += b[q][j];
    }
    if (A.out32) st_vec<V>(reinterpret_cast<float*>(A.out32) + static_cast<size_t>(r) * A.ld_32 + c, v);
    __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(A.out16) + static_cast<size_t>(r) * A.ld_16 + c;
#pragma unroll
    for (int j = 0; j < V; ++j)
      if (c + j < A.c16) o[j] = __float2bfloat16(v[j]);
  }
}

__device__ void tile_sum_slabs(const TileDesc& t, int tid) {
  const SumArgs* p = reinterpret_cast<const SumArgs*>(t.a[0]);
  if (((__ldcg(&p->cols) | __ldcg(&p->ld_in)) & 3) == 0) sum_rows<4>(t, tid);
  else sum_rows<1>(t, tid);
}

// ------------------------------------------------------------------ residual streams
// S is the largest number of streams an instance takes; the loops are guarded by the row's own number.
// One row of the streams by `width` threads of which this is thread `l`: update (or start) the streams, form the next
// sublayer's input u, and its norm.  kReg: u stays in registers (W <= 8 V width), else it is formed again from the
// stored streams.
template <int V, int S, bool kReg>
__device__ __forceinline__ void streams_row(const StreamArgs& A, uint32_t r, int token, int l, int width, bool block, int* scratch,
                                            const float (&w_in)[S], const float (&w_out)[S], const float (&mix)[S * S]) {
  constexpr int NU = 8;
  const int W = static_cast<int>(A.W), n = W / V, ns = static_cast<int>(A.streams);
  float* const xs = reinterpret_cast<float*>(A.xs) + static_cast<size_t>(r) * ns * W;
  float* const sum_out = A.sum_out ? reinterpret_cast<float*>(A.sum_out) + static_cast<size_t>(r) * W : nullptr;
  const int parts = static_cast<int>(A.y_parts);
  const size_t slab = static_cast<size_t>(A.y_rows) * W;
  float u_reg[kReg ? NU : 1][V];
  float ss = 0.f;
  auto column = [&](int c, float (&u)[V]) {
    float x[S][V];
    if (A.embed) {
      const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(A.embed) + static_cast<size_t>(token) * W + c * V;
#pragma unroll
      for (int j = 0; j < V; ++j) x[0][j] = __bfloat162float(e[j]);
#pragma unroll
      for (int s = 1; s < S; ++s)
#pragma unroll
        for (int j = 0; j < V; ++j) x[s][j] = x[0][j];
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (s < ns) ld_vec<V>(xs + s * W + c * V, x[s]);
        else
#pragma unroll
          for (int j = 0; j < V; ++j) x[s][j] = 0.f;
      }
    }
    float nx[S][V];
    if (parts > 0) {
      float y[V];
      const float* yp = f32p(A.y) + static_cast<size_t>(r) * W + c * V;
      ld_vec<V>(yp, y);
      for (int q0 = 1; q0 < parts; q0 += 4) {   // four slabs' loads are issued before the first is used
        float b[4][V];
#pragma unroll
        for (int i = 0; i < 4; ++i) ld_vec<V>(yp + min(q0 + i, parts - 1) * slab, b[i]);
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (q0 + i < parts)
#pragma unroll
            for (int j = 0; j < V; ++j) y[j] += b[i][j];
      }
#pragma unroll
      for (int to = 0; to < S; ++to)
#pragma unroll
        for (int j = 0; j < V; ++j) {
          float v = w_out[to] * y[j];
#pragma unroll
          for (int s = 0; s < S; ++s) v = fmaf(mix[s * S + to], x[s][j], v);
          nx[to][j] = v;
        }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int j = 0; j < V; ++j) nx[s][j] = x[s][j];
    }
    if (parts > 0 || A.embed)
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < ns) st_vec<V>(xs + s * W + c * V, nx[s]);
    float sum[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      u[j] = 0.f;
      sum[j] = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) {
        u[j] = fmaf(w_in[s], nx[s][j], u[j]);
        if (s < ns) sum[j] += nx[s][j];
      }
      ss = fmaf(u[j], u[j], ss);
    }
    if (sum_out) st_vec<V>(sum_out + c * V, sum);
  };
  if constexpr (kReg) {
#pragma unroll
    for (int i = 0; i < NU; ++i)
      if (l + i * width < n) column(l + i * width, u_reg[i]);
  } else {
    for (int c = l; c < n; c += width) column(c, u_reg[0]);
  }
  ss = warp_sum(ss);
  if (block) {
    float* const s_red = reinterpret_cast<float*>(scratch);
    if ((l & 31) == 0) s_red[l >> 5] = ss;
    exec_sync();
    ss = s_red[0] + s_red[1] + s_red[2] + s_red[3];
    exec_sync();
  }
  const float inv = 1.f / sqrtf(ss / static_cast<float>(W) + A.eps);
  const int g = A.gather ? reinterpret_cast<const int*>(A.gather)[r] : -1;
  auto finish = [&](int c, const float (&u)[V]) {
    float h[V];
    ld_vec<V>(f32p(A.w) + c * V, h);
#pragma unroll
    for (int j = 0; j < V; ++j) h[j] = u[j] * inv * h[j];
    if (A.h32) st_vec<V>(reinterpret_cast<float*>(A.h32) + static_cast<size_t>(r) * A.ld_h32 + c * V, h);
    if (g >= 0 && A.out32) st_vec<V>(reinterpret_cast<float*>(A.out32) + static_cast<size_t>(g) * A.ld_out + c * V, h);
    auto st16 = [&](unsigned long long base, size_t at) {
      __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(base) + at;
      if constexpr (V == 4) {
        const __nv_bfloat162 q[2] = {__floats2bfloat162_rn(h[0], h[1]), __floats2bfloat162_rn(h[2], h[3])};
        *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(q);
      } else {
        o[0] = __float2bfloat16(h[0]);
      }
    };
    if (g >= 0 && A.out16) st16(A.out16, static_cast<size_t>(g) * A.ld_out + c * V);
    if (A.h16) {
      const size_t at = static_cast<size_t>(r) * A.ld_h16 + c * V;
      st16(A.h16, at);
      for (uint32_t part = 1; part <= 2 && A.split; ++part) {   // what rounding has left, rounded again
#pragma unroll
        for (int j = 0; j < V; ++j) h[j] -= __bfloat162float(__float2bfloat16(h[j]));
        st16(A.h16, at + part * A.split);
      }
    }
  };
  if constexpr (kReg) {
#pragma unroll
    for (int i = 0; i < NU; ++i)
      if (l + i * width < n) finish(l + i * width, u_reg[i]);
  } else {
    for (int c = l; c < n; c += width) {
      float u[V];
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (s >= ns) break;
        float x[V];
        ld_vec<V>(xs + s * W + c * V, x);
#pragma unroll
        for (int j = 0; j < V; ++j) u[j] = fmaf(w_in[s], x[j], u[j]);
      }
      finish(c, u);
    }
  }
}

template <int V, int S>
__device__ __noinline__ void streams_rows(const TileDesc& t, int tid, int* scratch) {
  StreamArgs A;
  load_block(A, t.a[0]);
  float w_in[S], w_out[S], mix[S * S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    const int ns = static_cast<int>(A.streams);
    w_in[s] = s < ns ? f32p(A.hc_in)[s] : 0.f;
    w_out[s] = (A.y_parts && s < ns) ? f32p(A.hc_out)[s] : 0.f;
#pragma unroll
    for (int to = 0; to < S; ++to) mix[s * S + to] = (A.y_parts && s < ns && to < ns) ? f32p(A.hc_mix)[s * ns + to] : 0.f;
  }
  StepArgs St{};
  if (A.step) load_block(St, A.step);
  const int page = St.page_size ? static_cast<int>(St.page_size) : 64;
  const int warp = tid >> 5, lane = tid & 31;
  const bool block = t.i1 == 1;   // one row in the tile: the four warps share it
  const int width = block ? kExecThreads : 32, l = block ? tid : lane;
  const bool in_regs = static_cast<int>(A.W) <= 8 * V * width;
  for (uint32_t r = t.i0 + (block ? 0 : warp); r < t.i0 + t.i1; r += block ? 1 : kExecThreads / 32) {
    int token = 0;
    if (A.embed) token = A.step ? step_row(St, page, static_cast<int>(r), l) : reinterpret_cast<const int*>(A.tokens)[r];
    if (in_regs) streams_row<V, S, true>(A, r, token, l, width, block, scratch, w_in, w_out, mix);
    else streams_row<V, S, false>(A, r, token, l, width, block, scratch, w_in, w_out, mix);
  }
}

// Kind 53, StreamArgs: rows [i0, i0 + i1).
__device__ void tile_streams(const TileDesc& t, int tid, int* scratch) {
  const StreamArgs* p = reinterpret_cast<const StreamArgs*>(t.a[0]);
  if ((__ldcg(&p->W) & 3) == 0 && __ldcg(&p->streams) <= 4) streams_rows<4, 4>(t, tid, scratch);
  else streams_rows<1, kMaxStreams>(t, tid, scratch);
}

__device__ bool run_layer_tile(const TileDesc& t, int tid, const LayerCtx& ctx) {
  int* const scratch = ctx.scratch;
  switch (t.kind) {
    case kTileProduct32: tile_product32(t, tid, scratch); return true;
    case kTileGatedAct: tile_gated_act(t, tid); return true;
    case kTileStreams: tile_streams(t, tid, scratch); return true;
    case kTileConv: tile_conv(t, tid); return true;
    case kTileScan: return tile_scan(t, tid, ctx.ring);
    case kTileMemoryStep: return tile_memory_step(t, tid);
    case kTileScanStep: tile_scan_step(t, tid); return true;
    case kTileMemory: return tile_memory(t, tid, ctx.ring);
    case kTileHeadNorm: tile_head_norm(t, tid); return true;
    case kTileLatentKv: tile_latent_kv(t, tid); return true;
    case kTileLatentAttn: return tile_latent_attn(t, tid);
    case kTileLatentMma: return tile_latent_mma(t, tid, ctx);
    case kTileLatentDirect: return tile_latent_direct(t, tid, ctx);
    case kTileLatentMerge: tile_latent_merge(t, tid); return true;
    case kTileSumSlabs: tile_sum_slabs(t, tid); return true;
    case kTileResidual: tile_residual(t, tid, scratch); return true;
    case kTileDecay: tile_decay(t, tid); return true;
    case kTileGatedMemory: return tile_gated_memory(t, tid, ctx.ring);
    case kTileGatedStep: return tile_gated_step(t, tid, ctx);
    case kTileQkv: tile_qkv(t, tid); return true;
    case kTileGroupedAttn: return tile_grouped_attn(t, tid);
    case kTileHeadGate: tile_head_gate(t, tid); return true;
    default: return false;
  }
}

}  // namespace fab
}  // namespace mf
