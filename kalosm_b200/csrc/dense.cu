// Products with weights kept in raw row-major form (F32, F16, BF16, Q5_0, Q5_K).
//
// F16 / Q5_0: the reference's Tensor::q_mat_mul dequantises such a matrix and runs a dense matmul
// (fusor-ml/fusor/src/lib.rs:1184-1215); one warp forms one output with element-wise dequantisation and a
// fixed-order shuffle reduction. BF16 and F32 are the weight types of the hybrid decoders and have kernels of
// their own:
//  * dense_gemv_kernel (one activation row; HBM-bound: the matrix is streamed once): the row sits in shared
//    memory as f32 (RMSNorm runs in the prologue), a warp forms two output rows at a time -- or the gate row and
//    the up row of one SwiGLU output -- with 16-byte loads, KS warps of a CTA sharing a pair along K when
//    few rows are left. f32 activations, f32 accumulation, sums in a fixed order.
//  * dense_gemm_f32_kernel (F32 weights, any number of rows): a 64 x 64 register-blocked product in true f32.
//  * BF16 weights with more rows: dense_tc.cu.
#include <algorithm>

#include "dense.cuh"
#include "formats.cuh"
#include "qgemv_common.cuh"

namespace {

__global__ void dense_matmul_kernel(uint32_t type, const uint8_t* __restrict__ w,
                                    const float* __restrict__ x, uint64_t m, uint64_t n, uint64_t k,
                                    float* __restrict__ y) {
  const uint64_t warp = ((uint64_t)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (warp >= m * n) return;
  const uint64_t mi = warp / n, ni = warp % n;
  float acc = 0.f;
  for (uint64_t c = lane; c < k; c += 32)
    acc = fmaf(x[mi * k + c], fb::raw_elem(type, w, ni * k + c), acc);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xFFFFFFFFu, acc, o);
  if (lane == 0) y[mi * n + ni] = acc;
}

constexpr int GV_THREADS = 512, GV_WARPS = GV_THREADS / 32;

struct GemvArgs {
  const void* w;
  const float* x;
  const float* norm_w;
  const float* ff_norm_w;
  const float* add;
  const float* bias;
  float* y;
  float* z;
  int k, kx, row0, n_plain, gate0, up0, ff, act, ks, whole, units;
  float eps, alpha, softcap;
};

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// dot product pieces of one 16-byte piece of two weight rows
__device__ __forceinline__ void gv_fma(const uint4& u, const float4& x0, const float4& x1, float& acc, __nv_bfloat16) {
  acc = fmaf(__uint_as_float(u.x << 16), x0.x, acc);
  acc = fmaf(__uint_as_float(u.x & 0xFFFF0000u), x0.y, acc);
  acc = fmaf(__uint_as_float(u.y << 16), x0.z, acc);
  acc = fmaf(__uint_as_float(u.y & 0xFFFF0000u), x0.w, acc);
  acc = fmaf(__uint_as_float(u.z << 16), x1.x, acc);
  acc = fmaf(__uint_as_float(u.z & 0xFFFF0000u), x1.y, acc);
  acc = fmaf(__uint_as_float(u.w << 16), x1.z, acc);
  acc = fmaf(__uint_as_float(u.w & 0xFFFF0000u), x1.w, acc);
}
__device__ __forceinline__ void gv_fma(const uint4& u, const float4& x0, const float4&, float& acc, float) {
  acc = fmaf(__uint_as_float(u.x), x0.x, acc);
  acc = fmaf(__uint_as_float(u.y), x0.y, acc);
  acc = fmaf(__uint_as_float(u.z), x0.z, acc);
  acc = fmaf(__uint_as_float(u.w), x0.w, acc);
}

// value of a plain output row
__device__ __forceinline__ float plain_value(float acc, float alpha, const float* bias, const float* add, float softcap, int n) {
  float v = alpha * acc;
  if (bias) v += bias[n];
  if (add) v += add[n];
  return softcap > 0.f ? softcap * tanhf(v / softcap) : v;
}

// The activation row is kept as float4 planes: plane p holds elements 4 p .. 4 p + 3 of every 16-byte piece of a
// weight row (two planes for bf16 weights, one for f32), so that consecutive lanes read consecutive float4.
template <typename WT>
__global__ void __launch_bounds__(GV_THREADS, 2) dense_gemv_kernel(const GemvArgs a) {
  constexpr int E = 16 / (int)sizeof(WT), P = E / 4;  // elements and float4 planes per piece
  extern __shared__ __align__(16) float4 xs[];        // [P][k / E], twice where the feed-forward rows have their own norm
  __shared__ float red[2 * GV_WARPS];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pieces = a.k / E, plain_units = (a.n_plain + 1) >> 1;
  auto rows_of = [&](int u, int& r0, int& r1) {
    if (u < plain_units) {
      r0 = a.row0 + 2 * u;
      r1 = 2 * u + 1 < a.n_plain ? r0 + 1 : r0;
    } else if (a.act == FB200_FFN_GELU) {
      r0 = a.up0 + 2 * (u - plain_units);
      r1 = 2 * (u - plain_units) + 1 < a.ff ? r0 + 1 : r0;
    } else {
      r0 = a.gate0 + u - plain_units;
      r1 = a.up0 + u - plain_units;
    }
  };
  const uint4* w = reinterpret_cast<const uint4*>(a.w);
  // `whole` rounds in which every warp has a unit of its own, then one round of the rest, `ks` warps to a unit
  const int gw = (int)blockIdx.x * GV_WARPS + warp, warps = (int)gridDim.x * GV_WARPS;
  const int team = gw / a.ks, part = gw % a.ks, per = (pieces + a.ks - 1) / a.ks, rest = a.whole * warps + team;
  // weights do not depend on the kernel before this one: request the first pieces while it drains
  {
    const int u = a.whole ? gw : rest, p0 = a.whole ? 0 : part * per, p1 = min(pieces, a.whole ? 128 : p0 + min(per, 128));
    if (u < a.units) {
      int r0, r1;
      rows_of(u, r0, r1);
      for (int p = p0 + lane * 8; p < p1; p += 256) {
        asm volatile("prefetch.global.L2 [%0];" ::"l"(w + (size_t)r0 * pieces + p));
        asm volatile("prefetch.global.L2 [%0];" ::"l"(w + (size_t)r1 * pieces + p));
      }
    }
  }
  pdl_wait();
  // ---- the activation row: (RMS-normalised) f32, zero padding beyond kx
  auto root = [&](float ss) {  // of the mean square, over the CTA
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < GV_WARPS; ++i) ss += red[i];
    return sqrtf(ss / (float)a.kx + a.eps);
  };
  // four elements 4 i .. of the row into their plane
  auto put = [&](float4* to, int i, const float4& v) { to[((4 * i % E) >> 2) * pieces + 4 * i / E] = v; };
  auto times = [](const float4& v, float scale, const float4& n) {
    return make_float4((v.x / scale) * n.x, (v.y / scale) * n.y, (v.z / scale) * n.z, (v.w / scale) * n.w);
  };
  const bool vec = (a.kx & 3) == 0 && (reinterpret_cast<uintptr_t>(a.x) & 15u) == 0;
  const float4* x4 = reinterpret_cast<const float4*>(a.x);
  const int n4 = a.k >> 2, nx4 = a.kx >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  if (vec && a.norm_w && n4 <= 2 * GV_THREADS) {  // the row stays in registers between the sum of squares and the norm
    const float4 *n1 = reinterpret_cast<const float4*>(a.norm_w), *n2 = reinterpret_cast<const float4*>(a.ff_norm_w);
    float4 v[2], m1[2], m2[2];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = tid + j * GV_THREADS;
      v[j] = i < nx4 ? __ldcg(x4 + i) : zero;
      m1[j] = i < nx4 ? n1[i] : zero;
      m2[j] = n2 && i < nx4 ? n2[i] : zero;
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) ss = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, ss))));
    const float scale = root(ss);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = tid + j * GV_THREADS;
      if (i >= n4) continue;
      put(xs, i, times(v[j], scale, m1[j]));
      if (n2) put(xs + P * pieces, i, times(v[j], scale, m2[j]));
    }
  } else if (vec && !a.norm_w) {
#pragma unroll 4
    for (int i = tid; i < n4; i += GV_THREADS) put(xs, i, i < nx4 ? __ldcg(x4 + i) : zero);
  } else {
    float scale = 1.f;
    if (a.norm_w) {
      float ss = 0.f;
      for (int i = tid; i < a.kx; i += GV_THREADS) {
        const float v = __ldcg(a.x + i);
        ss = fmaf(v, v, ss);
      }
      scale = root(ss);
    }
    for (int i = tid; i < a.k; i += GV_THREADS) {
      float v = 0.f, v2 = 0.f;
      if (i < a.kx) {
        v = __ldcg(a.x + i);
        if (a.ff_norm_w) v2 = (v / scale) * a.ff_norm_w[i];
        if (a.norm_w) v = (v / scale) * a.norm_w[i];
      }
      const int piece = i / E, e = i % E, at = ((e >> 2) * pieces + piece) * 4 + (e & 3);
      reinterpret_cast<float*>(xs)[at] = v;
      if (a.ff_norm_w) reinterpret_cast<float*>(xs + P * pieces)[at] = v2;
    }
  }
  __syncthreads();

  // this lane's share of the two sums of unit u over pieces p0 .. p1
  auto dots = [&](int u, int p0, int p1, float& s0, float& s1) {
    int r0, r1;
    rows_of(u, r0, r1);
    const uint4* w0 = w + (size_t)r0 * pieces;
    const uint4* w1 = w + (size_t)r1 * pieces;
    const float4* xu = a.ff_norm_w && u >= plain_units ? xs + P * pieces : xs;
    int p = p0 + lane;
    for (; p + 96 < p1; p += 128) {
      uint4 b0[4], b1[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { b0[i] = __ldcs(w0 + p + 32 * i); b1[i] = __ldcs(w1 + p + 32 * i); }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 x0 = xu[p + 32 * i], x1 = P > 1 ? xu[(P - 1) * pieces + p + 32 * i] : x0;
        gv_fma(b0[i], x0, x1, s0, WT());
        gv_fma(b1[i], x0, x1, s1, WT());
      }
    }
    for (; p < p1; p += 32) {
      const uint4 b0 = __ldcs(w0 + p), b1 = __ldcs(w1 + p);
      const float4 x0 = xu[p], x1 = P > 1 ? xu[(P - 1) * pieces + p] : x0;
      gv_fma(b0, x0, x1, s0, WT());
      gv_fma(b1, x0, x1, s1, WT());
    }
  };
  auto total = [](float& s0, float& s1) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      s0 += __shfl_xor_sync(0xFFFFFFFFu, s0, o);
      s1 += __shfl_xor_sync(0xFFFFFFFFu, s1, o);
    }
  };
  auto store = [&](int u, float s0, float s1) {
    if (u < plain_units) {
      const int n = 2 * u;
      a.y[n] = plain_value(s0, a.alpha, a.bias, a.add, a.softcap, n);
      if (n + 1 < a.n_plain) a.y[n + 1] = plain_value(s1, a.alpha, a.bias, a.add, a.softcap, n + 1);
    } else if (a.act == FB200_FFN_GELU) {
      const int n = 2 * (u - plain_units);
      a.z[n] = fb_gelu_tanh(s0);
      if (n + 1 < a.ff) a.z[n + 1] = fb_gelu_tanh(s1);
    } else {
      a.z[u - plain_units] = silu_f(s0) * s1;
    }
  };
  for (int it = 0; it < a.whole; ++it) {
    const int u = it * warps + gw;
    float s0 = 0.f, s1 = 0.f;
    dots(u, 0, pieces, s0, s1);
    total(s0, s1);
    if (lane == 0) store(u, s0, s1);
  }
  // two CTAs fill an SM's registers: the next kernel is let in only when the last round begins
  pdl_launch_dependents();
  float s0 = 0.f, s1 = 0.f;
  if (rest < a.units) dots(rest, part * per, min(pieces, (part + 1) * per), s0, s1);
  total(s0, s1);
  if (a.ks > 1) {  // the parts of a unit meet in shared memory, added in part order
    __syncthreads();
    if (lane == 0) { red[2 * warp] = s0; red[2 * warp + 1] = s1; }
    __syncthreads();
    if (part == 0 && lane == 0) {
      s0 = s1 = 0.f;
      for (int i = 0; i < a.ks; ++i) { s0 += red[2 * (warp + i)]; s1 += red[2 * (warp + i) + 1]; }
    }
  }
  if (rest < a.units && part == 0 && lane == 0) store(rest, s0, s1);
}

// ---- F32 weights, many rows: 64 output rows x 64 activation rows per CTA, 4 x 4 per thread
constexpr int GF_T = 64, GF_K = 16;

struct GemmF32Args {
  const float* w;
  const float* x;
  const float* add;
  const float* bias;
  float* y;
  float* z;
  size_t ldx, ldy, ldadd, ldz, ff_off;
  int m, k, kx, row0, n_plain, gate0, up0, ff, act, plain_tiles;
  float alpha, softcap;
};

__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const GemmF32Args a) {
  __shared__ float ws[2][GF_K][GF_T + 4], xs[GF_K][GF_T + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;  // 4 output rows at tx * 4, 4 activation rows at ty * 4
  const bool ffn = (int)blockIdx.x >= a.plain_tiles, gelu = a.act == FB200_FFN_GELU, pair = ffn && !gelu;
  const int nt = ffn ? (int)blockIdx.x - a.plain_tiles : (int)blockIdx.x;
  const int r0 = (ffn ? gelu ? a.up0 : a.gate0 : a.row0) + nt * GF_T, r1 = a.up0 + nt * GF_T;
  const int lim = ffn ? a.ff - nt * GF_T : a.n_plain - nt * GF_T;  // rows of this tile that exist
  const float* x = ffn ? a.x + a.ff_off : a.x;
  const int m0 = (int)blockIdx.y * GF_T;
  float acc[2][4][4];
#pragma unroll
  for (int h = 0; h < 2; ++h)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[h][i][q] = 0.f;
  for (int k0 = 0; k0 < a.kx; k0 += GF_K) {
    for (int i = tid; i < GF_T * GF_K; i += 256) {
      const int r = i / GF_K, c = i % GF_K;
      const bool kin = k0 + c < a.kx;
      ws[0][c][r] = kin && r < lim ? a.w[(size_t)(r0 + r) * a.k + k0 + c] : 0.f;
      if (pair) ws[1][c][r] = kin && r < lim ? a.w[(size_t)(r1 + r) * a.k + k0 + c] : 0.f;
      xs[c][r] = kin && m0 + r < a.m ? x[(size_t)(m0 + r) * a.ldx + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < GF_K; ++c) {
      float xv[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = xs[c][ty * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i) wv[i] = ws[0][c][tx * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[0][i][q] = fmaf(wv[i], xv[q], acc[0][i][q]);
      if (pair) {
#pragma unroll
        for (int i = 0; i < 4; ++i) wv[i] = ws[1][c][tx * 4 + i];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int q = 0; q < 4; ++q) acc[1][i][q] = fmaf(wv[i], xv[q], acc[1][i][q]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const int m = m0 + ty * 4 + q;
    if (m >= a.m) continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = tx * 4 + i, n = nt * GF_T + r;
      if (r >= lim) continue;
      if (ffn) a.z[(size_t)m * a.ldz + n] = gelu ? fb_gelu_tanh(acc[0][i][q]) : silu_f(acc[0][i][q]) * acc[1][i][q];
      else a.y[(size_t)m * a.ldy + n] = plain_value(acc[0][i][q], a.alpha, a.bias, a.add ? a.add + (size_t)m * a.ldadd : nullptr, a.softcap, n);
    }
  }
}

// f32 rows -> (normalised) bf16 rows with zero padding, one CTA per row
__global__ void __launch_bounds__(256)
rows_to_bf16_kernel(const float* __restrict__ x, size_t ldx, const float* __restrict__ w, const float* __restrict__ w2, float eps,
                    int n, int np, __nv_bfloat16* __restrict__ y) {
  __shared__ float sh[8];
  const size_t row = blockIdx.x;
  const float* xr = x + row * ldx;
  y += row * (w2 ? 2 : 1) * (size_t)np;
  float rms = 1.f;
  if (w) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += 256) ss = fmaf(xr[i], xr[i], ss);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < 8; ++i) ss += sh[i];
    rms = sqrtf(ss / (float)n + eps);
  }
  for (int i = threadIdx.x; i < np; i += 256) {
    const float u = i < n ? xr[i] / rms : 0.f;
    y[i] = __float2bfloat16(w && i < n ? u * w[i] : u);
    if (w2) y[np + i] = __float2bfloat16(i < n ? u * w2[i] : 0.f);
  }
}

}  // namespace

int fb200_rows_to_bf16(fb200_device* dev, const float* x, size_t ldx, const float* w, const float* w2, float eps, size_t rows,
                       int n, int np, __nv_bfloat16* y) {
  if (rows == 0) return FB200_OK;
  rows_to_bf16_kernel<<<(unsigned)rows, 256, 0, dev->stream>>>(x, ldx, w, w2, eps, n, np, y);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}

int fb200_dense_gemv(fb200_device* dev, const fb200_dense_job& j) {
  const bool bf = j.w->type == FB200_BF16;
  const int e = bf ? 8 : 4;
  if (j.m != 1 || j.y_bf16 || j.w->k % e || j.w->k * 4 > 200 * 1024)
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "dense product: one row of %llu columns is not covered", (unsigned long long)j.w->k);
  if (j.ff && j.n_plain && (j.ff_off || (j.ff_norm_w && j.w->k * 8 > 200 * 1024))) {  // the two groups one after the other
    fb200_dense_job p = j, f = j;
    p.ff = 0;
    f.n_plain = 0;
    f.x = (const float*)j.x + j.ff_off;
    f.norm_w = j.ff_norm_w ? j.ff_norm_w : j.norm_w;
    p.ff_norm_w = f.ff_norm_w = nullptr;
    p.ff_off = f.ff_off = 0;
    const int rc = fb200_dense_gemv(dev, p);
    return rc ? rc : fb200_dense_gemv(dev, f);
  }
  GemvArgs a = {};
  a.w = j.w->data; a.x = (const float*)j.x; a.norm_w = j.norm_w; a.ff_norm_w = j.ff ? j.ff_norm_w : nullptr; a.add = j.add; a.bias = j.bias;
  a.y = (float*)j.y; a.z = (float*)j.z; a.alpha = j.alpha; a.softcap = j.softcap; a.act = j.act;
  a.k = (int)j.w->k; a.kx = j.kx; a.row0 = j.row0; a.n_plain = j.n_plain; a.gate0 = j.gate0; a.up0 = j.up0; a.ff = j.ff; a.eps = j.eps;
  a.units = (j.n_plain + 1) / 2 + (j.act == FB200_FFN_GELU ? (j.ff + 1) / 2 : j.ff);
  if (a.units == 0) return FB200_OK;
  const size_t smem = (size_t)j.w->k * (a.ff_norm_w ? 8 : 4);
  const int per_sm = smem <= 100 * 1024 ? 2 : 1;
  const int ctas = dev->sm_count * per_sm;
  // whole rounds, and for the units that are left the split of K that one round has warps for
  a.whole = a.units / (ctas * GV_WARPS);
  const int left = a.units - a.whole * ctas * GV_WARPS;
  a.ks = 1;
  while (a.ks < GV_WARPS && left * a.ks * 2 <= ctas * GV_WARPS && a.k / e >= a.ks * 2 * 32) a.ks *= 2;
  const int grid = a.whole ? ctas : (left * a.ks + GV_WARPS - 1) / GV_WARPS;
  static bool configured[64] = {false};
  if (!configured[dev->ordinal & 63]) {
    FB_CUDA(dev, cudaFuncSetAttribute(dense_gemv_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    FB_CUDA(dev, cudaFuncSetAttribute(dense_gemv_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    configured[dev->ordinal & 63] = true;
  }
  return fb200_launch(dev, bf ? dense_gemv_kernel<__nv_bfloat16> : dense_gemv_kernel<float>, dim3((unsigned)grid), dim3(GV_THREADS),
                      smem, true, a);
}

int fb200_dense_gemm_f32(fb200_device* dev, const fb200_dense_job& j) {
  if (j.w->type != FB200_F32 || j.norm_w || j.y_bf16)
    return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "dense product: f32 rows need F32 weights");
  GemmF32Args a = {};
  a.w = (const float*)j.w->data; a.x = (const float*)j.x; a.add = j.add; a.bias = j.bias; a.y = (float*)j.y; a.z = (float*)j.z;
  a.alpha = j.alpha; a.softcap = j.softcap; a.act = j.act; a.ff_off = j.ff_off;
  a.ldx = j.ldx; a.ldy = j.ldy; a.ldadd = j.ldadd; a.ldz = j.ldz;
  a.m = j.m; a.k = (int)j.w->k; a.kx = j.kx; a.row0 = j.row0; a.n_plain = j.n_plain; a.gate0 = j.gate0; a.up0 = j.up0; a.ff = j.ff;
  a.plain_tiles = (j.n_plain + GF_T - 1) / GF_T;
  const unsigned gx = (unsigned)(a.plain_tiles + (j.ff + GF_T - 1) / GF_T), gy = (unsigned)((j.m + GF_T - 1) / GF_T);
  if (gx == 0 || gy == 0) return FB200_OK;
  dense_gemm_f32_kernel<<<dim3(gx, gy), 256, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}

int fb200_dense_product(fb200_device* dev, const fb200_dense_job& j) {
  if (j.m <= 0) return FB200_OK;
  if (j.m == 1) return fb200_dense_gemv(dev, j);
  if (j.w->type == FB200_F32) return fb200_dense_gemm_f32(dev, j);
  return fb200_dense_gemm_tc(dev, j);
}

// q_mat_mul with an untiled matrix: y [m, n] = x [m, k] . W^T, f32 rows in and out
int fb200_dense_matmul(fb200_device* dev, const fb200_qmatrix* w, const float* x, size_t m, float* y) {
  const bool aligned = ((reinterpret_cast<uintptr_t>(w->data) | reinterpret_cast<uintptr_t>(x)) & 15u) == 0 && m < (1ull << 31);
  fb200_dense_job j;
  j.w = w; j.m = (int)m; j.x = x; j.ldx = w->k; j.kx = (int)w->k; j.n_plain = (int)w->n; j.y = y; j.ldy = w->n;
  if (aligned && w->type == FB200_F32 && m > 1) return fb200_dense_gemm_f32(dev, j);
  if (aligned && w->type == FB200_F32 && w->k % 4 == 0 && w->k * 4 <= 200 * 1024) return fb200_dense_gemv(dev, j);
  if (aligned && w->type == FB200_BF16 && w->k % 8 == 0) {
    if (m == 1 && w->k * 4 <= 200 * 1024) return fb200_dense_gemv(dev, j);
    int rc = fb200_ensure(dev, &dev->xpack, &dev->xpack_bytes, m * w->k * 2);
    if (rc) return rc;
    __nv_bfloat16* xb = (__nv_bfloat16*)dev->xpack;
    if ((rc = fb200_rows_to_bf16(dev, x, w->k, nullptr, nullptr, 0.f, m, (int)w->k, (int)w->k, xb))) return rc;
    j.x = xb;
    return fb200_dense_gemm_tc(dev, j);
  }
  const uint64_t warps = (uint64_t)m * w->n;
  const uint64_t blocks = (warps * 32 + 255) / 256;
  if (blocks >= (1ull << 31)) return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "dense matmul too large");
  dense_matmul_kernel<<<(unsigned)blocks, 256, 0, dev->stream>>>(w->type, w->data, x, m, w->n, w->k, y);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}
