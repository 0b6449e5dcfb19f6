// Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, the read-out normalised over all heads.
//
// The columns of S (one per value element) are independent: a group of lanes owns a column and keeps it in registers. All
// sums, states and decays are f32.
//  * linear_scan_kernel: token by token. One new token per sequence is one launch: the state is requested before the
//    projections are there, and the CTA that arrives last normalises the whole row and applies the gates. Bound: HBM on
//    the state, read and written once.
//  * linear_out_kernel: the normalisation and the gates of a prompt's rows.
#include <algorithm>

#include "mixers.cuh"
#include "qgemv_common.cuh"
#include "state_columns.cuh"

namespace {

constexpr int LS_THREADS = 256, LS_LPC = 16, LS_COLS = LS_THREADS / LS_LPC;

// o [h v] of one row: RMS norm over the heads together, weight, sigmoid gate, factor; all threads of the CTA
__device__ __forceinline__ void linear_finish_row(const fb200_linear_args& a, size_t row, float* red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = a.h * a.v;
  const float* o = a.o + row * n;
  const float* g = a.y + row * a.ldy + a.off_g;
  float ss = 0.f;
  for (int i = tid; i < n; i += LS_THREADS) {
    const float x = __ldcg(o + i);
    ss = fmaf(x, x, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < LS_THREADS / 32; ++i) ss += red[i];
  const float rms = sqrtf(ss / (float)n + a.eps);
  for (int i = tid; i < n; i += LS_THREADS) {
    const float x = (__ldcg(o + i) / rms) * a.out_norm[i] * dr_sigmoid(g[i]) * a.out_scale;
    if (a.z_bf16) reinterpret_cast<__nv_bfloat16*>(a.z)[row * a.ldz + i] = __float2bfloat16(x);
    else reinterpret_cast<float*>(a.z)[row * a.ldz + i] = x;
  }
}

__global__ void __launch_bounds__(LS_THREADS) linear_out_kernel(const fb200_linear_args a) {
  __shared__ float red[LS_THREADS / 32];
  linear_finish_row(a, blockIdx.x, red);
}

// CTA: LS_COLS columns of one head of one sequence. EPT elements of a column per lane; TOK tokens staged at a time.
template <int EPT, int TOK>
__global__ void __launch_bounds__(LS_THREADS) linear_scan_kernel(const fb200_linear_args a) {
  constexpr int DP = EPT * LS_LPC;
  __shared__ __align__(16) float ks[TOK][DP], qs[TOK][DP];
  __shared__ float vs[TOK][LS_COLS], red[LS_THREADS / 32];
  __shared__ int last;
  const int tid = threadIdx.x, p = tid % LS_LPC, cl = tid / LS_LPC, c0 = blockIdx.x * LS_COLS, c = c0 + cl, h = blockIdx.y, b = blockIdx.z;
  const int pos = *a.pos_dev, hv = a.h * a.v;
  float* st = a.state + (((size_t)b * a.h + h) * a.v + c) * (size_t)DP;
  const float decay = a.decay[(size_t)h * (FB200_LINEAR_CHUNK + 1) + 1];
  float2 s[EPT / 2];
  // an earlier pass wrote the state: its loads do not wait for this pass's projections
  if (c < a.v && pos > 0) {
    load_column<EPT, LS_LPC>(st, p, s);
  } else {
#pragma unroll
    for (int i = 0; i < EPT / 2; ++i) s[i] = make_float2(0.f, 0.f);
  }
  pdl_wait();
  pdl_launch_dependents();
  const float2 g2 = make_float2(decay, decay);
  for (int t0 = 0; t0 < a.s; t0 += TOK) {
    const int n = min(TOK, a.s - t0);
    for (int i = tid; i < n * DP; i += LS_THREADS) {
      const int t = i / DP, e = i % DP;
      const float* yr = a.y + ((size_t)b * a.s + t0 + t) * a.ldy + (size_t)h * a.d + e;
      qs[t][e] = e < a.d ? dr_silu(yr[0]) : 0.f;
      ks[t][e] = e < a.d ? dr_silu(yr[a.off_k]) : 0.f;
    }
    for (int i = tid; i < n * LS_COLS; i += LS_THREADS) {
      const int t = i / LS_COLS, cc = c0 + i % LS_COLS;
      vs[t][i % LS_COLS] = cc < a.v ? dr_silu(a.y[((size_t)b * a.s + t0 + t) * a.ldy + a.off_v + (size_t)h * a.v + cc]) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
      const float v = vs[t][cl];
      const float2 v2 = make_float2(v, v);
      float2 o0 = make_float2(0.f, 0.f), o1 = o0;
#pragma unroll
      for (int i = 0; i < EPT / 4; ++i) {
        const float4 k = *reinterpret_cast<const float4*>(&ks[t][4 * (i * LS_LPC + p)]);
        const float4 q = *reinterpret_cast<const float4*>(&qs[t][4 * (i * LS_LPC + p)]);
        s[2 * i] = fma2(make_float2(k.x, k.y), v2, mul2(s[2 * i], g2));
        s[2 * i + 1] = fma2(make_float2(k.z, k.w), v2, mul2(s[2 * i + 1], g2));
        o0 = fma2(s[2 * i], make_float2(q.x, q.y), o0);
        o1 = fma2(s[2 * i + 1], make_float2(q.z, q.w), o1);
      }
      float o = (o0.x + o0.y) + (o1.x + o1.y);
#pragma unroll
      for (int w = LS_LPC / 2; w > 0; w >>= 1) o += __shfl_xor_sync(0xFFFFFFFFu, o, w);
      if (p == 0 && c < a.v) a.o[((size_t)b * a.s + t0 + t) * hv + (size_t)h * a.v + c] = o;
    }
    __syncthreads();
  }
  if (c < a.v && a.commit) store_column<EPT, LS_LPC>(st, p, s);
  if (a.s > 1) return;
  // one token: the last CTA of the sequence finishes its row
  __threadfence();
  __syncthreads();
  if (tid == 0) last = atomicAdd(a.done + b, 1) == (int)(gridDim.x * gridDim.y) - 1;
  __syncthreads();
  if (!last) return;
  __threadfence();
  if (tid == 0) a.done[b] = 0;
  linear_finish_row(a, b, red);
}

int linear_scan(fb200_device* dev, const fb200_linear_args& a) {
  const dim3 grid((unsigned)((a.v + LS_COLS - 1) / LS_COLS), (unsigned)a.h, (unsigned)a.b), block(LS_THREADS);
  switch (a.dp) {
    case 64: return fb200_launch(dev, linear_scan_kernel<4, 16>, grid, block, 0, true, a);
    case 128: return fb200_launch(dev, linear_scan_kernel<8, 16>, grid, block, 0, true, a);
    case 256: return fb200_launch(dev, linear_scan_kernel<16, 8>, grid, block, 0, true, a);
    case 512: return fb200_launch(dev, linear_scan_kernel<32, 4>, grid, block, 0, true, a);
    default: return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "linear attention: head size %d", a.d);
  }
}

}  // namespace

int fb200_linear_dp(int d) {
  for (int dp : {64, 128, 256, 512})
    if (d <= dp) return dp;
  return 0;
}

int fb200_linear_step(fb200_device* dev, const fb200_linear_args& a) { return linear_scan(dev, a); }

int fb200_linear_prompt(fb200_device* dev, const fb200_linear_args& a) {
  const int rc = linear_scan(dev, a);
  if (rc) return rc;
  linear_out_kernel<<<(unsigned)(a.b * a.s), LS_THREADS, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}
