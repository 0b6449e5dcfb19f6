// Latent attention, row by row in the latent space.
//
// A cached position is one latent c (rk numbers) and one rotated key part (r numbers) shared by all heads; head n's
// key is (W_uk,n c, key part) and its value W_uv,n c. For a row of queries the expansions are applied to the query and
// to the read-out instead of to the keys:
//   q_n . k_n = (W_uk,n^T q_n) . c + q_rot,n . key part,      sum_j p_j W_uv,n c_j = W_uv,n (sum_j p_j c_j)
// so that a step reads the cache and the two expansion matrices once and nothing is expanded in memory.
//  * latent_query_kernel: rotation, W_uk^T q per head (x scale); one more CTA per row normalises the new latent, rotates the
//    new key part and appends both to the cache,
//  * latent_attn_kernel: scores, online softmax and read-out over the visible keys, split over CTAs,
//  * latent_out_kernel: merges the splits, W_uv, the sigmoid gate of the head.
// f32 arithmetic throughout (bf16 or f32 weights and cache). Decode steps run these for one row per sequence; prompts
// run them for F32 models and for shapes the tensor-core path does not cover.
#include <algorithm>

#include "mixers.cuh"
#include "qgemv_common.cuh"

namespace {

constexpr int LQ_THREADS = 256, LA_WARPS = 4, LO_THREADS = 256;

__device__ __forceinline__ float la_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
// the elements of a 16-byte piece as floats
__device__ __forceinline__ void unpack(const uint4& u, float (&f)[8], __nv_bfloat16) {
  f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xFFFF0000u);
  f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xFFFF0000u);
  f[4] = __uint_as_float(u.z << 16); f[5] = __uint_as_float(u.z & 0xFFFF0000u);
  f[6] = __uint_as_float(u.w << 16); f[7] = __uint_as_float(u.w & 0xFFFF0000u);
}
__device__ __forceinline__ void unpack(const uint4& u, float (&f)[4], float) {
  f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
}
__device__ __forceinline__ void store_elem(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void store_elem(float* p, float v) { *p = v; }

// T: element type of the expansion matrices and of the cache. CTAs 0 .. heads - 1 of a row take a query head each.
template <typename T>
__global__ void __launch_bounds__(LQ_THREADS) latent_query_kernel(const fb200_latent_args a, int heads) {
  constexpr int E = 16 / (int)sizeof(T);
  extern __shared__ __align__(16) float lsm[];  // query head [d + r], or partial sums [LQ_THREADS][E]
  __shared__ float red[LQ_THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.y, b = row / a.s;
  pdl_launch_dependents();
  pdl_wait();
  const int pos = *a.pos_dev + row % a.s;
  const float* yr = a.y + (size_t)row * a.ldy;
  const int half = a.r / 2;
  const float *cs = a.rope_cos + (size_t)pos * half, *sn = a.rope_sin + (size_t)pos * half;
  if ((int)blockIdx.x == heads) {  // the new position of a layer with a cache of its own
    const float* src = yr + a.off_dkv;
    T* dst = reinterpret_cast<T*>(a.cache) + ((size_t)b * a.cap + pos) * a.ldc;
    float ss = 0.f;
    for (int i = tid; i < a.rk; i += LQ_THREADS) ss = fmaf(src[i], src[i], ss);
    ss = la_warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < LQ_THREADS / 32; ++i) ss += red[i];
    const float rms = sqrtf(ss / (float)a.rk + a.eps);
    for (int i = tid; i < a.rk; i += LQ_THREADS) store_elem(dst + i, (src[i] / rms) * a.c_norm[i]);
    for (int i = tid; i < half; i += LQ_THREADS) {
      const float u = src[a.rk + i], v = src[a.rk + half + i];
      store_elem(dst + a.rk + i, u * cs[i] - v * sn[i]);
      store_elem(dst + a.rk + half + i, v * cs[i] + u * sn[i]);
    }
    return;
  }
  const int h = blockIdx.x;
  float* qs = lsm;
  float* part = lsm + ((a.d + 3) & ~3);
  const float* q = yr + (size_t)h * (a.d + a.r);
  float* out = a.qa + ((size_t)row * a.h + h) * (a.rk + a.r);
  for (int i = tid; i < a.d; i += LQ_THREADS) qs[i] = q[i];
  for (int i = tid; i < half; i += LQ_THREADS) {
    const float u = q[a.d + i], v = q[a.d + half + i];
    out[a.rk + i] = (u * cs[i] - v * sn[i]) * a.scale;
    out[a.rk + half + i] = (v * cs[i] + u * sn[i]) * a.scale;
  }
  __syncthreads();
  // W_uk^T q: a thread owns one 16-byte piece of the latent, groups of threads share the sum over d
  const int np = a.rkp / E;
  const T* w = reinterpret_cast<const T*>(a.w_ukv) + (size_t)h * a.d * a.rkp;
  for (int c0 = 0; c0 < np; c0 += LQ_THREADS) {
    const int nc = min(np - c0, LQ_THREADS), groups = LQ_THREADS / nc, c = tid % nc, gr = tid / nc;
    float acc[E];
#pragma unroll
    for (int e = 0; e < E; ++e) acc[e] = 0.f;
    if (gr < groups) {
#pragma unroll 4
      for (int i = gr; i < a.d; i += groups) {
        float f[E];
        unpack(*reinterpret_cast<const uint4*>(w + (size_t)i * a.rkp + (c0 + c) * E), f, T());
#pragma unroll
        for (int e = 0; e < E; ++e) acc[e] = fmaf(f[e], qs[i], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < E; ++e) part[(gr * nc + c) * E + e] = acc[e];
    }
    __syncthreads();
    for (int i = tid; i < nc * E; i += LQ_THREADS) {
      float s = 0.f;
      for (int k = 0; k < groups; ++k) s += part[k * nc * E + i];
      if (c0 * E + i < a.rk) out[c0 * E + i] = s * a.scale;
    }
    __syncthreads();
  }
}

__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) {
  const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xFFFF0000u));
}
__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }

// One CTA per (split of the visible keys, head, row); a warp takes 4 keys at a time, a lane the element pairs
// 2 lane + 64 i of a cache row. NI = 64-element pieces of a cache row.
template <typename T, int NI>
__global__ void __launch_bounds__(LA_WARPS * 32) latent_attn_kernel(const fb200_latent_args a) {
  extern __shared__ __align__(16) float lsm[];  // [LA_WARPS][rk]
  __shared__ float wm[LA_WARPS], wl[LA_WARPS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, row = blockIdx.z, b = row / a.s;
  pdl_launch_dependents();
  pdl_wait();
  const int pos = *a.pos_dev + row % a.s, n = a.rk + a.r;
  const int lo = a.window ? max(0, pos - a.window + 1) : 0, keys = pos + 1 - lo;
  const int per = (keys + a.nsplit - 1) / a.nsplit, k0 = lo + min(keys, (int)blockIdx.x * per), k1 = min(pos + 1, k0 + per);
  const float* qa = a.qa + ((size_t)row * a.h + h) * n;
  float2 q[NI], acc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int e = 2 * lane + 64 * i;
    q[i] = make_float2(e < n ? qa[e] : 0.f, e + 1 < n ? qa[e + 1] : 0.f);
    acc[i] = make_float2(0.f, 0.f);
  }
  const T* cache = reinterpret_cast<const T*>(a.cache) + (size_t)b * a.cap * a.ldc;
  float m = -INFINITY, l = 0.f;
  for (int k = k0 + 4 * warp; k < k1; k += 4 * LA_WARPS) {
    float2 c[4][NI];
    float s[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      s[j] = 0.f;
      const T* r = cache + (size_t)min(k + j, k1 - 1) * a.ldc;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int e = 2 * lane + 64 * i;
        c[j][i] = e < a.ldc ? load_pair(r + e) : make_float2(0.f, 0.f);
        s[j] = fmaf(c[j][i].x, q[i].x, s[j]);
        s[j] = fmaf(c[j][i].y, q[i].y, s[j]);
      }
    }
    float mx = m;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      s[j] = la_warp_sum(s[j]);
      if (k + j >= k1) s[j] = -INFINITY;
      mx = fmaxf(mx, s[j]);
    }
    const float alpha = expf(m - mx);
    m = mx;
    l *= alpha;
#pragma unroll
    for (int i = 0; i < NI; ++i) { acc[i].x *= alpha; acc[i].y *= alpha; }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float p = expf(s[j] - mx);
      l += p;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        acc[i].x = fmaf(p, c[j][i].x, acc[i].x);
        acc[i].y = fmaf(p, c[j][i].y, acc[i].y);
      }
    }
  }
  if (lane == 0) { wm[warp] = m; wl[warp] = l; }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int e = 2 * lane + 64 * i;
    if (e < a.rk) lsm[warp * a.rk + e] = acc[i].x;
    if (e + 1 < a.rk) lsm[warp * a.rk + e + 1] = acc[i].y;
  }
  __syncthreads();
  float mx = -INFINITY, w[LA_WARPS], lt = 0.f;
#pragma unroll
  for (int i = 0; i < LA_WARPS; ++i) mx = fmaxf(mx, wm[i]);
#pragma unroll
  for (int i = 0; i < LA_WARPS; ++i) {
    w[i] = wm[i] == -INFINITY ? 0.f : expf(wm[i] - mx);
    lt = fmaf(wl[i], w[i], lt);
  }
  float* out = a.part + (((size_t)row * a.h + h) * a.nsplit + blockIdx.x) * (a.rk + 2);
  for (int e = tid; e < a.rk; e += LA_WARPS * 32) {
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < LA_WARPS; ++i) v = fmaf(lsm[i * a.rk + e], w[i], v);
    out[e] = v;
  }
  if (tid == 0) { out[a.rk] = mx; out[a.rk + 1] = lt; }
}

template <typename T>
__global__ void __launch_bounds__(LO_THREADS) latent_out_kernel(const fb200_latent_args a) {
  constexpr int E = 16 / (int)sizeof(T);
  extern __shared__ __align__(16) float lsm[];  // merged read-out [rkp], split weights [nsplit]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, row = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const float* part = a.part + ((size_t)row * a.h + h) * a.nsplit * (a.rk + 2);
  float* wt = lsm + a.rkp;
  float mx = -INFINITY, l = 0.f;
  for (int s = 0; s < a.nsplit; ++s) mx = fmaxf(mx, part[(size_t)s * (a.rk + 2) + a.rk]);
  for (int s = 0; s < a.nsplit; ++s) {
    const float m = part[(size_t)s * (a.rk + 2) + a.rk];
    const float w = m == -INFINITY ? 0.f : expf(m - mx);
    l = fmaf(part[(size_t)s * (a.rk + 2) + a.rk + 1], w, l);
    if (tid == 0) wt[s] = w;
  }
  __syncthreads();
  const float inv = 1.0f / l;
  for (int e = tid; e < a.rkp; e += LO_THREADS) {
    float v = 0.f;
    if (e < a.rk)
      for (int s = 0; s < a.nsplit; ++s) v = fmaf(part[(size_t)s * (a.rk + 2) + e], wt[s], v);
    lsm[e] = v * inv;
  }
  __syncthreads();
  const T* w = reinterpret_cast<const T*>(a.w_ukv) + ((size_t)a.h * a.d + (size_t)h * a.v) * a.rkp;
  const float gate = 1.0f / (1.0f + expf(-a.y[(size_t)row * a.ldy + a.off_g + h]));
  const int np = a.rkp / E;
  for (int v = warp; v < a.v; v += LO_THREADS / 32) {
    float s = 0.f;
    for (int p = lane; p < np; p += 32) {
      float f[E];
      unpack(*reinterpret_cast<const uint4*>(w + (size_t)v * a.rkp + p * E), f, T());
#pragma unroll
      for (int e = 0; e < E; ++e) s = fmaf(f[e], lsm[p * E + e], s);
    }
    s = la_warp_sum(s);
    if (lane == 0) {
      const size_t zi = (size_t)row * a.ldz + h * a.v + v;
      if (a.z_bf16) reinterpret_cast<__nv_bfloat16*>(a.z)[zi] = __float2bfloat16(s * gate);
      else reinterpret_cast<float*>(a.z)[zi] = s * gate;
    }
  }
}

template <typename T>
int latent_rows(fb200_device* dev, const fb200_latent_args& a) {
  const unsigned rows = (unsigned)(a.b * a.s);
  constexpr int E = 16 / (int)sizeof(T);
  int rc;
  const size_t smem_q = (size_t)(((a.d + 3) & ~3) + LQ_THREADS * E) * 4;
  if ((rc = fb200_launch(dev, latent_query_kernel<T>, dim3((unsigned)(a.h + (a.off_dkv >= 0 ? 1 : 0)), rows), dim3(LQ_THREADS), smem_q, true, a, a.h)))
    return rc;
  const int n = (a.ldc + 63) / 64;
  const dim3 grid((unsigned)a.nsplit, (unsigned)a.h, rows);
  const size_t smem = (size_t)LA_WARPS * a.rk * 4;
  const dim3 block(LA_WARPS * 32);
  if (n <= 2) rc = fb200_launch(dev, latent_attn_kernel<T, 2>, grid, block, smem, true, a);
  else if (n <= 4) rc = fb200_launch(dev, latent_attn_kernel<T, 4>, grid, block, smem, true, a);
  else if (n <= 6) rc = fb200_launch(dev, latent_attn_kernel<T, 6>, grid, block, smem, true, a);
  else if (n <= 10) rc = fb200_launch(dev, latent_attn_kernel<T, 10>, grid, block, smem, true, a);
  else rc = fb200_launch(dev, latent_attn_kernel<T, 18>, grid, block, smem, true, a);
  if (rc) return rc;
  return fb200_launch(dev, latent_out_kernel<T>, dim3((unsigned)a.h, rows), dim3(LO_THREADS), (size_t)(a.rkp + a.nsplit) * 4, true, a);
}

}  // namespace

bool fb200_latent_covers(int d, int r, int v, int rk) {
  return d > 0 && v > 0 && rk > 0 && r >= 0 && r % 2 == 0 && d <= 4096 && rk + r <= 1144;
}

// Splits of the visible keys per head: enough CTAs for the GPU, at least 32 keys each.
int fb200_latent_nsplit(const fb200_device* dev, int b, int h, int window, int cap) {
  const int keys = window && window < cap ? window : cap;
  const int ns = std::min((keys + 31) / 32, 4 * dev->sm_count / std::max(1, b * h));
  return std::max(1, std::min(ns, 32));
}

int fb200_latent_append(fb200_device* dev, const fb200_latent_args& a) {
  if (a.off_dkv < 0) return FB200_OK;
  const dim3 grid(1, (unsigned)(a.b * a.s));
  if (a.b * a.s > 65535) return fb200_fail(dev, FB200_ERR_CAPACITY, "latent attention: at most 65535 rows per pass");
  if (a.cache_f32) return fb200_launch(dev, latent_query_kernel<float>, grid, dim3(LQ_THREADS), 16, true, a, 0);
  return fb200_launch(dev, latent_query_kernel<__nv_bfloat16>, grid, dim3(LQ_THREADS), 16, true, a, 0);
}

int fb200_latent_rows(fb200_device* dev, const fb200_latent_args& a) {
  if (a.b * a.s > 65535) return fb200_fail(dev, FB200_ERR_CAPACITY, "latent attention: at most 65535 rows per pass without the tensor-core path");
  return a.cache_f32 ? latent_rows<float>(dev, a) : latent_rows<__nv_bfloat16>(dev, a);
}
