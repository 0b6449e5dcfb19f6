// Latent attention, row by row in the latent space.
//
// A cached position is one latent c (rk numbers) and one rotated key part (r numbers) shared by all heads; head n's
// key is (W_uk,n c, key part) and its value W_uv,n c. For a row of queries the expansions are applied to the query and
// to the read-out instead of to the keys:
//   q_n . k_n = (W_uk,n^T q_n) . c + q_rot,n . key part,      sum_j p_j W_uv,n c_j = W_uv,n (sum_j p_j c_j)
// so that a step reads the cache and the two expansion matrices once and nothing is expanded in memory.
//  * latent_query_kernel: rotation, W_uk^T q per head (x scale); one more CTA per row normalises the new latent, rotates the
//    new key part and appends both to the cache,
//  * latent_attn_mma_kernel / latent_attn_kernel: scores, online softmax and read-out over the visible keys, split
//    over CTAs (bf16 tensor cores where the sizes allow, else plain f32),
//  * latent_out_kernel: merges the splits, W_uv, the sigmoid gate of the head.
// f32 arithmetic otherwise (bf16 or f32 weights and cache). Decode steps run these for one row per sequence; prompts
// run them for F32 models and for shapes the tensor-core path does not cover.
#include <algorithm>

#include "attn_mma.cuh"
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

// T: element type of the expansion matrices and of the cache. A row's CTAs take `csplit` column ranges of
// each query head, the last one the new position.
template <typename T>
__global__ void __launch_bounds__(LQ_THREADS) latent_query_kernel(const fb200_latent_args a, int heads, int csplit) {
  constexpr int E = 16 / (int)sizeof(T);
  extern __shared__ __align__(16) float lsm[];  // query head [d + r], or partial sums [LQ_THREADS][E]
  __shared__ float red[LQ_THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.y, b = row / a.s;
  pdl_wait();
  pdl_launch_dependents();
  const int pos = *a.pos_dev + row % a.s;
  const float* yr = a.y + (size_t)row * a.ldy;
  const int half = a.r / 2;
  const float *cs = a.rope_cos + (size_t)pos * half, *sn = a.rope_sin + (size_t)pos * half;
  if ((int)blockIdx.x == heads * csplit) {  // the new position of a layer with a cache of its own
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
  const int h = blockIdx.x / csplit, cs_i = blockIdx.x % csplit;
  float* qs = lsm;
  float* part = lsm + ((a.d + 3) & ~3);
  const float* q = yr + (size_t)h * (a.d + a.r);
  float* out = a.qa + ((size_t)row * a.h + h) * (a.rk + a.r);
  for (int i = tid; i < a.d; i += LQ_THREADS) qs[i] = q[i];
  for (int i = tid; i < half && cs_i == 0; i += LQ_THREADS) {
    const float u = q[a.d + i], v = q[a.d + half + i];
    out[a.rk + i] = (u * cs[i] - v * sn[i]) * a.scale;
    out[a.rk + half + i] = (v * cs[i] + u * sn[i]) * a.scale;
  }
  __syncthreads();
  // W_uk^T q: a thread owns one 16-byte piece of the latent, groups of threads share the sum over d
  const int np = a.rkp / E;
  const T* w = reinterpret_cast<const T*>(a.w_ukv) + (size_t)h * a.d * a.rkp;
  const int cper = (np + csplit - 1) / csplit, cend = min(np, (cs_i + 1) * cper);
  for (int c0 = cs_i * cper; c0 < cend; c0 += LQ_THREADS) {
    const int nc = min(cend - c0, LQ_THREADS), groups = LQ_THREADS / nc, c = tid % nc, gr = tid / nc;
    float acc[E];
#pragma unroll
    for (int e = 0; e < E; ++e) acc[e] = 0.f;
    if (gr < groups) {
#pragma unroll 8
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
  pdl_wait();
  pdl_launch_dependents();
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

// CTAs of a (head, row) take LO_ROWS value rows per warp each; the weights do not depend on the kernels before.
constexpr int LO_ROWS = 4;
template <typename T>
__global__ void __launch_bounds__(LO_THREADS) latent_out_kernel(const fb200_latent_args a) {
  constexpr int E = 16 / (int)sizeof(T), PRE = 2;  // pieces per lane requested ahead
  extern __shared__ __align__(16) float lsm[];     // merged read-out [rkp], split weights [nsplit]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, row = blockIdx.y;
  const int v0 = ((int)blockIdx.z * (LO_THREADS / 32) + warp) * LO_ROWS, np = a.rkp / E;
  const T* w = reinterpret_cast<const T*>(a.w_ukv) + ((size_t)a.h * a.d + (size_t)h * a.v) * a.rkp;
  uint4 pre[LO_ROWS][PRE];
#pragma unroll
  for (int i = 0; i < LO_ROWS; ++i)
#pragma unroll
    for (int k = 0; k < PRE; ++k) {
      pre[i][k] = make_uint4(0u, 0u, 0u, 0u);
      if (v0 + i < a.v && lane + 32 * k < np) pre[i][k] = *reinterpret_cast<const uint4*>(w + (size_t)(v0 + i) * a.rkp + (lane + 32 * k) * E);
    }
  pdl_wait();
  pdl_launch_dependents();
  const float* part = a.part + ((size_t)row * a.h + h) * a.nsplit * (a.rk + 2);
  float* wt = lsm + a.rkp;
  if (warp == 0) {  // weights of the splits, normalised
    float mx = -INFINITY, l = 0.f;
    for (int s = lane; s < a.nsplit; s += 32) mx = fmaxf(mx, part[(size_t)s * (a.rk + 2) + a.rk]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, o));
    for (int s = lane; s < a.nsplit; s += 32) {
      const float m = part[(size_t)s * (a.rk + 2) + a.rk], x = m == -INFINITY ? 0.f : expf(m - mx);
      wt[s] = x;
      l = fmaf(part[(size_t)s * (a.rk + 2) + a.rk + 1], x, l);
    }
    l = la_warp_sum(l);
    for (int s = lane; s < a.nsplit; s += 32) wt[s] *= 1.0f / l;
  }
  const float gate = 1.0f / (1.0f + expf(-a.y[(size_t)row * a.ldy + a.off_g + h]));
  __syncthreads();
  // merged read-out; an empty split (weight 0) left nothing behind
  if ((a.rk & 1) == 0) {
    for (int e = 2 * tid; e < a.rkp; e += 2 * LO_THREADS) {
      float2 v = make_float2(0.f, 0.f);
      if (e < a.rk) {
#pragma unroll 16
        for (int s = 0; s < a.nsplit; ++s) {
          const float2 x = *reinterpret_cast<const float2*>(part + (size_t)s * (a.rk + 2) + e);
          const float w = wt[s];
          v.x = fmaf(w != 0.f ? x.x : 0.f, w, v.x);
          v.y = fmaf(w != 0.f ? x.y : 0.f, w, v.y);
        }
      }
      *reinterpret_cast<float2*>(lsm + e) = v;
    }
  } else {
    for (int e = tid; e < a.rkp; e += LO_THREADS) {
      float v = 0.f;
      if (e < a.rk) {
#pragma unroll 8
        for (int s = 0; s < a.nsplit; ++s) {
          const float x = part[(size_t)s * (a.rk + 2) + e], w = wt[s];
          v = fmaf(w != 0.f ? x : 0.f, w, v);
        }
      }
      lsm[e] = v;
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < LO_ROWS; ++i) {
    const int v = v0 + i;
    if (v >= a.v) break;
    float s = 0.f;
    for (int p = lane, k = 0; p < np; p += 32, ++k) {
      float f[E];
      unpack(k == 0 ? pre[i][0] : k == 1 ? pre[i][1] : *reinterpret_cast<const uint4*>(w + (size_t)v * a.rkp + p * E), f, T());
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

// ---- the same attention on bf16 tensor cores (bf16 cache, aligned sizes) ------------------------------------------
// One CTA per (split of the visible keys, 16 heads, row): the heads are the rows of the MMA tiles, so a cached
// position is read once for all of them. Tiles of 64 positions come by cp.async. S = Q K^T: a warp takes 16 positions; the queries
// are split into a bf16 value and a bf16 remainder, so the scores keep them in (nearly) 32 bits. The row maxima meet in
// shared memory, P is rounded to bf16, and O += P C runs with the latent columns cut over the four warps. NT: 8-column
// tiles of the latent per warp at most. Positions before this pass are requested before the kernel in front has finished.
constexpr int LM_KEYS = 64, LM_THREADS = 128, LM_PS = LM_KEYS + 8;

template <int NT>
__global__ void __launch_bounds__(LM_THREADS) latent_attn_mma_kernel(const fb200_latent_args a) {
  extern __shared__ __align__(16) float lsm[];
  const int n = a.rk + a.r, stride = n + 8;  // elements of a staged row; 16 bytes of padding spread the rows over the banks
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(lsm);    // [64][stride]
  __nv_bfloat16* Qh = Ks + (size_t)LM_KEYS * stride;            // [16][stride] values
  __nv_bfloat16* Ql = Qh + 16 * (size_t)stride;                 // [16][stride] remainders
  __nv_bfloat16* Ps = Ql + 16 * (size_t)stride;                 // [16][LM_PS]
  __shared__ float wmax[4][16], wsum[4][16];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, j = lane >> 3, r8 = lane & 7;
  const int row = blockIdx.z, b = row / a.s, h0 = blockIdx.y * 16;
  const int base = *a.pos_dev, pos = base + row % a.s;
  const int lo = a.window ? max(0, pos - a.window + 1) : 0, keys = pos + 1 - lo;
  const int per = ((keys + a.nsplit - 1) / a.nsplit + LM_KEYS - 1) / LM_KEYS * LM_KEYS;
  const int k0 = lo + min(keys, (int)blockIdx.x * per), k1 = min(pos + 1, k0 + per);
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache) + (size_t)b * a.cap * a.ldc;
  const int chunks = n / 8;
  // rows of tile kt with old (position < base) == want, zeros beyond the split
  auto fetch = [&](int kt, bool old) {
    for (int i = tid; i < LM_KEYS * chunks; i += LM_THREADS) {
      const int kr = i / chunks, c = i % chunks, key = kt + kr;
      const bool valid = key < k1;
      if ((!valid || key < base) != old) continue;
      pf_cp16(pf_smem(Ks + (size_t)kr * stride + c * 8), cache + (size_t)(valid ? key : 0) * a.ldc + c * 8, valid);
    }
  };
  if (k0 < k1) fetch(k0, true);
  pdl_wait();
  pdl_launch_dependents();
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int wcols = a.rk / 4, ntiles = wcols / 8;  // this warp's latent columns
  if (k0 < k1) {
    fetch(k0, false);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int i = tid; i < 16 * n; i += LM_THREADS) {
      const int hr = i / n, e = i % n;
      const float q = h0 + hr < a.h ? a.qa[((size_t)row * a.h + h0 + hr) * n + e] : 0.f;
      const __nv_bfloat16 hi = __float2bfloat16(q);
      Qh[hr * stride + e] = hi;
      Ql[hr * stride + e] = __float2bfloat16(q - __bfloat162float(hi));
    }
  }
  constexpr float LOG2E = 1.4426950408889634f;
  for (int kt = k0; kt < k1; kt += LM_KEYS) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // ---- S of this warp's 16 positions (the scale is in q)
    float s[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const uint32_t qa_h = pf_smem(Qh + ((j & 1) * 8 + r8) * stride + (j >> 1) * 8), qa_l = pf_smem(Ql + ((j & 1) * 8 + r8) * stride + (j >> 1) * 8);
    const uint32_t kb = pf_smem(Ks + (size_t)(warp * 16 + (j >> 1) * 8 + r8) * stride + (j & 1) * 8);
#pragma unroll 4
    for (int ks = 0; ks < n / 16; ++ks) {
      uint32_t ah[4], al[4], bb[4];
      pf_ldsm4(qa_h + ks * 32, ah);
      pf_ldsm4(qa_l + ks * 32, al);
      pf_ldsm4(kb + ks * 32, bb);
      pf_mma_bf16(s[0], ah, bb[0], bb[1]);
      pf_mma_bf16(s[1], ah, bb[2], bb[3]);
      pf_mma_bf16(s[0], al, bb[0], bb[1]);
      pf_mma_bf16(s[1], al, bb[2], bb[3]);
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[nt][e] = kt + warp * 16 + nt * 8 + 2 * t + (e & 1) < k1 ? s[nt][e] * LOG2E : -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[nt][e]);
      }
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
      mx[hr] = fmaxf(mx[hr], __shfl_xor_sync(0xFFFFFFFFu, mx[hr], 1));
      mx[hr] = fmaxf(mx[hr], __shfl_xor_sync(0xFFFFFFFFu, mx[hr], 2));
      if (t == 0) wmax[warp][g + 8 * hr] = mx[hr];
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
      const int q = g + 8 * hr;
      const float m_new = fmaxf(fmaxf(fmaxf(wmax[0][q], wmax[1][q]), fmaxf(wmax[2][q], wmax[3][q])), m_run[hr]);  // finite: the tile has a key
      alpha[hr] = exp2f(m_run[hr] - m_new);
      m_run[hr] = m_new;
      l_run[hr] *= alpha[hr];
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int hr = 0; hr < 2; ++hr) {
        const float p0 = exp2f(s[nt][2 * hr] - m_run[hr]), p1 = exp2f(s[nt][2 * hr + 1] - m_run[hr]);
        l_run[hr] += p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(Ps + (g + 8 * hr) * LM_PS + warp * 16 + nt * 8 + 2 * t) = __floats2bfloat162_rn(p0, p1);
      }
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      o[i][0] *= alpha[0]; o[i][1] *= alpha[0];
      o[i][2] *= alpha[1]; o[i][3] *= alpha[1];
    }
    __syncthreads();
    // ---- O += P C over this warp's latent columns
    const uint32_t pa_base = pf_smem(Ps + ((j & 1) * 8 + r8) * LM_PS + (j >> 1) * 8);
    const uint32_t vb = pf_smem(Ks + (size_t)((j & 1) * 8 + r8) * stride + warp * wcols + (j >> 1) * 8);
#pragma unroll
    for (int ks = 0; ks < LM_KEYS / 16; ++ks) {
      uint32_t pa[4];
      pf_ldsm4(pa_base + ks * 32, pa);
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        if (i >= ntiles) break;
        uint32_t bb[4];
        pf_ldsm4_t(vb + (uint32_t)(ks * 16 * stride + i * 8) * 2, bb);
        pf_mma_bf16(o[i], pa, bb[0], bb[1]);
        if (i + 1 < NT) pf_mma_bf16(o[i + 1 < NT ? i + 1 : i], pa, bb[2], bb[3]);
      }
    }
    if (kt + LM_KEYS < k1) {
      __syncthreads();  // every warp is done with the tile
      fetch(kt + LM_KEYS, true);
      fetch(kt + LM_KEYS, false);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
  }
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    l_run[hr] += __shfl_xor_sync(0xFFFFFFFFu, l_run[hr], 1);
    l_run[hr] += __shfl_xor_sync(0xFFFFFFFFu, l_run[hr], 2);
    if (t == 0) wsum[warp][g + 8 * hr] = l_run[hr];
  }
  __syncthreads();
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    const int q = g + 8 * hr;
    if (h0 + q >= a.h) continue;
    float* out = a.part + (((size_t)row * a.h + h0 + q) * a.nsplit + blockIdx.x) * (a.rk + 2);
    if (warp == 0 && t == 0) {
      out[a.rk] = m_run[hr] == -INFINITY ? -INFINITY : m_run[hr] * 0.6931471805599453f;
      out[a.rk + 1] = ((wsum[0][q] + wsum[1][q]) + wsum[2][q]) + wsum[3][q];
    }
    if (k0 >= k1) continue;  // an empty split: the merge skips it
#pragma unroll
    for (int i = 0; i < NT; ++i)
      if (i < ntiles) *reinterpret_cast<float2*>(out + warp * wcols + i * 8 + 2 * t) = make_float2(o[i][2 * hr], o[i][2 * hr + 1]);
  }
}

bool latent_mma_covers(const fb200_latent_args& a) {
  return !a.cache_f32 && a.rk % 32 == 0 && a.rk <= 512 && a.r % 16 == 0 && a.ldc % 8 == 0;
}
size_t latent_mma_smem(const fb200_latent_args& a) { return ((size_t)(LM_KEYS + 32) * (a.rk + a.r + 8) + 16 * LM_PS) * 2; }

template <int NT>
int launch_attn_mma(fb200_device* dev, const fb200_latent_args& a) {
  const size_t smem = latent_mma_smem(a);
  static size_t configured[64] = {0};
  if (configured[dev->ordinal & 63] < smem) {
    FB_CUDA(dev, cudaFuncSetAttribute(latent_attn_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured[dev->ordinal & 63] = smem;
  }
  return fb200_launch(dev, latent_attn_mma_kernel<NT>, dim3((unsigned)a.nsplit, (unsigned)((a.h + 15) / 16), (unsigned)(a.b * a.s)),
                      dim3(LM_THREADS), smem, true, a);
}

template <typename T>
int latent_rows(fb200_device* dev, const fb200_latent_args& a) {
  const unsigned rows = (unsigned)(a.b * a.s);
  constexpr int E = 16 / (int)sizeof(T);
  int rc;
  const int csplit = (a.rkp / E + 15) / 16;
  const size_t smem_q = (size_t)(((a.d + 3) & ~3) + LQ_THREADS * E) * 4;
  if ((rc = fb200_launch(dev, latent_query_kernel<T>, dim3((unsigned)(a.h * csplit + (a.off_dkv >= 0 ? 1 : 0)), rows), dim3(LQ_THREADS), smem_q, true,
                         a, a.h, csplit)))
    return rc;
  if (latent_mma_covers(a)) {
    rc = a.rk <= 128 ? launch_attn_mma<4>(dev, a) : a.rk <= 256 ? launch_attn_mma<8>(dev, a) : launch_attn_mma<16>(dev, a);
  } else {
    const int n = (a.ldc + 63) / 64;
    const dim3 grid((unsigned)a.nsplit, (unsigned)a.h, rows), block(LA_WARPS * 32);
    const size_t smem = (size_t)LA_WARPS * a.rk * 4;
    if (n <= 2) rc = fb200_launch(dev, latent_attn_kernel<T, 2>, grid, block, smem, true, a);
    else if (n <= 4) rc = fb200_launch(dev, latent_attn_kernel<T, 4>, grid, block, smem, true, a);
    else if (n <= 6) rc = fb200_launch(dev, latent_attn_kernel<T, 6>, grid, block, smem, true, a);
    else if (n <= 10) rc = fb200_launch(dev, latent_attn_kernel<T, 10>, grid, block, smem, true, a);
    else rc = fb200_launch(dev, latent_attn_kernel<T, 18>, grid, block, smem, true, a);
  }
  if (rc) return rc;
  return fb200_launch(dev, latent_out_kernel<T>, dim3((unsigned)a.h, rows, (unsigned)((a.v + LO_ROWS * 8 - 1) / (LO_ROWS * 8))), dim3(LO_THREADS),
                      (size_t)(a.rkp + a.nsplit) * 4, true, a);
}

}  // namespace

bool fb200_latent_covers(int d, int r, int v, int rk) {
  return d > 0 && v > 0 && rk > 0 && r >= 0 && r % 2 == 0 && d <= 4096 && rk + r <= 1144;
}

// Splits of the visible keys per head: enough CTAs for the GPU, at least 64 keys each (b h splits <= max(b h, 8 SMs)).
int fb200_latent_nsplit(const fb200_device* dev, int b, int h, int window, int cap) {
  const int keys = window && window < cap ? window : cap;
  const int ns = std::min((keys + 63) / 64, 8 * dev->sm_count / std::max(1, b * h));
  return std::max(1, std::min(ns, 32));
}

int fb200_latent_append(fb200_device* dev, const fb200_latent_args& a) {
  if (a.off_dkv < 0) return FB200_OK;
  const dim3 grid(1, (unsigned)(a.b * a.s));
  if (a.b * a.s > 65535) return fb200_fail(dev, FB200_ERR_CAPACITY, "latent attention: at most 65535 rows per pass");
  if (a.cache_f32) return fb200_launch(dev, latent_query_kernel<float>, grid, dim3(LQ_THREADS), 16, true, a, 0, 1);
  return fb200_launch(dev, latent_query_kernel<__nv_bfloat16>, grid, dim3(LQ_THREADS), 16, true, a, 0, 1);
}

int fb200_latent_rows(fb200_device* dev, const fb200_latent_args& a) {
  if (a.b * a.s > 65535) return fb200_fail(dev, FB200_ERR_CAPACITY, "latent attention: at most 65535 rows per pass without the tensor-core path");
  return a.cache_f32 ? latent_rows<float>(dev, a) : latent_rows<__nv_bfloat16>(dev, a);
}
