// Grouped softmax attention, row by row: per-head norms, rotary positions, softcap, sliding window, sinks, head gates.
//
//  * attn_prep_kernel (prompts): a warp per head of a row normalises and rotates it; queries go to a scratch buffer, keys
//    and values into the cache.
//  * attn_rows_kernel: one CTA per (split of the visible keys, up to NQ query heads of one key/value head, row). A
//    group of LPK lanes reads a cached key and value in 16-byte pieces and serves all NQ heads with them; every group keeps a running
//    softmax of its own, merged at the end over lanes, warps and (by the CTA that arrives last) splits. f32 arithmetic,
//    bf16 or f32 cache. A step of one position per sequence prepares its heads here too: one kernel. Bound: HBM on the
//    cache. Prompts run it for F32 models, short passes and head sizes above those of the tensor-core kernel (latent_prefill.cu).
#include <algorithm>

#include "mixers.cuh"
#include "qgemv_common.cuh"

namespace {

constexpr int GA_WARPS = 4, GA_THREADS = GA_WARPS * 32, GA_MIN_KEYS = 32, GA_MAX_SPLITS = 32;

__device__ __forceinline__ float ga_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
__device__ __forceinline__ void ga_unpack(const uint4& u, float (&f)[8], __nv_bfloat16) {
  f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xFFFF0000u);
  f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xFFFF0000u);
  f[4] = __uint_as_float(u.z << 16); f[5] = __uint_as_float(u.z & 0xFFFF0000u);
  f[6] = __uint_as_float(u.w << 16); f[7] = __uint_as_float(u.w & 0xFFFF0000u);
}
__device__ __forceinline__ void ga_unpack(const uint4& u, float (&f)[4], float) {
  f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
}
__device__ __forceinline__ void ga_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void ga_store(float* p, float v) { *p = v; }

// exponentials and tanh in the precision of the cache: the bf16 form of tanh(z) is 1 - 2 / (1 + exp(2 z))
__device__ __forceinline__ float ga_exp(float x, __nv_bfloat16) { return __expf(x); }
__device__ __forceinline__ float ga_exp(float x, float) { return expf(x); }
__device__ __forceinline__ float ga_tanh(float z, __nv_bfloat16) { return 1.0f - __fdividef(2.0f, 1.0f + __expf(fminf(2.0f * z, 80.0f))); }
__device__ __forceinline__ float ga_tanh(float z, float) { return tanhf(z); }

// A warp writes one head of n elements: normalised under w (null: not), its first r dimensions rotated (cs, sn: this
// position's row of the tables), x mul; zeros up to np. `raw`: shared memory for the head, or null where x is read again.
template <typename T>
__device__ __forceinline__ void ga_head(const float* x, int n, int np, const float* w, float eps, const float* cs, const float* sn, int r,
                                        float mul, T* dst, float* raw = nullptr) {
  const int lane = threadIdx.x & 31, half = r >> 1;
  float rms = 1.f;
  if (w || raw) {
    float ss = 0.f;
#pragma unroll 4
    for (int i = lane; i < n; i += 32) {
      const float v = x[i];
      ss = fmaf(v, v, ss);
      if (raw) raw[i] = v;
    }
    if (w) rms = 1.0f / sqrtf(ga_warp_sum(ss) / (float)n + eps);
    if (raw) {
      __syncwarp();
      x = raw;
    }
  }
  auto value = [&](int i) { return w ? (x[i] * rms) * w[i] : x[i]; };
  for (int i = lane; i < half; i += 32) {
    const float u = value(i), v = value(i + half);
    ga_store(dst + i, (u * cs[i] - v * sn[i]) * mul);
    ga_store(dst + half + i, (v * cs[i] + u * sn[i]) * mul);
  }
  for (int i = r + lane; i < np; i += 32) ga_store(dst + i, i < n ? value(i) * mul : 0.f);
}

__device__ __forceinline__ void ga_store2(__nv_bfloat16* p, float x, float y) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x, y); }
__device__ __forceinline__ void ga_store2(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }

// ga_head for n and r multiples of 4, rows and heads 8-byte aligned: two elements per access, read once. J: pairs per lane.
template <int J, typename T>
__device__ __forceinline__ void ga_head_pairs(const float* x, int n, int np, const float* w, float eps, const float* cs, const float* sn, int r, T* dst) {
  const int lane = threadIdx.x & 31, hp = r >> 2, rp = r >> 1, pairs = n >> 1;  // pairs of the half, of the rotated part, of the head
  const float2 *x2 = reinterpret_cast<const float2*>(x), *w2 = reinterpret_cast<const float2*>(w);
  // lane's pair j: the first half of the rotated part (its partner hp pairs behind), then what does not rotate
  float2 u[J], v[J];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int i = lane + 32 * j, at = i < hp ? i : i + hp;
    u[j] = at < pairs ? x2[at] : make_float2(0.f, 0.f);
    v[j] = i < hp ? x2[i + hp] : make_float2(0.f, 0.f);
    ss = fmaf(u[j].x, u[j].x, fmaf(u[j].y, u[j].y, fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, ss))));
  }
  const float inv = w ? 1.0f / sqrtf(ga_warp_sum(ss) / (float)n + eps) : 1.f;
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int i = lane + 32 * j, at = i < hp ? i : i + hp;
    if (at >= (np >> 1)) continue;
    if (w && at < pairs) {
      const float2 f = w2[at];
      u[j] = make_float2(u[j].x * inv * f.x, u[j].y * inv * f.y);
    }
    if (i < hp) {
      if (w) {
        const float2 f = w2[i + hp];
        v[j] = make_float2(v[j].x * inv * f.x, v[j].y * inv * f.y);
      }
      const float2 c = reinterpret_cast<const float2*>(cs)[i], s = reinterpret_cast<const float2*>(sn)[i];
      ga_store2(dst + 2 * i, u[j].x * c.x - v[j].x * s.x, u[j].y * c.y - v[j].y * s.y);
      ga_store2(dst + 2 * i + rp, v[j].x * c.x + u[j].x * s.x, v[j].y * c.y + u[j].y * s.y);
    } else {
      ga_store2(dst + 2 * at, u[j].x, u[j].y);
    }
  }
}

template <typename T, typename QT>
__global__ void __launch_bounds__(256) attn_prep_kernel(const fb200_attn_args a) {
  const int slots = a.h + 2 * a.g;
  const uint32_t id = blockIdx.x * 8 + (threadIdx.x >> 5), total = (uint32_t)(a.b * a.s) * slots;
  pdl_wait();
  pdl_launch_dependents();
  if (id >= total) return;
  const uint32_t row = id / slots;
  const int slot = (int)(id % slots), b = (int)(row / a.s), pos = *a.pos_dev + (int)(row % a.s), half = a.r >> 1;
  const float* y = a.y + (size_t)row * a.ldy;
  const float *cs = a.rope_cos + (size_t)pos * half, *sn = a.rope_sin + (size_t)pos * half;
  T* cache = reinterpret_cast<T*>(a.cache) + ((size_t)b * a.cap + pos) * a.ldc;
  const bool pairs = ((a.d | a.v | a.r | a.off_k | a.off_v | (int)a.ldy) & 3) == 0 && a.d <= 256 && a.v <= 256 &&
                     (reinterpret_cast<uintptr_t>(a.y) & 7u) == 0;
  if (pairs) {  // heads are multiples of 4: the padding to dp and vp is at most two pairs
    const bool is_v = slot >= a.h + a.g;
    const int k = is_v ? slot - a.h - a.g : slot - a.h, n = is_v ? a.v : a.d;
    const float* x = slot < a.h ? y + (size_t)slot * a.d : is_v ? y + a.off_v + (size_t)k * a.v : y + a.off_k + (size_t)k * a.d;
    const float* w = slot < a.h ? a.q_norm : is_v ? nullptr : a.k_norm;
    const int r = is_v ? 0 : a.r;
    if (slot < a.h) {
      QT* dst = reinterpret_cast<QT*>(a.qn) + ((size_t)row * a.h + slot) * a.dp;
      if (n <= 128) ga_head_pairs<2>(x, n, a.dp, w, a.eps, cs, sn, r, dst);
      else ga_head_pairs<4>(x, n, a.dp, w, a.eps, cs, sn, r, dst);
    } else {
      T* dst = cache + (is_v ? a.g * a.dp + k * a.vp : k * a.dp);
      if (n <= 128) ga_head_pairs<2>(x, n, is_v ? a.vp : a.dp, w, a.eps, cs, sn, r, dst);
      else ga_head_pairs<4>(x, n, is_v ? a.vp : a.dp, w, a.eps, cs, sn, r, dst);
    }
  } else if (slot < a.h) {
    ga_head(y + (size_t)slot * a.d, a.d, a.dp, a.q_norm, a.eps, cs, sn, a.r, 1.f, reinterpret_cast<QT*>(a.qn) + ((size_t)row * a.h + slot) * a.dp);
  } else if (slot < a.h + a.g) {
    const int k = slot - a.h;
    ga_head(y + a.off_k + (size_t)k * a.d, a.d, a.dp, a.k_norm, a.eps, cs, sn, a.r, 1.f, cache + k * a.dp);
  } else {
    const int k = slot - a.h - a.g;
    ga_head(y + a.off_v + (size_t)k * a.v, a.v, a.vp, nullptr, 0.f, cs, sn, 0, 1.f, cache + a.g * a.dp + k * a.vp);
  }
}

// T: element type of the cache; a piece is 16 bytes, E elements; LPK lanes take NP pieces each of a key and of a value.
template <typename T, int NP, int NQ>
__global__ void __launch_bounds__(GA_THREADS) attn_rows_kernel(const fb200_attn_args a, int nsplit) {
  constexpr int E = 16 / (int)sizeof(T), LPK = 64 / E, KS = 32 / LPK, U = 2;  // U: keys per lane group in flight
  constexpr int STEP = GA_WARPS * KS * U, SETS = GA_WARPS * KS, COLS = 64 * NP;  // SETS: lane groups of the CTA
  // queries [NQ][COLS], later outputs [SETS][NQ][COLS]; in a step of one position also raw heads [GA_WARPS][max(dp, vp)], q_norm,
  // k_norm [dp], cos, sin [r / 2]
  extern __shared__ __align__(16) float gsm[];
  __shared__ float wm[SETS][NQ], wl[SETS][NQ], wt[NQ][32], top[NQ], tot[NQ];
  __shared__ int last;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, slot = lane / LPK, p = lane % LPK;
  const int split = (int)(blockIdx.x % nsplit), gq = a.h / a.g, hgroups = (gq + NQ - 1) / NQ, kvh = blockIdx.y / hgroups;
  const size_t row = blockIdx.x / nsplit;
  const int b = (int)(row / a.s), h0 = kvh * gq + ((int)blockIdx.y % hgroups) * NQ, nq = min(NQ, (kvh + 1) * gq - h0);
  const int pos = *a.pos_dev + (int)(row % a.s);
  const int lo = a.window ? max(0, pos - a.window + 1) : 0, keys = pos + 1 - lo;
  const int per = max(GA_MIN_KEYS, (keys + nsplit - 1) / nsplit), active = (keys + per - 1) / per;
  if (split >= active) return;
  const int k0 = lo + split * per, k1 = min(pos + 1, k0 + per);
  T* cache = reinterpret_cast<T*>(a.cache) + (size_t)b * a.cap * a.ldc;
  const T *kc = cache + kvh * a.dp, *vc = cache + a.g * a.dp + kvh * a.vp;
  uint4 kr[U][NP], vr[U][NP];
  auto fetch = [&](int key, int u) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int at = (i * LPK + p) * E;
      kr[u][i] = at < a.dp ? *reinterpret_cast<const uint4*>(kc + (size_t)key * a.ldc + at) : make_uint4(0u, 0u, 0u, 0u);
      vr[u][i] = at < a.vp ? *reinterpret_cast<const uint4*>(vc + (size_t)key * a.ldc + at) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  const int first = k0 + warp * KS * U;  // this warp's first keys
  const int half = a.r >> 1;
  const float inv_cap = a.softcap > 0.f ? 1.0f / a.softcap : 0.f;
  float* raw = gsm + SETS * NQ * COLS;
  float *qw = raw + GA_WARPS * max(a.dp, a.vp), *kw = qw + a.dp, *cs = kw + a.dp, *sn = cs + half;
  if (a.s == 1) {
    // cached rows, norms and rotation do not depend on the kernel in front: requested ahead of it
    if (first < k1)
#pragma unroll
      for (int u = 0; u < U; ++u) fetch(min(first + u * KS + slot, k1 - 1), u);
    for (int i = tid; i < a.d; i += GA_THREADS) {
      if (a.q_norm) qw[i] = a.q_norm[i];
      if (a.k_norm) kw[i] = a.k_norm[i];
    }
    for (int i = tid; i < half; i += GA_THREADS) {
      cs[i] = a.rope_cos[(size_t)pos * half + i];
      sn[i] = a.rope_sin[(size_t)pos * half + i];
    }
    __syncthreads();
  }
  pdl_wait();
  pdl_launch_dependents();
  if (a.s == 1) {  // this position's queries, and its key and value where this split holds it
    const float* y = a.y + row * a.ldy;
    float* mine = raw + warp * max(a.dp, a.vp);
    for (int job = warp; job < nq + (k1 == pos + 1 ? 2 : 0); job += GA_WARPS) {
      T* dst = cache + (size_t)pos * a.ldc;
      if (job < nq) ga_head(y + (size_t)(h0 + job) * a.d, a.d, a.dp, a.q_norm ? qw : nullptr, a.eps, cs, sn, a.r, a.scale, gsm + job * COLS, mine);
      else if (job == nq) ga_head(y + a.off_k + (size_t)kvh * a.d, a.d, a.dp, a.k_norm ? kw : nullptr, a.eps, cs, sn, a.r, 1.f, dst + kvh * a.dp, mine);
      else ga_head(y + a.off_v + (size_t)kvh * a.v, a.v, a.vp, nullptr, 0.f, cs, sn, 0, 1.f, dst + a.g * a.dp + kvh * a.vp);
    }
  } else {
    const float* q = reinterpret_cast<const float*>(a.qn) + (row * a.h + h0) * a.dp;
    for (int i = tid; i < nq * a.dp; i += GA_THREADS) gsm[i / a.dp * COLS + i % a.dp] = q[i] * a.scale;
  }
  for (int i = tid; i < NQ * COLS; i += GA_THREADS)
    if (i / COLS >= nq || i % COLS >= a.dp) gsm[i] = 0.f;
  __syncthreads();
  float q[NQ][NP * E], acc[NQ][NP * E], m[NQ], l[NQ];
#pragma unroll
  for (int n = 0; n < NQ; ++n) {
    m[n] = -INFINITY;
    l[n] = 0.f;
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
      for (int e = 0; e < E; e += 4) {
        *reinterpret_cast<float4*>(&q[n][i * E + e]) = *reinterpret_cast<const float4*>(gsm + n * COLS + (i * LPK + p) * E + e);
        *reinterpret_cast<float4*>(&acc[n][i * E + e]) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
  }
  __syncthreads();  // the outputs take the queries' place
  for (int kt = first; kt < k1; kt += STEP) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int key = min(kt + u * KS + slot, k1 - 1);
      if (a.s > 1 || kt != first || key == pos) fetch(key, u);  // (the new position was written after the first request)
    }
    float s[U][NQ];
#pragma unroll
    for (int u = 0; u < U; ++u) {
#pragma unroll
      for (int n = 0; n < NQ; ++n) s[u][n] = 0.f;
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        float f[E];
        ga_unpack(kr[u][i], f, T());
#pragma unroll
        for (int n = 0; n < NQ; ++n)
#pragma unroll
          for (int e = 0; e < E; ++e) s[u][n] = fmaf(f[e], q[n][i * E + e], s[u][n]);
      }
#pragma unroll
      for (int n = 0; n < NQ; ++n) {
#pragma unroll
        for (int o = LPK / 2; o > 0; o >>= 1) s[u][n] += __shfl_xor_sync(0xFFFFFFFFu, s[u][n], o);
        if (a.softcap > 0.f) s[u][n] = a.softcap * ga_tanh(s[u][n] * inv_cap, T());
        if (kt + u * KS + slot >= k1) s[u][n] = -INFINITY;
      }
    }
    float pr[U][NQ];
#pragma unroll
    for (int n = 0; n < NQ; ++n) {
      float mx = m[n];
#pragma unroll
      for (int u = 0; u < U; ++u) mx = fmaxf(mx, s[u][n]);
      const float base = mx == -INFINITY ? 0.f : mx, alpha = ga_exp(m[n] - base, T());
      m[n] = mx;
      l[n] *= alpha;
#pragma unroll
      for (int i = 0; i < NP * E; ++i) acc[n][i] *= alpha;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        pr[u][n] = ga_exp(s[u][n] - base, T());
        l[n] += pr[u][n];
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        float f[E];
        ga_unpack(vr[u][i], f, T());
#pragma unroll
        for (int n = 0; n < NQ; ++n)
#pragma unroll
          for (int e = 0; e < E; ++e) acc[n][i * E + e] = fmaf(pr[u][n], f[e], acc[n][i * E + e]);
      }
  }
  // ---- the lane groups' outputs meet in shared memory
  const int set = warp * KS + slot;
#pragma unroll
  for (int n = 0; n < NQ; ++n) {
    if (p == 0) { wm[set][n] = m[n]; wl[set][n] = l[n]; }
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
      for (int e = 0; e < E; e += 4)
        *reinterpret_cast<float4*>(gsm + (set * NQ + n) * COLS + (i * LPK + p) * E + e) = *reinterpret_cast<const float4*>(&acc[n][i * E + e]);
  }
  __syncthreads();
  if (warp < NQ) {
    const float ms = lane < SETS ? wm[lane % SETS][warp] : -INFINITY;
    float mx = ms;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, o));
    const float w = ms == -INFINITY ? 0.f : ga_exp(ms - mx, T());
    const float lt = ga_warp_sum(w != 0.f ? wl[lane % SETS][warp] * w : 0.f);
    wt[warp][lane] = w;
    if (lane == 0) { top[warp] = mx; tot[warp] = lt; }
  }
  __syncthreads();
  const float* y = a.y + row * a.ldy;
  auto put = [&](int n, int c, float v) {  // v: the output with weights of sum 1
    if (a.off_g >= 0) v *= 1.0f / (1.0f + expf(-y[a.off_g + h0 + n]));
    v *= a.out_scale;
    const size_t zi = row * a.ldz + (size_t)(h0 + n) * a.v + c;
    if (a.z_bf16) reinterpret_cast<__nv_bfloat16*>(a.z)[zi] = __float2bfloat16(v);
    else reinterpret_cast<float*>(a.z)[zi] = v;
  };
  float* part = a.part + ((row * a.h + h0) * (size_t)nsplit) * (a.v + 2);  // [head][split][v + 2]
  for (int i = tid; i < nq * a.v; i += GA_THREADS) {
    const int n = i / a.v, c = i % a.v;
    const float mx = top[n];
    float v = 0.f, lt = tot[n];
#pragma unroll 4
    for (int j = 0; j < SETS; ++j) v = fmaf(gsm[(j * NQ + n) * COLS + c], wt[n][j], v);
    if (active == 1) {
      if (a.sink) lt += expf(a.sink[h0 + n] - mx);
      put(n, c, v / lt);
    } else {
      float* out = part + ((size_t)n * nsplit + split) * (a.v + 2);
      out[c] = v;
      if (c == 0) { out[a.v] = mx; out[a.v + 1] = lt; }
    }
  }
  if (active == 1) return;
  // ---- the last split of these heads merges all of them
  __threadfence();
  __syncthreads();
  int* done = a.done + row * gridDim.y + blockIdx.y;
  if (tid == 0) last = atomicAdd(done, 1) == active - 1;
  __syncthreads();
  if (!last) return;
  __threadfence();
  if (tid == 0) *done = 0;
  for (int n = warp; n < nq; n += GA_WARPS) {
    const float* src = part + ((size_t)n * nsplit + lane) * (a.v + 2) + a.v;
    const float ms = lane < active ? __ldcg(src) : -INFINITY, ls = lane < active ? __ldcg(src + 1) : 0.f;
    float mx = ms;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, o));
    const float w = lane < active ? expf(ms - mx) : 0.f;
    float lt = ga_warp_sum(ls * w);
    wt[n][lane] = w;
    if (lane == 0) tot[n] = a.sink ? lt + expf(a.sink[h0 + n] - mx) : lt;
  }
  __syncthreads();
  for (int i = tid; i < nq * a.v; i += GA_THREADS) {
    const int n = i / a.v, c = i % a.v;
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < active; ++s) v = fmaf(__ldcg(part + ((size_t)n * nsplit + s) * (a.v + 2) + c), wt[n][s], v);
    put(n, c, v / tot[n]);
  }
}

// query heads per CTA: as many as the registers hold, no more than a group has
int ga_heads(int np, int gq) { return std::min(np <= 2 ? 4 : np <= 4 ? 2 : 1, gq >= 3 ? 4 : gq); }

template <typename T, int NP, int NQ>
int launch_rows(fb200_device* dev, const fb200_attn_args& a) {
  const int gq = a.h / a.g, gy = a.g * ((gq + NQ - 1) / NQ);
  const size_t rows = (size_t)a.b * a.s;
  const int keys = a.window && a.window < a.cap ? a.window : a.cap;
  // enough CTAs for two per SM; fb200_attn_part_floats counts on rows gy nsplit <= 2 SMs where nsplit > 1
  int ns = (int)std::min<size_t>(GA_MAX_SPLITS, 2 * (size_t)dev->sm_count / (rows * gy));
  ns = std::max(1, std::min(ns, (keys + GA_MIN_KEYS - 1) / GA_MIN_KEYS));
  constexpr int SETS = GA_WARPS * 32 * 16 / (int)sizeof(T) / 64;
  const size_t smem = ((size_t)SETS * NQ * 64 * NP + (a.s == 1 ? GA_WARPS * std::max(a.dp, a.vp) + 2 * a.dp + a.r : 0)) * 4;
  return fb200_launch(dev, attn_rows_kernel<T, NP, NQ>, dim3((unsigned)(rows * ns), (unsigned)gy), dim3(GA_THREADS), smem, true, a, ns);
}

template <typename T>
int attn_rows(fb200_device* dev, const fb200_attn_args& a) {
  int rc;
  if (a.s > 1 && (rc = fb200_attn_prepare(dev, a, false))) return rc;
  const int n = (std::max(a.dp, a.vp) + 63) / 64, np = n <= 1 ? 1 : n <= 2 ? 2 : n <= 4 ? 4 : 8, nq = ga_heads(np, a.h / a.g);
  switch (np * 8 + nq) {
    case 9: return launch_rows<T, 1, 1>(dev, a);
    case 10: return launch_rows<T, 1, 2>(dev, a);
    case 12: return launch_rows<T, 1, 4>(dev, a);
    case 17: return launch_rows<T, 2, 1>(dev, a);
    case 18: return launch_rows<T, 2, 2>(dev, a);
    case 20: return launch_rows<T, 2, 4>(dev, a);
    case 33: return launch_rows<T, 4, 1>(dev, a);
    case 34: return launch_rows<T, 4, 2>(dev, a);
    default: return launch_rows<T, 8, 1>(dev, a);
  }
}

}  // namespace

bool fb200_attn_covers(int d, int v) { return d > 0 && v > 0 && d <= 512 && v <= 512; }

size_t fb200_attn_part_floats(const fb200_device* dev, int v) { return (size_t)2 * dev->sm_count * 4 * (v + 2); }

int fb200_attn_prepare(fb200_device* dev, const fb200_attn_args& a, bool q_bf16) {
  const size_t warps = (size_t)a.b * a.s * (a.h + 2 * a.g);
  if (warps >= (1ull << 32)) return fb200_fail(dev, FB200_ERR_CAPACITY, "grouped attention: %d x %d rows of %d heads in one pass", a.b, a.s, a.h);
  const dim3 grid((unsigned)((warps + 7) / 8)), block(256);
  if (a.cache_f32) return fb200_launch(dev, attn_prep_kernel<float, float>, grid, block, 0, true, a);
  if (q_bf16) return fb200_launch(dev, attn_prep_kernel<__nv_bfloat16, __nv_bfloat16>, grid, block, 0, true, a);
  return fb200_launch(dev, attn_prep_kernel<__nv_bfloat16, float>, grid, block, 0, true, a);
}

int fb200_attn_rows(fb200_device* dev, const fb200_attn_args& a) {
  return a.cache_f32 ? attn_rows<float>(dev, a) : attn_rows<__nv_bfloat16>(dev, a);
}
