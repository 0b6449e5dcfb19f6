// Gated delta rule: short convolution, unit q / k, the recurrence and its gated, normalised read-out.
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// per head, with S [d, v] in 32-bit floats. The columns of S are independent, so a column (or a few) is
// what a group of lanes owns for the whole sequence: it stays in registers, k and q of a token come from shared
// memory, and both sums over d are formed in one pass from the state BEFORE the token,
//   S^T k -> g (S^T k),   o = g (S^T q) + u (k . q),
// which leaves one reduction over the lanes per token. Everything is f32, and a token is always processed the
// same way, so a sequence gives the same state however it is cut.
//
//  * delta_step_kernel: one new token per sequence. One CTA per (head, sequence): convolution, unit vectors,
//    decay, state update, read-out, RMSNorm and gate. Bound: HBM on the state (read and written once).
//  * prompts: delta_prep_kernel (convolution, SiLU, unit vectors, decay and write strength), delta_scan_kernel (the
//    recurrence; bound: f32 FMA issue, packed two-wide), delta_out_kernel (RMSNorm, gate) and
//    conv_ring_kernel (the convolution's memory).
#include "mixers.cuh"
#include "qgemv_common.cuh"

namespace {

constexpr float UNIT_EPS = 1e-6f;  // inside the root of the unit vectors

__device__ __forceinline__ float dr_silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float dr_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float dr_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float dr_decay(float a_log, float a, float dt) { return expf(-expf(a_log) * dr_softplus(a + dt)); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
// two f32 operations per instruction
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(reinterpret_cast<unsigned long long&>(r))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)),
        "l"(reinterpret_cast<unsigned long long&>(c)));
  return r;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 r;
  asm("mul.rn.f32x2 %0, %1, %2;"
      : "=l"(reinterpret_cast<unsigned long long&>(r))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)));
  return r;
}

// input of convolution channel c at position pos + t of sequence b (t < 0: earlier than this pass)
__device__ __forceinline__ float conv_in(const fb200_delta_args& a, int b, int c, int t, int pos) {
  if (t >= 0) return a.y[((size_t)b * a.s + t) * a.ldy + c];
  const int p = pos + t;
  if (p < 0) return 0.f;
  return a.ring[((size_t)b * a.taps + p % a.taps) * a.channels + c];
}
__device__ __forceinline__ float conv_silu(const fb200_delta_args& a, int b, int c, int t, int pos) {
  const float* w = a.conv_w + (size_t)c * a.taps;
  float acc = 0.f;
  for (int j = 0; j < a.taps; ++j) acc = fmaf(w[j], conv_in(a, b, c, t - (a.taps - 1) + j, pos), acc);
  return dr_silu(acc);
}

// A column's d elements lie over LPC lanes, EPT per lane: element 4 (i LPC + p) + j is float j of piece i of lane p.
template <int EPT, int LPC>
__device__ __forceinline__ void load_column(const float* col, int p, float2 (&s)[EPT / 2]) {
#pragma unroll
  for (int i = 0; i < EPT / 4; ++i) {
    const float4 v = *reinterpret_cast<const float4*>(col + 4 * (i * LPC + p));
    s[2 * i] = make_float2(v.x, v.y);
    s[2 * i + 1] = make_float2(v.z, v.w);
  }
}
template <int EPT, int LPC>
__device__ __forceinline__ void store_column(float* col, int p, const float2 (&s)[EPT / 2]) {
#pragma unroll
  for (int i = 0; i < EPT / 4; ++i)
    *reinterpret_cast<float4*>(col + 4 * (i * LPC + p)) = make_float4(s[2 * i].x, s[2 * i].y, s[2 * i + 1].x, s[2 * i + 1].y);
}
// sums of S k and S q over this lane's elements
template <int EPT, int LPC>
__device__ __forceinline__ void column_dots(const float2 (&s)[EPT / 2], const float* ks, const float* qs, int p, float& dk, float& dq) {
  float2 k0 = make_float2(0.f, 0.f), k1 = k0, q0 = k0, q1 = k0;
#pragma unroll
  for (int i = 0; i < EPT / 4; ++i) {
    const float4 k = *reinterpret_cast<const float4*>(ks + 4 * (i * LPC + p));
    const float4 q = *reinterpret_cast<const float4*>(qs + 4 * (i * LPC + p));
    k0 = fma2(s[2 * i], make_float2(k.x, k.y), k0);
    k1 = fma2(s[2 * i + 1], make_float2(k.z, k.w), k1);
    q0 = fma2(s[2 * i], make_float2(q.x, q.y), q0);
    q1 = fma2(s[2 * i + 1], make_float2(q.z, q.w), q1);
  }
  dk = (k0.x + k0.y) + (k1.x + k1.y);
  dq = (q0.x + q0.y) + (q1.x + q1.y);
#pragma unroll
  for (int o = LPC / 2; o > 0; o >>= 1) {
    dk += __shfl_xor_sync(0xFFFFFFFFu, dk, o);
    dq += __shfl_xor_sync(0xFFFFFFFFu, dq, o);
  }
}
// S <- g S + k u
template <int EPT, int LPC>
__device__ __forceinline__ void column_update(float2 (&s)[EPT / 2], const float* ks, int p, float g, float u) {
  const float2 g2 = make_float2(g, g), u2 = make_float2(u, u);
#pragma unroll
  for (int i = 0; i < EPT / 4; ++i) {
    const float4 k = *reinterpret_cast<const float4*>(ks + 4 * (i * LPC + p));
    s[2 * i] = fma2(make_float2(k.x, k.y), u2, mul2(s[2 * i], g2));
    s[2 * i + 1] = fma2(make_float2(k.z, k.w), u2, mul2(s[2 * i + 1], g2));
  }
}

// ---- one new token -------------------------------------------------------------------------------------
constexpr int ST_MAX_THREADS = 512;

template <int EPT, int LPC>
__global__ void __launch_bounds__(ST_MAX_THREADS) delta_step_kernel(const fb200_delta_args a) {
  extern __shared__ __align__(16) float dsm[];  // k, q [dp] (silu of the convolution), read-out [v]
  __shared__ float red[3 * 16], gbs[2];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x, nw = nt >> 5;
  float *ks = dsm, *qs = dsm + a.dp, *os = dsm + 2 * a.dp;
  const int group = a.h / a.hk, hk = h / group;
  const int pos = *a.pos_dev;
  const int p = tid % LPC, cols = nt / LPC, c0 = tid / LPC;
  float* st = a.state + ((size_t)b * a.h + h) * (size_t)a.v * a.dp;
  // the state was written by an earlier step: its loads do not wait for this step's projections
  float2 s[EPT / 2];
  const bool has0 = c0 < a.v && pos > 0;
  if (has0) load_column<EPT, LPC>(st + (size_t)c0 * a.dp, p, s);
  pdl_launch_dependents();
  pdl_wait();
  const float* yr = a.y + (size_t)b * a.ldy;
  float skk = 0.f, sqq = 0.f, skq = 0.f;
  for (int i = tid; i < a.dp; i += nt) {
    float k = 0.f, q = 0.f;
    if (i < a.d) {
      q = conv_silu(a, b, hk * a.d + i, 0, pos);
      k = conv_silu(a, b, (a.hk + hk) * a.d + i, 0, pos);
    }
    ks[i] = k;
    qs[i] = q;
    skk = fmaf(k, k, skk);
    sqq = fmaf(q, q, sqq);
    skq = fmaf(k, q, skq);
  }
  skk = warp_sum(skk);
  sqq = warp_sum(sqq);
  skq = warp_sum(skq);
  if (lane == 0) { red[warp] = skk; red[16 + warp] = sqq; red[32 + warp] = skq; }
  if (tid == 0) {
    gbs[0] = dr_decay(a.a_log[h], yr[a.off_a + h], a.dt_bias[h]);
    gbs[1] = dr_sigmoid(yr[a.off_b + h]);
  }
  __syncthreads();
  skk = sqq = skq = 0.f;
  for (int i = 0; i < nw; ++i) { skk += red[i]; sqq += red[16 + i]; skq += red[32 + i]; }
  const float ik = 1.0f / sqrtf(skk + UNIT_EPS), iq = (1.0f / sqrtf(sqq + UNIT_EPS)) / sqrtf((float)a.d);
  const float g = gbs[0], beta = gbs[1], kq = skq * ik * iq;
  float ss = 0.f;
  const int rounds = (a.v + cols - 1) / cols;
  for (int it = 0; it < rounds; ++it) {
    const int c = c0 + it * cols;
    const bool in = c < a.v;
    if (!(it == 0 && has0)) {
      if (in && pos > 0) {
        load_column<EPT, LPC>(st + (size_t)c * a.dp, p, s);
      } else {
#pragma unroll
        for (int i = 0; i < EPT / 2; ++i) s[i] = make_float2(0.f, 0.f);
      }
    }
    const float v = in ? conv_silu(a, b, a.off_v + h * a.v + c, 0, pos) : 0.f;
    float dk, dq;
    column_dots<EPT, LPC>(s, ks, qs, p, dk, dq);
    const float u = beta * (v - g * (dk * ik));
    const float o = fmaf(g, dq * iq, u * kq);
    if (in) {
      if (a.commit) {
        column_update<EPT, LPC>(s, ks, p, g, u * ik);
        store_column<EPT, LPC>(st + (size_t)c * a.dp, p, s);
      }
      if (p == 0) {
        os[c] = o;
        ss = fmaf(o, o, ss);
      }
    }
  }
  ss = warp_sum(ss);
  __syncthreads();
  if (lane == 0) red[warp] = ss;
  // this token's convolution inputs, into the slot that no convolution of this step reads
  float* ring = a.ring + ((size_t)b * a.taps + pos % a.taps) * a.channels;
  if (h % group == 0)
    for (int i = tid; i < a.d; i += nt) {
      ring[hk * a.d + i] = yr[hk * a.d + i];
      ring[(a.hk + hk) * a.d + i] = yr[(a.hk + hk) * a.d + i];
    }
  for (int i = tid; i < a.v; i += nt) ring[a.off_v + h * a.v + i] = yr[a.off_v + h * a.v + i];
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < nw; ++i) ss += red[i];
  const float rms = sqrtf(ss / (float)a.v + a.eps);
  for (int i = tid; i < a.v; i += nt) {
    const float val = (os[i] / rms) * a.out_norm[i] * dr_silu(yr[a.off_g + h * a.v + i]);
    const size_t zi = (size_t)b * a.ldz + h * a.v + i;
    if (a.z_bf16) reinterpret_cast<__nv_bfloat16*>(a.z)[zi] = __float2bfloat16(val);
    else reinterpret_cast<float*>(a.z)[zi] = val;
  }
}

// ---- prompts ---------------------------------------------------------------------------------------------
constexpr int PREP_T = 16, PREP_WARPS = 4, PREP_VCH = 128;

// A warp per (unit, 16 tokens): units 0 .. hk are the q and k vectors of a q/k head, then blocks of 128 v channels, then
// the decays and write strengths of all heads. NE = channels of a q/k head per lane.
template <int NE>
__global__ void __launch_bounds__(PREP_WARPS * 32) delta_prep_kernel(const fb200_delta_args a) {
  const int lane = threadIdx.x & 31, b = blockIdx.z, t0 = blockIdx.x * PREP_T, t1 = min(a.s, t0 + PREP_T);
  const int hv = a.h * a.v, vblocks = (hv + PREP_VCH - 1) / PREP_VCH;
  int unit = blockIdx.y * PREP_WARPS + (threadIdx.x >> 5);
  const int pos = *a.pos_dev;
  if (unit < a.hk) {
    const float qscale = 1.0f / sqrtf((float)a.d);
    for (int t = t0; t < t1; ++t) {
      float q[NE], k[NE], skk = 0.f, sqq = 0.f, skq = 0.f;
#pragma unroll
      for (int i = 0; i < NE; ++i) {
        const int c = lane + 32 * i;
        q[i] = k[i] = 0.f;
        if (c < a.d) {
          q[i] = conv_silu(a, b, unit * a.d + c, t, pos);
          k[i] = conv_silu(a, b, (a.hk + unit) * a.d + c, t, pos);
        }
        skk = fmaf(k[i], k[i], skk);
        sqq = fmaf(q[i], q[i], sqq);
        skq = fmaf(k[i], q[i], skq);
      }
      skk = warp_sum(skk);
      sqq = warp_sum(sqq);
      skq = warp_sum(skq);
      const float ik = 1.0f / sqrtf(skk + UNIT_EPS), iq = (1.0f / sqrtf(sqq + UNIT_EPS)) * qscale;
      const size_t row = ((size_t)b * a.s + t) * a.hk + unit;
#pragma unroll
      for (int i = 0; i < NE; ++i) {
        const int c = lane + 32 * i;
        if (c < a.dp) {
          a.qn[row * a.dp + c] = q[i] * iq;
          a.kn[row * a.dp + c] = k[i] * ik;
        }
      }
      if (lane == 0) a.kq[row] = skq * ik * iq;
    }
    return;
  }
  unit -= a.hk;
  if (unit < vblocks) {
    for (int t = t0; t < t1; ++t)
#pragma unroll
      for (int i = 0; i < PREP_VCH / 32; ++i) {
        const int c = unit * PREP_VCH + lane + 32 * i;
        if (c < hv) a.vn[((size_t)b * a.s + t) * hv + c] = conv_silu(a, b, a.off_v + c, t, pos);
      }
    return;
  }
  if (unit > vblocks) return;
  for (int i = lane; i < (t1 - t0) * a.h; i += 32) {
    const int t = t0 + i / a.h, h = i % a.h;
    const size_t row = (size_t)b * a.s + t;
    const float* yr = a.y + row * a.ldy;
    a.gb[(row * a.h + h) * 2] = dr_decay(a.a_log[h], yr[a.off_a + h], a.dt_bias[h]);
    a.gb[(row * a.h + h) * 2 + 1] = dr_sigmoid(yr[a.off_b + h]);
  }
}

constexpr int SC_WARPS = 4;

template <int EPT, int LPC, int TOK>
__global__ void __launch_bounds__(SC_WARPS * 32) delta_scan_kernel(const fb200_delta_args a) {
  constexpr int DP = EPT * LPC, COLS = SC_WARPS * 32 / LPC, THREADS = SC_WARPS * 32;
  constexpr int STAGE = TOK * (2 * DP + COLS + 4);  // floats: k, q [TOK][DP], v [TOK][COLS], (g, beta, kq, -) [TOK][4]
  extern __shared__ __align__(16) float dsm[];
  const int tid = threadIdx.x, h = blockIdx.y, b = blockIdx.z, group = a.h / a.hk, hk = h / group, hv = a.h * a.v;
  const int p = tid % LPC, cl = tid / LPC, c = blockIdx.x * COLS + cl;
  const int pos = *a.pos_dev;
  const size_t row0 = (size_t)b * a.s;
  auto cp4 = [](uint32_t dst, const void* src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory"); };
  auto cp16 = [](uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); };
  auto fetch = [&](int t0, int stage) {
    float* sb = dsm + stage * STAGE;
    const int n = min(TOK, a.s - t0);
    for (int i = tid; i < n * (DP / 4); i += THREADS) {
      const int t = i / (DP / 4), e = (i % (DP / 4)) * 4;
      const size_t src = ((row0 + t0 + t) * a.hk + hk) * (size_t)DP + e;
      cp16(smem_u32(sb + t * DP + e), a.kn + src);
      cp16(smem_u32(sb + (TOK + t) * DP + e), a.qn + src);
    }
    float* vb = sb + 2 * TOK * DP;
    for (int i = tid; i < n * COLS; i += THREADS) {
      const int t = i / COLS, cc = i % COLS, col = blockIdx.x * COLS + cc;
      if (col < a.v) cp4(smem_u32(vb + i), a.vn + (row0 + t0 + t) * hv + h * a.v + col);
    }
    float* gs = vb + TOK * COLS;
    for (int i = tid; i < n * 3; i += THREADS) {
      const int t = i / 3, f = i % 3;
      const size_t r = row0 + t0 + t;
      cp4(smem_u32(gs + t * 4 + f), f < 2 ? a.gb + (r * a.h + h) * 2 + f : a.kq + r * a.hk + hk);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  float2 s[EPT / 2];
  float* col = a.state + (((size_t)b * a.h + h) * a.v + c) * a.dp;
  if (c < a.v && pos > 0) {
    load_column<EPT, LPC>(col, p, s);
  } else {
#pragma unroll
    for (int i = 0; i < EPT / 2; ++i) s[i] = make_float2(0.f, 0.f);
  }
  const int chunks = (a.s + TOK - 1) / TOK;
  for (int ch = 0; ch < chunks; ++ch) {
    if (ch + 1 < chunks) {
      fetch((ch + 1) * TOK, (ch + 1) & 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* sb = dsm + (ch & 1) * STAGE;
    const float *vb = sb + 2 * TOK * DP, *gs = vb + TOK * COLS;
    const int n = min(TOK, a.s - ch * TOK);
    float* orow = a.o + (row0 + ch * TOK) * hv + h * a.v + c;
    for (int t = 0; t < n; ++t) {
      const float *ks = sb + t * DP, *qs = sb + (TOK + t) * DP;
      const float4 gk = *reinterpret_cast<const float4*>(gs + t * 4);
      float dk, dq;
      column_dots<EPT, LPC>(s, ks, qs, p, dk, dq);
      const float u = gk.y * (vb[t * COLS + cl] - gk.x * dk);
      column_update<EPT, LPC>(s, ks, p, gk.x, u);
      if (p == 0 && c < a.v) orow[(size_t)t * hv] = fmaf(gk.x, dq, u * gk.z);
    }
    __syncthreads();  // the stage is free before the chunk after next lands in it
  }
  if (c < a.v) store_column<EPT, LPC>(col, p, s);
}

// A warp per (row, head): RMSNorm over v, the plain weight, the SiLU gate.
__global__ void __launch_bounds__(256) delta_out_kernel(const fb200_delta_args a) {
  const int lane = threadIdx.x & 31;
  const size_t id = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= (size_t)a.b * a.s * a.h) return;
  const size_t row = id / a.h;
  const int h = (int)(id % a.h);
  const float* o = a.o + id * a.v;
  const float* g = a.y + row * a.ldy + a.off_g + h * a.v;
  float ss = 0.f;
  for (int i = lane; i < a.v; i += 32) ss = fmaf(o[i], o[i], ss);
  const float rms = sqrtf(warp_sum(ss) / (float)a.v + a.eps);
  for (int i = lane; i < a.v; i += 32) {
    const float val = (o[i] / rms) * a.out_norm[i] * dr_silu(g[i]);
    const size_t zi = row * a.ldz + h * a.v + i;
    if (a.z_bf16) reinterpret_cast<__nv_bfloat16*>(a.z)[zi] = __float2bfloat16(val);
    else reinterpret_cast<float*>(a.z)[zi] = val;
  }
}

// The last min(s, taps) inputs of every sequence into their slots (after every convolution of the pass has run).
__global__ void conv_ring_kernel(const fb200_delta_args a) {
  const int n = min(a.s, a.taps), pos = *a.pos_dev;
  const size_t total = (size_t)a.b * n * a.channels;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const int c = (int)(i % a.channels), t = a.s - 1 - (int)(i / a.channels % n), b = (int)(i / a.channels / n);
    a.ring[((size_t)b * a.taps + (pos + t) % a.taps) * a.channels + c] = a.y[((size_t)b * a.s + t) * a.ldy + c];
  }
}

template <int EPT, int LPC>
int launch_step(fb200_device* dev, const fb200_delta_args& a) {
  int threads = (a.v * LPC + 31) / 32 * 32;
  threads = threads > ST_MAX_THREADS ? ST_MAX_THREADS : threads < 64 ? 64 : threads;
  const size_t smem = (size_t)(2 * a.dp + a.v) * 4;
  return fb200_launch(dev, delta_step_kernel<EPT, LPC>, dim3((unsigned)a.h, (unsigned)a.b), dim3((unsigned)threads), smem, true, a);
}

template <int EPT, int LPC, int TOK>
int launch_scan(fb200_device* dev, const fb200_delta_args& a) {
  constexpr int DP = EPT * LPC, COLS = SC_WARPS * 32 / LPC;
  constexpr size_t smem = (size_t)2 * TOK * (2 * DP + COLS + 4) * 4;
  static bool configured[64] = {false};
  if (!configured[dev->ordinal & 63]) {
    FB_CUDA(dev, cudaFuncSetAttribute(delta_scan_kernel<EPT, LPC, TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured[dev->ordinal & 63] = true;
  }
  delta_scan_kernel<EPT, LPC, TOK><<<dim3((unsigned)((a.v + COLS - 1) / COLS), (unsigned)a.h, (unsigned)a.b), SC_WARPS * 32, smem, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}

template <int NE>
int launch_prep(fb200_device* dev, const fb200_delta_args& a) {
  const int units = a.hk + (a.h * a.v + PREP_VCH - 1) / PREP_VCH + 1;
  delta_prep_kernel<NE><<<dim3((unsigned)((a.s + PREP_T - 1) / PREP_T), (unsigned)((units + PREP_WARPS - 1) / PREP_WARPS), (unsigned)a.b),
                          PREP_WARPS * 32, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}

}  // namespace

int fb200_delta_dp(int d) {
  for (int dp : {32, 64, 128, 256, 512, 1024})
    if (d <= dp) return dp;
  return 0;
}

int fb200_delta_step(fb200_device* dev, const fb200_delta_args& a) {
  switch (a.dp) {
    case 32: return launch_step<8, 4>(dev, a);
    case 64: return launch_step<16, 4>(dev, a);
    case 128: return launch_step<32, 4>(dev, a);
    case 256: return launch_step<32, 8>(dev, a);
    case 512: return launch_step<32, 16>(dev, a);
    case 1024: return launch_step<32, 32>(dev, a);
    default: return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "delta rule: head size %d", a.d);
  }
}

int fb200_delta_prompt(fb200_device* dev, const fb200_delta_args& a) {
  int rc;
  switch (a.dp) {
    case 32: rc = launch_prep<1>(dev, a); break;
    case 64: rc = launch_prep<2>(dev, a); break;
    case 128: rc = launch_prep<4>(dev, a); break;
    case 256: rc = launch_prep<8>(dev, a); break;
    case 512: rc = launch_prep<16>(dev, a); break;
    case 1024: rc = launch_prep<32>(dev, a); break;
    default: return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "delta rule: head size %d", a.d);
  }
  if (rc) return rc;
  switch (a.dp) {
    case 32: rc = launch_scan<8, 4, 16>(dev, a); break;
    case 64: rc = launch_scan<16, 4, 16>(dev, a); break;
    case 128: rc = launch_scan<32, 4, 16>(dev, a); break;
    case 256: rc = launch_scan<32, 8, 16>(dev, a); break;
    case 512: rc = launch_scan<32, 16, 4>(dev, a); break;
    default: rc = launch_scan<32, 32, 4>(dev, a); break;
  }
  if (rc) return rc;
  const size_t warps = (size_t)a.b * a.s * a.h;
  delta_out_kernel<<<(unsigned)((warps + 7) / 8), 256, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  conv_ring_kernel<<<(unsigned)(a.channels / 256 + 1), 256, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}
