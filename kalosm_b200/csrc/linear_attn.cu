// Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, the read-out normalised over all heads.
//
// The columns of S (one per value element) are independent: a group of lanes owns a column and keeps it in registers. All
// sums, states and decays are f32.
//  * linear_scan_kernel: token by token. One new token per sequence is one launch: the state is requested before the
//    projections are there, and the CTA that arrives last normalises the whole row and applies the gates. Bound: HBM on
//    the state, read and written once.
//  * bf16 prompts work on chunks of tokens with tensor cores: with S the state before a chunk of n tokens and tokens i, j of it,
//      o_i = decay^(i+1) S^T q_i + sum_(j<=i) decay^(i-j) (q_i . k_j) v_j,   S <- decay^n S + sum_i k_i (decay^(n-1-i) v_i)^T,
//    the same recurrence. q, k and v are bf16 (linear_prep_kernel makes them); what the recurrence adds to them (the state, the
//    decayed values, the decayed products q . k) enters the tensor cores as a bf16 value and a bf16 remainder, sums and the
//    state itself are f32. Bound: HBM on the operands and the read-out. Heads of up to 128 run linear_prefill.cu (tcgen05),
//    wider ones linear_chunk_kernel (mma.sync, 64 tokens at a time).
//  * linear_out_kernel: the normalisation and the gates of a prompt's rows.
#include <algorithm>

#include "attn_mma.cuh"
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
  const float inv = 1.0f / sqrtf(ss / (float)n + a.eps);
  if ((n & 3) == 0 && (reinterpret_cast<uintptr_t>(g) & 15u) == 0 && (a.ldz & 3) == 0 && (reinterpret_cast<uintptr_t>(a.z) & 15u) == 0) {
    for (int i = 4 * tid; i < n; i += 4 * LS_THREADS) {
      const float4 x = __ldcg(reinterpret_cast<const float4*>(o + i)), w = *reinterpret_cast<const float4*>(a.out_norm + i);
      const float4 y = *reinterpret_cast<const float4*>(g + i);
      const float v0 = x.x * inv * w.x * dr_sigmoid(y.x) * a.out_scale, v1 = x.y * inv * w.y * dr_sigmoid(y.y) * a.out_scale;
      const float v2 = x.z * inv * w.z * dr_sigmoid(y.z) * a.out_scale, v3 = x.w * inv * w.w * dr_sigmoid(y.w) * a.out_scale;
      if (a.z_bf16) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v0, v1), hi = __floats2bfloat162_rn(v2, v3);
        *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(a.z) + row * a.ldz + i) =
            make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
      } else {
        *reinterpret_cast<float4*>(reinterpret_cast<float*>(a.z) + row * a.ldz + i) = make_float4(v0, v1, v2, v3);
      }
    }
    return;
  }
  for (int i = tid; i < n; i += LS_THREADS) {
    const float x = __ldcg(o + i) * inv * a.out_norm[i] * dr_sigmoid(g[i]) * a.out_scale;
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

// ---- prompts on tensor cores -----------------------------------------------------------------------------------
constexpr int LC = 64, LC_VS = 32, LC_VP = LC_VS + 8, LC_THREADS = 256;

// A thread per 8 elements: q and k heads (zeros from d to dp), then v heads (to vp).
__global__ void __launch_bounds__(256) linear_prep_kernel(const fb200_linear_args a, int vp) {
  const int qp = a.dp / 8, per_head = 2 * qp + vp / 8;
  const size_t id = (size_t)blockIdx.x * 256 + threadIdx.x, per_row = (size_t)a.h * per_head;
  if (id >= (size_t)a.b * a.s * per_row) return;
  const size_t row = id / per_row;
  const int rem = (int)(id % per_row), h = rem / per_head, c = rem % per_head;
  const bool is_v = c >= 2 * qp, is_k = !is_v && c >= qp;
  const int e0 = 8 * (is_v ? c - 2 * qp : is_k ? c - qp : c), n = is_v ? a.v : a.d;
  const float* src = a.y + row * a.ldy + (is_v ? a.off_v : is_k ? a.off_k : 0) + (size_t)h * n + e0;
  float x[8];
  if (e0 + 8 <= n && (reinterpret_cast<uintptr_t>(src) & 15u) == 0) {
    *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(src);
    *reinterpret_cast<float4*>(x + 4) = *reinterpret_cast<const float4*>(src + 4);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = dr_silu(x[e]);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = e0 + e < n ? dr_silu(src[e]) : 0.f;
  }
  uint32_t w[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const __nv_bfloat162 t = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
    w[e] = *reinterpret_cast<const uint32_t*>(&t);
  }
  __nv_bfloat16* dst = is_v ? a.v16 + (row * a.h + h) * vp : (is_k ? a.k16 : a.q16) + (row * a.h + h) * a.dp;
  *reinterpret_cast<uint4*>(dst + e0) = make_uint4(w[0], w[1], w[2], w[3]);
}

// two f32 as bf16 values and bf16 remainders
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 bf2(uint32_t u) { return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xFFFF0000u)); }

template <int DP>
struct LcShape {
  static constexpr int STRIDE = DP + 8;  // elements of a staged q / k row: 16 bytes of padding spread the rows over the banks
  static constexpr int QK = LC * STRIDE, V = LC * LC_VP, STAGE = 2 * QK + V, ST = DP * LC_VP;  // elements
  static constexpr int SMEM = (2 * STAGE + 4 * ST) * 2;
};

// CTA: LC_VS value columns of one head of one sequence. Warps 0..3 form the read-out of 16 tokens each, warps 4..7 carry the
// state, DP / 4 rows of it each in accumulators, and hand it over through shared memory one chunk ahead of its use.
template <int DP>
__global__ void __launch_bounds__(LC_THREADS) linear_chunk_kernel(const fb200_linear_args a, int vp) {
  using S = LcShape<DP>;
  constexpr int MT = DP / 64, NT = LC_VS / 8;  // state tiles of a warp: MT x NT of 16 x 8
  extern __shared__ __align__(16) __nv_bfloat16 csm[];
  __shared__ float pw[LC + 1];
  __nv_bfloat16* st = csm + 2 * S::STAGE;  // [buffer][value, remainder][DP][LC_VP]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, j = lane >> 3, r8 = lane & 7;
  const int c0 = blockIdx.x * LC_VS, h = blockIdx.y, b = blockIdx.z, hv = a.h * a.v, w = warp & 3;
  const int pos = *a.pos_dev, chunks = (a.s + LC - 1) / LC;
  for (int i = tid; i <= LC; i += LC_THREADS) pw[i] = a.decay[(size_t)h * (FB200_LINEAR_CHUNK + 1) + i];
  const size_t row0 = (size_t)b * a.s;
  auto fetch = [&](int ch) {
    __nv_bfloat16* dst = csm + (ch & 1) * S::STAGE;
    constexpr int P = DP / 8, VPC = LC_VS / 8;
    for (int i = tid; i < 2 * LC * P; i += LC_THREADS) {
      const int m = i / (LC * P), r = i / P % LC, e = (i % P) * 8, tok = ch * LC + r;
      const bool in = tok < a.s;
      pf_cp16(pf_smem(dst + m * S::QK + r * S::STRIDE + e), (m ? a.k16 : a.q16) + ((row0 + (in ? tok : 0)) * a.h + h) * DP + e, in);
    }
    for (int i = tid; i < LC * VPC; i += LC_THREADS) {
      const int r = i / VPC, e = (i % VPC) * 8, tok = ch * LC + r;
      const bool in = tok < a.s && c0 + e < vp;
      pf_cp16(pf_smem(dst + 2 * S::QK + r * LC_VP + e), a.v16 + ((row0 + (in ? tok : 0)) * a.h + h) * vp + (in ? c0 + e : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  float s[MT][NT][4];
  float* state = a.state + (((size_t)b * a.h + h) * a.v + c0) * (size_t)DP;
  // element e of tile (mi, nt): row d, column v
  auto at = [&](int mi, int nt, int e, int& d, int& v) {
    d = (w * MT + mi) * 16 + g + 8 * (e >> 1);
    v = nt * 8 + 2 * t + (e & 1);
  };
  auto hand_over = [&](int buf) {
    __nv_bfloat16* dst = st + buf * 2 * S::ST;
#pragma unroll
    for (int mi = 0; mi < MT; ++mi)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          int d, v;
          at(mi, nt, e, d, v);
          uint32_t hi, lo;
          split2(s[mi][nt][e], s[mi][nt][e + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(dst + d * LC_VP + v) = hi;
          *reinterpret_cast<uint32_t*>(dst + S::ST + d * LC_VP + v) = lo;
        }
  };
  if (warp >= 4) {
#pragma unroll
    for (int mi = 0; mi < MT; ++mi)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          int d, v;
          at(mi, nt, e, d, v);
          s[mi][nt][e] = pos > 0 && c0 + v < a.v ? state[(size_t)v * DP + d] : 0.f;
        }
    hand_over(0);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  for (int ch = 0; ch < chunks; ++ch) {
    const int n = min(LC, a.s - ch * LC);
    if (ch + 1 < chunks) fetch(ch + 1);
    const __nv_bfloat16 *Q = csm + (ch & 1) * S::STAGE, *K = Q + S::QK, *V = K + S::QK;
    if (warp >= 4) {
      // ---- S <- decay^n S + sum_i k_i (decay^(n-1-i) v_i)^T
      const float dn = pw[n];
#pragma unroll
      for (int mi = 0; mi < MT; ++mi)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[mi][nt][e] *= dn;
#pragma unroll
      for (int ks = 0; ks < LC / 16; ++ks) {
        uint32_t vh[NT][2], vl[NT][2];
        float f[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) f[e] = pw[max(0, n - 1 - (ks * 16 + 2 * t + (e & 1) + 8 * (e >> 1)))];
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t bb[4];
          pf_ldsm4_t(pf_smem(V + (ks * 16 + (j & 1) * 8 + r8) * LC_VP + nt * 8 + (j >> 1) * 8), bb);
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const float2 x = bf2(bb[q]);
            split2(x.x * f[(q & 1) * 2], x.y * f[(q & 1) * 2 + 1], vh[nt + (q >> 1)][q & 1], vl[nt + (q >> 1)][q & 1]);
          }
        }
#pragma unroll
        for (int mi = 0; mi < MT; ++mi) {
          uint32_t aa[4];
          pf_ldsm4_t(pf_smem(K + (ks * 16 + (j >> 1) * 8 + r8) * S::STRIDE + (w * MT + mi) * 16 + (j & 1) * 8), aa);
#pragma unroll
          for (int nt = 0; nt < NT; ++nt) {
            pf_mma_bf16(s[mi][nt], aa, vh[nt][0], vh[nt][1]);
            pf_mma_bf16(s[mi][nt], aa, vl[nt][0], vl[nt][1]);
          }
        }
      }
      if (ch + 1 < chunks) hand_over((ch + 1) & 1);
    } else {
      // ---- read-out of tokens 16 w .. 16 w + 15: first the state's share
      const __nv_bfloat16* sh = st + (ch & 1) * 2 * S::ST;
      float o[NT][4], p[8][4];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) p[nt][0] = p[nt][1] = p[nt][2] = p[nt][3] = 0.f;
      const uint32_t qb = pf_smem(Q + (w * 16 + (j & 1) * 8 + r8) * S::STRIDE + (j >> 1) * 8);
#pragma unroll 4
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t aa[4];
        pf_ldsm4(qb + ks * 32, aa);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int nt = 0; nt < NT; nt += 2) {
            uint32_t bb[4];
            pf_ldsm4_t(pf_smem(sh + part * S::ST + (ks * 16 + (j & 1) * 8 + r8) * LC_VP + nt * 8 + (j >> 1) * 8), bb);
            pf_mma_bf16(o[nt], aa, bb[0], bb[1]);
            pf_mma_bf16(o[nt + 1], aa, bb[2], bb[3]);
          }
#pragma unroll
        for (int kt = 0; kt < 4; ++kt)  // q . k for the keys in front of this warp's last token
          if (kt <= w) {
            uint32_t bb[4];
            pf_ldsm4(pf_smem(K + (kt * 16 + (j >> 1) * 8 + r8) * S::STRIDE + ks * 16 + (j & 1) * 8), bb);
            pf_mma_bf16(p[2 * kt], aa, bb[0], bb[1]);
            pf_mma_bf16(p[2 * kt + 1], aa, bb[2], bb[3]);
          }
      }
      const float d0 = pw[w * 16 + g + 1], d1 = pw[w * 16 + g + 9];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        o[nt][0] *= d0;
        o[nt][1] *= d0;
        o[nt][2] *= d1;
        o[nt][3] *= d1;
      }
#pragma unroll
      for (int kt = 0; kt < 4; ++kt)
        if (kt <= w) {
          uint32_t ph[4], pl[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {  // rows g + 8 (q & 1), keys 16 kt + 8 (q >> 1) + 2 t, + 1
            const int i = w * 16 + g + 8 * (q & 1), k = kt * 16 + 8 * (q >> 1) + 2 * t;
            const float x = k <= i ? p[2 * kt + (q >> 1)][2 * (q & 1)] * pw[i - k] : 0.f;
            const float y = k < i ? p[2 * kt + (q >> 1)][2 * (q & 1) + 1] * pw[i - k - 1] : 0.f;
            split2(x, y, ph[q], pl[q]);
          }
#pragma unroll
          for (int nt = 0; nt < NT; nt += 2) {
            uint32_t bb[4];
            pf_ldsm4_t(pf_smem(V + (kt * 16 + (j & 1) * 8 + r8) * LC_VP + nt * 8 + (j >> 1) * 8), bb);
            pf_mma_bf16(o[nt], ph, bb[0], bb[1]);
            pf_mma_bf16(o[nt + 1], ph, bb[2], bb[3]);
            pf_mma_bf16(o[nt], pl, bb[0], bb[1]);
            pf_mma_bf16(o[nt + 1], pl, bb[2], bb[3]);
          }
        }
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int i = w * 16 + g + 4 * e, v = c0 + nt * 8 + 2 * t;
          if (i >= n) continue;
          float* dst = a.o + (row0 + ch * LC + i) * hv + (size_t)h * a.v + v;
          if (v + 1 < a.v && (hv & 1) == 0 && (a.v & 1) == 0) *reinterpret_cast<float2*>(dst) = make_float2(o[nt][e], o[nt][e + 1]);
          else {
            if (v < a.v) dst[0] = o[nt][e];
            if (v + 1 < a.v) dst[1] = o[nt][e + 1];
          }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
  }
  if (warp >= 4) {
#pragma unroll
    for (int mi = 0; mi < MT; ++mi)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          int d, v;
          at(mi, nt, e, d, v);
          if (c0 + v < a.v) state[(size_t)v * DP + d] = s[mi][nt][e];
        }
  }
}

template <int DP>
int linear_chunks(fb200_device* dev, const fb200_linear_args& a) {
  const int vp = (a.v + 7) / 8 * 8;
  static bool configured[64] = {false};
  if (!configured[dev->ordinal & 63]) {
    FB_CUDA(dev, cudaFuncSetAttribute(linear_chunk_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, LcShape<DP>::SMEM));
    configured[dev->ordinal & 63] = true;
  }
  linear_chunk_kernel<DP><<<dim3((unsigned)((a.v + LC_VS - 1) / LC_VS), (unsigned)a.h, (unsigned)a.b), LC_THREADS, LcShape<DP>::SMEM, dev->stream>>>(a, vp);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
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
  int rc;
  if (a.bf16 && a.s >= 16 && a.dp <= 256) {
    const int vp = (a.v + 7) / 8 * 8;
    const size_t threads = (size_t)a.b * a.s * a.h * (2 * a.dp + vp) / 8;
    linear_prep_kernel<<<(unsigned)((threads + 255) / 256), 256, 0, dev->stream>>>(a, vp);
    FB_LAUNCH_CHECK(dev);
    rc = fb200_linear_prefill_covers(a) ? fb200_linear_prefill(dev, a) : linear_chunks<256>(dev, a);
  } else {
    rc = linear_scan(dev, a);
  }
  if (rc) return rc;
  linear_out_kernel<<<(unsigned)(a.b * a.s), LS_THREADS, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}
