// Gated delta rule: short convolution, unit q / k, the recurrence and its gated, normalised read-out.
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// per head, with S [d, v] in 32-bit floats. The columns of S are independent, so a column (or a few) is
// what a group of lanes owns for the whole sequence: it stays in registers, k and q come from shared memory.
// Both sums over d are formed in one pass from the state BEFORE the token,
//   S^T k -> g (S^T k),   o = g (S^T q) + u (k . q),
// and in a prompt four tokens share a pass: with a_i = S^T k_i, c_i = S^T q_i from the state before the four,
// G_i = g_0 .. g_i and w_j = (g_(j+1) .. g_i) u_j,
//   u_i = beta_i (v_i - G_i a_i - sum_(j<i) (k_j . k_i) w_j),   o_i = G_i c_i + sum_(j<=i) (k_j . q_i) w_j,
//   S <- G_3 S + sum_j k_j w_j,
// the same recurrence with one reduction over the lanes per four tokens. Everything is f32.
//
//  * delta_step_kernel: one new token per sequence. One CTA per (head, sequence): convolution, unit vectors,
//    decay, state update, read-out, RMSNorm and gate. Bound: HBM on the state (read and written once).
//  * prompts: delta_prep_kernel (convolution, SiLU, unit vectors, products of the four tokens' k and q, decay and
//    write strength), delta_scan_kernel (the recurrence; bound: f32 FMA issue, packed two-wide), delta_out_kernel (RMSNorm, gate) and
//    conv_ring_kernel (the convolution's memory).
#include "mixers.cuh"
#include "qgemv_common.cuh"
#include "state_columns.cuh"

namespace {

constexpr float UNIT_EPS = 1e-6f;  // inside the root of the unit vectors

__device__ __forceinline__ float dr_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float dr_decay(float a_log, float a, float dt) { return expf(-expf(a_log) * dr_softplus(a + dt)); }
// input of convolution channel c at position pos + t of sequence b (t < 0: earlier than this pass)
__device__ __forceinline__ float conv_in(const fb200_delta_args& a, int b, int c, int t, int pos) {
  if (t >= 0) return a.y[((size_t)b * a.s + t) * a.ldy + c];
  const int p = pos + t;
  if (p < 0) return 0.f;
  return a.ring[((size_t)b * a.taps + p % a.taps) * a.channels + c];
}
__device__ __forceinline__ float conv_silu(const fb200_delta_args& a, int b, int c, int t, int pos) {
  float acc = 0.f;
  for (int j = 0; j < a.taps; ++j) acc = fmaf(a.conv_w[(size_t)j * a.channels + c], conv_in(a, b, c, t - (a.taps - 1) + j, pos), acc);
  return dr_silu(acc);
}

// what the cached inputs contribute to the convolution of channel c at position pos
__device__ __forceinline__ float conv_past(const fb200_delta_args& a, int b, int c, int pos) {
  float acc = 0.f;
#pragma unroll 4
  for (int j = 0; j < a.taps - 1; ++j) {
    const int p = pos - (a.taps - 1) + j;
    if (p >= 0) acc = fmaf(a.conv_w[(size_t)j * a.channels + c], a.ring[((size_t)b * a.taps + p % a.taps) * a.channels + c], acc);
  }
  return acc;
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
  // so were the convolution's older inputs: threads take q [dp] | k [dp], and a lane per column its v channel
  auto qk_channel = [&](int i) { return i < a.dp ? (i < a.d ? hk * a.d + i : -1) : (i - a.dp < a.d ? (a.hk + hk) * a.d + i - a.dp : -1); };
  const int ch0 = tid < 2 * a.dp ? qk_channel(tid) : -1;
  const float past0 = ch0 >= 0 ? conv_past(a, b, ch0, pos) : 0.f, w0 = ch0 >= 0 ? a.conv_w[(size_t)(a.taps - 1) * a.channels + ch0] : 0.f;
  float vpast = 0.f, vw = 0.f;
  if (p == 0 && c0 < a.v) {
    vpast = conv_past(a, b, a.off_v + h * a.v + c0, pos);
    vw = a.conv_w[(size_t)(a.taps - 1) * a.channels + a.off_v + h * a.v + c0];
  }
  pdl_wait();
  pdl_launch_dependents();
  const float* yr = a.y + (size_t)b * a.ldy;
  float v0 = 0.f;
  if (p == 0 && c0 < a.v) v0 = dr_silu(fmaf(vw, yr[a.off_v + h * a.v + c0], vpast));
  v0 = __shfl_sync(0xFFFFFFFFu, v0, lane & ~(LPC - 1));
  for (int i = tid; i < 2 * a.dp; i += nt) {
    const int ch = i == tid ? ch0 : qk_channel(i);
    float x = 0.f;
    if (ch >= 0) x = i == tid ? dr_silu(fmaf(w0, yr[ch], past0)) : conv_silu(a, b, ch, 0, pos);
    (i < a.dp ? qs : ks - a.dp)[i] = x;
  }
  __syncthreads();
  float skk = 0.f, sqq = 0.f, skq = 0.f;
  for (int i = tid; i < a.dp; i += nt) {
    const float k = ks[i], q = qs[i];
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
    const float v = it == 0 ? v0 : in ? conv_silu(a, b, a.off_v + h * a.v + c, 0, pos) : 0.f;
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
constexpr int CH = 4;  // tokens per pass of the recurrence
constexpr int PREP_WARPS = 4, PREP_VCH = 128;
constexpr int PAIRS = 16;  // k_j . k_i (j < i): 6 values, then k_j . q_i (j <= i): 10 values, i-major
// (j, i) of pair p, two bits each
constexpr uint32_t PAIR_J = 0u | 0u << 2 | 1u << 4 | 0u << 6 | 1u << 8 | 2u << 10 | 0u << 12 | 0u << 14 | 1u << 16 | 0u << 18 | 1u << 20 |
                            2u << 22 | 0u << 24 | 1u << 26 | 2u << 28 | 3u << 30;
constexpr uint32_t PAIR_I = 1u | 2u << 2 | 2u << 4 | 3u << 6 | 3u << 8 | 3u << 10 | 0u << 12 | 1u << 14 | 1u << 16 | 2u << 18 | 2u << 20 |
                            2u << 22 | 3u << 24 | 3u << 26 | 3u << 28 | 3u << 30;

// convolution + SiLU of channel c for the CH tokens from t0 (zeros from token s on); inputs before this pass come
// from the ring. Addresses are selected, not branched on, so that a channel's loads go out together.
__device__ __forceinline__ void conv_chunk(const fb200_delta_args& a, int b, int c, int t0, int pos, float (&out)[CH]) {
#pragma unroll
  for (int i = 0; i < CH; ++i) out[i] = 0.f;
  for (int j0 = 0; j0 < a.taps; j0 += 4) {  // four taps at a time meet seven inputs
    float w[4], x[CH + 3];
#pragma unroll
    for (int j = 0; j < 4; ++j) w[j] = j0 + j < a.taps ? a.conv_w[(size_t)(j0 + j) * a.channels + c] : 0.f;
#pragma unroll
    for (int r = 0; r < CH + 3; ++r) {
      const int t = t0 - (a.taps - 1) + j0 + r, p = pos + t;
      const bool valid = j0 + r < a.taps + CH - 1 && t < a.s && p >= 0;
      const float* src = t >= 0 ? a.y + ((size_t)b * a.s + t) * a.ldy + c : a.ring + ((size_t)b * a.taps + (valid ? p % a.taps : 0)) * a.channels + c;
      x[r] = valid ? *src : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < CH; ++i) out[i] = fmaf(w[j], x[i + j], out[i]);
  }
#pragma unroll
  for (int i = 0; i < CH; ++i) out[i] = t0 + i < a.s ? dr_silu(out[i]) : 0.f;
}

// Sums v[0..31] over the lanes of a warp; lane l returns the total of v[l].
__device__ __forceinline__ float warp_sum32(float (&v)[32]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, o);
    }
  }
  return v[0];
}

// A warp per (unit, CH tokens): units 0 .. hk are the q and k vectors of a q/k head, then blocks of 128 v channels, then
// the decays and write strengths of all heads. NE = channels of a q/k head per lane.
template <int NE>
__global__ void __launch_bounds__(PREP_WARPS * 32) delta_prep_kernel(const fb200_delta_args a) {
  const int lane = threadIdx.x & 31, b = blockIdx.z, t0 = blockIdx.x * CH, n = min(CH, a.s - t0);
  const int hv = a.h * a.v, vblocks = (hv + PREP_VCH - 1) / PREP_VCH;
  int unit = blockIdx.y * PREP_WARPS + (threadIdx.x >> 5);
  const int pos = *a.pos_dev;
  if (unit < a.hk) {
    float q[NE][CH], k[NE][CH], sum[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) sum[i] = 0.f;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int c = lane + 32 * e;
#pragma unroll
      for (int i = 0; i < CH; ++i) q[e][i] = k[e][i] = 0.f;
      if (c < a.d) {
        conv_chunk(a, b, unit * a.d + c, t0, pos, q[e]);
        conv_chunk(a, b, (a.hk + unit) * a.d + c, t0, pos, k[e]);
      }
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        sum[i] = fmaf(k[e][i], k[e][i], sum[i]);
        sum[4 + i] = fmaf(q[e][i], q[e][i], sum[4 + i]);
      }
#pragma unroll
      for (int p = 0; p < PAIRS; ++p) {
        const int j = (PAIR_J >> (2 * p)) & 3, i = (PAIR_I >> (2 * p)) & 3;
        sum[8 + p] = fmaf(k[e][j], p < 6 ? k[e][i] : q[e][i], sum[8 + p]);
      }
    }
    const float total = warp_sum32(sum);
    const float inv = (1.0f / sqrtf(total + UNIT_EPS)) * (lane >= 4 ? 1.0f / sqrtf((float)a.d) : 1.0f);  // lanes 0..3: k, 4..7: q
    const int p = lane - 8;
    const float sj = __shfl_sync(0xFFFFFFFFu, inv, (PAIR_J >> (2 * (p & 15))) & 3);
    const float si = __shfl_sync(0xFFFFFFFFu, inv, ((PAIR_I >> (2 * (p & 15))) & 3) + (p < 6 ? 0 : 4));
    if (p >= 0 && p < PAIRS) a.kq[(((size_t)b * gridDim.x + blockIdx.x) * a.hk + unit) * PAIRS + p] = total * sj * si;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const float ik = __shfl_sync(0xFFFFFFFFu, inv, i), iq = __shfl_sync(0xFFFFFFFFu, inv, 4 + i);
      if (i >= n) continue;
      const size_t row = ((size_t)b * a.s + t0 + i) * a.hk + unit;
#pragma unroll
      for (int e = 0; e < NE; ++e) {
        const int c = lane + 32 * e;
        if (c < a.dp) {
          a.qn[row * a.dp + c] = q[e][i] * iq;
          a.kn[row * a.dp + c] = k[e][i] * ik;
        }
      }
    }
    return;
  }
  unit -= a.hk;
  if (unit < vblocks) {
    float v[PREP_VCH / 32][CH];
#pragma unroll
    for (int e = 0; e < PREP_VCH / 32; ++e) {
      const int c = unit * PREP_VCH + lane + 32 * e;
      if (c < hv) conv_chunk(a, b, a.off_v + c, t0, pos, v[e]);
    }
#pragma unroll
    for (int e = 0; e < PREP_VCH / 32; ++e) {
      const int c = unit * PREP_VCH + lane + 32 * e;
#pragma unroll
      for (int i = 0; i < CH; ++i)
        if (c < hv && i < n) a.vn[((size_t)b * a.s + t0 + i) * hv + c] = v[e][i];
    }
    return;
  }
  if (unit > vblocks) return;
  for (int i = lane; i < n * a.h; i += 32) {
    const int t = t0 + i / a.h, h = i % a.h;
    const size_t row = (size_t)b * a.s + t;
    const float* yr = a.y + row * a.ldy;
    a.gb[(row * a.h + h) * 2] = dr_decay(a.a_log[h], yr[a.off_a + h], a.dt_bias[h]);
    a.gb[(row * a.h + h) * 2 + 1] = dr_sigmoid(yr[a.off_b + h]);
  }
}

constexpr int SC_WARPS = 4, CPT = 4;  // columns per group of lanes

// A group of LPC lanes owns CPT columns of S: k and q read from shared memory serve all of them, and the sums are
// reduced so that lane p ends up with those of column p % 4, so one pass over the four tokens does all columns.
// TOK tokens make a shared-memory stage (a multiple of CH).
template <int EPT, int LPC, int TOK>
__global__ void __launch_bounds__(SC_WARPS * 32) delta_scan_kernel(const fb200_delta_args a) {
  constexpr int DP = EPT * LPC, GROUPS = SC_WARPS * 32 / LPC, COLS = GROUPS * CPT, THREADS = SC_WARPS * 32, NC = TOK / CH;
  // floats of a stage: k, q [TOK][DP], v [COLS][TOK], pairs [NC][PAIRS], g [TOK], beta [TOK]
  constexpr int OV = 2 * TOK * DP, OP = OV + COLS * TOK, OG = OP + NC * PAIRS, STAGE = OG + 2 * TOK;
  constexpr bool KEEP = EPT <= 16;  // k of the four tokens stays in registers for the update
  extern __shared__ __align__(16) float dsm[];
  const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.y, b = blockIdx.z, group = a.h / a.hk, hk = h / group, hv = a.h * a.v;
  const int p = tid % LPC, cl = tid / LPC, c = blockIdx.x * COLS + cl;  // columns c, c + GROUPS, ..
  const int pos = *a.pos_dev, nchunks = (a.s + CH - 1) / CH;
  const size_t row0 = (size_t)b * a.s;
  auto cp4 = [](const float* dst, const float* src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory"); };
  auto cp16 = [](const float* dst, const float* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory"); };
  auto fetch = [&](int t0, int stage) {
    float* sb = dsm + stage * STAGE;
    const int n = min(TOK, a.s - t0);
    for (int i = tid; i < TOK * (DP / 4); i += THREADS) {
      const int t = i / (DP / 4), e = (i % (DP / 4)) * 4;
      if (t < n) {
        const size_t src = ((row0 + t0 + t) * a.hk + hk) * (size_t)DP + e;
        cp16(sb + t * DP + e, a.kn + src);
        cp16(sb + (TOK + t) * DP + e, a.qn + src);
      } else {  // beyond the last token: k = q = v = 0, g = 1, beta = 0 change nothing
        *reinterpret_cast<float4*>(sb + t * DP + e) = make_float4(0.f, 0.f, 0.f, 0.f);
        *reinterpret_cast<float4*>(sb + (TOK + t) * DP + e) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    for (int i = tid; i < TOK * COLS; i += THREADS) {
      const int t = i / COLS, cc = i % COLS, col = blockIdx.x * COLS + cc;
      if (t < n && col < a.v) cp4(sb + OV + cc * TOK + t, a.vn + (row0 + t0 + t) * hv + h * a.v + col);
      else sb[OV + cc * TOK + t] = 0.f;
    }
    for (int i = tid; i < NC * (PAIRS / 4); i += THREADS) {
      const int ch = t0 / CH + i / (PAIRS / 4), e = (i % (PAIRS / 4)) * 4;
      if (ch < nchunks) cp16(sb + OP + (i / (PAIRS / 4)) * PAIRS + e, a.kq + (((size_t)b * nchunks + ch) * a.hk + hk) * PAIRS + e);
      else *reinterpret_cast<float4*>(sb + OP + (i / (PAIRS / 4)) * PAIRS + e) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int i = tid; i < 2 * TOK; i += THREADS) {
      const int t = i % TOK, f = i / TOK;
      if (t < n) cp4(sb + OG + i, a.gb + ((row0 + t0 + t) * a.h + h) * 2 + f);
      else sb[OG + i] = f ? 0.f : 1.f;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  float2 s[CPT][EPT / 2];
  float* state = a.state + ((size_t)b * a.h + h) * (size_t)a.v * a.dp;
#pragma unroll
  for (int cc = 0; cc < CPT; ++cc) {
    if (c + cc * GROUPS < a.v && pos > 0) {
      load_column<EPT, LPC>(state + (size_t)(c + cc * GROUPS) * a.dp, p, s[cc]);
    } else {
#pragma unroll
      for (int i = 0; i < EPT / 2; ++i) s[cc][i] = make_float2(0.f, 0.f);
    }
  }
  const int stages = (a.s + TOK - 1) / TOK;
  for (int st = 0; st < stages; ++st) {
    if (st + 1 < stages) {
      fetch((st + 1) * TOK, (st + 1) & 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* sb = dsm + (st & 1) * STAGE;
#pragma unroll 1
    for (int ch = 0; ch < NC; ++ch) {
      const int t0 = st * TOK + ch * CH;
      if (t0 >= a.s) break;
      const float *kb = sb + ch * CH * DP, *qb = sb + (TOK + ch * CH) * DP;
      // ---- a_i = S^T k_i, c_i = S^T q_i over this lane's elements
      float2 kf[KEEP ? CH : 1][EPT / 2];
      float val[CPT][2 * CH];
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        float2 ka[CPT], qa[CPT];
#pragma unroll
        for (int cc = 0; cc < CPT; ++cc) ka[cc] = qa[cc] = make_float2(0.f, 0.f);
#pragma unroll
        for (int e = 0; e < EPT / 4; ++e) {
          const float4 k = *reinterpret_cast<const float4*>(kb + i * DP + 4 * (e * LPC + p));
          const float4 q = *reinterpret_cast<const float4*>(qb + i * DP + 4 * (e * LPC + p));
#pragma unroll
          for (int cc = 0; cc < CPT; ++cc) {
            ka[cc] = fma2(s[cc][2 * e], make_float2(k.x, k.y), ka[cc]);
            qa[cc] = fma2(s[cc][2 * e], make_float2(q.x, q.y), qa[cc]);
            ka[cc] = fma2(s[cc][2 * e + 1], make_float2(k.z, k.w), ka[cc]);
            qa[cc] = fma2(s[cc][2 * e + 1], make_float2(q.z, q.w), qa[cc]);
          }
          if (KEEP) {
            kf[KEEP ? i : 0][2 * e] = make_float2(k.x, k.y);
            kf[KEEP ? i : 0][2 * e + 1] = make_float2(k.z, k.w);
          }
        }
#pragma unroll
        for (int cc = 0; cc < CPT; ++cc) {
          val[cc][i] = ka[cc].x + ka[cc].y;
          val[cc][CH + i] = qa[cc].x + qa[cc].y;
        }
      }
      // ---- totals over the LPC lanes: two halving steps leave lane p with column p % 4, the rest adds up its lanes
#pragma unroll
      for (int x = 0; x < 2 * CH; ++x) {
        const bool odd = lane & 1, high = lane & 2;
        const float s01 = odd ? val[0][x] : val[1][x], k01 = odd ? val[1][x] : val[0][x];
        const float s23 = odd ? val[2][x] : val[3][x], k23 = odd ? val[3][x] : val[2][x];
        const float c01 = k01 + __shfl_xor_sync(0xFFFFFFFFu, s01, 1), c23 = k23 + __shfl_xor_sync(0xFFFFFFFFu, s23, 1);
        float t = (high ? c23 : c01) + __shfl_xor_sync(0xFFFFFFFFu, high ? c01 : c23, 2);
#pragma unroll
        for (int o = 4; o < LPC; o <<= 1) t += __shfl_xor_sync(0xFFFFFFFFu, t, o);
        val[0][x] = t;
      }
      // ---- the four tokens in order
      float pr[PAIRS];
#pragma unroll
      for (int i = 0; i < PAIRS / 4; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(sb + OP + ch * PAIRS + 4 * i);
        pr[4 * i] = x.x; pr[4 * i + 1] = x.y; pr[4 * i + 2] = x.z; pr[4 * i + 3] = x.w;
      }
      const float4 g4 = *reinterpret_cast<const float4*>(sb + OG + ch * CH), b4 = *reinterpret_cast<const float4*>(sb + OG + TOK + ch * CH);
      const float gi[CH] = {g4.x, g4.y, g4.z, g4.w}, bi[CH] = {b4.x, b4.y, b4.z, b4.w};
      const float2 G2 = make_float2(((g4.x * g4.y) * g4.z) * g4.w, ((g4.x * g4.y) * g4.z) * g4.w);
      const int mycol = cl + (p & 3) * GROUPS;
      const float4 v4 = *reinterpret_cast<const float4*>(sb + OV + mycol * TOK + ch * CH);
      const float vi[CH] = {v4.x, v4.y, v4.z, v4.w};
      float u[CH], out[CH], G = 1.f;
      int pk = 0, pq = 6;
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        G *= gi[i];
        float uk = G * val[0][i], o = G * val[0][CH + i];
#pragma unroll
        for (int j = 0; j < CH; ++j)
          if (j < i) {
            u[j] *= gi[i];
            uk = fmaf(pr[pk++], u[j], uk);
            o = fmaf(pr[pq++], u[j], o);
          }
        u[i] = bi[i] * (vi[i] - uk);
        out[i] = fmaf(pr[pq++], u[i], o);
      }
      if (p < 8 && blockIdx.x * COLS + mycol < a.v) {  // lanes 0..3 store tokens 0 and 1, lanes 4..7 tokens 2 and 3
        const int i0 = p < 4 ? 0 : 2;
        float* dst = a.o + (row0 + t0 + i0) * hv + h * a.v + blockIdx.x * COLS + mycol;
        if (t0 + i0 < a.s) dst[0] = p < 4 ? out[0] : out[2];
        if (t0 + i0 + 1 < a.s) dst[hv] = p < 4 ? out[1] : out[3];
      }
      float w[CPT][CH];
#pragma unroll
      for (int cc = 0; cc < CPT; ++cc)
#pragma unroll
        for (int i = 0; i < CH; ++i) w[cc][i] = __shfl_sync(0xFFFFFFFFu, u[i], (lane & ~3) | cc);
      // ---- S <- G S + sum_j k_j w_j
#pragma unroll
      for (int cc = 0; cc < CPT; ++cc)
#pragma unroll
        for (int e = 0; e < EPT / 2; ++e) s[cc][e] = mul2(s[cc][e], G2);
#pragma unroll
      for (int i = 0; i < CH; ++i) {
#pragma unroll
        for (int e = 0; e < EPT / 4; ++e) {
          float2 k0, k1;
          if (KEEP) {
            k0 = kf[KEEP ? i : 0][2 * e];
            k1 = kf[KEEP ? i : 0][2 * e + 1];
          } else {
            const float4 k = *reinterpret_cast<const float4*>(kb + i * DP + 4 * (e * LPC + p));
            k0 = make_float2(k.x, k.y);
            k1 = make_float2(k.z, k.w);
          }
#pragma unroll
          for (int cc = 0; cc < CPT; ++cc) {
            const float2 w2 = make_float2(w[cc][i], w[cc][i]);
            s[cc][2 * e] = fma2(k0, w2, s[cc][2 * e]);
            s[cc][2 * e + 1] = fma2(k1, w2, s[cc][2 * e + 1]);
          }
        }
      }
    }
    __syncthreads();  // the stage is free before the one after next lands in it
  }
#pragma unroll
  for (int cc = 0; cc < CPT; ++cc)
    if (c + cc * GROUPS < a.v) store_column<EPT, LPC>(state + (size_t)(c + cc * GROUPS) * a.dp, p, s[cc]);
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
  constexpr int DP = EPT * LPC, COLS = SC_WARPS * 32 / LPC * CPT;
  constexpr size_t smem = (size_t)2 * (2 * TOK * DP + COLS * TOK + TOK / CH * PAIRS + 2 * TOK) * 4;
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
  delta_prep_kernel<NE><<<dim3((unsigned)((a.s + CH - 1) / CH), (unsigned)((units + PREP_WARPS - 1) / PREP_WARPS), (unsigned)a.b),
                          PREP_WARPS * 32, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}

}  // namespace

int fb200_delta_dp(int d) {
  for (int dp : {32, 64, 128, 256, 512})
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
    default: return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "delta rule: head size %d", a.d);
  }
  if (rc) return rc;
  switch (a.dp) {
    case 32: rc = launch_scan<4, 8, 16>(dev, a); break;
    case 64: rc = launch_scan<4, 16, 16>(dev, a); break;
    case 128:
      // 16 lanes per column group do less per token (fewer shuffles); 32 lanes make more CTAs where there are few heads
      if ((a.v + 15) / 16 * a.h * a.b <= dev->sm_count) rc = launch_scan<4, 32, 16>(dev, a);
      else rc = launch_scan<8, 16, 16>(dev, a);
      break;
    case 256: rc = launch_scan<8, 32, 16>(dev, a); break;
    default: rc = launch_scan<16, 32, 8>(dev, a); break;
  }
  if (rc) return rc;
  const size_t warps = (size_t)a.b * a.s * a.h;
  delta_out_kernel<<<(unsigned)((warps + 7) / 8), 256, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  conv_ring_kernel<<<(unsigned)(a.channels / 256 + 1), 256, 0, dev->stream>>>(a);
  FB_LAUNCH_CHECK(dev);
  return FB200_OK;
}
