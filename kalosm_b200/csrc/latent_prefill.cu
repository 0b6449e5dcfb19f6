// Attention of a prompt pass of the token-mixer layers on the 5th-generation tensor cores: latent attention and grouped
// attention.
//
// Latent attention: for many query rows the keys and values are expanded once, K | V = W_ukv c for the visible positions (a
// bf16 product, dense_tc.cu), and the attention runs over them; the rotated key part, shared by the heads, is read
// from the cache as it is. Bound: tensor cores, 2 (d + r + v) flops per head and visible (query, key) pair.
// Grouped attention: keys and values are the cache rows themselves, queries come prepared (normalised, rotated, bf16).
//
// mixer_prefill_kernel: the scheme of attn_prefill_tc.cu (128 query rows of one head: a softmax thread per row; a
// warp that issues the MMAs, a warp that requests the tiles; S = Q K^T double-buffered in TMEM, P written back
// over S, O accumulated in TMEM and rescaled lazily), with
//  * one or two groups of 128 rows per CTA (G): two groups share every key and value tile and take turns, one group's
//    products run under the other's softmax; each group visits only its own range of tiles,
//  * keys of two parts: NK boxes of 64 columns per 64-key tile, the first na from the expanded keys (columns h d ..; a
//    box may run into the next head's columns, which meet zero columns of Q), the rest from the cache's key part,
//  * a sliding window: tiles in front of the first visible key are never visited, and only tiles that touch the
//    diagonal or the window's edge run the mask arithmetic,
//  * latent queries: rotary positions applied while Q is staged,
//  * an optional softcap c tanh(. / c) of the scores, with tanh(z) = 1 - 2 / (1 + exp(2 z)); bound then: exponentials and
//    reciprocals, three per score,
//  * an optional sink in the denominator, the head's sigmoid gate applied to O, bf16 rows out.
// Waits are bounded as in attn_prefill_tc.cu.
#include <algorithm>

#include "dense.cuh"
#include "mixers.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int LP_Q = 128, LP_K = 64, LP_THREADS = 128;
constexpr uint32_t LP_BOX = LP_K * 64 * 2;  // bytes of one box: 64 keys x 64 columns of bf16
constexpr int LP_TAIL = 256;
constexpr float LP_RESCALE = 8.0f;  // log2 of the growth of a row maximum that triggers a rescale of O
constexpr uint32_t LP_SW128 = 2;    // layout code of the 128-byte swizzle

enum { LP_LATENT = 0, LP_GROUPED = 1, LP_GROUPED_CAP = 2 };

struct LpArgs {
  const float* y;  // projections: q at column 0 (latent), gate at off_g (-1: none)
  size_t ldy;
  const __nv_bfloat16* q16;  // grouped: prepared queries [rows][h][dq]
  const float *rope_cos, *rope_sin, *sink;
  __nv_bfloat16* z;
  size_t ldz;
  // d: columns of a head's keys in kvmap, heads dk apart, `group` query heads per key head; v_col: first value column,
  // heads dv apart; kv_rows: rows of kvmap per sequence
  int off_g, s, h, d, r, v, na, nk, rk, window, pos, kbase, cap, v_col, group, dq, dk, dv, kv_rows, z_vec;
  float scale_log2, cap_in, cap_out, out_scale;  // softcap in exponents of two: s -> cap_out tanh(log(2) / 2 cap_in s)
  int* status;
};

__device__ __forceinline__ uint32_t lp_pack(float lo, float hi) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&t);
}

__device__ __forceinline__ float lp_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// KIND: LP_*; NV: 64-column boxes of a value tile; KB, VB: key and value tiles in shared memory; G: groups of 128 query rows
template <int KIND, int NV, int KB, int VB, int G>
__global__ void __launch_bounds__(G * LP_THREADS + 64)
mixer_prefill_kernel(const LpArgs a, const __grid_constant__ CUtensorMap kvmap, const __grid_constant__ CUtensorMap cmap) {
  // TMEM of a group: S buffers in columns 0..63 and 64..127, O from 128
  constexpr int GCOLS = NV <= 2 ? 256 : 512, COLS = G * GCOLS;
  static_assert(COLS <= 512, "two groups need values of at most 128 columns");
  constexpr int SOFT = G * LP_THREADS;  // softmax threads
  extern __shared__ uint8_t sm_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(sm_raw) + 1023) & ~(uintptr_t)1023);
  const int kbytes = a.nk * (int)LP_BOX, kchunks = a.nk * 8, qbytes = LP_Q * a.nk * 128;
  uint8_t* Ks = sm;                             // [KB][nk boxes]
  uint8_t* Vs = Ks + KB * kbytes;               // [VB][NV boxes]
  uint8_t* Qs = Vs + VB * NV * (int)LP_BOX;     // [G][128][64 nk], core-matrix layout
  uint64_t* bars = reinterpret_cast<uint64_t*>(Qs + G * qbytes);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 25);
  volatile int* dead = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = __shfl_sync(0xFFFFFFFFu, tid >> 5, 0), lane = tid & 31;
  // per group: S done [2] (one per S buffer), O += P V done, P written [2]; per tile buffer: keys landed [3], values landed [2]; per
  // group and tile buffer: keys read [3], values read [2]. No barrier may run a phase ahead of its waiter: each of these
  // completes again only after what its waiter does next
  const uint32_t bar_s = smem_u32(bars), bar_o = smem_u32(bars + 4), bar_pfull = smem_u32(bars + 6), bar_kfull = smem_u32(bars + 10),
                 bar_vfull = smem_u32(bars + 13), bar_kfree = smem_u32(bars + 15), bar_vfree = smem_u32(bars + 21);
  const int qt = gridDim.x - 1 - blockIdx.x;  // longest key ranges first
  const int head = blockIdx.y, b = blockIdx.z;
  const int q0 = qt * LP_Q * G;
  // keys are counted from kbase: key j is row j - kbase of the expansions. Tiles tf[g] .. tl[g] hold the visible keys of
  // group g; the groups' ranges start and end in order and leave no tile between them out.
  int tf[G], tl[G];
  const int t_first = max(0, (a.window ? a.pos + q0 - a.window + 1 : 0) - a.kbase) / LP_K;
  int t_last = t_first;
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int qg = q0 + g * LP_Q;
    tf[g] = max(0, (a.window ? a.pos + qg - a.window + 1 : 0) - a.kbase) / LP_K;
    tl[g] = qg < a.s ? (min(a.s, qg + LP_Q) - 1 + a.pos - a.kbase) / LP_K : tf[g] - 1;
    t_last = max(t_last, tl[g]);
  }
  const int ntiles = t_last - t_first + 1;

  if (tid == 0) {
    *dead = 0;
    for (int g = 0; g < G; ++g) {
      mbar_init(bar_s + 16 * g, 1);
      mbar_init(bar_s + 16 * g + 8, 1);
      mbar_init(bar_o + 8 * g, 1);
      mbar_init(bar_pfull + 16 * g, LP_THREADS);
      mbar_init(bar_pfull + 16 * g + 8, LP_THREADS);
      for (int i = 0; i < KB; ++i) mbar_init(bar_kfree + 24 * g + 8 * i, 1);
      for (int i = 0; i < VB; ++i) mbar_init(bar_vfree + 16 * g + 8 * i, 1);
    }
    for (int i = 0; i < KB; ++i) mbar_init(bar_kfull + 8 * i, 1);
    for (int i = 0; i < VB; ++i) mbar_init(bar_vfull + 8 * i, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "n"(COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  // ---- Q, bf16, K-major operand layout
  if (KIND != LP_LATENT) {
    if (tid < SOFT) {  // [d, zeros to 64 nk]: eight threads take one 16-byte column piece of eight rows (one core matrix)
      const __nv_bfloat16* q = a.q16 + ((size_t)b * a.s + q0) * a.h * a.dq + (size_t)head * a.dq;
#pragma unroll 4
      for (int id = tid; id < G * LP_Q * kchunks; id += SOFT) {
        const int row = (id & 7) + ((id / (8 * kchunks)) << 3), c = (id >> 3) % kchunks;
        uint4 x = make_uint4(0u, 0u, 0u, 0u);
        if (q0 + row < a.s && c * 8 < a.dq) x = *reinterpret_cast<const uint4*>(q + (size_t)row * a.h * a.dq + c * 8);
        *reinterpret_cast<uint4*>(Qs + (row >> 7) * qbytes + x_kmajor(row & 127, c, kchunks)) = x;
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // these stores -> tensor-core reads
    }
  } else if (tid < SOFT) {  // rotary positions; [d, zeros to 64 na | r, zeros]
    const int half = a.r / 2, nchunks = a.na * 8, rchunks = kchunks - nchunks;
    const bool vec = ((a.d + a.r) & 3) == 0;
    auto put = [&](int row, int c, const float (&x)[8]) {
      *reinterpret_cast<uint4*>(Qs + (row >> 7) * qbytes + x_kmajor(row & 127, c, kchunks)) =
          make_uint4(lp_pack(x[0], x[1]), lp_pack(x[2], x[3]), lp_pack(x[4], x[5]), lp_pack(x[6], x[7]));
    };
    auto q_row = [&](int row) { return a.y + ((size_t)b * a.s + q0 + row) * a.ldy + (size_t)head * (a.d + a.r); };
    // eight threads take one 16-byte column piece of eight rows (one core matrix)
    if (vec) {
#pragma unroll 6
      for (int id = tid; id < G * LP_Q * nchunks; id += SOFT) {
        const int row = (id & 7) + ((id / (8 * nchunks)) << 3), c = (id >> 3) % nchunks;
        const bool in = q0 + row < a.s && c * 8 < a.d;  // d is a multiple of 8
        const float4* q = reinterpret_cast<const float4*>(in ? q_row(row) + c * 8 : a.y);
        const float4 x0 = q[0], x1 = q[1];
        const float m = in ? 1.f : 0.f;
        const float x[8] = {in ? x0.x : m, in ? x0.y : m, in ? x0.z : m, in ? x0.w : m, in ? x1.x : m, in ? x1.y : m, in ? x1.z : m, in ? x1.w : m};
        put(row, c, x);
      }
    } else {
      for (int id = tid; id < G * LP_Q * nchunks; id += SOFT) {
        const int row = (id & 7) + ((id / (8 * nchunks)) << 3), c = (id >> 3) % nchunks;
        float x[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = q0 + row < a.s && c * 8 + e < a.d ? q_row(row)[c * 8 + e] : 0.f;
        put(row, c, x);
      }
    }
    if (vec && (half & 7) == 0) {  // a thread rotates eight pairs: two pieces
      const int pchunks = half / 8, zchunks = rchunks - 2 * pchunks;
#pragma unroll 2
      for (int id = tid; id < G * LP_Q * pchunks; id += SOFT) {
        const int row = (id & 7) + ((id / (8 * pchunks)) << 3), c = (id >> 3) % pchunks;
        const bool in = q0 + row < a.s;
        const float4* u4 = reinterpret_cast<const float4*>(in ? q_row(row) + a.d + c * 8 : a.y);
        const float4* v4 = reinterpret_cast<const float4*>(in ? q_row(row) + a.d + half + c * 8 : a.y);
        const size_t tp = (size_t)(a.pos + (in ? q0 + row : 0)) * half + c * 8;
        const float4 *c4 = reinterpret_cast<const float4*>(a.rope_cos + tp), *s4 = reinterpret_cast<const float4*>(a.rope_sin + tp);
        float u[8], v[8], cs[8], sn[8], xu[8], xv[8];
        *reinterpret_cast<float4*>(u) = u4[0]; *reinterpret_cast<float4*>(u + 4) = u4[1];
        *reinterpret_cast<float4*>(v) = v4[0]; *reinterpret_cast<float4*>(v + 4) = v4[1];
        *reinterpret_cast<float4*>(cs) = c4[0]; *reinterpret_cast<float4*>(cs + 4) = c4[1];
        *reinterpret_cast<float4*>(sn) = s4[0]; *reinterpret_cast<float4*>(sn + 4) = s4[1];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          xu[e] = in ? u[e] * cs[e] - v[e] * sn[e] : 0.f;
          xv[e] = in ? v[e] * cs[e] + u[e] * sn[e] : 0.f;
        }
        put(row, nchunks + c, xu);
        put(row, nchunks + pchunks + c, xv);
      }
      const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      for (int id = tid; id < G * LP_Q * zchunks; id += SOFT)
        put((id & 7) + ((id / (8 * zchunks)) << 3), nchunks + 2 * pchunks + (id >> 3) % zchunks, zero);
    } else {
      for (int id = tid; id < G * LP_Q * rchunks; id += SOFT) {
        const int row = (id & 7) + ((id / (8 * rchunks)) << 3), c = (id >> 3) % rchunks;
        float x[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int i = c * 8 + e;
          x[e] = 0.f;
          if (q0 + row >= a.s || i >= a.r) continue;
          const float* q = q_row(row) + a.d;
          const size_t tp = (size_t)(a.pos + q0 + row) * half;
          x[e] = i < half ? q[i] * a.rope_cos[tp + i] - q[half + i] * a.rope_sin[tp + i]
                          : q[i] * a.rope_cos[tp + i - half] + q[i - half] * a.rope_sin[tp + i - half];
        }
        put(row, nchunks + c, x);
      }
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // these stores -> tensor-core reads
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();  // barriers initialised, TMEM columns allocated, Q staged
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = __shfl_sync(0xFFFFFFFFu, *tmem_slot, 0);
  // instruction descriptors: fp32 accumulator, bf16 operands, M = 128; S: N = 64, both K-major; O: N = 64 NV, B MN-major
  constexpr uint32_t IDESC_S = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LP_K >> 3) << 17) | ((uint32_t)(LP_Q >> 4) << 24);
  constexpr uint32_t IDESC_O = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(NV * 8) << 17) | ((uint32_t)(LP_Q >> 4) << 24);
  auto in_range = [&](int g, int t) { return t >= tf[g] && t <= tl[g]; };

  if (warp == SOFT / 32 + 1) {
    // ---- copy requester; tile u of the CTA is tile t_first + u
    if (lane == 0) {
      const int ky = b * a.kv_rows, cy = b * a.cap, kvh = head / a.group;
      auto fetch_k = [&](int u) {
        const uint32_t dst = smem_u32(Ks) + (uint32_t)((u % KB) * kbytes), bar = bar_kfull + 8 * (u % KB);
        const int j0 = (t_first + u) * LP_K;
        mbar_expect_tx(bar, (uint32_t)kbytes);
        for (int i = 0; i < a.na; ++i) x_tma_box2(dst + i * LP_BOX, &kvmap, kvh * a.dk + 64 * i, ky + j0, bar);
        for (int i = a.na; i < a.nk; ++i) x_tma_box2(dst + i * LP_BOX, &cmap, a.rk + 64 * (i - a.na), cy + j0, bar);
      };
      auto fetch_v = [&](int u) {
        const uint32_t dst = smem_u32(Vs) + (uint32_t)((u % VB) * NV) * LP_BOX, bar = bar_vfull + 8 * (u % VB);
        const int j0 = (t_first + u) * LP_K;
        mbar_expect_tx(bar, NV * LP_BOX);
        for (int i = 0; i < NV; ++i) x_tma_box2(dst + i * LP_BOX, &kvmap, a.v_col + kvh * a.dv + 64 * i, ky + j0, bar);
      };
      int nkt = 0, nvt = 0;  // tiles requested
      while (nkt < KB && nkt < ntiles) fetch_k(nkt++);
      while (nvt < VB && nvt < ntiles) fetch_v(nvt++);
      bool ok = true;
      int kread[G] = {}, vread[G] = {};  // per group: bit i = parity of the next phase of buffer i
      for (int u = 0; u + VB < ntiles && ok; ++u) {
        const int t = t_first + u;
        if (u + KB < ntiles) {
#pragma unroll
          for (int g = 0; g < G; ++g)  // S of every group that uses the tile is done: its key buffer is free
            if (in_range(g, t)) {
              ok = ok && x_wait(bar_kfree + 24 * g + 8 * (u % KB), (uint32_t)(kread[g] >> (u % KB)) & 1, dead, a.status);
              kread[g] ^= 1 << (u % KB);
            }
          if (ok) fetch_k(nkt++);
        }
#pragma unroll
        for (int g = 0; g < G; ++g)  // and O: its value buffer is free
          if (in_range(g, t)) {
            ok = ok && x_wait(bar_vfree + 16 * g + 8 * (u % VB), (uint32_t)(vread[g] >> (u % VB)) & 1, dead, a.status);
            vread[g] ^= 1 << (u % VB);
          }
        if (ok) fetch_v(nvt++);
      }
      if (*dead) {
        for (int u = max(0, nkt - KB); u < nkt; ++u) x_drain(bar_kfull + 8 * (u % KB), (uint32_t)((u / KB) & 1));
        for (int u = max(0, nvt - VB); u < nvt; ++u) x_drain(bar_vfull + 8 * (u % VB), (uint32_t)((u / VB) & 1));
      }
    }
  } else if (warp == SOFT / 32) {
    // ---- MMA issuer: per tile and group, S of the next tile (under the softmax of this one), then O += P V
    {  // the whole warp runs these loops, one lane issues
      uint64_t qdesc[G], kdesc[KB], vdesc[VB];  // a descriptor's low bits hold its address / 16
#pragma unroll
      for (int g = 0; g < G; ++g) qdesc[g] = x_desc(smem_u32(Qs) + (uint32_t)(g * qbytes), 128, (uint32_t)kchunks * 128);
#pragma unroll
      for (int i = 0; i < KB; ++i) kdesc[i] = x_desc(smem_u32(Ks) + (uint32_t)(i * kbytes), 16, 1024, LP_SW128);
#pragma unroll
      for (int i = 0; i < VB; ++i) vdesc[i] = x_desc(smem_u32(Vs) + (uint32_t)(i * NV) * LP_BOX, LP_BOX, 1024, LP_SW128);
      auto issue_s = [&](int g, int u) {
        const int tg = t_first + u - tf[g];
        w_wait(bar_kfull + 8 * (u % KB), (uint32_t)((u / KB) & 1), dead, a.status);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        uint64_t qd = qdesc[0], kd = kdesc[0];
#pragma unroll
        for (int i = 1; i < G; ++i) qd = g == i ? qdesc[i] : qd;
#pragma unroll
        for (int i = 1; i < KB; ++i) kd = u % KB == i ? kdesc[i] : kd;
        const uint32_t dst = tmem + (uint32_t)(g * GCOLS + (tg & 1) * LP_K);
        for (int i = 0; i < a.nk; ++i, qd += 4 * 256 / 16, kd += LP_BOX / 16)  // a box is four steps of 16 columns (zero columns of Q where it is wider)
#pragma unroll
          for (int s = 0; s < 4; ++s) w_mma(dst, qd + s * (256 / 16), kd + s * (32 / 16), IDESC_S, (i | s) ? 1u : 0u);
        w_commit(bar_s + 16 * g + 8 * (tg & 1));
        w_commit(bar_kfree + 24 * g + 8 * (u % KB));
      };
#pragma unroll
      for (int g = 0; g < G; ++g)
        if (in_range(g, t_first)) issue_s(g, 0);
      for (int u = 0; u < ntiles; ++u) {
        const int t = t_first + u;
#pragma unroll
        for (int g = 0; g < G; ++g) {
          if (u + 1 < ntiles && in_range(g, t + 1)) issue_s(g, u + 1);
          if (!in_range(g, t)) continue;
          const int tg = t - tf[g];
          w_wait(bar_pfull + 16 * g + 8 * (tg & 1), (uint32_t)((tg >> 1) & 1), dead, a.status);
          w_wait(bar_vfull + 8 * (u % VB), (uint32_t)((u / VB) & 1), dead, a.status);
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const uint32_t tm = tmem + (uint32_t)(g * GCOLS), pa = tm + (uint32_t)((tg & 1) * LP_K);
          const uint64_t vd = VB > 1 && (u & 1) ? vdesc[VB - 1] : vdesc[0];
#pragma unroll
          for (int s = 0; s < LP_K / 16; ++s)  // 16 keys = 16 rows of 128 bytes further
            w_mma_ta(tm + 2 * LP_K, pa + (uint32_t)(s * 8), vd + s * (2048 / 16), IDESC_O, (tg | s) ? 1u : 0u);
          w_commit(bar_o + 8 * g);
          w_commit(bar_vfree + 16 * g + 8 * (u % VB));
        }
      }
    }
  } else {
    // ---- softmax threads: thread r of group g owns query row q0 + 128 g + r = TMEM lane r
    const int g = G > 1 ? warp >> 2 : 0, r = tid & 127;
    const int t0 = G > 1 && g ? tf[G - 1] : tf[0], n = (G > 1 && g ? tl[G - 1] : tl[0]) - t0 + 1;
    const uint32_t tl_base = tmem + (uint32_t)(g * GCOLS) + ((uint32_t)(32 * (warp & 3)) << 16);
    const uint32_t my_s = bar_s + 16 * g, my_o = bar_o + 8 * g, my_p = bar_pfull + 16 * g;
    float m_ref = -INFINITY, l_run = 0.f;
    const int qg = q0 + g * LP_Q, row = qg + r;
    const int hi = a.pos + row - a.kbase;                      // last visible key of this row
    const int lo = a.window ? hi - a.window + 1 : -(1 << 30);  // first visible key
    const int hi_min = a.pos + qg - a.kbase;                   // of the group's rows
    const int lo_max = a.window ? min(a.s, qg + LP_Q) - 1 + a.pos - a.kbase - a.window + 1 : -(1 << 30);
    for (int t = 0; t < n; ++t) {
      const int sb = t & 1, kt = (t0 + t) * LP_K;
      x_wait(my_s + 8 * sb, (uint32_t)((t >> 1) & 1), dead, a.status);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      uint32_t sv[2][32];
      x_ld32(tl_base + (uint32_t)(sb * LP_K), sv[0]);
      x_ld32(tl_base + (uint32_t)(sb * LP_K + 32), sv[1]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      if (KIND == LP_GROUPED_CAP) {
#pragma unroll
        for (int j = 0; j < LP_K; ++j) {
          const float e = x_ex2(__uint_as_float(sv[j >> 5][j & 31]) * a.cap_in);
          sv[j >> 5][j & 31] = __float_as_uint(fmaf(-2.0f * a.cap_out, lp_rcp(1.0f + e), a.cap_out));
        }
      }
      if (kt + LP_K - 1 > hi_min || kt < lo_max) {  // the tile touches the diagonal or the window's edge of some row
#pragma unroll
        for (int j = 0; j < LP_K; ++j)
          if (kt + j > hi || kt + j < lo) sv[j >> 5][j & 31] = 0xFF800000u;  // -inf
      }
      float mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < LP_K; ++j) mx = fmaxf(mx, __uint_as_float(sv[j >> 5][j & 31]));
      const float sl2 = KIND == LP_GROUPED_CAP ? 1.0f : a.scale_log2;
      const float m_new = fmaxf(m_ref, mx * sl2);
      const bool grow = m_new > m_ref + LP_RESCALE;  // also true for the first finite maximum
      const float alpha = grow ? x_ex2(m_ref - m_new) : 1.0f;
      if (grow) m_ref = m_new;
      const float msafe = m_ref == -INFINITY ? 0.f : m_ref;
      float psum = 0.f;
      uint32_t pk[LP_K / 2];  // P as bf16 pairs
#pragma unroll
      for (int j = 0; j < LP_K / 2; ++j) {
        const float e0 = x_ex2(fmaf(__uint_as_float(sv[(2 * j) >> 5][(2 * j) & 31]), sl2, -msafe));
        const float e1 = x_ex2(fmaf(__uint_as_float(sv[(2 * j + 1) >> 5][(2 * j + 1) & 31]), sl2, -msafe));
        psum += e0 + e1;
        pk[j] = lp_pack(e0, e1);
      }
      l_run = l_run * alpha + psum;
      x_st32(tl_base + (uint32_t)(sb * LP_K), pk);
      if (t > 0 && __any_sync(0xFFFFFFFFu, grow)) {  // O is rescaled behind the previous tile's product
        x_wait(my_o, (uint32_t)((t - 1) & 1), dead, a.status);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t ov[32];
          x_ld32(tl_base + 2 * LP_K + 32 * c, ov);
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
          for (int i = 0; i < 32; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha);
          x_st32(tl_base + 2 * LP_K + 32 * c, ov);
        }
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      // before the last product can start, the one before it is seen complete: the final wait below then is for the
      // phase in progress (a parity wait must be neither two phases early nor two late)
      if (t > 0 && t == n - 1) x_wait(my_o, (uint32_t)((t - 1) & 1), dead, a.status);
      mbar_arrive(my_p + 8 * sb);
    }
    if (n > 0) {
      x_wait(my_o, (uint32_t)((n - 1) & 1), dead, a.status);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const bool store = row < a.s && !*dead;
      float scale = 0.f;
      if (store) {
        if (KIND != LP_LATENT && a.sink) l_run += exp2f(a.sink[head] * 1.4426950408889634f - m_ref);
        scale = a.out_scale / l_run;
        if (a.off_g >= 0) scale /= 1.0f + expf(-a.y[((size_t)b * a.s + row) * a.ldy + a.off_g + head]);
      }
      __nv_bfloat16* dst = a.z + ((size_t)b * a.s + row) * a.ldz + (size_t)head * a.v;
#pragma unroll
      for (int c = 0; c < NV * 2; ++c) {
        uint32_t ov[32];
        x_ld32(tl_base + 2 * LP_K + 32 * c, ov);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (store && KIND != LP_LATENT && !a.z_vec) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (32 * c + i < a.v) dst[32 * c + i] = __float2bfloat16(__uint_as_float(ov[i]) * scale);
        } else if (store) {
#pragma unroll
          for (int i = 0; i < 4; ++i)  // v is a multiple of 8: whole 16-byte pieces
            if (32 * c + 8 * i < a.v) {
              uint32_t w[4];
#pragma unroll
              for (int e = 0; e < 4; ++e)
                w[e] = lp_pack(__uint_as_float(ov[8 * i + 2 * e]) * scale, __uint_as_float(ov[8 * i + 2 * e + 1]) * scale);
              *reinterpret_cast<uint4*>(dst + 32 * c + 8 * i) = make_uint4(w[0], w[1], w[2], w[3]);
            }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 0)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(COLS) : "memory");
}

size_t lp_smem(int nk, int nv, int kb, int vb, int g) {
  size_t n = (size_t)kb * nk * LP_BOX + (size_t)vb * nv * LP_BOX + (size_t)g * LP_Q * nk * 128 + LP_TAIL + 1024;
  if (nv > 2 || g > 1) n = std::max(n, (size_t)120 * 1024);  // all 512 TMEM columns: one CTA per SM
  return n;
}

template <int KIND, int NV, int KB, int VB, int G>
int launch_lp(fb200_device* dev, const LpArgs& a, int b, const CUtensorMap& kvmap, const CUtensorMap& cmap) {
  const size_t smem = lp_smem(a.nk, NV, KB, VB, G);
  static size_t configured[64] = {0};
  if (configured[dev->ordinal & 63] < smem) {
    FB_CUDA(dev, cudaFuncSetAttribute(mixer_prefill_kernel<KIND, NV, KB, VB, G>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured[dev->ordinal & 63] = smem;
  }
  return fb200_launch(dev, mixer_prefill_kernel<KIND, NV, KB, VB, G>, dim3((unsigned)((a.s + LP_Q * G - 1) / (LP_Q * G)), (unsigned)a.h, (unsigned)b),
                      dim3(G * LP_THREADS + 64), smem, false, a, kvmap, cmap);
}

constexpr float LP_LOG2E = 1.4426950408889634f;

template <int KIND>
int launch_kind(fb200_device* dev, const LpArgs& p, int b, const CUtensorMap& kvmap, const CUtensorMap& cmap) {
  const int nv = (p.v + 63) / 64;
  // two groups of rows per CTA once one per CTA would not fit the SMs at a time anyway; three key and two value tiles
  // where they fit
  const long ctas = (long)((p.s + LP_Q - 1) / LP_Q) * p.h * b;
  if (nv <= 2 && ctas > dev->sm_count && lp_smem(p.nk, nv, 3, 2, 2) <= 227 * 1024)
    return nv == 1 ? launch_lp<KIND, 1, 3, 2, 2>(dev, p, b, kvmap, cmap) : launch_lp<KIND, 2, 3, 2, 2>(dev, p, b, kvmap, cmap);
  const bool deep = lp_smem(p.nk, nv, 3, 2, 1) <= 227 * 1024;
  switch (nv * 2 + (deep ? 1 : 0)) {
    case 2: return launch_lp<KIND, 1, 2, 1, 1>(dev, p, b, kvmap, cmap);
    case 3: return launch_lp<KIND, 1, 3, 2, 1>(dev, p, b, kvmap, cmap);
    case 4: return launch_lp<KIND, 2, 2, 1, 1>(dev, p, b, kvmap, cmap);
    case 5: return launch_lp<KIND, 2, 3, 2, 1>(dev, p, b, kvmap, cmap);
    case 6: return launch_lp<KIND, 3, 2, 1, 1>(dev, p, b, kvmap, cmap);
    case 7: return launch_lp<KIND, 3, 3, 2, 1>(dev, p, b, kvmap, cmap);
    case 8: return launch_lp<KIND, 4, 2, 1, 1>(dev, p, b, kvmap, cmap);
    default: return launch_lp<KIND, 4, 3, 2, 1>(dev, p, b, kvmap, cmap);
  }
}

}  // namespace

// Shapes the tensor-core path covers: 16-byte aligned columns and a tile that fits shared memory.
bool fb200_latent_prefill_covers(int h, int d, int r, int v, int rk, float scale) {
  return d % 8 == 0 && v % 8 == 0 && rk % 8 == 0 && d <= 256 && r <= 128 && v <= 256 && h <= 65535 && scale > 0.f &&
         lp_smem((d + 63) / 64 + (r + 63) / 64, (v + 63) / 64, 2, 1, 1) <= 227 * 1024;
}

// The new positions' latents must already be in the cache. a.kvx holds b * keys rows of kv_ld elements.
int fb200_latent_prefill(fb200_device* dev, const fb200_latent_args& a, const fb200_qmatrix* w_ukv) {
  const int kbase = a.window ? std::max(0, a.pos - a.window + 1) : 0, keys = a.pos + a.s - kbase;
  const int kv_ld = a.h * (a.d + a.v);  // a multiple of 8
  int rc;
  for (int b = 0; b < a.b; ++b) {
    fb200_dense_job j;
    j.w = w_ukv; j.m = keys; j.kx = a.rk; j.ldx = a.ldc;
    j.x = (const __nv_bfloat16*)a.cache + ((size_t)b * a.cap + kbase) * a.ldc;
    j.n_plain = kv_ld; j.y = a.kvx + (size_t)b * keys * kv_ld; j.ldy = kv_ld; j.y_bf16 = 1;
    if ((rc = fb200_dense_gemm_tc(dev, j))) return rc;
  }
  CUtensorMap kvmap, cmap;
  if (!fb200_make_map_2d(&kvmap, a.kvx, 1, (uint64_t)kv_ld, (uint64_t)a.b * keys, (uint64_t)kv_ld * 2, LP_K) ||
      !fb200_make_map_2d(&cmap, (const __nv_bfloat16*)a.cache + (size_t)kbase * a.ldc, 1, (uint64_t)(a.rk + a.r),
                         (uint64_t)(a.b - 1) * a.cap + keys, (uint64_t)a.ldc * 2, LP_K))
    return fb200_fail(dev, FB200_ERR_CUDA, "latent attention: tensor map refused");
  LpArgs p = {};
  p.y = a.y; p.ldy = a.ldy; p.rope_cos = a.rope_cos; p.rope_sin = a.rope_sin; p.z = (__nv_bfloat16*)a.z; p.ldz = a.ldz; p.off_g = a.off_g;
  p.s = a.s; p.h = a.h; p.d = a.d; p.r = a.r; p.v = a.v; p.na = (a.d + 63) / 64; p.nk = p.na + (a.r + 63) / 64; p.rk = a.rk;
  p.window = a.window; p.pos = a.pos; p.kbase = kbase; p.kv_rows = keys; p.cap = a.cap; p.v_col = a.h * a.d;
  p.group = 1; p.dk = a.d; p.dv = a.v; p.z_vec = 1; p.out_scale = 1.f;
  p.scale_log2 = a.scale * LP_LOG2E; p.status = dev->status;
  return launch_kind<LP_LATENT>(dev, p, a.b, kvmap, cmap);
}

bool fb200_attn_prefill_covers(int h, int d, int v, float scale) {
  return d <= 256 && v <= 256 && h <= 65535 && scale > 0.f && lp_smem((d + 63) / 64, (v + 63) / 64, 2, 1, 1) <= 227 * 1024;
}

// a.qn holds b * s rows of prepared bf16 queries; keys and values are the cache rows.
int fb200_attn_prefill(fb200_device* dev, const fb200_attn_args& a) {
  int rc;
  if ((rc = fb200_attn_prepare(dev, a, true))) return rc;
  const int kbase = a.window ? std::max(0, a.pos - a.window + 1) : 0, keys = a.pos + a.s - kbase;
  CUtensorMap map;
  if (!fb200_make_map_2d(&map, (const __nv_bfloat16*)a.cache + (size_t)kbase * a.ldc, 1, (uint64_t)a.ldc, (uint64_t)(a.b - 1) * a.cap + keys,
                         (uint64_t)a.ldc * 2, LP_K))
    return fb200_fail(dev, FB200_ERR_CUDA, "grouped attention: tensor map refused");
  LpArgs p = {};
  p.y = a.y; p.ldy = a.ldy; p.q16 = (const __nv_bfloat16*)a.qn; p.sink = a.sink; p.z = (__nv_bfloat16*)a.z; p.ldz = a.ldz; p.off_g = a.off_g;
  p.s = a.s; p.h = a.h; p.d = a.d; p.v = a.v; p.na = p.nk = (a.d + 63) / 64; p.window = a.window; p.pos = a.pos; p.kbase = kbase;
  p.cap = p.kv_rows = a.cap; p.v_col = a.g * a.dp; p.group = a.h / a.g; p.dq = p.dk = a.dp; p.dv = a.vp;
  p.z_vec = a.v % 8 == 0 && a.ldz % 8 == 0 && ((uintptr_t)a.z & 15u) == 0; p.out_scale = a.out_scale;
  p.scale_log2 = a.scale * LP_LOG2E; p.status = dev->status;
  if (a.softcap > 0.f) {
    p.cap_in = 2.f * LP_LOG2E * a.scale / a.softcap;
    p.cap_out = a.softcap * LP_LOG2E;
    return launch_kind<LP_GROUPED_CAP>(dev, p, a.b, map, map);
  }
  return launch_kind<LP_GROUPED>(dev, p, a.b, map, map);
}
