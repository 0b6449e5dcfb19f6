// Linear attention of a prompt pass on the 5th-generation tensor cores (heads of up to 128).
//
// A CTA walks one head of one sequence in chunks of 128 tokens, 64 value columns wide. With S [d][64] the state before a
// chunk of n tokens, D_ij = decay^(i-j) for j <= i and else 0,
//   A = Q K^T,   O = diag(decay^(i+1)) Q S + (D * A) V,   S <- decay^n S + K^T diag(decay^(n-1-i)) V.
// A, the two parts of O and S are f32 accumulators in tensor memory. S, D * A and the decayed V enter their products as a bf16
// value and a bf16 remainder each (two products), so that beside the bf16 q, k and v everything keeps (nearly) 32 bits.
// Roles, coupled only by mbarriers:
//  * four groups of four warps: (P) D * A, written over A in tensor memory; (S) the state: hands it to the next chunk as an
//    operand in shared memory and scales the accumulator; (V) the decayed values, in shared memory; (O) the read-out to global memory;
//  * copy requester: q, k and v of a chunk by tensor TMA (128-byte swizzle), two chunks in shared memory;
//  * MMA issuer: A of the next chunk, then Q S, K^T V and (D * A) V of this one.
// Every wait is bounded (2^22 polls); a wait that gives up sets the device status word and makes the other roles leave.
#include <algorithm>

#include "dense.cuh"
#include "mixers.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int LT_C = FB200_LINEAR_CHUNK, LT_GROUP = 128, LT_THREADS = 4 * LT_GROUP + 64;
constexpr uint32_t LT_BOX = 128 * 64 * 2;  // 128 tokens (or rows of S) x 64 columns of bf16, rows of 128 bytes
constexpr uint32_t LT_STAGE = 5 * LT_BOX;  // q, q, k, k, v
constexpr uint32_t LT_VT = 2 * LT_STAGE, LT_ST = LT_VT + 2 * LT_BOX, LT_BARS = LT_ST + 2 * LT_BOX;
constexpr int LT_NBARS = 14;
constexpr uint32_t LT_TABLE = LT_BARS + 8 * LT_NBARS + 16;
constexpr uint32_t LT_SMEM = LT_TABLE + (2 * LT_C + 1) * 4 + 1024;
static_assert(LT_C == 128 && LT_SMEM <= 227 * 1024, "shared memory of a CTA");
// columns in tensor memory: A of even and odd chunks, Q S, (D * A) V, S
constexpr uint32_t TM_A = 0, TM_O1 = 256, TM_O2 = 320, TM_S = 384, TM_COLS = 512;
constexpr uint32_t SW128 = 2;

// byte offset of the 16-byte piece c of row r in a box (128-byte swizzle)
__device__ __forceinline__ uint32_t box_at(int r, int c) { return (uint32_t)(r * 128 + ((c ^ (r & 7)) << 4)); }
// two f32 as bf16 values and bf16 remainders
__device__ __forceinline__ void lt_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

__global__ void __launch_bounds__(LT_THREADS, 1)
linear_prefill_kernel(const fb200_linear_args a, int vp, int* status, const __grid_constant__ CUtensorMap qmap,
                      const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap) {
  extern __shared__ uint8_t sm_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(sm_raw) + 1023) & ~(uintptr_t)1023);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(sm + LT_BARS + 8 * LT_NBARS);
  volatile int* dead = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* table = reinterpret_cast<float*>(sm + LT_TABLE);  // zeros in front of the powers 0 .. 128
  const float* pw = table + LT_C;
  const uint32_t base = smem_u32(sm), bars = base + LT_BARS;
  // tiles landed [2], chunk finished [2], A done [2], P written [2]; one phase per chunk: S handed over, V decayed, state updated,
  // O done, O read; end
  const uint32_t b_full = bars, b_free = bars + 16, b_a = bars + 32, b_p = bars + 48, b_st = bars + 64, b_vt = bars + 72, b_kv = bars + 80,
                 b_o = bars + 88, b_read = bars + 96, b_end = bars + 104;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, group = warp >> 2, r = tid & 127;
  const int c0 = blockIdx.x * 64, h = blockIdx.y, b = blockIdx.z, chunks = (a.s + LT_C - 1) / LT_C, nkb = a.dp / 64, row0 = b * a.s;
  for (int i = tid; i <= 2 * LT_C; i += LT_THREADS) table[i] = i < LT_C ? 0.f : a.decay[(size_t)h * (LT_C + 1) + i - LT_C];
  if (tid == 0) {
    *dead = 0;
    for (int i = 0; i < 2; ++i) {
      mbar_init(b_full + 8 * i, 1);
      mbar_init(b_free + 8 * i, 1);
      mbar_init(b_a + 8 * i, 1);
      mbar_init(b_p + 8 * i, LT_GROUP);
    }
    mbar_init(b_st, LT_GROUP);
    mbar_init(b_vt, LT_GROUP);
    mbar_init(b_kv, 1);
    mbar_init(b_o, 1);
    mbar_init(b_read, LT_GROUP);
    mbar_init(b_end, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "n"(TM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (nkb == 1) {  // the rows 64 .. 127 of S come from the second box of k: zeros
    for (int i = tid; i < 2 * (int)LT_BOX / 16; i += LT_THREADS)
      *reinterpret_cast<uint4*>(sm + (i / (LT_BOX / 16)) * LT_STAGE + 3 * LT_BOX + (i % (LT_BOX / 16)) * 16) = make_uint4(0u, 0u, 0u, 0u);
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *tmem_slot, lanes = (uint32_t)(32 * (warp & 3)) << 16;
  auto tokens_of = [&](int c) { return min(LT_C, a.s - c * LT_C); };

  if (warp == 16) {
    // ---- copy requester
    if (lane == 0) {
      int issued = 0;
      for (int c = 0; c < chunks; ++c, ++issued) {
        const int s = c & 1;
        if (c >= 2 && !x_wait(b_free + 8 * s, (uint32_t)((c >> 1) - 1) & 1, dead, status)) break;
        const uint32_t dst = base + s * LT_STAGE, bar = b_full + 8 * s;
        mbar_expect_tx(bar, (uint32_t)(2 * nkb + 1) * LT_BOX);
        for (int i = 0; i < nkb; ++i) {
          x_tma_box2(dst + i * LT_BOX, &qmap, h * a.dp + 64 * i, row0 + c * LT_C, bar);
          x_tma_box2(dst + (2 + i) * LT_BOX, &kmap, h * a.dp + 64 * i, row0 + c * LT_C, bar);
        }
        x_tma_box2(dst + 4 * LT_BOX, &vmap, h * vp + c0, row0 + c * LT_C, bar);
      }
      if (*dead)
        for (int c = max(0, issued - 2); c < issued; ++c) x_drain(b_full + 8 * (c & 1), (uint32_t)(c >> 1) & 1);
    }
  } else if (warp == 17) {
    // ---- MMA issuer. bf16 operands, f32 accumulator, M = 128; bit 15 / 16: A / B rows run along K (MN-major)
    if (lane == 0) {
      constexpr uint32_t ID = (1u << 4) | (1u << 7) | (1u << 10) | (8u << 24);
      constexpr uint32_t ID_A = ID | (16u << 17), ID_O = ID | (8u << 17) | (1u << 16), ID_S = ID | (8u << 17) | (1u << 16) | (1u << 15);
      const int ksteps = a.dp / 16;
      auto kmajor = [&](uint32_t at, int k) { return x_desc(at + (uint32_t)(k >> 2) * LT_BOX, 16, 1024, SW128) + (uint64_t)((k & 3) * 2); };
      auto mnmajor = [&](uint32_t at, int k) { return x_desc(at, LT_BOX, 1024, SW128) + (uint64_t)(k * (2048 / 16)); };
      auto issue_a = [&](int c) {
        const int s = c & 1;
        if (!x_wait(b_full + 8 * s, (uint32_t)(c >> 1) & 1, dead, status)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t q = base + s * LT_STAGE, k = q + 2 * LT_BOX;
        for (int i = 0; i < ksteps; ++i) x_mma(tmem + TM_A + (uint32_t)s * 128, kmajor(q, i), kmajor(k, i), ID_A, i ? 1u : 0u);
        x_commit(b_a + 8 * s);
        return true;
      };
      bool ok = issue_a(0);
      for (int c = 0; c < chunks && ok; ++c) {
        const int s = c & 1;
        const uint32_t q = base + s * LT_STAGE, k = q + 2 * LT_BOX, v = q + 4 * LT_BOX;
        // the other A buffer is free: the product that read it was issued before
        if (c + 1 < chunks) ok = issue_a(c + 1);
        ok = ok && x_wait(b_st, (uint32_t)c & 1, dead, status);
        ok = ok && (c == 0 || x_wait(b_read, (uint32_t)(c - 1) & 1, dead, status));
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (int p = 0; p < 2; ++p)
          for (int i = 0; i < ksteps; ++i)
            x_mma(tmem + TM_O1, kmajor(q, i), mnmajor(base + LT_ST + p * LT_BOX, i), ID_O, (p | i) ? 1u : 0u);
        ok = x_wait(b_vt, (uint32_t)c & 1, dead, status);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (int p = 0; p < 2; ++p)
          for (int i = 0; i < LT_C / 16; ++i) x_mma(tmem + TM_S, mnmajor(k, i), mnmajor(base + LT_VT + p * LT_BOX, i), ID_S, 1u);
        x_commit(b_kv);
        ok = x_wait(b_p + 8 * s, (uint32_t)(c >> 1) & 1, dead, status);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (int p = 0; p < 2; ++p)
          for (int i = 0; i < LT_C / 16; ++i)  // 32 keys: 16 columns of values, 16 of remainders
            x_mma_ta(tmem + TM_O2, tmem + TM_A + (uint32_t)(s * 128 + (i >> 1) * 32 + (i & 1) * 8 + p * 16), mnmajor(v, i), ID_O, (p | i) ? 1u : 0u);
        x_commit(b_o);
        x_commit(b_free + 8 * s);
      }
      x_commit(b_end);
      x_drain(b_end, 0);
    }
  } else if (group == 0) {
    // ---- P: row r of D * A over row r of A
    for (int c = 0; c < chunks; ++c) {
      const int s = c & 1;
      if (!x_wait(b_a + 8 * s, (uint32_t)(c >> 1) & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t at = tmem + lanes + TM_A + (uint32_t)s * 128;
#pragma unroll 1
      for (int kb = 0; kb < 4; ++kb) {
        uint32_t w[32];
        if (kb <= warp) {  // some of the keys 32 kb .. are in front of this warp's rows
          uint32_t x[32];
          x_ld32(at + 32 * kb, x);
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
          const float* d = pw + r - 32 * kb;
#pragma unroll
          for (int e = 0; e < 16; ++e)
            lt_split(__uint_as_float(x[2 * e]) * d[-2 * e], __uint_as_float(x[2 * e + 1]) * d[-2 * e - 1], w[e], w[16 + e]);
        } else {
#pragma unroll
          for (int e = 0; e < 32; ++e) w[e] = 0u;
        }
        x_st32(at + 32 * kb, w);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(b_p + 8 * s);
    }
  } else if (group == 1) {
    // ---- S: row r (a dimension of k) of the state
    const uint32_t at = tmem + lanes + TM_S;
    float* state = a.state + (((size_t)b * a.h + h) * a.v + c0) * (size_t)a.dp + r;
    const int cols = min(64, a.v - c0);
    const bool row_in = r < a.dp, old = *a.pos_dev > 0;
    // 32 columns: operand for the next chunk, and the accumulator scaled by its decay
    auto hand_over = [&](uint32_t (&x)[32], int half, float f) {
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) lt_split(__uint_as_float(x[8 * p + 2 * e]), __uint_as_float(x[8 * p + 2 * e + 1]), hi[e], lo[e]);
        const uint32_t off = box_at(r, half * 4 + p);
        *reinterpret_cast<uint4*>(sm + LT_ST + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(sm + LT_ST + LT_BOX + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
#pragma unroll
      for (int e = 0; e < 32; ++e) x[e] = __float_as_uint(__uint_as_float(x[e]) * f);
      x_st32(at + 32 * half, x);
    };
    auto ready = [&]() {
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(b_st);
    };
#pragma unroll 1
    for (int half = 0; half < 2; ++half) {
      uint32_t x[32];
#pragma unroll
      for (int e = 0; e < 32; ++e) x[e] = old && row_in && 32 * half + e < cols ? __float_as_uint(state[(size_t)(32 * half + e) * a.dp]) : 0u;
      hand_over(x, half, pw[tokens_of(0)]);
    }
    ready();
    for (int c = 0; c < chunks; ++c) {
      if (!x_wait(b_kv, (uint32_t)c & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const bool end = c + 1 == chunks;
      const float f = end ? 0.f : pw[tokens_of(c + 1)];
#pragma unroll 1
      for (int half = 0; half < 2; ++half) {
        uint32_t x[32];
        x_ld32(at + 32 * half, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (!end) {
          hand_over(x, half, f);
        } else if (row_in) {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if (32 * half + e < cols) state[(size_t)(32 * half + e) * a.dp] = __uint_as_float(x[e]);
        }
      }
      if (!end) ready();
    }
  } else if (group == 2) {
    // ---- V: token r of the decayed values
    for (int c = 0; c < chunks; ++c) {
      if (!x_wait(b_full + 8 * (c & 1), (uint32_t)(c >> 1) & 1, dead, status)) break;
      if (c && !x_wait(b_kv, (uint32_t)(c - 1) & 1, dead, status)) break;
      const uint8_t* v = sm + (c & 1) * LT_STAGE + 4 * LT_BOX;
      const int n = tokens_of(c);
      const float f = r < n ? pw[n - 1 - r] : 0.f;
#pragma unroll
      for (int p = 0; p < 8; ++p) {
        const uint32_t off = box_at(r, p);
        const uint4 x = *reinterpret_cast<const uint4*>(v + off);
        const uint32_t u[4] = {x.x, x.y, x.z, x.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          lt_split(r < n ? __uint_as_float(u[e] << 16) * f : 0.f, r < n ? __uint_as_float(u[e] & 0xFFFF0000u) * f : 0.f, hi[e], lo[e]);
        *reinterpret_cast<uint4*>(sm + LT_VT + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(sm + LT_VT + LT_BOX + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      mbar_arrive(b_vt);
    }
  } else {
    // ---- O: token r of the read-out
    const int hv = a.h * a.v, cols = min(64, a.v - c0);
    const bool vec = a.v % 4 == 0;
    const float f = pw[r + 1];
    for (int c = 0; c < chunks; ++c) {
      if (!x_wait(b_o, (uint32_t)c & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      float o[64];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t x[32], y[32];
        x_ld32(tmem + lanes + TM_O1 + 32 * half, x);
        x_ld32(tmem + lanes + TM_O2 + 32 * half, y);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int e = 0; e < 32; ++e) o[32 * half + e] = fmaf(__uint_as_float(x[e]), f, __uint_as_float(y[e]));
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(b_read);
      if (r < tokens_of(c)) {
        float* dst = a.o + (size_t)(row0 + c * LT_C + r) * hv + (size_t)h * a.v + c0;
#pragma unroll
        for (int e = 0; e < 64; e += 4) {
          if (vec && e < cols) *reinterpret_cast<float4*>(dst + e) = make_float4(o[e], o[e + 1], o[e + 2], o[e + 3]);
          if (!vec) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (e + i < cols) dst[e + i] = o[e + i];
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(TM_COLS) : "memory");
}

}  // namespace

bool fb200_linear_prefill_covers(const fb200_linear_args& a) { return a.bf16 && (a.dp == 64 || a.dp == 128) && a.h <= 65535 && a.b <= 65535; }

int fb200_linear_prefill(fb200_device* dev, const fb200_linear_args& a) {
  const int vp = (a.v + 7) / 8 * 8;
  const uint64_t rows = (uint64_t)a.b * a.s;
  CUtensorMap q, k, v;
  if (!fb200_make_map_2d(&q, a.q16, 1, (uint64_t)a.h * a.dp, rows, (uint64_t)a.h * a.dp * 2, LT_C) ||
      !fb200_make_map_2d(&k, a.k16, 1, (uint64_t)a.h * a.dp, rows, (uint64_t)a.h * a.dp * 2, LT_C) ||
      !fb200_make_map_2d(&v, a.v16, 1, (uint64_t)a.h * vp, rows, (uint64_t)a.h * vp * 2, LT_C))
    return fb200_fail(dev, FB200_ERR_CUDA, "linear attention: tensor map refused");
  static bool configured[64] = {false};
  if (!configured[dev->ordinal & 63]) {
    FB_CUDA(dev, cudaFuncSetAttribute(linear_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM));
    configured[dev->ordinal & 63] = true;
  }
  return fb200_launch(dev, linear_prefill_kernel, dim3((unsigned)((a.v + 63) / 64), (unsigned)a.h, (unsigned)a.b), dim3(LT_THREADS), LT_SMEM, false, a,
                      vp, dev->status, q, k, v);
}
