// Linear attention of a prompt pass on the 5th-generation tensor cores (heads of up to 128).
//
// A CTA walks one head of one sequence in chunks of 128 tokens, 64 value columns wide. With S [d][64] the state before a
// chunk of n tokens, D_ij = decay^(i-j) for j <= i and else 0,
//   A = Q K^T,   O = diag(decay^(i+1)) Q S + (D * A) V,   S <- decay^n S + K^T diag(decay^(n-1-i)) V.
// A, the two parts of O and S are f32 accumulators in tensor memory. S, D * A and the decayed V enter their products as a bf16
// value and a bf16 remainder each (two products), so that beside the bf16 q, k and v everything keeps (nearly) 32 bits.
// Roles, coupled only by mbarriers:
//  * four groups of four warps: (P) D * A, written over A in tensor memory; (S) the state: hands it to the next chunk as an
//    operand in shared memory and scales the accumulator; (V) the decayed values, in shared memory; (O) the read-out: Q S times the
//    decays, onto which (D * A) V is accumulated, and the sum to global memory;
//  * copy requester: q, k and v of a chunk by tensor TMA (128-byte swizzle), two chunks in shared memory;
//  * two MMA issuers: one the state's way round (Q S and K^T V of a chunk), one A of the next chunk and (D * A) V of this one.
// Few heads leave SMs idle, so a long prompt is cut into segments that run side by side: a first launch forms what every
// segment adds to the state (K^T V alone, the decays counted to the segment's end), and a segment of the second launch starts
// from the state those give.
// Every wait is bounded (2^22 polls); a wait that gives up sets the device status word and makes the other roles leave.
#include <algorithm>

#include "dense.cuh"
#include "mixers.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int LT_C = FB200_LINEAR_CHUNK, LT_GROUP = 128, LT_THREADS = 4 * LT_GROUP + 96;
constexpr uint32_t LT_BOX = 128 * 64 * 2;  // 128 tokens (or rows of S) x 64 columns of bf16, rows of 128 bytes
constexpr uint32_t LT_STAGE = 5 * LT_BOX;  // q, q, k, k, v
constexpr uint32_t LT_VT = 2 * LT_STAGE, LT_ST = LT_VT + 2 * LT_BOX, LT_BARS = LT_ST + 2 * LT_BOX;
constexpr int LT_NBARS = 20;
constexpr uint32_t LT_TABLE = LT_BARS + 8 * LT_NBARS + 16;
constexpr uint32_t LT_SMEM = LT_TABLE + (2 * LT_C + 1) * 4 + 1024;
static_assert(LT_C == 128 && LT_SMEM <= 227 * 1024, "shared memory of a CTA");
// columns in tensor memory: A of even and odd chunks, Q S (values, remainders of S), O, S
constexpr uint32_t TM_A = 0, TM_O1 = 256, TM_O2 = 384, TM_S = 448, TM_COLS = 512;
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

// STATE: the first launch of a prompt in segments (`per` chunks each); NKB: 64-element boxes of a q or k row
template <bool STATE, int NKB>
__global__ void __launch_bounds__(LT_THREADS, 1)
linear_prefill_kernel(const fb200_linear_args a, int vp, int nseg, int per, int* status, const __grid_constant__ CUtensorMap qmap,
                      const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap) {
  extern __shared__ uint8_t sm_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(sm_raw) + 1023) & ~(uintptr_t)1023);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(sm + LT_BARS + 8 * LT_NBARS);
  volatile int* dead = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* table = reinterpret_cast<float*>(sm + LT_TABLE);  // zeros in front of the powers 0 .. 128
  const float* pw = table + LT_C;
  const uint32_t base = smem_u32(sm), bars = base + LT_BARS;
  // q and k landed [2], v landed [2], q and k free [2], v free [2], A done [2], P written [2], V decayed [2]; one phase per chunk: S
  // handed over, state updated, O done, Q S taken over into O; end
  const uint32_t b_qk = bars, b_v = bars + 16, b_qkfree = bars + 32, b_vfree = bars + 48, b_a = bars + 64, b_p = bars + 80, b_vt = bars + 96,
                 b_st = bars + 112, b_kv = bars + 120, b_o = bars + 128, b_read = bars + 136, b_end = bars + 144;
  const int tid = threadIdx.x, warp = __shfl_sync(0xFFFFFFFFu, tid >> 5, 0), lane = tid & 31, group = warp >> 2, r = tid & 127;
  const int seg = (int)blockIdx.x % nseg, c0 = (int)blockIdx.x / nseg * 64, h = blockIdx.y, b = blockIdx.z;
  const int all = (a.s + LT_C - 1) / LT_C, ch0 = seg * per, chunks = min(per, all - ch0);
  const int row0 = b * a.s + ch0 * LT_C, tokens = a.s - ch0 * LT_C;  // first row; tokens from there on
  const size_t state_at = (((size_t)b * a.h + h) * a.v + c0) * (size_t)a.dp + r, seg_size = (size_t)a.b * a.h * a.v * a.dp;
  const int cols = min(64, a.v - c0);
  const bool row_in = r < a.dp;
  if (STATE && seg == nseg - 1) {  // nobody starts from the last segment's end; the state in front of the prompt, for all of them
    const bool old = *a.pos_dev > 0;
    if (group == 0 && row_in)
      for (int v = 0; v < cols; ++v) a.seg[state_at + (size_t)v * a.dp] = old ? a.state[state_at + (size_t)v * a.dp] : 0.f;
    return;
  }
  for (int i = tid; i <= 2 * LT_C; i += LT_THREADS) table[i] = i < LT_C ? 0.f : a.decay[(size_t)h * (LT_C + 1) + i - LT_C];
  if (tid == 0) {
    *dead = 0;
    for (int i = 0; i < 2; ++i) {
      for (uint32_t bar : {b_qk, b_v, b_vfree, b_a}) mbar_init(bar + 8 * i, 1);
      mbar_init(b_qkfree + 8 * i, STATE ? 1 : 2);
      mbar_init(b_p + 8 * i, LT_GROUP);
      mbar_init(b_vt + 8 * i, LT_GROUP);
    }
    mbar_init(b_st, LT_GROUP);
    mbar_init(b_kv, 1);
    mbar_init(b_o, 1);
    mbar_init(b_read, LT_GROUP);
    mbar_init(b_end, STATE ? 1 : 2);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "n"(TM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (NKB == 1) {  // the rows 64 .. 127 of S come from the second box of k: zeros
    for (int i = tid; i < 2 * (int)LT_BOX / 16; i += LT_THREADS)
      *reinterpret_cast<uint4*>(sm + (i / (LT_BOX / 16)) * LT_STAGE + 3 * LT_BOX + (i % (LT_BOX / 16)) * 16) = make_uint4(0u, 0u, 0u, 0u);
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = __shfl_sync(0xFFFFFFFFu, *tmem_slot, 0), lanes = (uint32_t)(32 * (warp & 3)) << 16;
  auto tokens_of = [&](int c) { return min(LT_C, tokens - c * LT_C); };
  // where the decayed values of a chunk lie: the first launch has no use for the operand form of S
  auto vt_at = [&](int c) { return STATE && (c & 1) ? LT_ST : LT_VT; };

  if (warp == 16) {
    // ---- copy requester
    if (lane == 0) {
      int issued = 0;
      for (int c = 0; c < chunks; ++c, ++issued) {
        const int s = c & 1, y = row0 + c * LT_C;
        const uint32_t dst = base + s * LT_STAGE, again = (uint32_t)((c >> 1) - 1) & 1;
        if (c >= 2 && !x_wait(b_qkfree + 8 * s, again, dead, status)) break;
        mbar_expect_tx(b_qk + 8 * s, (uint32_t)((STATE ? 1 : 2) * NKB) * LT_BOX);
#pragma unroll
        for (int i = 0; i < NKB; ++i) {
          if (!STATE) x_tma_box2(dst + i * LT_BOX, &qmap, h * a.dp + 64 * i, y, b_qk + 8 * s);
          x_tma_box2(dst + (2 + i) * LT_BOX, &kmap, h * a.dp + 64 * i, y, b_qk + 8 * s);
        }
        // (a give-up between the two copies of a chunk leaves the first one in flight: drained here, the others below)
        if (c >= 2 && !x_wait(b_vfree + 8 * s, again, dead, status)) {
          x_drain(b_qk + 8 * s, (uint32_t)(c >> 1) & 1);
          break;
        }
        mbar_expect_tx(b_v + 8 * s, LT_BOX);
        x_tma_box2(dst + 4 * LT_BOX, &vmap, h * vp + c0, y, b_v + 8 * s);
      }
      if (*dead)
        for (int c = max(0, issued - 2); c < issued; ++c) {
          x_drain(b_qk + 8 * (c & 1), (uint32_t)(c >> 1) & 1);
          x_drain(b_v + 8 * (c & 1), (uint32_t)(c >> 1) & 1);
        }
    }
  } else if (warp >= 17) {
    // ---- MMA issuers. bf16 operands, f32 accumulator, M = 128; bit 15 / 16: A / B rows run along K (MN-major)
    if (!(STATE && warp == 18)) {
      constexpr uint32_t ID = (1u << 4) | (1u << 7) | (1u << 10) | (8u << 24);
      constexpr uint32_t ID_A = ID | (16u << 17), ID_O1 = ID_A | (1u << 16), ID_O2 = ID | (8u << 17) | (1u << 16), ID_S = ID_O2 | (1u << 15);
      // the whole warp runs these loops, one lane issues. Descriptors: bases here, constant steps in unrolled loops. A step of 16
      // elements of K is 32 bytes inside the rows of a K-major box and 16 rows of an MN-major one
      uint64_t qk[2], kk[2], kn[2], vn[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const uint32_t at = base + i * LT_STAGE;
        qk[i] = x_desc(at, 16, 1024, SW128);
        kk[i] = x_desc(at + 2 * LT_BOX, 16, 1024, SW128);
        kn[i] = x_desc(at + 2 * LT_BOX, LT_BOX, 1024, SW128);
        vn[i] = x_desc(at + 4 * LT_BOX, LT_BOX, 1024, SW128);
      }
      const uint64_t vt0 = x_desc(base + LT_VT, LT_BOX, 1024, SW128), st0 = x_desc(base + LT_ST, LT_BOX, 1024, SW128);
      auto kstep = [](int i) { return (uint64_t)((i >> 2) * (LT_BOX / 16) + (i & 3) * 2); };
      auto nstep = [](int i) { return (uint64_t)(i * (2048 / 16)); };
      auto wait = [&](uint32_t bar, int phase) { return w_wait(bar, (uint32_t)phase & 1, dead, status); };
      auto landed = [&](int c) {
        if (!wait(b_qk + 8 * (c & 1), c >> 1)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        return true;
      };
      auto issue_a = [&](int c) {
        if (!landed(c)) return false;
        const uint64_t q = c & 1 ? qk[1] : qk[0], k = c & 1 ? kk[1] : kk[0];
        const uint32_t d = tmem + TM_A + (uint32_t)(c & 1) * 128;
#pragma unroll
        for (int i = 0; i < 4 * NKB; ++i) w_mma(d, q + kstep(i), k + kstep(i), ID_A, i ? 1u : 0u);
        w_commit(b_a + 8 * (c & 1));
        w_commit(b_qkfree + 8 * (c & 1));
        return true;
      };
      auto issue_s = [&](int c) {
        const uint64_t k = c & 1 ? kn[1] : kn[0], vt = STATE && (c & 1) ? st0 : vt0;
#pragma unroll
        for (int i = 0; i < 2 * LT_C / 16; ++i)
          w_mma(tmem + TM_S, k + nstep(i & 7), vt + (i >> 3) * (LT_BOX / 16) + nstep(i & 7), ID_S, STATE && (c | i) == 0 ? 0u : 1u);
      };
      if (warp == 17) {
        for (int c = 0; c < chunks; ++c) {
          const int s = c & 1;
          if (!landed(c)) break;
          if (!STATE) {
            if (!wait(b_st, c) || (c && !wait(b_read, c - 1))) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint64_t q = s ? qk[1] : qk[0];
#pragma unroll
            for (int i = 0; i < 4 * NKB; ++i) w_mma(tmem + TM_O1, q + kstep(i), st0 + nstep(i), ID_O1, i ? 1u : 0u);
          }
          if (!wait(b_vt + 8 * s, c >> 1)) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          issue_s(c);
          w_commit(STATE ? b_vfree + 8 * s : b_kv);
          w_commit(b_qkfree + 8 * s);
        }
        if (STATE) w_commit(b_o);
      }
      bool ok = warp == 18 && issue_a(0);
      for (int c = 0; c < chunks && ok; ++c) {
        const int s = c & 1;
        // the other A buffer is free: the product that read it was issued before
        if (c + 1 < chunks) ok = issue_a(c + 1);
        ok = ok && wait(b_p + 8 * s, c >> 1) && wait(b_read, c);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint64_t v = s ? vn[1] : vn[0];
        const uint32_t pa = tmem + TM_A + (uint32_t)s * 128;
#pragma unroll
        for (int i = 0; i < 2 * LT_C / 16; ++i)  // 16 keys: 8 columns of values, 8 of remainders
          w_mma_ta(tmem + TM_O2, pa + (uint32_t)((i >> 1) * 16 + (i & 1) * 8), v + nstep(i >> 1), ID_O2, 1u);
        w_commit(b_o);
        w_commit(b_vfree + 8 * s);
      }
      w_commit(b_end);
      x_drain(b_end, 0);
    }
  } else if (STATE && group != 2) {
    if (group == 1 && x_wait(b_o, 0, dead, status)) {  // what the segment adds to the state
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll 1
      for (int half = 0; half < 2; ++half) {
        uint32_t x[32];
        x_ld32(tmem + lanes + TM_S + 32 * half, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int e = 0; e < 32; ++e)
          if (row_in && 32 * half + e < cols) a.seg[(seg + 1) * seg_size + state_at + (size_t)(32 * half + e) * a.dp] = __uint_as_float(x[e]);
      }
    }
  } else if (group == 0) {
    // ---- P: row r of D * A over row r of A (short loops: the roles share the instruction caches)
    for (int c = 0; c < chunks; ++c) {
      const int s = c & 1;
      if (!x_wait(b_a + 8 * s, (uint32_t)(c >> 1) & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t at = tmem + lanes + TM_A + (uint32_t)s * 128;
#pragma unroll 1
      for (int kb = 0; kb < 8; ++kb) {
        uint32_t w[16];
        if (kb < 2 * warp + 2) {  // some of the keys 16 kb .. are in front of this warp's rows
          uint32_t x[16];
          x_ld16(at + 16 * kb, x);
          const float* d = pw + r - 16 * kb;
          float f[16];
#pragma unroll
          for (int e = 0; e < 16; ++e) f[e] = d[-e];
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
          for (int e = 0; e < 8; ++e) lt_split(__uint_as_float(x[2 * e]) * f[2 * e], __uint_as_float(x[2 * e + 1]) * f[2 * e + 1], w[e], w[8 + e]);
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e) w[e] = 0u;
        }
        x_st16(at + 16 * kb, w);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(b_p + 8 * s);
    }
  } else if (group == 1) {
    // ---- S: row r (a dimension of k) of the state
    const uint32_t at = tmem + lanes + TM_S;
    float* state = a.state + state_at;
    const bool old = *a.pos_dev > 0;
    // 16 columns: operand for the next chunk, and the accumulator scaled by its decay
    auto hand_over = [&](uint32_t (&x)[16], int q, float f) {
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) lt_split(__uint_as_float(x[8 * p + 2 * e]), __uint_as_float(x[8 * p + 2 * e + 1]), hi[e], lo[e]);
        const uint32_t off = box_at(r, q * 2 + p);
        *reinterpret_cast<uint4*>(sm + LT_ST + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(sm + LT_ST + LT_BOX + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
#pragma unroll
      for (int e = 0; e < 16; ++e) x[e] = __float_as_uint(__uint_as_float(x[e]) * f);
      x_st16(at + 16 * q, x);
    };
    auto ready = [&]() {
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(b_st);
    };
    // the state in front of this segment
    float whole = 1.f;  // decay over a segment
    for (int j = 0; j < per && nseg > 1; ++j) whole *= pw[LT_C];
#pragma unroll 1
    for (int q = 0; q < 4; ++q) {
      uint32_t x[16];
      auto load = [&](const float* from, float decay) {  // x = decay x + the columns at `from`
        float v[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) v[e] = row_in && 16 * q + e < cols ? from[state_at + (size_t)(16 * q + e) * a.dp] : 0.f;
#pragma unroll
        for (int e = 0; e < 16; ++e) x[e] = __float_as_uint(fmaf(decay, __uint_as_float(x[e]), v[e]));
      };
#pragma unroll
      for (int e = 0; e < 16; ++e) x[e] = 0u;
      if (nseg > 1)
        for (int j = 0; j <= seg; ++j) load(a.seg + j * seg_size, whole);
      else if (old) load(a.state, 0.f);
      hand_over(x, q, pw[tokens_of(0)]);
    }
    ready();
    for (int c = 0; c < chunks; ++c) {
      if (!x_wait(b_kv, (uint32_t)c & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const bool end = c + 1 == chunks;
      const float f = end ? 0.f : pw[tokens_of(c + 1)];
#pragma unroll 1
      for (int q = 0; q < 4; ++q) {
        uint32_t x[16];
        x_ld16(at + 16 * q, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (!end) {
          hand_over(x, q, f);
        } else if (row_in && seg == nseg - 1) {
#pragma unroll
          for (int e = 0; e < 16; ++e)
            if (16 * q + e < cols) state[(size_t)(16 * q + e) * a.dp] = __uint_as_float(x[e]);
        }
      }
      if (!end) ready();
    }
  } else if (group == 2) {
    // ---- V: token r of the decayed values
    for (int c = 0; c < chunks; ++c) {
      if (!x_wait(b_v + 8 * (c & 1), (uint32_t)(c >> 1) & 1, dead, status)) break;
      const uint8_t* v = sm + (c & 1) * LT_STAGE + 4 * LT_BOX;
      uint8_t* vt = sm + vt_at(c);
      const int n = tokens_of(c);
      float f = r < n ? pw[n - 1 - r] : 0.f;
      if (STATE)  // to the end of the segment, which is whole: n = 128
        for (int j = c + 1; j < chunks; ++j) f *= pw[LT_C];
      uint32_t hi[32], lo[32];
#pragma unroll
      for (int p = 0; p < 8; ++p) {
        uint4 x = *reinterpret_cast<const uint4*>(v + box_at(r, p));
        if (r >= n) x = make_uint4(0u, 0u, 0u, 0u);  // a row of another sequence
        const uint32_t u[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) lt_split(__uint_as_float(u[e] << 16) * f, __uint_as_float(u[e] & 0xFFFF0000u) * f, hi[4 * p + e], lo[4 * p + e]);
      }
      // the place is free: the products that read it are done
      if (STATE ? c >= 2 && !x_wait(b_qkfree + 8 * (c & 1), (uint32_t)((c >> 1) - 1) & 1, dead, status)
                : c && !x_wait(b_kv, (uint32_t)(c - 1) & 1, dead, status)) break;
#pragma unroll
      for (int p = 0; p < 8; ++p) {
        const uint32_t off = box_at(r, p);
        *reinterpret_cast<uint4*>(vt + off) = make_uint4(hi[4 * p], hi[4 * p + 1], hi[4 * p + 2], hi[4 * p + 3]);
        *reinterpret_cast<uint4*>(vt + LT_BOX + off) = make_uint4(lo[4 * p], lo[4 * p + 1], lo[4 * p + 2], lo[4 * p + 3]);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      mbar_arrive(b_vt + 8 * (c & 1));
    }
  } else {
    // ---- O: token r; in the last step a lane stores pairs of columns of rows l / 4 + 8 k of its warp
    const int hv = a.h * a.v;
    const bool vec = a.v % 2 == 0;
    const float f = pw[r + 1];
    for (int c = 0; c < chunks; ++c) {
      if (!x_wait(b_kv, (uint32_t)c & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll 1
      for (int q = 0; q < 64; q += 16) {
        uint32_t x[16], y[16];
        x_ld16(tmem + lanes + TM_O1 + q, x);
        x_ld16(tmem + lanes + TM_O1 + 64 + q, y);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int e = 0; e < 16; ++e) x[e] = __float_as_uint(f * (__uint_as_float(x[e]) + __uint_as_float(y[e])));
        x_st16(tmem + lanes + TM_O2 + q, x);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(b_read);
      if (!x_wait(b_o, (uint32_t)c & 1, dead, status)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const int n = tokens_of(c);
#pragma unroll 1
      for (int part = 0; part < 2; ++part) {
        uint32_t x[32];
        x_ld16x256(tmem + lanes + ((uint32_t)(16 * part) << 16) + TM_O2, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        const int row = 32 * (warp & 3) + 16 * part + (lane >> 2), col = 2 * (lane & 3);
        float* dst = a.o + (size_t)(row0 + c * LT_C + row) * hv + (size_t)h * a.v + c0 + col;
#pragma unroll
        for (int k = 0; k < 2; ++k) {  // rows row and row + 8
          if (row + 8 * k >= n) continue;
          float* d = dst + (size_t)(8 * k) * hv;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const float u = __uint_as_float(x[4 * i + 2 * k]), w = __uint_as_float(x[4 * i + 2 * k + 1]);
            if (vec && 8 * i + col < cols) *reinterpret_cast<float2*>(d + 8 * i) = make_float2(u, w);
            if (!vec && 8 * i + col < cols) d[8 * i] = u;
            if (!vec && 8 * i + col + 1 < cols) d[8 * i + 1] = w;
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(TM_COLS) : "memory");
}

template <int NKB>
int launch_prefill(fb200_device* dev, const fb200_linear_args& a, int vp, int nseg, int per, const CUtensorMap& q, const CUtensorMap& k,
                   const CUtensorMap& v) {
  static bool configured[64] = {false};
  if (!configured[dev->ordinal & 63]) {
    FB_CUDA(dev, cudaFuncSetAttribute(linear_prefill_kernel<false, NKB>, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM));
    FB_CUDA(dev, cudaFuncSetAttribute(linear_prefill_kernel<true, NKB>, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM));
    configured[dev->ordinal & 63] = true;
  }
  const dim3 grid((unsigned)((a.v + 63) / 64 * nseg), (unsigned)a.h, (unsigned)a.b), block(LT_THREADS);
  int rc;
  if (nseg > 1 && (rc = fb200_launch(dev, linear_prefill_kernel<true, NKB>, grid, block, LT_SMEM, false, a, vp, nseg, per, dev->status, q, k, v))) return rc;
  return fb200_launch(dev, linear_prefill_kernel<false, NKB>, grid, block, LT_SMEM, false, a, vp, nseg, per, dev->status, q, k, v);
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
  // segments of at least four chunks, as many as the SMs take side by side
  const int slices = (a.v + 63) / 64, chunks = (a.s + LT_C - 1) / LT_C;
  int nseg = (int)std::min<long>(std::min(FB200_LINEAR_SEGMENTS, chunks / 4), dev->sm_count / ((long)slices * a.h * a.b));
  nseg = std::max(nseg, 1);
  const int per = (chunks + nseg - 1) / nseg;
  nseg = (chunks + per - 1) / per;
  return a.dp == 64 ? launch_prefill<1>(dev, a, vp, nseg, per, q, k, v) : launch_prefill<2>(dev, a, vp, nseg, per, q, k, v);
}
