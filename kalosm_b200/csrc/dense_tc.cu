// Products of many activation rows with BF16 weights on the 5th-generation tensor cores.
//
// Bound: tensor cores (2 M N K flops) for prompts, HBM (the matrix is read once) for a few rows.
// A CTA computes NH x 128 weight rows by BM activation rows of Y^T = W . X^T; the fp32 accumulators
// (NH x BM columns of 128 lanes) live in tensor memory. Roles, coupled only by mbarriers:
//  * copy requester (one thread): a stage is the NH weight boxes (64 columns x 128 rows) and the activation
//    box (64 columns x BM rows) of one 64-wide K block, by tensor TMA with 128-byte swizzle; rows and columns
//    outside the matrices arrive as zeros;
//  * MMA issuer (one thread): 4 NH tcgen05.mma (M = 128, N = BM, K = 16, kind::f16 with bf16 operands and fp32
//    accumulation) per stage, tcgen05.commit hands the stage back;
//  * epilogue (8 warps): tcgen05.ld, then f32 or bf16 rows (factor, bias, residual, softcap), gelu rows, or SwiGLU:
//    gate and up rows of an output are the two halves of the same CTA, so they sit in the same TMEM lane BM columns apart.
// Every wait is bounded (2^22 polls): a wait that gives up sets the device status word and a flag that makes the
// other roles leave; TMEM is released on every path.
#include <algorithm>

#include "dense.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int TC_BN = 128, TC_BK = 64, TC_EPI_WARPS = 8, TC_THREADS = (TC_EPI_WARPS + 2) * 32;
constexpr int TC_MAX_STAGES = 6, TC_TAIL = 256;

template <int BM, int NH>
struct TcShape {
  static constexpr int A_BYTES = NH * TC_BN * TC_BK * 2, B_BYTES = BM * TC_BK * 2, STAGE = A_BYTES + B_BYTES;
  static constexpr int COLS = NH * BM < 32 ? 32 : NH * BM;
  // small tiles leave room for two CTAs on an SM
  static constexpr int BUDGET = BM <= 64 ? 112 * 1024 : 224 * 1024;
  static constexpr int STAGES_FIT = (BUDGET - TC_TAIL - 1024) / STAGE;
  static constexpr int STAGES = STAGES_FIT > TC_MAX_STAGES ? TC_MAX_STAGES : STAGES_FIT;
  static constexpr int SMEM = STAGES * STAGE + TC_TAIL + 1024;
  // instruction descriptor: fp32 accumulator, bf16 A and B, both K-major, N = BM, M = 128
  static constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BM >> 3) << 17) | ((uint32_t)(TC_BN >> 4) << 24);
};

struct DenseTcArgs {
  float* y;
  __nv_bfloat16* yb;
  const float* add;
  const float* bias;
  __nv_bfloat16* z;
  size_t ldy, ldadd, ldz;
  int m, kblocks, row0, n_plain, gate0, up0, ff, gelu, ff_col, plain_tiles, m_tiles;
  float alpha, softcap;
  int* status;
};

// K-major operand with 128-byte swizzle: rows of 128 bytes, groups of 8 rows 1024 bytes apart, descriptor version 1
__device__ __forceinline__ uint64_t dt_desc(uint32_t saddr) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
template <int BM, int NH>
__global__ void __launch_bounds__(TC_THREADS, BM <= 64 ? 2 : 1)
dense_tc_kernel(const DenseTcArgs a, const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap) {
  using S = TcShape<BM, NH>;
  extern __shared__ uint8_t sm_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(sm_raw) + 1023) & ~(uintptr_t)1023);
  uint64_t* bars = reinterpret_cast<uint64_t*>(sm + S::STAGES * S::STAGE);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * TC_MAX_STAGES + 1);
  volatile int* dead = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const uint32_t full = smem_u32(bars), empty = full + 8 * TC_MAX_STAGES, done = full + 16 * TC_MAX_STAGES;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // activation tiles fastest: the CTAs that run together share their weight rows in L2
  const int mt = (int)blockIdx.x % a.m_tiles, nt = (int)blockIdx.x / a.m_tiles;
  const bool ffn = nt >= a.plain_tiles, pair = ffn && !a.gelu;
  const int n0 = ffn ? (nt - a.plain_tiles) * TC_BN * (pair ? 1 : NH) : nt * TC_BN * NH;  // first output row of the tile
  const int m0 = mt * BM;
  if (tid == 0) {
    *dead = 0;
    for (int i = 0; i < S::STAGES; ++i) { mbar_init(full + 8 * i, 1); mbar_init(empty + 8 * i, 1); }
    mbar_init(done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "n"(S::COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *tmem_slot;

  if (warp == TC_EPI_WARPS) {
    if (lane == 0) {
      const int r0 = (pair ? a.gate0 : ffn ? a.up0 : a.row0) + n0, r1 = pair ? a.up0 + n0 : r0 + TC_BN, xc = ffn ? a.ff_col : 0;
      int issued = 0;
      for (int kb = 0; kb < a.kblocks; ++kb, ++issued) {
        const int s = kb % S::STAGES;
        if (kb >= S::STAGES && !x_wait(empty + 8 * s, (uint32_t)((kb / S::STAGES - 1) & 1), dead, a.status)) break;
        const uint32_t dst = smem_u32(sm + s * S::STAGE), bar = full + 8 * s;
        mbar_expect_tx(bar, S::STAGE);
        x_tma_box2(dst, &wmap, kb * TC_BK, r0, bar);
        if (NH == 2) x_tma_box2(dst + TC_BN * TC_BK * 2, &wmap, kb * TC_BK, r1, bar);
        x_tma_box2(dst + S::A_BYTES, &xmap, xc + kb * TC_BK, m0, bar);
      }
      if (*dead)
        for (int kb = max(0, issued - S::STAGES); kb < issued; ++kb) x_drain(full + 8 * (kb % S::STAGES), (uint32_t)((kb / S::STAGES) & 1));
    }
  } else if (warp == TC_EPI_WARPS + 1) {
    if (lane == 0) {
      bool ok = true;
      for (int kb = 0; kb < a.kblocks && ok; ++kb) {
        const int s = kb % S::STAGES;
        ok = x_wait(full + 8 * s, (uint32_t)((kb / S::STAGES) & 1), dead, a.status);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t st = smem_u32(sm + s * S::STAGE);
#pragma unroll
        for (int k = 0; k < TC_BK / 16; ++k)  // 32 bytes further inside the 128-byte rows per K step
#pragma unroll
          for (int h = 0; h < NH; ++h)
            x_mma(tmem + (uint32_t)(h * BM), dt_desc(st + h * TC_BN * TC_BK * 2 + k * 32), dt_desc(st + S::A_BYTES + k * 32), S::IDESC,
                   (kb | k) ? 1u : 0u);
        x_commit(empty + 8 * s);
      }
      x_commit(done);
    }
  } else {
    // ---- epilogue: warp w reads TMEM lanes 32 (w % 4) .., columns of one half of the activation rows
    const int quad = warp & 3, ch = warp >> 2;
    x_wait(done, 0, dead, a.status);
    if (*dead) x_drain(done, 0);
    else {
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t tl = tmem + ((uint32_t)(32 * quad) << 16);
      const int r = quad * 32 + lane;
#pragma unroll 1
      for (int c = ch * (BM / 2); c < (ch + 1) * (BM / 2); c += 16) {
        if (m0 + c >= a.m) break;
        const int lim = min(16, a.m - (m0 + c));
        uint32_t v0[16], v1[16];
        x_ld16(tl + (uint32_t)c, v0);
        if (NH == 2) x_ld16(tl + (uint32_t)(BM + c), v1);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (pair) {
          if (n0 + r < a.ff) {
            __nv_bfloat16* zp = a.z + (size_t)(m0 + c) * a.ldz + n0 + r;
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (i < lim) {
                const float g = __uint_as_float(v0[i]);
                zp[(size_t)i * a.ldz] = __float2bfloat16(g / (1.0f + __expf(-g)) * __uint_as_float(v1[i]));
              }
          }
        } else {
#pragma unroll
          for (int h = 0; h < NH; ++h) {
            const int n = n0 + h * TC_BN + r;
            if (n >= (ffn ? a.ff : a.n_plain)) continue;
            uint32_t (&v)[16] = h ? v1 : v0;
            if (ffn) {
              __nv_bfloat16* zp = a.z + (size_t)(m0 + c) * a.ldz + n;
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (i < lim) {
                  const float t = __uint_as_float(v[i]), u = 0.7978845608028654f * fmaf(0.044715f * t * t, t, t);
                  zp[(size_t)i * a.ldz] = __float2bfloat16(__fdividef(t, 1.0f + __expf(-2.0f * u)));
                }
              continue;
            }
            const float bias = a.bias ? a.bias[n] : 0.f;
#pragma unroll
            for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(fmaf(a.alpha, __uint_as_float(v[i]), bias));
            if (a.softcap > 0.f) {  // of a product without a residual
#pragma unroll
              for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(a.softcap * tanhf(__uint_as_float(v[i]) / a.softcap));
            }
            if (a.yb) {
              __nv_bfloat16* yp = a.yb + (size_t)(m0 + c) * a.ldy + n;
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (i < lim) yp[(size_t)i * a.ldy] = __float2bfloat16(__uint_as_float(v[i]));
            } else if (a.add) {
              const float* ap = a.add + (size_t)(m0 + c) * a.ldadd + n;
              float* yp = a.y + (size_t)(m0 + c) * a.ldy + n;
              float r0[16];
#pragma unroll
              for (int i = 0; i < 16; ++i) r0[i] = i < lim ? ap[(size_t)i * a.ldadd] : 0.f;
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (i < lim) yp[(size_t)i * a.ldy] = __uint_as_float(v[i]) + r0[i];
            } else {
              float* yp = a.y + (size_t)(m0 + c) * a.ldy + n;
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (i < lim) yp[(size_t)i * a.ldy] = __uint_as_float(v[i]);
            }
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 0)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(S::COLS) : "memory");
}

typedef CUresult (*encode_fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                              const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                              CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// feed-forward tiles: a gated pair takes both halves of a tile
int tc_ff_tiles(const fb200_dense_job& j, int nh) {
  const int rows = j.act == FB200_FFN_GELU ? TC_BN * nh : TC_BN;
  return (j.ff + rows - 1) / rows;
}

template <int BM, int NH>
int launch_tc(fb200_device* dev, const fb200_dense_job& j, DenseTcArgs a) {
  using S = TcShape<BM, NH>;
  static_assert(S::STAGES >= 2, "at least two stages");
  CUtensorMap wmap, xmap;
  if (!fb200_make_map_2d(&wmap, j.w->data, 1, j.w->k, j.w->n, j.w->k * 2, TC_BN) ||
      !fb200_make_map_2d(&xmap, j.x, 1, (uint64_t)(j.ff_off + j.kx), (uint64_t)j.m, j.ldx * 2, BM))
    return fb200_fail(dev, FB200_ERR_CUDA, "dense product: tensor map refused (w %llu x %llu, x %d x %d stride %zu)",
                      (unsigned long long)j.w->n, (unsigned long long)j.w->k, j.m, j.kx, j.ldx);
  a.plain_tiles = (j.n_plain + TC_BN * NH - 1) / (TC_BN * NH);
  a.m_tiles = (j.m + BM - 1) / BM;
  const int tiles = a.plain_tiles + tc_ff_tiles(j, NH);
  if (tiles == 0) return FB200_OK;
  static bool configured[64] = {false};
  if (!configured[dev->ordinal & 63]) {
    FB_CUDA(dev, cudaFuncSetAttribute(dense_tc_kernel<BM, NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::SMEM));
    configured[dev->ordinal & 63] = true;
  }
  return fb200_launch(dev, dense_tc_kernel<BM, NH>, dim3((unsigned)(tiles * a.m_tiles)), dim3(TC_THREADS), (size_t)S::SMEM, false, a,
                      wmap, xmap);
}

}  // namespace

bool fb200_make_map_2d(CUtensorMap_st* map, const void* base, int bf16, uint64_t cols, uint64_t rows, uint64_t row_stride_bytes,
                       uint32_t box_rows) {
  static encode_fn enc = [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
      p = nullptr;
    return reinterpret_cast<encode_fn>(p);
  }();
  if (!enc) return false;
  const cuuint64_t dims[2] = {cols, rows}, strides[1] = {row_stride_bytes};
  const cuuint32_t box[2] = {64, box_rows}, estr[2] = {1, 1};
  return enc(map, bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2, const_cast<void*>(base), dims, strides, box,
             estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

int fb200_dense_gemm_tc(fb200_device* dev, const fb200_dense_job& j) {
  if (j.w->type != FB200_BF16 || j.norm_w || j.w->k % 8 || j.ldx % 8 || ((uintptr_t)j.x & 15u) || j.ff_off % 8 ||
      (j.ff_off && j.ff_off + (size_t)j.kx > j.ldx))
    return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "dense product: bf16 rows and BF16 weights of an aligned width needed");
  DenseTcArgs a = {};
  if (j.y_bf16) a.yb = (__nv_bfloat16*)j.y;
  else a.y = (float*)j.y;
  a.add = j.add; a.z = (__nv_bfloat16*)j.z; a.ldy = j.ldy; a.ldadd = j.ldadd; a.ldz = j.ldz;
  a.bias = j.bias; a.alpha = j.alpha; a.softcap = j.softcap; a.gelu = j.act == FB200_FFN_GELU; a.ff_col = (int)j.ff_off;
  a.m = j.m; a.kblocks = (j.kx + TC_BK - 1) / TC_BK; a.row0 = j.row0; a.n_plain = j.n_plain; a.gate0 = j.gate0; a.up0 = j.up0; a.ff = j.ff;
  a.status = dev->status;
  // tile shape by a small cost model: rounds of CTAs over the SMs x time of one tile (relative to 256 x 256)
  auto cost = [&](int bm, int nh, double tile) {
    if (nh == 1 && j.ff && j.act != FB200_FFN_GELU) return 1e30;
    const long tiles = (long)((j.n_plain + TC_BN * nh - 1) / (TC_BN * nh) + tc_ff_tiles(j, nh)) * ((j.m + bm - 1) / bm);
    const int slots = dev->sm_count * (bm <= 64 ? 2 : 1);
    const long full = tiles / slots, rest = tiles % slots;
    // two small tiles on one SM share it: a last round that half fills the slots takes half a round's time
    double rounds = (double)full;
    if (rest) rounds += bm <= 64 ? (rest > dev->sm_count ? 1.0 : 0.5) : 1.0;
    return rounds * tile * (bm <= 64 ? 2.0 : 1.0);
  };
  struct Cand { int bm, nh; double tile; };
  const Cand cands[] = {{256, 2, 1.0}, {256, 1, 0.62}, {128, 2, 0.62}, {128, 1, 0.38}, {64, 2, 0.42}, {64, 1, 0.24}, {32, 2, 0.36}, {32, 1, 0.19}};
  int pick = 0;
  double best = 1e31;
  for (int i = 0; i < 8; ++i) {
    const double c = cost(cands[i].bm, cands[i].nh, cands[i].tile);
    if (c < best) { best = c; pick = i; }
  }
  switch (pick) {
    case 0: return launch_tc<256, 2>(dev, j, a);
    case 1: return launch_tc<256, 1>(dev, j, a);
    case 2: return launch_tc<128, 2>(dev, j, a);
    case 3: return launch_tc<128, 1>(dev, j, a);
    case 4: return launch_tc<64, 2>(dev, j, a);
    case 5: return launch_tc<64, 1>(dev, j, a);
    case 6: return launch_tc<32, 2>(dev, j, a);
    default: return launch_tc<32, 1>(dev, j, a);
  }
}
