// Products with dense (BF16 or F32) weight matrices, as the hybrid decoder layers use them: the rows
// of several projections that read the same input are stacked into ONE matrix, so a layer is one
// product in front of its mixer and one behind it.
#pragma once

#include "common.cuh"

// One product y = W . x over m activation rows, with up to two groups of output rows:
//  * plain rows 0 .. n_plain: y[m * ldy + n] = alpha * acc (+ bias[n]) (+ add[m * ldadd + n]), as f32 or (y_bf16) bf16;
//    with a softcap c: c tanh(. / c) of that;
//  * feed-forward rows i < ff: z[m * ldz + i] = silu(W[gate0 + i] . x') * (W[up0 + i] . x'), or (FB200_FFN_GELU)
//    gelu(W[up0 + i] . x') with the tanh form of gelu. x' is x, or rows of their own: ff_off elements behind x (a column
//    offset inside the rows for bf16 operands), and for one row x under the norm ff_norm_w.
// W is untiled row-major [w->n, w->k]; w->k is padded to a multiple of 64, the columns from kx on are zero.
// Operand rows: one row (m == 1) or F32 weights read f32 rows x[m * ldx + c], c < kx, optionally RMS-normalised
// first (norm_w, m == 1 only); BF16 weights with m > 1 read bf16 rows of kx elements at stride ldx.
// z holds f32 when the operand rows are f32, bf16 otherwise.
struct fb200_dense_job {
  const fb200_qmatrix* w = nullptr;
  int m = 0;
  const void* x = nullptr;
  size_t ldx = 0;
  int kx = 0;
  const float* norm_w = nullptr;
  const float* ff_norm_w = nullptr;  // m == 1: the norm of the feed-forward rows' operand where it differs
  float eps = 0.f;
  int row0 = 0;  // first plain row (a sub-range of the stacked matrix)
  int n_plain = 0;
  void* y = nullptr;
  size_t ldy = 0;
  int y_bf16 = 0;
  const float* add = nullptr;
  size_t ldadd = 0;
  const float* bias = nullptr;
  float alpha = 1.f, softcap = 0.f;
  int gate0 = 0, up0 = 0, ff = 0, act = 0;  // act: fb200_ffn_act
  size_t ff_off = 0;
  void* z = nullptr;
  size_t ldz = 0;
};

int fb200_dense_product(fb200_device* dev, const fb200_dense_job& j);
int fb200_dense_gemv(fb200_device* dev, const fb200_dense_job& j);      // m == 1
int fb200_dense_gemm_f32(fb200_device* dev, const fb200_dense_job& j);  // F32 weights
int fb200_dense_gemm_tc(fb200_device* dev, const fb200_dense_job& j);   // BF16 weights, tcgen05
// f32 rows (n elements at stride ldx) -> bf16 rows of np elements (zeros from n on), RMS-normalised when w is given.
// With w2 an output row is 2 np elements: the row under w, then the row under w2.
int fb200_rows_to_bf16(fb200_device* dev, const float* x, size_t ldx, const float* w, const float* w2, float eps, size_t rows,
                       int n, int np, __nv_bfloat16* y);

// gelu in its tanh form: 0.5 v (1 + tanh(u)) = v / (1 + exp(-2 u)), u = sqrt(2 / pi) (v + 0.044715 v^3)
__device__ __forceinline__ float fb_gelu_tanh(float v) {
  const float u = 0.7978845608028654f * fmaf(0.044715f * v * v, v, v);
  return v / (1.0f + expf(-2.0f * u));
}

// cuTensorMapEncodeTiled of the driver, looked up once (the library does not link against libcuda); a 2-D map of
// 2-byte elements, 128-byte swizzle, boxes of 64 columns x box_rows rows, zeros outside.
struct CUtensorMap_st;
bool fb200_make_map_2d(CUtensorMap_st* map, const void* base, int bf16, uint64_t cols, uint64_t rows, uint64_t row_stride_bytes,
                       uint32_t box_rows);
