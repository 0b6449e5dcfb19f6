// Pieces shared by the mixers that carry a matrix state per head (delta_rule.cu, linear_attn.cu): a state is [v][dp] in
// 32-bit floats, and a group of lanes owns a column (one v) for as long as it works on it.
#pragma once

#include <cuda_runtime.h>

namespace {

__device__ __forceinline__ float dr_silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float dr_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
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

}  // namespace
