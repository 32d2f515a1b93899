// Helpers shared by the attention kernels.
#pragma once
#include "sm100.cuh"

namespace gb {

// tanh(x), absolute error below 3e-7: 1 - 2 / (1 + e^2x).
__device__ __forceinline__ float tanh_wide(float x) {
  return 1.0f - __fdividef(2.0f, 1.0f + fast_exp2(2.885390081777927f * x));
}

// tanh(x) for |x| <= 1, relative error below 1e-7: an odd polynomial (minimax fit of tanh(x) / x over x^2 by Remez's exchange), no special function unit.
__device__ __forceinline__ float tanh_unit(float x) {
  const float y = x * x;
  float p = fmaf(0.00104102258568f, y, -0.00620337898208f);
  p = fmaf(p, y, 0.0202899803204f);
  p = fmaf(p, y, -0.053457029549f);
  p = fmaf(p, y, 0.133252040772f);
  p = fmaf(p, y, -0.333328391536f);
  p = fmaf(p, y, 0.999999950241f);
  return x * p;
}

// Reduce 16 per-lane values over the 32 lanes of a warp with 16 shuffles (a reduce-scatter: 8 + 4 + 2 + 1 exchanges, then one
// more between neighbours): lane L returns the result for index L >> 1.
#define GB_RS_STEP(IN, OUT, N, BIT, OP)                                                       \
  _Pragma("unroll") for (int i = 0; i < N; ++i) {                                            \
    const bool up = (lane & BIT) != 0;                                                       \
    const float send = up ? IN[i] : IN[N + i], keep = up ? IN[N + i] : IN[i];                 \
    OUT[i] = OP(keep, __shfl_xor_sync(0xffffffffu, send, BIT));                               \
  }
__device__ __forceinline__ float rs_max(float a, float b) { return fmaxf(a, b); }
__device__ __forceinline__ float rs_add(float a, float b) { return a + b; }
__device__ __forceinline__ float warp_reduce16_max(const float* v, int lane) {
  float a[8], b[4], c[2], d[1];
  GB_RS_STEP(v, a, 8, 16, rs_max) GB_RS_STEP(a, b, 4, 8, rs_max) GB_RS_STEP(b, c, 2, 4, rs_max) GB_RS_STEP(c, d, 1, 2, rs_max)
  return fmaxf(d[0], __shfl_xor_sync(0xffffffffu, d[0], 1));
}
__device__ __forceinline__ float warp_reduce16_sum(const float* v, int lane) {
  float a[8], b[4], c[2], d[1];
  GB_RS_STEP(v, a, 8, 16, rs_add) GB_RS_STEP(a, b, 4, 8, rs_add) GB_RS_STEP(b, c, 2, 4, rs_add) GB_RS_STEP(c, d, 1, 2, rs_add)
  return d[0] + __shfl_xor_sync(0xffffffffu, d[0], 1);
}

}  // namespace gb
