// Element access and gate arithmetic shared by the recurrent mixers' kernels.
#pragma once
#include "sm100.cuh"

namespace gb {

__device__ __forceinline__ float ldv(const float* p) { return *p; }
__device__ __forceinline__ float ldv(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stv(float* p, float v) { *p = v; }
__device__ __forceinline__ void stv(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// V neighbouring elements (V = 4: aligned to four elements)
template <int V>
__device__ __forceinline__ void load_cols(const float* p, float* v) {
  if constexpr (V == 4) { const float4 q = *reinterpret_cast<const float4*>(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
  else v[0] = *p;
}
template <int V>
__device__ __forceinline__ void load_cols(const __nv_bfloat16* p, float* v) {
  if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else v[0] = __bfloat162float(*p);
}
template <int V>
__device__ __forceinline__ void store_cols(float* p, const float* v) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V>
__device__ __forceinline__ void store_cols(__nv_bfloat16* p, const float* v) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  else *p = __float2bfloat16(v[0]);
}

__device__ __forceinline__ float softplus_exact(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// f = low + (1 - low) sigmoid(z); also its complement 1 - f = (1 - low) sigmoid(-z), without cancellation.
__device__ __forceinline__ float forget_gate(float z, float low, float& complement) {
  const float e = expf(-fabsf(z)), big = 1.0f / (1.0f + e), small = e * big;       // sigmoid(|z|), sigmoid(-|z|)
  complement = (1.0f - low) * (z >= 0.f ? small : big);
  return fmaf(1.0f - low, z >= 0.f ? big : small, low);
}

// x = hi + lo in bf16, for two neighbours
__device__ __forceinline__ void split_bf16x2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  lo = pack_bf16x2(a - h.x, b - h.y);
}

// Bounded wait of a whole warp: its lanes leave a failed wait together (the tcgen05 loads that follow need all of them).
__device__ __forceinline__ bool warp_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, KernelStatus* st, int where, int aux) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, st, where, aux));
}

}  // namespace gb
