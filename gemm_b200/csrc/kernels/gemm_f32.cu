// Linear layer in true 32-bit floats (FFMA, no reduced-precision tensor-core mode): Out[m, n] = sum_k X[m, k] W[n, k] (+ bias[n]).
// The path of the "f32" weight format, which exists to check the 16-bit kernels against; any sizes, any row pitches.
#include "sm100.cuh"
#include "host_common.h"

namespace gb {

constexpr int kSgT = 64, kSgK = 16;       // output tile 64 x 64, K step 16; 256 threads, 4 x 4 results each

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ out, int m, int n, int k,
                int ldx, int ldw, int ldo) {
  pdl_wait();
  pdl_trigger();
  __shared__ float sx[kSgK][kSgT + 4], sw[kSgK][kSgT + 4];
  const int m0 = blockIdx.y * kSgT, n0 = blockIdx.x * kSgT, tid = threadIdx.x;
  const int tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += kSgK) {
    for (int i = tid; i < kSgT * kSgK; i += 256) {
      const int r = i / kSgK, c = i % kSgK;
      sx[c][r] = (m0 + r < m && k0 + c < k) ? x[(size_t)(m0 + r) * ldx + k0 + c] : 0.f;
      sw[c][r] = (n0 + r < n && k0 + c < k) ? w[(size_t)(n0 + r) * ldw + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kSgK; ++c) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[c][tr]), b = *reinterpret_cast<const float4*>(&sw[c][tc]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = m0 + tr + i, c = n0 + tc + j;
      if (r < m && c < n) out[(size_t)r * ldo + c] = acc[i][j] + (bias != nullptr ? bias[c] : 0.f);
    }
}

}  // namespace gb

using namespace gb;

GB_API int gb_gemm_f32(const float* x, const float* w, const float* bias, float* out, int m, int n, int k, int ldx, int ldw, int ldo, cudaStream_t stream) {
  if (m <= 0 || n <= 0) return 0;
  if (k < 1 || ldx < k || ldw < k || ldo < n) return fail("gemm_f32: bad sizes%s");
  if ((m + kSgT - 1) / kSgT > 65535) return fail("gemm_f32: too many rows%s");
  launch_k(gemm_f32_kernel, dim3((unsigned)((n + kSgT - 1) / kSgT), (unsigned)((m + kSgT - 1) / kSgT)), 256, 0, stream, x, w, bias, out, m, n, k, ldx, ldw, ldo);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}
