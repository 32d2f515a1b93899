// Linear layer in true 32-bit floats (FFMA, no reduced-precision tensor-core mode): Out[m, n] = sum_k X[m, k] W[n, k] (+ bias[n]).
// The path of the "f32" weight format, which exists to check the 16-bit kernels against; any sizes, any row pitches.
#include "sm100.cuh"
#include "host_common.h"

namespace gb {

constexpr int kSgT = 64, kSgK = 16;       // output tile 64 x 64, K step 16; 256 threads, 4 x 4 results each

// Plain: one product.  Batched (stride_*): product b of blockIdx.z.  Grouped (seg_start != null): the 64-row tiles of x belong to the group whose
// segment they lie in (segments start at multiples of 64); rows behind a segment's count are not written.
struct GemmF32Args {
  const float* x; const float* w; const float* bias; float* out;
  int m, n, k, ldx, ldw, ldo;
  long stride_x, stride_w, stride_o;
  const int* seg_start; const int* seg_count; int groups;
  const int* row_src;           // x row of tile row r (negative: zeros); null = r itself
};

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const GemmF32Args a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float sx[kSgK][kSgT + 4], sw[kSgK][kSgT + 4];
  __shared__ int s_group;
  const int m0 = blockIdx.y * kSgT, n0 = blockIdx.x * kSgT, tid = threadIdx.x;
  const int tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  const float* x = a.x + (size_t)blockIdx.z * a.stride_x;
  const float* w = a.w + (size_t)blockIdx.z * a.stride_w;
  float* out = a.out + (size_t)blockIdx.z * a.stride_o;
  int m = a.m;
  if (a.seg_start != nullptr) {
    if (tid == 0) s_group = -1;
    __syncthreads();
    for (int g = tid; g < a.groups; g += 256) { const int s = a.seg_start[g]; if (m0 >= s && m0 < s + a.seg_count[g]) s_group = g; }
    __syncthreads();
    const int g = s_group;
    if (g < 0) return;
    w += (size_t)g * a.stride_w;
    m = min(m, a.seg_start[g] + a.seg_count[g]);
  }
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.k; k0 += kSgK) {
    for (int i = tid; i < kSgT * kSgK; i += 256) {
      const int r = i / kSgK, c = i % kSgK;
      int xr = m0 + r < m ? m0 + r : -1;
      if (a.row_src != nullptr && xr >= 0) xr = a.row_src[xr];
      sx[c][r] = (xr >= 0 && k0 + c < a.k) ? x[(size_t)xr * a.ldx + k0 + c] : 0.f;
      sw[c][r] = (n0 + r < a.n && k0 + c < a.k) ? w[(size_t)(n0 + r) * a.ldw + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kSgK; ++c) {
      const float4 p = *reinterpret_cast<const float4*>(&sx[c][tr]), q = *reinterpret_cast<const float4*>(&sw[c][tc]);
      const float av[4] = {p.x, p.y, p.z, p.w}, bv[4] = {q.x, q.y, q.z, q.w};
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
      if (r < m && c < a.n) out[(size_t)r * a.ldo + c] = acc[i][j] + (a.bias != nullptr ? a.bias[c] : 0.f);
    }
}

static int gemm_f32_launch(const GemmF32Args& a, int batch, cudaStream_t stream) {
  if (a.m <= 0 || a.n <= 0 || batch <= 0) return 0;
  if (a.k < 1 || a.ldx < a.k || a.ldw < a.k || a.ldo < a.n) return fail("gemm_f32: bad sizes%s");
  if ((a.m + kSgT - 1) / kSgT > 65535 || batch > 65535) return fail("gemm_f32: too many rows%s");
  launch_k(gemm_f32_kernel, dim3((unsigned)((a.n + kSgT - 1) / kSgT), (unsigned)((a.m + kSgT - 1) / kSgT), (unsigned)batch), 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

GB_API int gb_gemm_f32(const float* x, const float* w, const float* bias, float* out, int m, int n, int k, int ldx, int ldw, int ldo, cudaStream_t stream) {
  GemmF32Args a = {x, w, bias, out, m, n, k, ldx, ldw, ldo, 0, 0, 0, nullptr, nullptr, 0, nullptr};
  return gemm_f32_launch(a, 1, stream);
}

// out[b] = x[b] w[b]^T for b < batch, matrices stride_* elements apart.
GB_API int gb_gemm_f32_batched(const float* x, const float* w, float* out, int batch, int m, int n, int k, int ldx, int ldw, int ldo, long stride_x, long stride_w,
                               long stride_o, cudaStream_t stream) {
  GemmF32Args a = {x, w, nullptr, out, m, n, k, ldx, ldw, ldo, stride_x, stride_w, stride_o, nullptr, nullptr, 0, nullptr};
  return gemm_f32_launch(a, batch, stream);
}

// x by segments (device arrays, starts multiples of 64), w [groups, n, k] -> out [rows, n]; row r of the segments is x[row_src[r]] (null: x[r]).
GB_API int gb_gemm_f32_grouped(const float* x, const float* w, float* out, const int* seg_start, const int* seg_count, int groups, int rows, int n, int k, int ldx,
                               const int* row_src, cudaStream_t stream) {
  if (groups < 1 || seg_start == nullptr || seg_count == nullptr) return fail("gemm_f32: no groups%s");
  GemmF32Args a = {x, w, nullptr, out, rows, n, k, ldx, k, n, 0, (long)n * k, 0, seg_start, seg_count, groups, row_src};
  return gemm_f32_launch(a, 1, stream);
}
