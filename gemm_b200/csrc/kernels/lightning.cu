// Lightning (decayed linear) attention, per head:  S_t = decay S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t,
// with q, k, v = SiLU of the columns of the mixer's input projection.  The state S [dim, vdim] is f32 and lives in a slot per sequence.
//
// lightning_step_kernel: token by token.  One CTA per (sequence, head, slice of value columns); a lane owns VEC value columns, the
// eight warps split the key rows, so a state row is read and written as whole 128-byte (VEC = 1) or 512-byte (VEC = 4) lines.
// A decode step is one pass over the state: all of a thread's state loads are in flight at once.
#include "sm100.cuh"
#include "host_common.h"

namespace gb {

struct LightningArgs {
  const void* proj;             // [n_part][tokens, ld]: columns [q heads x dim | k heads x dim | v heads x vdim | ...]
  int n_part; long part_stride; int ld;
  const float* decay;           // [heads]
  float* state;                 // [slots, heads, dim, vdim]
  int n_slots;
  const int* cu_q; const int* seq_slots;
  float* out; int ld_out;       // [tokens, heads * vdim] f32
  int heads, dim, vdim;
  int raw;                      // != 0: the columns are pre-activations (one bf16 slab of activated columns otherwise)
};

__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float ldp(const float* p) { return *p; }
__device__ __forceinline__ float ldp(const __nv_bfloat16* p) { return __bfloat162float(*p); }

template <typename TI>
__device__ __forceinline__ float proj_silu(const LightningArgs& a, size_t tok, int col) {
  const TI* p = (const TI*)a.proj + tok * a.ld + col;
  float s = ldp(p);
  for (int i = 1; i < a.n_part; ++i) s += ldp(p + (size_t)i * a.part_stride);
  return a.raw ? silu_exact(s) : s;
}

template <typename TI, int VEC, int R>             // dim <= 8 * R
__global__ void __launch_bounds__(256)
lightning_step_kernel(const LightningArgs a) {
  __shared__ float sq[8 * R], sk[8 * R];
  __shared__ float red[8][32 * VEC];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, s = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = a.cu_q[s], t1 = a.cu_q[s + 1];
  const int slot = a.seq_slots[s];
  if (t1 <= t0 || slot < 0 || slot >= a.n_slots) return;
  const int e0 = (blockIdx.y * 32 + lane) * VEC;
  const bool live = e0 < a.vdim;                   // VEC > 1 only when vdim % VEC == 0
  float* st = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim + e0;
  float S[R][VEC];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = warp + 8 * r;
#pragma unroll
    for (int j = 0; j < VEC; ++j) S[r][j] = 0.f;
    if (live && d < a.dim) {
      if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(st + (size_t)d * a.vdim);
        S[r][0] = v.x; S[r][1] = v.y; S[r][2] = v.z; S[r][3] = v.w;
      } else S[r][0] = st[(size_t)d * a.vdim];
    }
  }
  const float dec = a.decay[h];
  const int hd = a.heads * a.dim;
  for (int t = t0; t < t1; ++t) {
    for (int i = threadIdx.x; i < 2 * a.dim; i += 256) {
      const bool isk = i >= a.dim;
      const int c = isk ? i - a.dim : i;
      const float v = proj_silu<TI>(a, t, (isk ? hd : 0) + h * a.dim + c);
      if (isk) sk[c] = v; else sq[c] = v;
    }
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = live ? proj_silu<TI>(a, t, 2 * hd + h * a.vdim + e0 + j) : 0.f;
    __syncthreads();
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = warp + 8 * r;
      if (d < a.dim) {
        const float kd = sk[d], qd = sq[d];
#pragma unroll
        for (int j = 0; j < VEC; ++j) { S[r][j] = fmaf(dec, S[r][j], kd * v[j]); o[j] = fmaf(S[r][j], qd, o[j]); }
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) red[warp][lane * VEC + j] = o[j];
    __syncthreads();
    if (threadIdx.x < 32 * VEC) {
      float acc = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) acc += red[w][threadIdx.x];
      const int e = blockIdx.y * 32 * VEC + threadIdx.x;
      if (e < a.vdim) a.out[(size_t)t * a.ld_out + h * a.vdim + e] = acc;
    }
    // sq / sk / red are rewritten only after every thread has passed the barriers of the next token: sq / sk were last read before the
    // second barrier above, red is read before the first barrier of the next token by the threads that write it after that barrier
  }
  if (live) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = warp + 8 * r;
      if (d < a.dim) {
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(st + (size_t)d * a.vdim) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
        else st[(size_t)d * a.vdim] = S[r][0];
      }
    }
  }
}

template <typename TI>
static int lightning_step_launch(const LightningArgs& a, int n_seqs, cudaStream_t stream) {
  const bool vec = a.vdim % 4 == 0 && a.vdim > 32 && a.dim <= 256;
  const int cols = vec ? 128 : 32;
  const dim3 grid((unsigned)a.heads, (unsigned)((a.vdim + cols - 1) / cols), (unsigned)n_seqs);
#define GB_LS(VECV, RV) launch_k(lightning_step_kernel<TI, VECV, RV>, grid, 256, 0, stream, a)
  if (vec) {
    if (a.dim <= 32) GB_LS(4, 4); else if (a.dim <= 64) GB_LS(4, 8); else if (a.dim <= 128) GB_LS(4, 16); else GB_LS(4, 32);
  } else {
    if (a.dim <= 64) GB_LS(1, 8); else if (a.dim <= 256) GB_LS(1, 32); else GB_LS(1, 64);
  }
#undef GB_LS
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

// raw != 0: SiLU is applied here; else the columns carry it already.
GB_API int gb_lightning_step(const void* proj, int proj_f32, int raw, int n_part, long part_stride, int ld, const float* decay, float* state, int n_slots,
                             const int* cu_q, const int* seq_slots, float* out, int ld_out, int heads, int dim, int vdim, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || n_part < 1 || ld < 2 * heads * dim + heads * vdim || ld_out < heads * vdim) return fail("lightning: bad sizes%s");
  if (dim > 512) return fail("lightning: a key dimension of at most 512%s");
  if (n_seqs > 65535) return fail("lightning: too many sequences%s");
  LightningArgs a;
  a.raw = raw; a.proj = proj; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.decay = decay; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q;
  a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out; a.heads = heads; a.dim = dim; a.vdim = vdim;
  return proj_f32 ? lightning_step_launch<float>(a, n_seqs, stream) : lightning_step_launch<__nv_bfloat16>(a, n_seqs, stream);
}
