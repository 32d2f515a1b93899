// Token-wise kernels of models that keep their residual stream in 32-bit floats (models described layer by layer):
//   embed_f32           rows of a bf16 / f32 embedding table -> f32 stream
//   stream_norm         stream += pending update (bf16, f32, or K-split fp32 partial sums of a projection) [+ a vector added to
//                       every row], then RMSNorm of the row with an f32 weight -> bf16 or f32 rows for the next projection
//   stream_dyt          the same with Dynamic Tanh, tanh(alpha x) w + b, in place of the norm, and one of its own over the update, which
//                       may also be the router-weighted sum of expert outputs (formed here)
//   stream_rms2         stream_norm for an update with an RMSNorm of its own, a row added per token, and a second set of normalised rows
//   stream_join         stream += factor * result, for up to three pending results; a copy of the rows for a projection of the stream itself
//   stream_depth        stream += results as in stream_join; the new stream is kept, and a weighted sum of it and of earlier kept ones goes on, RMSNormed
//   depth_base          the part of later sums that is known already, for several of them in one pass
//   qk_unit_store       fused Q | K | V rows -> Q / K divided by their root mean square per head (no weight), K / V into their
//                       cache slots, Q scaled (by a function of the position, too) and laid out for the attention kernels
//   gated_norm          RMSNorm over all heads' outputs together, times sigmoid(gate): the tail of a linear-attention mixer
//   part_norm           RMSNorm of equal parts of a row, after (or before) SiLU(gate) if there is one: the tail of Mamba-2, HGRN2 and RWKV mixers
//   sigmoid_gate        the heads' outputs of an attention, times sigmoid(gate)
//   token_gate          GELU(z) times a row of a table, by token
//   gelu_f32            the exact GELU of f32 values (the 32-bit path)
//   act_mul             act(gate) * up of f32 rows (the 32-bit path; the bf16 path has it in the GEMM epilogue)
// One pass over HBM each; sizes are arbitrary (vector paths when they divide).  Output rows may be wider than the data (padding to
// the 16-byte row pitch the TMA descriptors of the next GEMM need); the padding is written as zero.
//
// The bf16-stream counterparts are in elementwise.cu (reference: common/transformer.h:593-637, :1281-1315).
#include "sm100.cuh"
#include "host_common.h"
#include <algorithm>

namespace gb {

__device__ __forceinline__ float ld_f(const float* p) { return *p; }
__device__ __forceinline__ float ld_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// four consecutive elements (aligned)
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// Sum over the block (256 threads); every thread gets it.
__device__ __forceinline__ float block_sum_256(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) s += red[i];
  return s;
}

// ------------------------------------------------------------------------------------------ embed
template <typename T>
__global__ void embed_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int width, int vocab, float scale) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) id = 0;
  for (int i = threadIdx.x; i < width; i += blockDim.x) out[(size_t)t * width + i] = ld_f(table + (size_t)id * width + i) * scale;
}

// ------------------------------------------------------------------------------------------ stream norm
struct StreamNormArgs {
  float* x;                     // stream [rows, width]
  const void* delta;            // pending update: f32 / bf16 [n_part][rows, ld_delta]; null = none
  int n_part; long part_stride; // K-split partial sums: slabs `part_stride` elements apart, added in order
  int ld_delta;
  float factor;                 // of the update
  const float* add;             // vector added to every row after the update; null = none
  const float* weight;          // f32 [width]
  const float* dot; float* gate;   // gate[r] = sigmoid(sum of x / rms(x) * dot) of output row r; null = none
  const long long* rows;        // output row r comes from stream row rows[r] (then the stream is not written); null = all rows in place
  void* out; int ld_out;        // normalised rows, ld_out >= width, the columns behind `width` are zeroed; null = only update the stream
  int width; float eps;
};

template <typename TD, typename TO, int VPT>       // VPT float4 per thread, width <= 1024 * VPT and width % 4 == 0
__global__ void __launch_bounds__(256)
stream_norm_vec_kernel(const StreamNormArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][8];
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  float* x = a.x + src * a.width;
  const TD* d = a.delta != nullptr ? (const TD*)a.delta + src * a.ld_delta : nullptr;
  const int nv = a.width >> 2;
  float4 v[VPT];
  float ss = 0.f, sd = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nv) continue;
    v[i] = ld4(x + c * 4);
    if (d != nullptr) {
      float4 s = ld4(d + c * 4);
      for (int p = 1; p < a.n_part; ++p) {
        const float4 q = ld4(d + (size_t)p * a.part_stride + c * 4);
        s.x += q.x; s.y += q.y; s.z += q.z; s.w += q.w;
      }
      v[i].x = fmaf(a.factor, s.x, v[i].x); v[i].y = fmaf(a.factor, s.y, v[i].y); v[i].z = fmaf(a.factor, s.z, v[i].z); v[i].w = fmaf(a.factor, s.w, v[i].w);
    }
    if (a.add != nullptr) {
      const float4 q = ld4(a.add + c * 4);
      v[i].x += q.x; v[i].y += q.y; v[i].z += q.z; v[i].w += q.w;
    }
    if (a.rows == nullptr && (d != nullptr || a.add != nullptr)) st4(x + c * 4, v[i]);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    if (a.dot != nullptr) {
      const float4 q = ld4(a.dot + c * 4);
      sd += v[i].x * q.x + v[i].y * q.y + v[i].z * q.z + v[i].w * q.w;
    }
  }
  if (a.out == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red[0]) / (float)a.width + a.eps);
  if (a.dot != nullptr) {
    const float g = block_sum_256(sd, red[1]) * inv;
    if (threadIdx.x == 0) a.gate[r] = 1.0f / (1.0f + expf(-g));
  }
  TO* o = (TO*)a.out + r * a.ld_out;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nv) continue;
    const float4 w = ld4(a.weight + c * 4);
    st4(o + c * 4, make_float4(v[i].x * inv * w.x, v[i].y * inv * w.y, v[i].z * inv * w.z, v[i].w * inv * w.w));
  }
  for (int c = a.width + threadIdx.x; c < a.ld_out; c += 256) st_f(o + c, 0.f);
}

template <typename TD, typename TO>                // any width
__global__ void __launch_bounds__(256)
stream_norm_any_kernel(const StreamNormArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][8];
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  float* x = a.x + src * a.width;
  const TD* d = a.delta != nullptr ? (const TD*)a.delta + src * a.ld_delta : nullptr;
  auto value = [&](int c) {
    float v = x[c];
    if (d != nullptr) {
      float s = ld_f(d + c);
      for (int p = 1; p < a.n_part; ++p) s += ld_f(d + (size_t)p * a.part_stride + c);
      v = fmaf(a.factor, s, v);
    }
    if (a.add != nullptr) v += a.add[c];
    return v;
  };
  const bool in_place = a.rows == nullptr;
  float ss = 0.f, sd = 0.f;
  for (int c = threadIdx.x; c < a.width; c += 256) {
    const float v = value(c);
    if (in_place) x[c] = v;
    ss += v * v;
    if (a.dot != nullptr) sd += v * a.dot[c];
  }
  if (a.out == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red[0]) / (float)a.width + a.eps);
  if (a.dot != nullptr) {
    const float g = block_sum_256(sd, red[1]) * inv;
    if (threadIdx.x == 0) a.gate[r] = 1.0f / (1.0f + expf(-g));
  }
  TO* o = (TO*)a.out + r * a.ld_out;
  for (int c = threadIdx.x; c < a.width; c += 256) st_f(o + c, (in_place ? x[c] : value(c)) * inv * a.weight[c]);
  for (int c = a.width + threadIdx.x; c < a.ld_out; c += 256) st_f(o + c, 0.f);
}

// ------------------------------------------------------------------------------------------ stream norm, normed update, two outputs
struct StreamRms2Args {
  float* x;                     // stream [rows, width]
  const void* delta; int n_part; long part_stride; int ld_delta;   // as in StreamNormArgs
  const float* post_w; float post_eps;                             // the update is divided by its root mean square and multiplied by this (null: added as it is)
  const float* add;             // [rows, width], added after the update; null = none
  const float* w[2];            // weights of the two outputs
  const long long* rows;        // as in StreamNormArgs
  void* out[2]; int ld_out;     // out[1] null = one output
  int width; float eps;
};

template <typename TD, typename TO, int VPT>       // VPT float4 per thread, width <= 1024 * VPT and width % 4 == 0
__global__ void __launch_bounds__(256)
stream_rms2_vec_kernel(const StreamRms2Args a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][8];
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  float* x = a.x + src * a.width;
  const int nv = a.width >> 2;
  float4 v[VPT], u[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    v[i] = u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nv) v[i] = ld4(x + c * 4);
  }
  if (a.delta != nullptr) {
    const TD* d = (const TD*)a.delta + src * a.ld_delta;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c >= nv) continue;
      u[i] = ld4(d + c * 4);
      for (int p = 1; p < a.n_part; ++p) {
        const float4 q = ld4(d + (size_t)p * a.part_stride + c * 4);
        u[i].x += q.x; u[i].y += q.y; u[i].z += q.z; u[i].w += q.w;
      }
      ss += u[i].x * u[i].x + u[i].y * u[i].y + u[i].z * u[i].z + u[i].w * u[i].w;
    }
    const bool post = a.post_w != nullptr;
    const float inv = post ? 1.0f / sqrtf(block_sum_256(ss, red[0]) / (float)a.width + a.post_eps) : 1.0f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c >= nv) continue;
      const float4 w = post ? ld4(a.post_w + c * 4) : make_float4(1.f, 1.f, 1.f, 1.f);
      v[i].x += u[i].x * inv * w.x; v[i].y += u[i].y * inv * w.y; v[i].z += u[i].z * inv * w.z; v[i].w += u[i].w * inv * w.w;
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nv) continue;
    if (a.add != nullptr) {
      const float4 q = ld4(a.add + src * a.width + c * 4);
      v[i].x += q.x; v[i].y += q.y; v[i].z += q.z; v[i].w += q.w;
    }
    if (a.rows == nullptr && (a.delta != nullptr || a.add != nullptr)) st4(x + c * 4, v[i]);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  }
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red[1]) / (float)a.width + a.eps);
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    if (a.out[y] == nullptr) continue;
    TO* o = (TO*)a.out[y] + r * a.ld_out;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c >= nv) continue;
      const float4 w = ld4(a.w[y] + c * 4);
      st4(o + c * 4, make_float4(v[i].x * inv * w.x, v[i].y * inv * w.y, v[i].z * inv * w.z, v[i].w * inv * w.w));
    }
    for (int c = a.width + threadIdx.x; c < a.ld_out; c += 256) st_f(o + c, 0.f);
  }
}

template <typename TD, typename TO>                // any width
__global__ void __launch_bounds__(256)
stream_rms2_any_kernel(const StreamRms2Args a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][8];
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  float* x = a.x + src * a.width;
  const TD* d = a.delta != nullptr ? (const TD*)a.delta + src * a.ld_delta : nullptr;
  auto update = [&](int c) {
    float s = ld_f(d + c);
    for (int p = 1; p < a.n_part; ++p) s += ld_f(d + (size_t)p * a.part_stride + c);
    return s;
  };
  float ud = 1.0f;
  if (d != nullptr && a.post_w != nullptr) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.width; c += 256) { const float u = update(c); ss += u * u; }
    ud = 1.0f / sqrtf(block_sum_256(ss, red[0]) / (float)a.width + a.post_eps);
  }
  auto value = [&](int c) {
    float v = x[c];
    if (d != nullptr) v += update(c) * ud * (a.post_w != nullptr ? a.post_w[c] : 1.0f);
    if (a.add != nullptr) v += a.add[src * a.width + c];
    return v;
  };
  const bool in_place = a.rows == nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.width; c += 256) {
    const float v = value(c);
    if (in_place) x[c] = v;
    ss += v * v;
  }
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red[1]) / (float)a.width + a.eps);
  for (int c = threadIdx.x; c < a.ld_out; c += 256) {
    const float v = c < a.width ? (in_place ? x[c] : value(c)) * inv : 0.f;
    for (int y = 0; y < 2; ++y)
      if (a.out[y] != nullptr) st_f((TO*)a.out[y] + r * a.ld_out + c, c < a.width ? v * a.w[y][c] : 0.f);
  }
}

// ------------------------------------------------------------------------------------------ several pending results into the stream
struct JoinPart {               // mirrored by ops/stream.py
  const void* p;                // f32 / bf16 [n_part][rows, ld], or expert outputs [*, ld] when pair_row is set
  const int* pair_row; const float* weights;         // as in DytArgs
  long stride;
  int f32, n_part, ld, k;
  float scale;
  const float* row_scale;       // one more factor per row (null = none)
};

// x[0 .. V - 1] (columns c ... of row r) += the part's result
template <int V>
__device__ __forceinline__ void add_part(const JoinPart& d, size_t r, int c, float* x) {
  float u[V];
#pragma unroll
  for (int j = 0; j < V; ++j) u[j] = 0.f;
  auto load = [&](const auto* p, float* v) {
    if constexpr (V == 4) { const float4 q = ld4(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
    else v[0] = ld_f(p);
  };
  auto add = [&](size_t off, float w) {
    float q[V];
    if (d.f32) load((const float*)d.p + off + c, q); else load((const __nv_bfloat16*)d.p + off + c, q);
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] = fmaf(w, q[j], u[j]);
  };
  if (d.pair_row != nullptr) {
#pragma unroll 4
    for (int e = 0; e < d.k; ++e) {
      const int row = d.pair_row[r * d.k + e];
      if (row >= 0) add((size_t)row * d.ld, d.weights[r * d.k + e]);
    }
  } else {
#pragma unroll 4
    for (int p = 0; p < d.n_part; ++p) add((size_t)p * d.stride + r * d.ld, 1.0f);
  }
  const float f = d.row_scale != nullptr ? d.scale * d.row_scale[r] : d.scale;
#pragma unroll
  for (int j = 0; j < V; ++j) x[j] = fmaf(f, u[j], x[j]);
}

struct JoinArgs {
  float* x;
  JoinPart part[3]; int n;
  void* out; int ld_out;        // copy of the new rows (null = none), zero behind `width`
  int width;
};

template <typename TO, int V>                      // V neighbouring columns per thread
__global__ void __launch_bounds__(256)
stream_join_kernel(const JoinArgs a) {
  pdl_wait();
  pdl_trigger();
  const size_t r = blockIdx.x;
  const int c = (blockIdx.y * 256 + threadIdx.x) * V;
  if (c >= a.width) {                              // padding (V == 4: width % 4 == 0)
    if (a.out != nullptr) {
#pragma unroll
      for (int i = 0; i < V; ++i) if (c + i < a.ld_out) st_f((TO*)a.out + r * a.ld_out + c + i, 0.f);
    }
    return;
  }
  float x[V];
  auto load = [&](const auto* p, float* v) {
    if constexpr (V == 4) { const float4 q = ld4(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
    else v[0] = ld_f(p);
  };
  load(a.x + r * a.width + c, x);
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    if (i >= a.n) break;
    add_part<V>(a.part[i], r, c, x);
  }
  if constexpr (V == 4) {
    const float4 y = make_float4(x[0], x[1], x[2], x[3]);
    st4(a.x + r * a.width + c, y);
    if (a.out != nullptr) st4((TO*)a.out + r * a.ld_out + c, y);
  } else {
    a.x[r * a.width + c] = x[0];
    if (a.out != nullptr) st_f((TO*)a.out + r * a.ld_out + c, x[0]);
  }
}

// ------------------------------------------------------------------------------------------ averages over the stream at earlier places
struct DepthArgs {
  float* x;                     // stream [rows, width]; becomes the average
  JoinPart part[3]; int n;
  float* hist; long stride;     // [places][rows, width], `stride` elements apart: the streams kept so far; the new one goes to place `at`
  const float* base; int first; // the sum over the places below `first` [rows, width] (null: first = 0)
  int at; const float* w;       // the average is the sum of w[j] * place j, j = 0 .. at
  const float* weight;          // f32 [width], of the norm
  const long long* rows;        // output row r comes from stream row rows[r] (then neither stream nor history is written); null = all rows in place
  void* out; int ld_out;        // normalised rows, zero behind `width`; null = only the average
  int width; float eps;
};

template <typename TO, int VPT>                    // VPT float4 per thread, width <= 1024 * VPT and width % 4 == 0
__global__ void __launch_bounds__(256)
stream_depth_vec_kernel(const DepthArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  const int nv = a.width >> 2;
  const float w_at = a.w[a.at];
  float4 x[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c >= nv) continue;
    float v[4];
    *reinterpret_cast<float4*>(v) = ld4(a.x + src * a.width + c * 4);
#pragma unroll
    for (int p = 0; p < 3; ++p) if (p < a.n) add_part<4>(a.part[p], src, c * 4, v);
    x[i] = make_float4(v[0], v[1], v[2], v[3]);
    if (a.rows == nullptr) st4(a.hist + (size_t)a.at * a.stride + src * a.width + c * 4, x[i]);
    x[i].x *= w_at; x[i].y *= w_at; x[i].z *= w_at; x[i].w *= w_at;
    if (a.base != nullptr) {
      const float4 q = ld4(a.base + src * a.width + c * 4);
      x[i].x += q.x; x[i].y += q.y; x[i].z += q.z; x[i].w += q.w;
    }
  }
#pragma unroll 4
  for (int j = a.first; j < a.at; ++j) {
    const float w = a.w[j];
    const float* h = a.hist + (size_t)j * a.stride + src * a.width;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c >= nv) continue;
      const float4 q = ld4(h + c * 4);
      x[i].x = fmaf(w, q.x, x[i].x); x[i].y = fmaf(w, q.y, x[i].y); x[i].z = fmaf(w, q.z, x[i].z); x[i].w = fmaf(w, q.w, x[i].w);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
    if (c < nv && a.rows == nullptr) st4(a.x + src * a.width + c * 4, x[i]);
  }
  if (a.out == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red) / (float)a.width + a.eps);
  TO* o = (TO*)a.out + r * a.ld_out;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nv) continue;
    const float4 w = ld4(a.weight + c * 4);
    st4(o + c * 4, make_float4(x[i].x * inv * w.x, x[i].y * inv * w.y, x[i].z * inv * w.z, x[i].w * inv * w.w));
  }
  for (int c = a.width + threadIdx.x; c < a.ld_out; c += 256) st_f(o + c, 0.f);
}

template <typename TO>                             // any width
__global__ void __launch_bounds__(256)
stream_depth_any_kernel(const DepthArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  const size_t at = src * a.width;
  const bool in_place = a.rows == nullptr;
  auto average = [&](int c) {
    float x = a.x[at + c];
    for (int p = 0; p < a.n; ++p) add_part<1>(a.part[p], src, c, &x);
    if (in_place) a.hist[(size_t)a.at * a.stride + at + c] = x;
    float s = x * a.w[a.at];
    if (a.base != nullptr) s += a.base[at + c];
    for (int j = a.first; j < a.at; ++j) s = fmaf(a.w[j], a.hist[(size_t)j * a.stride + at + c], s);
    return s;
  };
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.width; c += 256) {
    const float v = average(c);
    if (in_place) a.x[at + c] = v;
    ss += v * v;
  }
  if (a.out == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red) / (float)a.width + a.eps);
  TO* o = (TO*)a.out + r * a.ld_out;
  for (int c = threadIdx.x; c < a.width; c += 256) st_f(o + c, (in_place ? a.x[at + c] : average(c)) * inv * a.weight[c]);
  for (int c = a.width + threadIdx.x; c < a.ld_out; c += 256) st_f(o + c, 0.f);
}

// base[k] = sum of w[k][j] * place j over j < places, for k < K: every place is read once.
constexpr int kDepthBlock = 8;
struct DepthBaseArgs { const float* hist; long stride; int places; const float* w[kDepthBlock]; float* base; long n; };

template <int V>
__global__ void __launch_bounds__(256)
depth_base_kernel(const DepthBaseArgs a, int k_n) {
  pdl_wait();
  pdl_trigger();
  const long i = ((long)blockIdx.x * 256 + threadIdx.x) * V;
  if (i >= a.n) return;
  float acc[kDepthBlock][V];
#pragma unroll
  for (int k = 0; k < kDepthBlock; ++k)
#pragma unroll
    for (int y = 0; y < V; ++y) acc[k][y] = 0.f;
#pragma unroll 4
  for (int j = 0; j < a.places; ++j) {
    float q[V];
    const float* p = a.hist + (size_t)j * a.stride + i;
    if constexpr (V == 4) { const float4 f = ld4(p); q[0] = f.x; q[1] = f.y; q[2] = f.z; q[3] = f.w; }
    else q[0] = *p;
#pragma unroll
    for (int k = 0; k < kDepthBlock; ++k) {
      const float w = k < k_n ? a.w[k][j] : 0.f;
#pragma unroll
      for (int y = 0; y < V; ++y) acc[k][y] = fmaf(w, q[y], acc[k][y]);
    }
  }
#pragma unroll
  for (int k = 0; k < kDepthBlock; ++k)
    if (k < k_n) {
      float* p = a.base + (size_t)k * a.n + i;
      if constexpr (V == 4) st4(p, make_float4(acc[k][0], acc[k][1], acc[k][2], acc[k][3]));
      else *p = acc[k][0];
    }
}

// ------------------------------------------------------------------------------------------ gates
struct HeadGateArgs {
  void* a;                      // [rows, heads, dvp], in place
  const void* gate; int n_part; long part_stride; int ld_gate;     // pre-activations [n_part][rows, ld_gate]: heads x dv columns
  long n; int heads, dv, dvp;
};

template <typename TA, typename TG, int V>         // V neighbouring values of a head per thread
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(const HeadGateArgs a) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * 256 + threadIdx.x;
  if (i >= a.n) return;
  const int per = a.dv / V;
  const long rh = i / per;                         // row * heads + head
  const int c = (int)(i - rh * per) * V;
  const long r = rh / a.heads;
  const int h = (int)(rh - r * a.heads);
  TA* p = (TA*)a.a + (size_t)rh * a.dvp + c;
  const TG* g = (const TG*)a.gate + (size_t)r * a.ld_gate + (size_t)h * a.dv + c;
  if constexpr (V == 4) {
    float4 z = ld4(g);
    for (int q = 1; q < a.n_part; ++q) {
      const float4 y = ld4(g + (size_t)q * a.part_stride);
      z.x += y.x; z.y += y.y; z.z += y.z; z.w += y.w;
    }
    const float4 v = ld4(p);
    st4(p, make_float4(v.x / (1.0f + expf(-z.x)), v.y / (1.0f + expf(-z.y)), v.z / (1.0f + expf(-z.z)), v.w / (1.0f + expf(-z.w))));
  } else {
    float z = ld_f(g);
    for (int q = 1; q < a.n_part; ++q) z += ld_f(g + (size_t)q * a.part_stride);
    st_f(p, ld_f(p) / (1.0f + expf(-z)));
  }
}

struct TokenGateArgs {
  const void* z; int n_part; long part_stride; int ld_z;           // [n_part][rows, ld_z]
  const int* ids; const void* table; int table_f32, ld_t, col, vocab;
  void* out; int ld_out; long total; int n;
};

template <typename TZ, typename TO>
__global__ void __launch_bounds__(256)
token_gate_kernel(const TokenGateArgs a) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * 256 + threadIdx.x;
  if (i >= a.total) return;
  const long r = i / a.ld_out;
  const int c = (int)(i - r * a.ld_out);
  float y = 0.f;
  if (c < a.n) {
    const TZ* p = (const TZ*)a.z + (size_t)r * a.ld_z + c;
    float z = ld_f(p);
    for (int q = 1; q < a.n_part; ++q) z += ld_f(p + (size_t)q * a.part_stride);
    int id = a.ids[r];
    if (id < 0 || id >= a.vocab) id = 0;
    const size_t off = (size_t)id * a.ld_t + a.col + c;
    const float e = a.table_f32 ? ((const float*)a.table)[off] : __bfloat162float(((const __nv_bfloat16*)a.table)[off]);
    y = 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))) * e;
  }
  st_f((TO*)a.out + i, y);
}

// ------------------------------------------------------------------------------------------ stream with Dynamic Tanh
struct DytArgs {
  float* x;                     // stream [rows, width]
  const void* delta;            // update: f32 / bf16 [n_part][rows, ld_delta], or expert outputs [*, ld_delta] when pair_row is set; null = none
  int n_part; long part_stride; int ld_delta;
  const int* pair_row; const float* weights; int k;      // update of row r = sum_j weights[r k + j] * delta[pair_row[r k + j]] (negative row: nothing)
  float post_alpha; const float* post_w; const float* post_b;   // the update passes tanh(alpha u) w + b before it is added; null = it does not
  float alpha; const float* w; const float* b;
  const long long* rows;        // as in StreamNormArgs
  void* out; int ld_out;        // null = only update the stream
  int width;
};

__device__ __forceinline__ float dyt(float x, float alpha, float w, float b) { return fmaf(tanhf(alpha * x), w, b); }

// One thread per V neighbouring columns of a row (nothing is reduced over a row).
template <typename TD, typename TO, int V>
__global__ void __launch_bounds__(256)
stream_dyt_kernel(const DytArgs a) {
  pdl_wait();
  pdl_trigger();
  const size_t r = blockIdx.x, src = a.rows != nullptr ? (size_t)a.rows[r] : r;
  const int c = (blockIdx.y * 256 + threadIdx.x) * V;
  const int end = a.out != nullptr ? a.ld_out : a.width;
  if (c >= end) return;
  if (c >= a.width) {                              // padding (width % V == 0)
#pragma unroll
    for (int i = 0; i < V; ++i) if (c + i < end) st_f((TO*)a.out + r * a.ld_out + c + i, 0.f);
    return;
  }
  float x[V];
  auto load = [&](const auto* p, float* v) {
    if constexpr (V == 4) { const float4 q = ld4(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
    else v[0] = ld_f(p);
  };
  load(a.x + src * a.width + c, x);
  if (a.delta != nullptr) {
    float u[V];
    if (a.pair_row != nullptr) {
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = 0.f;
      const int* pr = a.pair_row + src * a.k;
      for (int j = 0; j < a.k; ++j) {
        const int row = pr[j];
        if (row < 0) continue;
        const float w = a.weights[src * a.k + j];
        float q[V];
        load((const TD*)a.delta + (size_t)row * a.ld_delta + c, q);
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] = fmaf(w, q[i], u[i]);
      }
    } else {
      const TD* d = (const TD*)a.delta + src * a.ld_delta + c;
      load(d, u);
      for (int p = 1; p < a.n_part; ++p) {
        float q[V];
        load(d + (size_t)p * a.part_stride, q);
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] += q[i];
      }
    }
    if (a.post_w != nullptr) {
      float w[V], b[V];
      load(a.post_w + c, w);
      load(a.post_b + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = dyt(u[i], a.post_alpha, w[i], b[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] += u[i];
    if (a.rows == nullptr) {
      if constexpr (V == 4) st4(a.x + src * a.width + c, make_float4(x[0], x[1], x[2], x[3]));
      else a.x[src * a.width + c] = x[0];
    }
  }
  if (a.out == nullptr) return;
  float w[V], b[V];
  load(a.w + c, w);
  load(a.b + c, b);
  TO* o = (TO*)a.out + r * a.ld_out + c;
#pragma unroll
  for (int i = 0; i < V; ++i) x[i] = dyt(x[i], a.alpha, w[i], b[i]);
  if constexpr (V == 4) st4(o, make_float4(x[0], x[1], x[2], x[3]));
  else st_f(o, x[0]);
}

// ------------------------------------------------------------------------------------------ Q / K unit norm + cache store
struct QkUnitArgs {
  const void* qkv;              // [n_part][tokens, ld]: rows [Q heads | K heads | V heads]
  int n_part; long part_stride; int ld;
  const int* slots;             // [tokens] cache slot (-1 = not stored)
  void* q_out;                  // [tokens, hq, dkp]
  void* k_cache; void* v_cache; // [slots, hkv, dkp] / [slots, hkv, dvp]
  long num_slots;
  int hq, hkv, dk, dv, dkp, dvp;
  float eps, q_scale;
  int unit;                     // 0: no normalisation
  const int* positions; float temp; double every;    // Q times 1 + temp ln(floor((position + 1) / every) + 1); null = not
};

// One warp per (token, head): heads 0 .. hq-1 are queries, then hkv keys, then hkv values.
template <typename TI, typename TC>
__global__ void __launch_bounds__(256)
qk_unit_store_kernel(const QkUnitArgs a, long n_items) {
  pdl_wait();
  pdl_trigger();
  const long w = ((long)blockIdx.x * 256 + threadIdx.x) >> 5;
  if (w >= n_items) return;
  const int lane = threadIdx.x & 31;
  const int per = a.hq + 2 * a.hkv;
  const long t = w / per;
  const int h = (int)(w - t * per);
  const bool is_q = h < a.hq, is_k = !is_q && h < a.hq + a.hkv;
  const int d = (is_q || is_k) ? a.dk : a.dv, dp = (is_q || is_k) ? a.dkp : a.dvp;
  const int col = is_q ? h * a.dk : is_k ? a.hq * a.dk + (h - a.hq) * a.dk : (a.hq + a.hkv) * a.dk + (h - a.hq - a.hkv) * a.dv;
  const TI* src = (const TI*)a.qkv + (size_t)t * a.ld + col;
  TC* dst;
  if (is_q) dst = (TC*)a.q_out + ((size_t)t * a.hq + h) * a.dkp;
  else {
    const int slot = a.slots[t];
    if (slot < 0 || slot >= a.num_slots) return;
    dst = is_k ? (TC*)a.k_cache + ((size_t)slot * a.hkv + (h - a.hq)) * a.dkp
               : (TC*)a.v_cache + ((size_t)slot * a.hkv + (h - a.hq - a.hkv)) * a.dvp;
  }
  auto value = [&](int c) {
    float s = ld_f(src + c);
    for (int p = 1; p < a.n_part; ++p) s += ld_f(src + (size_t)p * a.part_stride + c);
    return s;
  };
  const bool norm = a.unit && (is_q || is_k);
  const float q_scale = is_q && a.positions != nullptr ? a.q_scale * fmaf(a.temp, logf((float)floor((double)(a.positions[t] + 1) / a.every) + 1.0f), 1.0f) : a.q_scale;
  if (d <= 128) {               // the head's values stay in registers
    float v[4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) { const int c = lane + 32 * i; v[i] = c < d ? value(c) : 0.f; ss += v[i] * v[i]; }
    float sc = 1.0f;
    if (norm) sc = 1.0f / sqrtf(warp_sum(ss) / (float)d + a.eps);
    if (is_q) sc *= q_scale;
#pragma unroll
    for (int i = 0; i < 4; ++i) { const int c = lane + 32 * i; if (c < dp) st_f(dst + c, v[i] * sc); }
    return;
  }
  float sc = 1.0f;
  if (norm) {
    float ss = 0.f;
    for (int c = lane; c < d; c += 32) { const float v = value(c); ss += v * v; }
    sc = 1.0f / sqrtf(warp_sum(ss) / (float)d + a.eps);
  }
  if (is_q) sc *= q_scale;
  for (int c = lane; c < dp; c += 32) st_f(dst + c, c < d ? value(c) * sc : 0.f);
}

// ------------------------------------------------------------------------------------------ gated norm
struct GatedNormArgs {
  const float* o; int ld_o;     // [rows, n] f32
  const void* gate; int n_part; long part_stride; int ld_gate;     // gate pre-activations (columns of the mixer's input projection)
  const float* weight;          // f32 [n]
  void* out; int ld_out; int n; float eps;
};

template <typename TG, typename TO, int VPT>       // n % 4 == 0 and n <= 1024 * VPT
__global__ void __launch_bounds__(256)
gated_norm_vec_kernel(const GatedNormArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  const size_t r = blockIdx.x;
  const float* o = a.o + r * a.ld_o;
  const TG* g = (const TG*)a.gate + r * a.ld_gate;
  const int nv = a.n >> 2;
  float4 v[VPT], gv[VPT];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nv) continue;
    v[i] = ld4(o + c * 4);
    gv[i] = ld4(g + c * 4);
    for (int p = 1; p < a.n_part; ++p) {
      const float4 q = ld4(g + (size_t)p * a.part_stride + c * 4);
      gv[i].x += q.x; gv[i].y += q.y; gv[i].z += q.z; gv[i].w += q.w;
    }
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  }
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red) / (float)a.n + a.eps);
  TO* out = (TO*)a.out + r * a.ld_out;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nv) continue;
    const float4 w = ld4(a.weight + c * 4);
    st4(out + c * 4, make_float4(v[i].x * inv * w.x / (1.0f + expf(-gv[i].x)), v[i].y * inv * w.y / (1.0f + expf(-gv[i].y)),
                                 v[i].z * inv * w.z / (1.0f + expf(-gv[i].z)), v[i].w * inv * w.w / (1.0f + expf(-gv[i].w))));
  }
  for (int c = a.n + threadIdx.x; c < a.ld_out; c += 256) st_f(out + c, 0.f);
}

template <typename TG, typename TO>
__global__ void __launch_bounds__(256)
gated_norm_any_kernel(const GatedNormArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  const size_t r = blockIdx.x;
  const float* o = a.o + r * a.ld_o;
  const TG* g = (const TG*)a.gate + r * a.ld_gate;
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.n; c += 256) { const float v = o[c]; ss += v * v; }
  const float inv = 1.0f / sqrtf(block_sum_256(ss, red) / (float)a.n + a.eps);
  TO* out = (TO*)a.out + r * a.ld_out;
  for (int c = threadIdx.x; c < a.n; c += 256) {
    float gv = ld_f(g + c);
    for (int p = 1; p < a.n_part; ++p) gv += ld_f(g + (size_t)p * a.part_stride + c);
    st_f(out + c, o[c] * inv * a.weight[c] / (1.0f + expf(-gv)));
  }
  for (int c = a.n + threadIdx.x; c < a.ld_out; c += 256) st_f(out + c, 0.f);
}

// ------------------------------------------------------------------------------------------ norm of equal parts
struct PartNormArgs {
  const float* o; int ld_o;     // [rows, n] f32
  const void* gate; int n_part; long part_stride; int ld_gate;     // gate pre-activations (null = none)
  int gate_after;               // the gate multiplies the normalised values instead of the values
  const float* weight; int n_weight;   // f32, column c uses weight[c % n_weight]
  void* out; int ld_out; int n, parts; float eps; long items;
};

// G threads (a warp or a CTA) per (row, part), values in registers: parts of 4 G VPT columns at most, a multiple of 4; one weight per column of the row
// or of the part.
template <typename TG, typename TO, int G, int VPT>
__global__ void __launch_bounds__(256)
part_norm_vec_kernel(const PartNormArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  const long item = (long)blockIdx.x * (256 / G) + threadIdx.x / G;
  const bool live = item < a.items;
  const long r = live ? item / a.parts : 0;
  const int part = live ? (int)(item - r * a.parts) : 0, lane = threadIdx.x % G;
  const int len = a.n / a.parts, c0 = part * len, nv = live ? len >> 2 : 0;
  const float* o = a.o + (size_t)r * a.ld_o + c0;
  const TG* g = (const TG*)a.gate + (size_t)r * a.ld_gate + c0;
  float4 v[VPT], z[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = lane + i * G;
    v[i] = z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nv) { v[i] = ld4(o + c * 4); if (a.gate != nullptr) z[i] = ld4(g + c * 4); }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = lane + i * G;
    if (a.gate != nullptr && c < nv) {
      for (int p = 1; p < a.n_part; ++p) {
        const float4 q = ld4(g + (size_t)p * a.part_stride + c * 4);
        z[i].x += q.x; z[i].y += q.y; z[i].z += q.z; z[i].w += q.w;
      }
      z[i].x /= 1.0f + expf(-z[i].x); z[i].y /= 1.0f + expf(-z[i].y);
      z[i].z /= 1.0f + expf(-z[i].z); z[i].w /= 1.0f + expf(-z[i].w);
      if (!a.gate_after) { v[i].x *= z[i].x; v[i].y *= z[i].y; v[i].z *= z[i].z; v[i].w *= z[i].w; }
    }
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  }
  if constexpr (G == 32) ss = warp_sum(ss);
  else ss = block_sum_256(ss, red);
  if (!live) return;
  const float inv = 1.0f / sqrtf(ss / (float)len + a.eps);
  TO* out = (TO*)a.out + (size_t)r * a.ld_out;
  const float* w = a.weight + (a.n_weight == a.n ? c0 : 0);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = lane + i * G;
    if (c >= nv) continue;
    float4 q = ld4(w + c * 4);
    if (a.gate_after) { q.x *= z[i].x; q.y *= z[i].y; q.z *= z[i].z; q.w *= z[i].w; }
    st4(out + c0 + c * 4, make_float4(v[i].x * inv * q.x, v[i].y * inv * q.y, v[i].z * inv * q.z, v[i].w * inv * q.w));
  }
  if (part == a.parts - 1)
    for (int c = a.n + lane; c < a.ld_out; c += G) st_f(out + c, 0.f);
}

// Any sizes.
template <typename TG, typename TO, int G>
__global__ void __launch_bounds__(256)
part_norm_kernel(const PartNormArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  constexpr int kKeep = 8;                         // values per thread kept in registers
  const long item = (long)blockIdx.x * (256 / G) + threadIdx.x / G;
  const bool live = item < a.items;
  const long r = live ? item / a.parts : 0;
  const int part = live ? (int)(item - r * a.parts) : 0, lane = threadIdx.x % G;
  const int len = a.n / a.parts, c0 = part * len;
  const float* o = a.o + (size_t)r * a.ld_o + c0;
  const TG* g = a.gate != nullptr ? (const TG*)a.gate + (size_t)r * a.ld_gate + c0 : nullptr;
  auto gate = [&](int c) {
    float z = ld_f(g + c);
    for (int p = 1; p < a.n_part; ++p) z += ld_f(g + (size_t)p * a.part_stride + c);
    return z / (1.0f + expf(-z));
  };
  auto value = [&](int c) { return g != nullptr && !a.gate_after ? o[c] * gate(c) : o[c]; };
  float keep[kKeep];
  float ss = 0.f;
  if (live) {
#pragma unroll
    for (int i = 0; i < kKeep; ++i) { const int c = lane + i * G; if (c < len) { keep[i] = value(c); ss += keep[i] * keep[i]; } }
    for (int c = lane + kKeep * G; c < len; c += G) { const float v = value(c); ss += v * v; }
  }
  if constexpr (G == 32) ss = warp_sum(ss);
  else ss = block_sum_256(ss, red);
  if (!live) return;
  const float inv = 1.0f / sqrtf(ss / (float)len + a.eps);
  TO* out = (TO*)a.out + (size_t)r * a.ld_out;
  auto w = [&](int c) { return a.weight[(c0 + c) % a.n_weight] * (a.gate_after ? gate(c) : 1.0f); };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) { const int c = lane + i * G; if (c < len) st_f(out + c0 + c, keep[i] * inv * w(c)); }
  for (int c = lane + kKeep * G; c < len; c += G) st_f(out + c0 + c, value(c) * inv * w(c));
  if (part == a.parts - 1)
    for (int c = a.n + lane; c < a.ld_out; c += G) st_f(out + c, 0.f);
}

// ------------------------------------------------------------------------------------------ activations, f32
__global__ void gelu_f32_kernel(const float* __restrict__ x, float* __restrict__ out, long n) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) out[i] = 0.5f * x[i] * (1.0f + erff(x[i] * 0.70710678118654752f));
}

__global__ void act_mul_f32_kernel(const float* __restrict__ gu, float* __restrict__ out, long n, int inter, int ld, int act, float cap) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const long r = i / inter;
  const int c = (int)(i - r * inter);
  float g = gu[r * ld + c], u = gu[r * ld + inter + c];
  if (act == 2) {
    g = fminf(g, cap);
    out[r * inter + c] = g / (1.0f + expf(-1.702f * g)) * (fminf(fmaxf(u, -cap), cap) + 1.0f);
    return;
  }
  const float y = act == 1 ? 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) : g / (1.0f + expf(-g));
  out[r * inter + c] = y * u;
}

}  // namespace gb

using namespace gb;

GB_API int gb_embed_f32(const int* ids, const void* table, int table_f32, float* out, int n_tok, int width, int vocab, float scale,
                        cudaStream_t stream) {
  if (n_tok <= 0) return 0;
  if (table_f32) launch_k(embed_f32_kernel<float>, (unsigned)n_tok, 256, 0, stream, ids, (const float*)table, out, width, vocab, scale);
  else launch_k(embed_f32_kernel<__nv_bfloat16>, (unsigned)n_tok, 256, 0, stream, ids, (const __nv_bfloat16*)table, out, width, vocab, scale);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename TD, typename TO>
static int stream_norm_launch(const StreamNormArgs& a, int n_rows, cudaStream_t stream) {
  const size_t ed = sizeof(TD) * 4, eo = sizeof(TO) * 4;
  const bool vec = a.width % 4 == 0 && a.width <= 16384 && (a.delta == nullptr || (a.ld_delta % 4 == 0 && a.part_stride % 4 == 0 && (uintptr_t)a.delta % ed == 0)) &&
                   (a.out == nullptr || (a.ld_out % 4 == 0 && (uintptr_t)a.out % eo == 0)) && (uintptr_t)a.x % 16 == 0 && (uintptr_t)a.weight % 16 == 0 &&
                   (uintptr_t)a.add % 16 == 0 && (uintptr_t)a.dot % 16 == 0;
  if (!vec) launch_k(stream_norm_any_kernel<TD, TO>, (unsigned)n_rows, 256, 0, stream, a);
  else if (a.width <= 1024) launch_k(stream_norm_vec_kernel<TD, TO, 1>, (unsigned)n_rows, 256, 0, stream, a);
  else if (a.width <= 4096) launch_k(stream_norm_vec_kernel<TD, TO, 4>, (unsigned)n_rows, 256, 0, stream, a);
  else launch_k(stream_norm_vec_kernel<TD, TO, 16>, (unsigned)n_rows, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See StreamNormArgs.  delta_f32 / out_f32 give the element types; `rows` (int64, device) selects stream rows.
GB_API int gb_stream_norm(float* x, const void* delta, int delta_f32, int n_part, long part_stride, int ld_delta, float factor, const float* add, const float* weight,
                          const float* dot, float* gate, const long long* rows, void* out, int out_f32, int ld_out, int n_rows, int width, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || (out != nullptr && (ld_out < width || weight == nullptr)) || (delta != nullptr && (ld_delta < width || n_part < 1)))
    return fail("stream_norm: bad widths%s");
  StreamNormArgs a;
  if (dot != nullptr && (gate == nullptr || rows != nullptr || out == nullptr)) return fail("stream_norm: a gate goes with all rows%s");
  a.x = x; a.delta = delta; a.n_part = n_part; a.part_stride = part_stride; a.ld_delta = ld_delta; a.add = add; a.weight = weight; a.rows = rows;
  a.factor = factor; a.dot = dot; a.gate = gate;
  a.out = out; a.ld_out = ld_out; a.width = width; a.eps = eps;
  if (delta_f32) return out_f32 ? stream_norm_launch<float, float>(a, n_rows, stream) : stream_norm_launch<float, __nv_bfloat16>(a, n_rows, stream);
  return out_f32 ? stream_norm_launch<__nv_bfloat16, float>(a, n_rows, stream) : stream_norm_launch<__nv_bfloat16, __nv_bfloat16>(a, n_rows, stream);
}

template <typename TD, typename TO>
static int stream_dyt_launch(const DytArgs& a, int n_rows, cudaStream_t stream) {
  const size_t ed = sizeof(TD) * 4, eo = sizeof(TO) * 4;
  const auto ok16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = a.width % 4 == 0 && (a.delta == nullptr || (a.ld_delta % 4 == 0 && a.part_stride % 4 == 0 && (uintptr_t)a.delta % ed == 0)) &&
                   (a.out == nullptr || (a.ld_out % 4 == 0 && (uintptr_t)a.out % eo == 0)) && ok16(a.x) && ok16(a.w) && ok16(a.b) && ok16(a.post_w) && ok16(a.post_b);
  const int cols = a.out != nullptr ? a.ld_out : a.width;
  if (vec) launch_k(stream_dyt_kernel<TD, TO, 4>, dim3((unsigned)n_rows, (unsigned)((cols + 1023) / 1024)), 256, 0, stream, a);
  else launch_k(stream_dyt_kernel<TD, TO, 1>, dim3((unsigned)n_rows, (unsigned)((cols + 255) / 256)), 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See DytArgs.
GB_API int gb_stream_dyt(float* x, const void* delta, int delta_f32, int n_part, long part_stride, int ld_delta, const int* pair_row, const float* weights, int k,
                         float post_alpha, const float* post_w, const float* post_b, float alpha, const float* w, const float* b, const long long* rows, void* out,
                         int out_f32, int ld_out, int n_rows, int width, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || (out != nullptr && (ld_out < width || w == nullptr || b == nullptr)) || (delta != nullptr && (ld_delta < width || n_part < 1)) ||
      (pair_row != nullptr && (weights == nullptr || k < 1)) || (post_w != nullptr && post_b == nullptr))
    return fail("stream_dyt: bad arguments%s");
  DytArgs a;
  a.x = x; a.delta = delta; a.n_part = n_part; a.part_stride = part_stride; a.ld_delta = ld_delta; a.pair_row = pair_row; a.weights = weights; a.k = k;
  a.post_alpha = post_alpha; a.post_w = post_w; a.post_b = post_b; a.alpha = alpha; a.w = w; a.b = b; a.rows = rows; a.out = out; a.ld_out = ld_out; a.width = width;
  if (delta_f32) return out_f32 ? stream_dyt_launch<float, float>(a, n_rows, stream) : stream_dyt_launch<float, __nv_bfloat16>(a, n_rows, stream);
  return out_f32 ? stream_dyt_launch<__nv_bfloat16, float>(a, n_rows, stream) : stream_dyt_launch<__nv_bfloat16, __nv_bfloat16>(a, n_rows, stream);
}

template <typename TG, typename TO>
static int part_norm_launch(const PartNormArgs& a, cudaStream_t stream) {
  const int len = a.n / a.parts;
  const size_t eg = sizeof(TG) * 4, eo = sizeof(TO) * 4;
  const bool vec = len % 4 == 0 && len <= 4096 && (a.n_weight == a.n || a.n_weight == len) && a.ld_o % 4 == 0 && a.ld_out % 4 == 0 && (uintptr_t)a.o % 16 == 0 &&
                   (uintptr_t)a.weight % 16 == 0 && (uintptr_t)a.out % eo == 0 &&
                   (a.gate == nullptr || (a.ld_gate % 4 == 0 && a.part_stride % 4 == 0 && (uintptr_t)a.gate % eg == 0));
  const unsigned warps = (unsigned)((a.items + 7) / 8);
  if (vec && len <= 128) launch_k(part_norm_vec_kernel<TG, TO, 32, 1>, warps, 256, 0, stream, a);
  else if (vec && len <= 512) launch_k(part_norm_vec_kernel<TG, TO, 32, 4>, warps, 256, 0, stream, a);
  else if (vec && len <= 1024) launch_k(part_norm_vec_kernel<TG, TO, 256, 1>, (unsigned)a.items, 256, 0, stream, a);
  else if (vec) launch_k(part_norm_vec_kernel<TG, TO, 256, 4>, (unsigned)a.items, 256, 0, stream, a);
  else if (len <= 512) launch_k(part_norm_kernel<TG, TO, 32>, (unsigned)((a.items + 7) / 8), 256, 0, stream, a);
  else launch_k(part_norm_kernel<TG, TO, 256>, (unsigned)a.items, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

GB_API int gb_part_norm(const float* o, int ld_o, const void* gate, int gate_f32, int n_part, long part_stride, int ld_gate, const float* weight, int n_weight,
                        void* out, int out_f32, int ld_out, int rows, int n, int parts, float eps, int gate_after, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (gate_after && gate == nullptr) return fail("part_norm: no gate%s");
  if (n < 1 || parts < 1 || n % parts || n_weight < 1 || n % n_weight || ld_o < n || ld_out < n || n_part < 1) return fail("part_norm: bad sizes%s");
  PartNormArgs a;
  a.o = o; a.ld_o = ld_o; a.gate = gate; a.n_part = n_part; a.part_stride = part_stride; a.ld_gate = ld_gate; a.weight = weight; a.n_weight = n_weight;
  a.out = out; a.ld_out = ld_out; a.n = n; a.parts = parts; a.eps = eps; a.items = (long)rows * parts; a.gate_after = gate_after;
  if (gate_f32) return out_f32 ? part_norm_launch<float, float>(a, stream) : part_norm_launch<float, __nv_bfloat16>(a, stream);
  return out_f32 ? part_norm_launch<__nv_bfloat16, float>(a, stream) : part_norm_launch<__nv_bfloat16, __nv_bfloat16>(a, stream);
}

// See QkUnitArgs.  in_f32: element type of qkv; cache_f32: element type of q_out and the caches.
GB_API int gb_qk_unit_store(const void* qkv, int in_f32, int n_part, long part_stride, int ld, const int* slots, void* q_out, void* k_cache, void* v_cache,
                            int cache_f32, long num_slots, int tokens, int hq, int hkv, int dk, int dv, int dkp, int dvp, float eps, float q_scale,
                            int unit, const int* positions, float temp, double every, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (hq < 1 || hkv < 1 || hq % hkv || dk < 1 || dv < 1 || dkp < dk || dvp < dv || n_part < 1) return fail("qk_unit_store: bad sizes%s");
  if ((dk <= 128 && dkp > 128) || (dv <= 128 && dvp > 128)) return fail("qk_unit_store: padding beyond 128%s");
  QkUnitArgs a;
  a.qkv = qkv; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.slots = slots; a.q_out = q_out; a.k_cache = k_cache; a.v_cache = v_cache;
  a.num_slots = num_slots; a.hq = hq; a.hkv = hkv; a.dk = dk; a.dv = dv; a.dkp = dkp; a.dvp = dvp; a.eps = eps; a.q_scale = q_scale; a.unit = unit;
  if (positions != nullptr && !(every > 0.0)) return fail("qk_unit_store: bad temperature%s");
  a.positions = positions; a.temp = temp; a.every = every;
  const long n = (long)tokens * (hq + 2 * hkv);
  const unsigned grid = (unsigned)((n + 7) / 8);
  if (in_f32 && cache_f32) launch_k(qk_unit_store_kernel<float, float>, grid, 256, 0, stream, a, n);
  else if (in_f32) launch_k(qk_unit_store_kernel<float, __nv_bfloat16>, grid, 256, 0, stream, a, n);
  else if (cache_f32) return fail("qk_unit_store: a 32-bit cache takes 32-bit rows%s");
  else launch_k(qk_unit_store_kernel<__nv_bfloat16, __nv_bfloat16>, grid, 256, 0, stream, a, n);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename TG, typename TO>
static int gated_norm_launch(const GatedNormArgs& a, int rows, cudaStream_t stream) {
  const size_t eg = sizeof(TG) * 4, eo = sizeof(TO) * 4;
  const bool vec = a.n % 4 == 0 && a.n <= 16384 && a.ld_o % 4 == 0 && a.ld_gate % 4 == 0 && a.part_stride % 4 == 0 && a.ld_out % 4 == 0 &&
                   (uintptr_t)a.o % 16 == 0 && (uintptr_t)a.gate % eg == 0 && (uintptr_t)a.out % eo == 0 && (uintptr_t)a.weight % 16 == 0;
  if (!vec) launch_k(gated_norm_any_kernel<TG, TO>, (unsigned)rows, 256, 0, stream, a);
  else if (a.n <= 1024) launch_k(gated_norm_vec_kernel<TG, TO, 1>, (unsigned)rows, 256, 0, stream, a);
  else if (a.n <= 4096) launch_k(gated_norm_vec_kernel<TG, TO, 4>, (unsigned)rows, 256, 0, stream, a);
  else launch_k(gated_norm_vec_kernel<TG, TO, 16>, (unsigned)rows, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

GB_API int gb_gated_norm(const float* o, int ld_o, const void* gate, int gate_f32, int n_part, long part_stride, int ld_gate, const float* weight,
                         void* out, int out_f32, int ld_out, int rows, int n, float eps, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (n < 1 || ld_o < n || ld_out < n || n_part < 1) return fail("gated_norm: bad sizes%s");
  GatedNormArgs a;
  a.o = o; a.ld_o = ld_o; a.gate = gate; a.n_part = n_part; a.part_stride = part_stride; a.ld_gate = ld_gate; a.weight = weight; a.out = out;
  a.ld_out = ld_out; a.n = n; a.eps = eps;
  if (gate_f32) return out_f32 ? gated_norm_launch<float, float>(a, rows, stream) : gated_norm_launch<float, __nv_bfloat16>(a, rows, stream);
  return out_f32 ? gated_norm_launch<__nv_bfloat16, float>(a, rows, stream) : gated_norm_launch<__nv_bfloat16, __nv_bfloat16>(a, rows, stream);
}

// act(gate) * up over f32 rows [gate | up]; act 0 = SiLU, 1 = the tanh form of GELU, 2 = g sigmoid(1.702 g) (u + 1), bounded by cap.
GB_API int gb_act_mul_f32(const float* gate_up, float* out, long rows, int inter, int ld, int act, float cap, cudaStream_t stream) {
  const long n = rows * inter;
  if (n <= 0) return 0;
  launch_k(act_mul_f32_kernel, (unsigned)((n + 255) / 256), 256, 0, stream, gate_up, out, n, inter, ld, act, cap);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename TD, typename TO>
static int stream_rms2_launch(const StreamRms2Args& a, int n_rows, cudaStream_t stream) {
  const size_t ed = sizeof(TD) * 4, eo = sizeof(TO) * 4;
  const auto ok16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = a.width % 4 == 0 && a.width <= 16384 && (a.delta == nullptr || (a.ld_delta % 4 == 0 && a.part_stride % 4 == 0 && (uintptr_t)a.delta % ed == 0)) &&
                   a.ld_out % 4 == 0 && (uintptr_t)a.out[0] % eo == 0 && (uintptr_t)a.out[1] % eo == 0 && ok16(a.x) && ok16(a.w[0]) && ok16(a.w[1]) && ok16(a.post_w) && ok16(a.add);
  if (!vec) launch_k(stream_rms2_any_kernel<TD, TO>, (unsigned)n_rows, 256, 0, stream, a);
  else if (a.width <= 1024) launch_k(stream_rms2_vec_kernel<TD, TO, 1>, (unsigned)n_rows, 256, 0, stream, a);
  else if (a.width <= 2048) launch_k(stream_rms2_vec_kernel<TD, TO, 2>, (unsigned)n_rows, 256, 0, stream, a);
  else if (a.width <= 4096) launch_k(stream_rms2_vec_kernel<TD, TO, 4>, (unsigned)n_rows, 256, 0, stream, a);
  else launch_k(stream_rms2_vec_kernel<TD, TO, 16>, (unsigned)n_rows, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See StreamRms2Args.
GB_API int gb_stream_rms2(float* x, const void* delta, int delta_f32, int n_part, long part_stride, int ld_delta, const float* post_w, float post_eps, const float* add,
                          const float* w0, const float* w1, const long long* rows, void* out0, void* out1, int out_f32, int ld_out, int n_rows, int width, float eps,
                          cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || out0 == nullptr || w0 == nullptr || (out1 != nullptr && w1 == nullptr) || ld_out < width || (delta != nullptr && (ld_delta < width || n_part < 1)))
    return fail("stream_rms2: bad arguments%s");
  StreamRms2Args a;
  a.x = x; a.delta = delta; a.n_part = n_part; a.part_stride = part_stride; a.ld_delta = ld_delta; a.post_w = post_w; a.post_eps = post_eps; a.add = add;
  a.w[0] = w0; a.w[1] = w1; a.rows = rows; a.out[0] = out0; a.out[1] = out1; a.ld_out = ld_out; a.width = width; a.eps = eps;
  if (delta_f32) return out_f32 ? stream_rms2_launch<float, float>(a, n_rows, stream) : stream_rms2_launch<float, __nv_bfloat16>(a, n_rows, stream);
  return out_f32 ? stream_rms2_launch<__nv_bfloat16, float>(a, n_rows, stream) : stream_rms2_launch<__nv_bfloat16, __nv_bfloat16>(a, n_rows, stream);
}

// x [n_rows, width] += sum of parts[0 .. n - 1] (host array of three); out: see JoinArgs.
GB_API int gb_stream_join(float* x, const JoinPart* parts, int n, void* out, int out_f32, int ld_out, int n_rows, int width, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || n < 1 || n > 3 || (out != nullptr && ld_out < width)) return fail("stream_join: bad sizes%s");
  JoinArgs a;
  bool vec = width % 4 == 0 && ((uintptr_t)x & 15) == 0 && (out == nullptr || (ld_out % 4 == 0 && (uintptr_t)out % (out_f32 ? 16 : 8) == 0));
  for (int i = 0; i < 3; ++i) {
    a.part[i] = parts[i];
    if (i >= n) continue;
    const JoinPart& d = parts[i];
    if (d.p == nullptr || d.ld < width || d.n_part < 1 || (d.pair_row != nullptr && (d.weights == nullptr || d.k < 1))) return fail("stream_join: bad part%s");
    vec = vec && d.ld % 4 == 0 && d.stride % 4 == 0 && (uintptr_t)d.p % (d.f32 ? 16 : 8) == 0;
  }
  a.x = x; a.n = n; a.out = out; a.ld_out = ld_out; a.width = width;
  const int cols = out != nullptr ? ld_out : width;
  const dim3 grid((unsigned)n_rows, (unsigned)((cols + (vec ? 1023 : 255)) / (vec ? 1024 : 256)));
  if (out_f32) { if (vec) launch_k(stream_join_kernel<float, 4>, grid, 256, 0, stream, a); else launch_k(stream_join_kernel<float, 1>, grid, 256, 0, stream, a); }
  else { if (vec) launch_k(stream_join_kernel<__nv_bfloat16, 4>, grid, 256, 0, stream, a); else launch_k(stream_join_kernel<__nv_bfloat16, 1>, grid, 256, 0, stream, a); }
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename TO>
static int stream_depth_launch(const DepthArgs& a, bool vec, int n_rows, cudaStream_t stream) {
  const unsigned g = (unsigned)n_rows;
  if (vec && a.width <= 1024) launch_k(stream_depth_vec_kernel<TO, 1>, g, 256, 0, stream, a);
  else if (vec && a.width <= 2048) launch_k(stream_depth_vec_kernel<TO, 2>, g, 256, 0, stream, a);
  else if (vec && a.width <= 4096) launch_k(stream_depth_vec_kernel<TO, 4>, g, 256, 0, stream, a);
  else if (vec && a.width <= 16384) launch_k(stream_depth_vec_kernel<TO, 16>, g, 256, 0, stream, a);
  else launch_k(stream_depth_any_kernel<TO>, g, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See DepthArgs; parts: host array of three.
GB_API int gb_stream_depth(float* x, const JoinPart* parts, int n, float* hist, long stride, const float* base, int first, int at, const float* w, const float* weight,
                           const long long* rows, void* out, int out_f32, int ld_out, int n_rows, int width, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || n < 1 || n > 3 || at < 1 || first < 0 || first > at || (base == nullptr) != (first == 0) || (out != nullptr && (ld_out < width || weight == nullptr)))
    return fail("stream_depth: bad arguments%s");
  DepthArgs a;
  const auto ok16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  bool vec = width % 4 == 0 && stride % 4 == 0 && ok16(x) && ok16(hist) && ok16(base) && ok16(weight) && (out == nullptr || (ld_out % 4 == 0 && (uintptr_t)out % (out_f32 ? 16 : 8) == 0));
  for (int i = 0; i < 3; ++i) {
    a.part[i] = parts[i];
    if (i >= n) continue;
    const JoinPart& d = parts[i];
    if (d.p == nullptr || d.ld < width || d.n_part < 1 || (d.pair_row != nullptr && (d.weights == nullptr || d.k < 1))) return fail("stream_depth: bad part%s");
    vec = vec && d.ld % 4 == 0 && d.stride % 4 == 0 && (uintptr_t)d.p % (d.f32 ? 16 : 8) == 0;
  }
  a.x = x; a.n = n; a.hist = hist; a.stride = stride; a.base = base; a.first = first; a.at = at; a.w = w; a.weight = weight; a.rows = rows; a.out = out; a.ld_out = ld_out;
  a.width = width; a.eps = eps;
  return out_f32 ? stream_depth_launch<float>(a, vec, n_rows, stream) : stream_depth_launch<__nv_bfloat16>(a, vec, n_rows, stream);
}

// base [k_n][n] from `places` blocks of n elements, `stride` apart; w: host array of k_n device pointers to at least `places` weights.
GB_API int gb_depth_base(const float* hist, long stride, int places, const float* const* w, int k_n, float* base, long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (places < 1 || k_n < 1 || k_n > kDepthBlock) return fail("depth_base: bad sizes%s");
  DepthBaseArgs a;
  for (int k = 0; k < kDepthBlock; ++k) a.w[k] = k < k_n ? w[k] : nullptr;
  a.hist = hist; a.stride = stride; a.places = places; a.base = base; a.n = n;
  const bool vec = n % 4 == 0 && stride % 4 == 0 && ((uintptr_t)hist & 15) == 0 && ((uintptr_t)base & 15) == 0;
  if (vec) launch_k(depth_base_kernel<4>, (unsigned)((n / 4 + 255) / 256), 256, 0, stream, a, k_n);
  else launch_k(depth_base_kernel<1>, (unsigned)((n + 255) / 256), 256, 0, stream, a, k_n);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

GB_API int gb_gelu_f32(const float* x, float* out, long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  launch_k(gelu_f32_kernel, (unsigned)((n + 255) / 256), 256, 0, stream, x, out, n);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename TA, typename TG>
static int sigmoid_gate_launch(HeadGateArgs a, long rows, cudaStream_t stream) {
  const bool vec = a.dv % 4 == 0 && a.dvp % 4 == 0 && a.ld_gate % 4 == 0 && a.part_stride % 4 == 0 && (uintptr_t)a.a % (4 * sizeof(TA)) == 0 && (uintptr_t)a.gate % (4 * sizeof(TG)) == 0;
  a.n = rows * a.heads * (a.dv / (vec ? 4 : 1));
  const unsigned grid = (unsigned)((a.n + 255) / 256);
  if (vec) launch_k(sigmoid_gate_kernel<TA, TG, 4>, grid, 256, 0, stream, a);
  else launch_k(sigmoid_gate_kernel<TA, TG, 1>, grid, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See HeadGateArgs.
GB_API int gb_sigmoid_gate(void* a_, int a_f32, const void* gate, int gate_f32, int n_part, long part_stride, int ld_gate, int rows, int heads, int dv, int dvp,
                           cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (heads < 1 || dv < 1 || dvp < dv || n_part < 1 || ld_gate < heads * dv) return fail("sigmoid_gate: bad sizes%s");
  HeadGateArgs a;
  a.a = a_; a.gate = gate; a.n_part = n_part; a.part_stride = part_stride; a.ld_gate = ld_gate; a.heads = heads; a.dv = dv; a.dvp = dvp; a.n = 0;
  if (a_f32) return gate_f32 ? sigmoid_gate_launch<float, float>(a, rows, stream) : sigmoid_gate_launch<float, __nv_bfloat16>(a, rows, stream);
  return gate_f32 ? sigmoid_gate_launch<__nv_bfloat16, float>(a, rows, stream) : sigmoid_gate_launch<__nv_bfloat16, __nv_bfloat16>(a, rows, stream);
}

// out [rows, ld_out] = gelu(z) * table[ids[row], col ...], zero behind n columns.
GB_API int gb_token_gate(const void* z, int z_f32, int n_part, long part_stride, int ld_z, const int* ids, const void* table, int table_f32, int ld_t, int col, int vocab,
                         void* out, int out_f32, int ld_out, int rows, int n, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (n < 1 || ld_out < n || ld_z < n || n_part < 1 || col < 0 || col + n > ld_t || vocab < 1) return fail("token_gate: bad sizes%s");
  TokenGateArgs a;
  a.z = z; a.n_part = n_part; a.part_stride = part_stride; a.ld_z = ld_z; a.ids = ids; a.table = table; a.table_f32 = table_f32; a.ld_t = ld_t; a.col = col; a.vocab = vocab;
  a.out = out; a.ld_out = ld_out; a.n = n; a.total = (long)rows * ld_out;
  const unsigned grid = (unsigned)((a.total + 255) / 256);
  if (z_f32) {
    if (out_f32) launch_k(token_gate_kernel<float, float>, grid, 256, 0, stream, a);
    else launch_k(token_gate_kernel<float, __nv_bfloat16>, grid, 256, 0, stream, a);
  } else {
    if (out_f32) launch_k(token_gate_kernel<__nv_bfloat16, float>, grid, 256, 0, stream, a);
    else launch_k(token_gate_kernel<__nv_bfloat16, __nv_bfloat16>, grid, 256, 0, stream, a);
  }
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}
