// What lies between the projection of an attention mixer and its attention kernel, for models described layer by layer (the per-head norm is in
// stream_ops.cu, the one of the Qwen families in elementwise.cu):
//   qk_rows_store       RMSNorm with weights over all heads of Q together, and of K together; K / V to their cache slots, Q scaled and laid out
//   rotary_table        cos and sin of the step's positions, formed once for all layers with the same rotation
//   conv_rotary_store   short causal convolution over time of Q and K (the last inputs carried per sequence), rotation of neighbouring pairs; the
//                       rotated K and, as values, the K before the rotation to their cache slots
// Rows come as bf16, f32 or K-split partial sums of the projection, added here.
#include "sm100.cuh"
#include "host_common.h"
#include "recurrent.cuh"

namespace gb {

template <typename T, int V>
__device__ __forceinline__ void load_sum(const T* p, int n_part, long stride, float* v) {
  load_cols<V>(p, v);
  for (int q = 1; q < n_part; ++q) {
    float y[V];
    load_cols<V>(p + (size_t)q * stride, y);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] += y[i];
  }
}

// ------------------------------------------------------------------------------------------ norm over all heads
struct QkRowsArgs {
  const void* qkv; int n_part; long part_stride; int ld;       // [n_part][tokens, ld]: [Q heads | K heads | V heads | ...]
  const int* slots;
  const float* q_norm; const float* k_norm;                    // [hq * dk], [hkv * dk]
  void* q_out; void* k_cache; void* v_cache; long num_slots;   // as in gb_qk_unit_store
  int hq, hkv, dk, dv, dkp, dvp;
  float eps, q_scale;
};

// V neighbouring columns of a head (dk % V == 0, dv % V == 0); NT threads, of which each keeps KEEP vectors in registers between the two passes.
template <typename TI, typename TC, int V, int NT, int KEEP>
__global__ void __launch_bounds__(NT)
qk_rows_store_kernel(const QkRowsArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][NT / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  const TI* row = (const TI*)a.qkv + (size_t)t * a.ld;
  const int nq = a.hq * a.dk / V, nk = a.hkv * a.dk / V, nv = a.hkv * a.dv / V;     // vectors: Q, then K, then V, as the columns lie
  const int slot = a.slots[t];
  const bool store = slot >= 0 && slot < a.num_slots;
  const int n = store ? nq + nk + nv : nq;
  float keep[KEEP][V], sq = 0.f, sk = 0.f;
  auto square = [&](int x, const float* v) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) s += v[j] * v[j];
    if (x < nq) sq += s; else sk += s;
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int x = tid + i * NT;
    if (x >= n) continue;
    load_sum<TI, V>(row + (size_t)x * V, a.n_part, a.part_stride, keep[i]);
    if (x < nq + nk) square(x, keep[i]);
  }
  for (int x = tid + KEEP * NT; x < min(n, nq + nk); x += NT) {
    float v[V];
    load_sum<TI, V>(row + (size_t)x * V, a.n_part, a.part_stride, v);
    square(x, v);
  }
  sq = warp_sum(sq); sk = warp_sum(sk);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float iq = a.q_scale / sqrtf(sq / (float)(a.hq * a.dk) + a.eps), ik = 1.0f / sqrtf(sk / (float)(a.hkv * a.dk) + a.eps);
  auto put = [&](int x, float* v) {
    TC* dst;
    if (x < nq) {
      const int c = x * V, h = c / a.dk;
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] *= iq * a.q_norm[c + j];
      dst = (TC*)a.q_out + ((size_t)t * a.hq + h) * a.dkp + (c - h * a.dk);
    } else if (x < nq + nk) {
      const int c = (x - nq) * V, h = c / a.dk;
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] *= ik * a.k_norm[c + j];
      dst = (TC*)a.k_cache + ((size_t)slot * a.hkv + h) * a.dkp + (c - h * a.dk);
    } else {
      const int c = (x - nq - nk) * V, h = c / a.dv;
      dst = (TC*)a.v_cache + ((size_t)slot * a.hkv + h) * a.dvp + (c - h * a.dv);
    }
    store_cols<V>(dst, v);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) { const int x = tid + i * NT; if (x < n) put(x, keep[i]); }
  for (int x = tid + KEEP * NT; x < n; x += NT) {
    float v[V];
    load_sum<TI, V>(row + (size_t)x * V, a.n_part, a.part_stride, v);
    put(x, v);
  }
  // padding of the heads
  if (a.dkp > a.dk) {
    const int pad = a.dkp - a.dk;
    for (int x = tid; x < (a.hq + (store ? a.hkv : 0)) * pad; x += NT) {
      const int h = x / pad, c = a.dk + x % pad;
      stv(h < a.hq ? (TC*)a.q_out + ((size_t)t * a.hq + h) * a.dkp + c : (TC*)a.k_cache + ((size_t)slot * a.hkv + h - a.hq) * a.dkp + c, 0.f);
    }
  }
  if (store && a.dvp > a.dv) {
    const int pad = a.dvp - a.dv;
    for (int x = tid; x < a.hkv * pad; x += NT) stv((TC*)a.v_cache + ((size_t)slot * a.hkv + x / pad) * a.dvp + a.dv + x % pad, 0.f);
  }
}

template <typename TI, typename TC>
static int qk_rows_launch(const QkRowsArgs& a, int tokens, cudaStream_t stream) {
  const bool vec = a.dk % 4 == 0 && a.dv % 4 == 0 && a.dkp % 4 == 0 && a.dvp % 4 == 0 && a.ld % 4 == 0 && a.part_stride % 4 == 0 && (uintptr_t)a.qkv % (4 * sizeof(TI)) == 0;
  // few tokens: more threads per token; many: more loads in flight per thread
  if (vec && tokens <= 64) launch_k(qk_rows_store_kernel<TI, TC, 4, 512, 4>, (unsigned)tokens, 512, 0, stream, a);
  else if (vec) launch_k(qk_rows_store_kernel<TI, TC, 4, 256, 8>, (unsigned)tokens, 256, 0, stream, a);
  else launch_k(qk_rows_store_kernel<TI, TC, 1, 256, 8>, (unsigned)tokens, 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// ------------------------------------------------------------------------------------------ rotation
__global__ void __launch_bounds__(256)
rotary_table_kernel(const int* __restrict__ positions, const double* __restrict__ freq, float mag, float2* __restrict__ out, long n, int pairs) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const long t = i / pairs;
  const double turn = 6.283185307179586476925286766559, inv_turn = 0.15915494309189533576888376337251;
  double a = (double)positions[t] * freq[i - t * pairs];
  a = fma(-turn, rint(a * inv_turn), a);                       // reduced in 64-bit floats
  float c, s;
  sincosf((float)a, &s, &c);
  out[i] = make_float2(c * mag, s * mag);
}

// ------------------------------------------------------------------------------------------ convolution, rotation, store
struct ConvRotaryArgs {
  const void* x; int n_part; long part_stride; int ld;         // [n_part][tokens, ld]: [Q heads | K heads]
  const float2* table; int dims;                               // [tokens, dims / 2]
  const int* slots;
  const float* w; int taps;                                    // [channels, taps]
  float* state; int n_slots;                                   // [slots, taps - 1, channels], oldest row first
  const int* cu_q; const int* seq_slots;
  void* q_out; void* k_cache; void* v_cache; long num_slots;
  int hq, hkv, d, dkp, dvp;
  float q_scale;
};

constexpr int kCrTile = 32, kCrTaps = 16;                      // tokens per CTA (at least the longest history); most taps

// A thread owns V neighbouring columns of one (padded) head: whole pairs of the rotation.  ODD: V = 2, any alignment and head size (the last column of an odd one is alone).
// Only a sequence's first tile reads the old state (a tile is longer than the history), and the same threads write the new one.
template <typename TI, typename TC, int V, bool ODD, int MT>   // taps <= MT
__global__ void __launch_bounds__(128)
conv_rotary_kernel(const ConvRotaryArgs a) {
  pdl_wait();
  pdl_trigger();
  const int s = blockIdx.z, t0 = a.cu_q[s], t1 = a.cu_q[s + 1];
  const int tb = t0 + blockIdx.y * kCrTile, te = min(t1, tb + kCrTile);
  const int st_slot = a.seq_slots[s];
  const int per = (a.dkp + V - 1) / V, item = blockIdx.x * 128 + threadIdx.x;
  const int h = item / per, c = (item - h * per) * V;          // head (queries, then keys), column in it
  if (h >= a.hq + a.hkv || tb >= t1 || st_slot < 0 || st_slot >= a.n_slots) return;
  const bool is_q = h < a.hq;
  const int n = min(V, a.d - c);                               // live columns (0: padding)
  const int channels = (a.hq + a.hkv) * a.d, ch = h * a.d + c, nh = a.taps - 1;
  const int n_pad = min(V, a.dkp - c);
  float* st = a.state + (size_t)st_slot * nh * channels + ch;
  auto row = [&](const auto* p, float* v) {
    if constexpr (ODD) { v[0] = ldv(p); v[1] = n > 1 ? ldv(p + 1) : 0.f; }
    else load_cols<V>(p, v);
  };
  auto input = [&](int t, float* v) {
    const TI* p = (const TI*)a.x + (size_t)t * a.ld + ch;
    row(p, v);
    for (int q = 1; q < a.n_part; ++q) {
      float y[V];
      row(p + (size_t)q * a.part_stride, y);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += y[i];
    }
  };
  float w[MT][V], win[MT][V];                                  // win[i]: the input nh - i tokens in front of the current one
#pragma unroll
  for (int k = 0; k < MT; ++k)
#pragma unroll
    for (int i = 0; i < V; ++i) { w[k][i] = k < a.taps && i < n ? a.w[(size_t)(ch + i) * a.taps + k] : 0.f; win[k][i] = 0.f; }
  if (n > 0) {
#pragma unroll
    for (int k = 0; k < MT - 1; ++k)
      if (k < nh) {
        const int t = tb - nh + k;
        if (t >= t0) input(t, win[k]);
        else row(st + (size_t)(t - t0 + nh) * channels, win[k]);
      }
    if (blockIdx.y == 0) {                                     // the history behind the sequence's last token
      float keep[MT][V];
#pragma unroll
      for (int k = 0; k < MT - 1; ++k)
        if (k < nh) {
          const int t = t1 - nh + k;
          if (t >= t0) input(t, keep[k]);
          else row(st + (size_t)(t - t0 + nh) * channels, keep[k]);
        }
#pragma unroll
      for (int k = 0; k < MT - 1; ++k)
        if (k < nh) {
          float* p = st + (size_t)k * channels;
          if constexpr (ODD) { p[0] = keep[k][0]; if (n > 1) p[1] = keep[k][1]; }
          else store_cols<V>(p, keep[k]);
        }
    }
  }
  auto put = [&](TC* p, const float* v, int count) {           // count columns of the padded head
    if constexpr (V == 4) store_cols<4>(p, v);
    else { stv(p, v[0]); if (count > 1) stv(p + 1, v[1]); }
  };
  for (int t = tb; t < te; ++t) {
    float y[V];
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = 0.f;
    if (n > 0) {
      float cur[V];
      input(t, cur);
#pragma unroll
      for (int k = 0; k < MT; ++k) {
        if (k < nh) {
#pragma unroll
          for (int i = 0; i < V; ++i) y[i] = fmaf(w[k][i], win[k][i], y[i]);
        } else if (k == nh) {
#pragma unroll
          for (int i = 0; i < V; ++i) y[i] = fmaf(w[k][i], cur[i], y[i]);
        }
      }
#pragma unroll
      for (int k = 0; k < MT - 1; ++k)
        if (k < nh)
#pragma unroll
          for (int i = 0; i < V; ++i) win[k][i] = k + 1 < nh ? win[k + 1][i] : cur[i];
    }
    const int slot = is_q ? 0 : a.slots[t];
    if (slot < 0 || slot >= a.num_slots) continue;
    if (!is_q && c < a.dvp) put((TC*)a.v_cache + ((size_t)slot * a.hkv + h - a.hq) * a.dvp + c, y, min(V, a.dvp - c));
#pragma unroll
    for (int i = 0; i < V; i += 2)
      if (c + i < a.dims) {
        const float2 cs = a.table[(size_t)t * (a.dims >> 1) + ((c + i) >> 1)];
        const float u = y[i], v = y[i + 1];
        y[i] = u * cs.x - v * cs.y;
        y[i + 1] = v * cs.x + u * cs.y;
      }
    if (is_q) {
#pragma unroll
      for (int i = 0; i < V; ++i) y[i] *= a.q_scale;
      put((TC*)a.q_out + ((size_t)t * a.hq + h) * a.dkp + c, y, n_pad);
    } else put((TC*)a.k_cache + ((size_t)slot * a.hkv + h - a.hq) * a.dkp + c, y, n_pad);
  }
}

template <typename TI, typename TC>
static int conv_rotary_launch(const ConvRotaryArgs& a, int max_tokens, int n_seqs, cudaStream_t stream) {
  const int channels = (a.hq + a.hkv) * a.d;
  const bool vec = a.taps <= 4 && a.d % 4 == 0 && a.dkp % 4 == 0 && a.dvp % 4 == 0 && a.ld % 4 == 0 && a.part_stride % 4 == 0 && channels % 4 == 0 &&
                   (uintptr_t)a.x % (4 * sizeof(TI)) == 0 && ((uintptr_t)a.state & 15) == 0;
  const int v = vec ? 4 : 2, items = (a.hq + a.hkv) * ((a.dkp + v - 1) / v);
  const dim3 grid((unsigned)((items + 127) / 128), (unsigned)((max_tokens + kCrTile - 1) / kCrTile), (unsigned)n_seqs);
  if (vec) launch_k(conv_rotary_kernel<TI, TC, 4, false, 4>, grid, 128, 0, stream, a);
  else launch_k(conv_rotary_kernel<TI, TC, 2, true, kCrTaps>, grid, 128, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

// See QkRowsArgs.  in_f32: element type of qkv; cache_f32: of q_out and the caches.
GB_API int gb_qk_rows_store(const void* qkv, int in_f32, int n_part, long part_stride, int ld, const int* slots, const float* q_norm, const float* k_norm, void* q_out,
                            void* k_cache, void* v_cache, int cache_f32, long num_slots, int tokens, int hq, int hkv, int dk, int dv, int dkp, int dvp, float eps,
                            float q_scale, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (hq < 1 || hkv < 1 || hq % hkv || dk < 1 || dv < 1 || dkp < dk || dvp < dv || n_part < 1 || ld < (hq + hkv) * dk + hkv * dv) return fail("qk_rows_store: bad sizes%s");
  QkRowsArgs a;
  a.qkv = qkv; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.slots = slots; a.q_norm = q_norm; a.k_norm = k_norm; a.q_out = q_out; a.k_cache = k_cache;
  a.v_cache = v_cache; a.num_slots = num_slots; a.hq = hq; a.hkv = hkv; a.dk = dk; a.dv = dv; a.dkp = dkp; a.dvp = dvp; a.eps = eps; a.q_scale = q_scale;
  if (in_f32) return cache_f32 ? qk_rows_launch<float, float>(a, tokens, stream) : qk_rows_launch<float, __nv_bfloat16>(a, tokens, stream);
  if (cache_f32) return fail("qk_rows_store: a 32-bit cache takes 32-bit rows%s");
  return qk_rows_launch<__nv_bfloat16, __nv_bfloat16>(a, tokens, stream);
}

// out [tokens, pairs, 2] = {cos, sin} of position * freq, times mag.
GB_API int gb_rotary_table(const int* positions, const double* freq, float mag, float* out, int tokens, int pairs, cudaStream_t stream) {
  const long n = (long)tokens * pairs;
  if (n <= 0) return 0;
  launch_k(rotary_table_kernel, (unsigned)((n + 255) / 256), 256, 0, stream, positions, freq, mag, (float2*)out, n, pairs);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See ConvRotaryArgs.  max_tokens: of the longest sequence.
GB_API int gb_conv_rotary_store(const void* x, int in_f32, int n_part, long part_stride, int ld, const float* table, int dims, const int* slots, const float* w, int taps,
                                float* state, int n_slots, const int* cu_q, const int* seq_slots, void* q_out, void* k_cache, void* v_cache, int cache_f32, long num_slots,
                                int hq, int hkv, int d, int dkp, int dvp, float q_scale, int max_tokens, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0 || max_tokens <= 0) return 0;
  if (hq < 1 || hkv < 1 || hq % hkv || d < 1 || dkp < d || dvp < d || dvp > dkp || n_part < 1 || ld < (hq + hkv) * d) return fail("conv_rotary: bad sizes%s");
  if (dims < 0 || dims % 2 || dims > d) return fail("conv_rotary: a rotation over an even part of the head%s");
  if (taps < 1 || taps > kCrTaps) return fail("conv_rotary: at most 16 taps%s");
  if (n_seqs > 65535 || (max_tokens + kCrTile - 1) / kCrTile > 65535) return fail("conv_rotary: too many tokens%s");
  ConvRotaryArgs a;
  a.x = x; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.table = (const float2*)table; a.dims = dims; a.slots = slots; a.w = w; a.taps = taps; a.state = state;
  a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.q_out = q_out; a.k_cache = k_cache; a.v_cache = v_cache; a.num_slots = num_slots; a.hq = hq; a.hkv = hkv;
  a.d = d; a.dkp = dkp; a.dvp = dvp; a.q_scale = q_scale;
  if (in_f32) return cache_f32 ? conv_rotary_launch<float, float>(a, max_tokens, n_seqs, stream) : conv_rotary_launch<float, __nv_bfloat16>(a, max_tokens, n_seqs, stream);
  if (cache_f32) return fail("conv_rotary: a 32-bit cache takes 32-bit rows%s");
  return conv_rotary_launch<__nv_bfloat16, __nv_bfloat16>(a, max_tokens, n_seqs, stream);
}
