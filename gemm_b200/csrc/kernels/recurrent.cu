// Recurrent mixers with input-dependent decay, token by token (decode steps, short portions, the 32-bit format):
//   causal_conv   depthwise causal convolution with bias + SiLU over packed tokens, the last taps - 1 inputs carried per sequence
//   ssd           Mamba-2:  S_t = exp(a dt_t) S_{t-1} + dt_t B_t x_t^T,  y_t = S_t^T C_t + D x_t, one scalar decay per head and token
//   gla           HGRN2:    S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,  o_t = S_t^T q_t, one decay per key channel
//   rwkv          o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,  S_t = diag(w_t) S_{t-1} + k_t v_t^T, w = exp(-exp(z)) per key channel
//   token_shift   mixes of a token's row and the one in front of it, the last row carried per sequence
//   tanh_rows     tanh of a projection's result (the middle of a low-rank projection)
// The state S [dim, vdim] is f32 and lives in a slot per sequence.  The chunked forms for prompts are in lightning_chunk.cu (Mamba-2) and
// gla_chunk.cu (HGRN2, RWKV).
//
// The step kernel has the layout of lightning.cu: one CTA per (sequence, head, slice of value columns); a lane owns VEC value columns, the eight
// warps split the key rows, and a decode step is one pass over the state with all of a thread's loads in flight at once.
#include "sm100.cuh"
#include "host_common.h"
#include "recurrent.cuh"

namespace gb {

// ------------------------------------------------------------------------------------------ convolution
struct CausalConvArgs {
  const void* x; int n_part; long part_stride; int ld_x;      // [n_part][tokens, ld_x], the channels are the first columns
  const float* w; const float* b;                             // [channels, taps], [channels]
  float* state; int n_slots;                                  // [slots, taps - 1, channels], oldest row first
  const int* cu_q; const int* seq_slots;
  void* out; int ld_out;                                      // activated channels
  int channels, taps;
};

constexpr int kConvTile = 32;                                 // tokens per CTA, at least the longest history
constexpr int kMaxTaps = 16;

// V neighbouring channels per thread.  Only a sequence's first tile reads the old state (a tile is longer than the history), and the same
// threads write the new one, so nothing races.
template <typename TI, typename TO, int V, int MT>            // taps <= MT
__global__ void __launch_bounds__(128)
causal_conv_kernel(const CausalConvArgs a) {
  pdl_wait();
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, s = blockIdx.z;
  const int t0 = a.cu_q[s], t1 = a.cu_q[s + 1];
  const int tb = t0 + blockIdx.y * kConvTile, te = min(t1, tb + kConvTile);
  const int slot = a.seq_slots[s];
  if (c >= a.channels || tb >= t1 || slot < 0 || slot >= a.n_slots) return;
  const int nh = a.taps - 1;
  float* st = a.state + (size_t)slot * nh * a.channels + c;
  float w[MT][V], b[V], win[MT][V];                           // win[i]: the input nh - i tokens in front of the current one
  auto input = [&](int t, float* v) {
    const TI* p = (const TI*)a.x + (size_t)t * a.ld_x + c;
    load_cols<V>(p, v);
    for (int q = 1; q < a.n_part; ++q) {
      float y[V];
      load_cols<V>(p + (size_t)q * a.part_stride, y);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += y[i];
    }
  };
#pragma unroll
  for (int i = 0; i < V; ++i) b[i] = a.b[c + i];
#pragma unroll
  for (int k = 0; k < MT; ++k)
#pragma unroll
    for (int i = 0; i < V; ++i) { w[k][i] = k < a.taps ? a.w[(size_t)(c + i) * a.taps + k] : 0.f; win[k][i] = 0.f; }
#pragma unroll
  for (int k = 0; k < MT - 1; ++k)
    if (k < nh) {
      const int t = tb - nh + k;
      if (t >= t0) input(t, win[k]);
      else load_cols<V>(st + (size_t)(t - t0 + nh) * a.channels, win[k]);
    }
  if (blockIdx.y == 0) {                                      // the history behind the sequence's last token
    float keep[MT][V];
#pragma unroll
    for (int k = 0; k < MT - 1; ++k)
      if (k < nh) {
        const int t = t1 - nh + k;
        if (t >= t0) input(t, keep[k]);
        else load_cols<V>(st + (size_t)(t - t0 + nh) * a.channels, keep[k]);
      }
#pragma unroll
    for (int k = 0; k < MT - 1; ++k)
      if (k < nh) store_cols<V>(st + (size_t)k * a.channels, keep[k]);
  }
  for (int t = tb; t < te; ++t) {
    float cur[V], y[V];
    input(t, cur);
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = b[i];
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
    for (int i = 0; i < V; ++i) y[i] = y[i] / (1.0f + expf(-y[i]));
    store_cols<V>((TO*)a.out + (size_t)t * a.ld_out + c, y);
#pragma unroll
    for (int k = 0; k < MT - 1; ++k)
      if (k < nh)
#pragma unroll
        for (int i = 0; i < V; ++i) win[k][i] = k + 1 < nh ? win[k + 1][i] : cur[i];
  }
}

// ------------------------------------------------------------------------------------------ recurrence
struct RecurrentArgs {
  // ssd: activated channels of the convolution [tokens, ld]: [x heads x vdim | B groups x dim | C groups x dim] (one slab)
  // gla: input projection [n_part][tokens, ld]: q heads x dim from column 0, v heads x vdim behind it
  // rwkv: r, k, v as three blocks of rows [tokens, ld], `part_stride` elements apart (one slab)
  const void* in; int n_part; long part_stride; int ld;
  // the gate's pre-activations, [g_part][tokens, g_ld] f32: dt (heads columns) or f (heads x dim columns)
  const float* gate; int g_part; long g_stride; int g_ld;
  const float* gate_bias;       // ssd: dt_bias [heads]; gla, rwkv: [heads * dim]
  const float* par;             // ssd: a [heads], negative; gla: lower bound [heads * dim]; rwkv: u [heads * dim]
  const float* d_skip;          // ssd: [heads]
  float* state; int n_slots;    // [slots, heads, dim, vdim]
  const int* cu_q; const int* seq_slots;
  float* out; int ld_out;       // [tokens, heads * vdim]
  int heads, groups, dim, vdim;
  int q_raw;                    // gla: != 0: q has no SiLU yet
  // kRwkvLow: gate holds the middle of a low-rank projection, [g_part][tokens, g_ld] with `rank` columns, before its tanh; its second matrix
  int rank; const __nv_bfloat16* w2;    // is w2 [heads * dim, rank]
};

constexpr int kMaxRank = 256;

template <typename TI>
__device__ __forceinline__ float in_col(const RecurrentArgs& a, size_t tok, long col) {
  const TI* p = (const TI*)a.in + tok * a.ld + col;
  float s = ldv(p);
  for (int i = 1; i < a.n_part; ++i) s += ldv(p + (size_t)i * a.part_stride);
  return s;
}
__device__ __forceinline__ float gate_col(const RecurrentArgs& a, size_t tok, int col) {
  const float* p = a.gate + tok * a.g_ld + col;
  float s = *p;
  for (int i = 1; i < a.g_part; ++i) s += p[(size_t)i * a.g_stride];
  return s;
}

enum RecurrentKind { kSsd = 0, kGla = 1, kRwkv = 2, kRwkvLow = 3 };       // kRwkvLow: forms the decays from the middle of their low-rank projection

template <typename TI, int KIND, int VEC, int R>   // dim <= 8 * R
__global__ void __launch_bounds__(256)
recurrent_step_kernel(const RecurrentArgs a) {
  constexpr bool GLA = KIND == kGla, RWKV = KIND >= kRwkv, LOW = KIND == kRwkvLow, CHAN = GLA || RWKV;       // CHAN: a decay per key channel
  __shared__ float sq[8 * R], sk[8 * R], sf[CHAN ? 8 * R : 1], su[RWKV ? 8 * R : 1];
  __shared__ float s_low[LOW ? kMaxRank : 1];
  __shared__ float red[8][32 * VEC];
  __shared__ float s_dec;
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
    if (live && d < a.dim) load_cols<VEC>(st + (size_t)d * a.vdim, S[r]);
  }
  const int nv = a.heads * a.vdim, grp = h / (a.heads / a.groups);
  const long q_col = CHAN ? h * a.dim : nv + (a.groups + grp) * a.dim, k_col = RWKV ? a.part_stride + h * a.dim : nv + grp * a.dim;
  const long v_col = (RWKV ? 2 * a.part_stride : GLA ? a.heads * a.dim : 0) + h * a.vdim + e0;
  const float a_h = CHAN ? 0.f : a.par[h], bias_h = CHAN ? 0.f : a.gate_bias[h], skip = CHAN ? 0.f : a.d_skip[h];
  for (int t = t0; t < t1; ++t) {
    float dt = 0.f;
    if constexpr (!CHAN) {
      dt = softplus_exact(gate_col(a, t, h) + bias_h);
      if (threadIdx.x == 0) s_dec = expf(a_h * dt);
    }
    if constexpr (LOW) {
      for (int i = threadIdx.x; i < a.rank; i += 256) s_low[i] = tanhf(gate_col(a, t, i));
      __syncthreads();
      for (int c0 = 0; c0 < a.dim; c0 += 128) {             // two threads per channel
        const int c = c0 + (threadIdx.x >> 1);
        float z = 0.f;
        if (c < a.dim) {
          const __nv_bfloat16* w = a.w2 + (size_t)(h * a.dim + c) * a.rank;
          if (a.rank % 16 == 0) {
            for (int x = (threadIdx.x & 1) * 8; x < a.rank; x += 16) {
              const uint4 q = *reinterpret_cast<const uint4*>(w + x);
              const uint32_t u[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
              for (int y = 0; y < 4; ++y) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[y]));
                z = fmaf(f.x, s_low[x + 2 * y], z);
                z = fmaf(f.y, s_low[x + 2 * y + 1], z);
              }
            }
          } else {
            for (int x = threadIdx.x & 1; x < a.rank; x += 2) z = fmaf(__bfloat162float(w[x]), s_low[x], z);
          }
        }
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        if (c < a.dim && (threadIdx.x & 1) == 0) sf[c] = expf(-expf(z + a.gate_bias[h * a.dim + c]));
      }
    }
    for (int i = threadIdx.x; i < 2 * a.dim; i += 256) {
      const bool isk = i >= a.dim;
      const int c = isk ? i - a.dim : i;
      if constexpr (GLA) {
        if (isk) {
          const float z = gate_col(a, t, h * a.dim + c) + a.gate_bias[h * a.dim + c], low = a.par[h * a.dim + c];
          sf[c] = forget_gate(z, low, sk[c]);
        } else {
          const float q = in_col<TI>(a, t, q_col + c);
          sq[c] = a.q_raw ? q / (1.0f + expf(-q)) : q;
        }
      } else if constexpr (RWKV) {
        if (isk) {
          const float k = in_col<TI>(a, t, k_col + c);
          sk[c] = k;
          su[c] = k * a.par[h * a.dim + c];
          if constexpr (!LOW) sf[c] = expf(-expf(gate_col(a, t, h * a.dim + c) + a.gate_bias[h * a.dim + c]));
        } else sq[c] = in_col<TI>(a, t, q_col + c);
      } else {
        if (isk) sk[c] = in_col<TI>(a, t, k_col + c) * dt; else sq[c] = in_col<TI>(a, t, q_col + c);
      }
    }
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = live ? in_col<TI>(a, t, v_col + j) : 0.f;
    __syncthreads();
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    const float dec = CHAN ? 0.f : s_dec;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = warp + 8 * r;
      if (d < a.dim) {
        const float kd = sk[d], qd = sq[d], f = CHAN ? sf[CHAN ? d : 0] : dec;
        if constexpr (RWKV) {                      // the output reads the state in front of the token
          const float ud = su[d];
#pragma unroll
          for (int j = 0; j < VEC; ++j) { o[j] = fmaf(fmaf(ud, v[j], S[r][j]), qd, o[j]); S[r][j] = fmaf(f, S[r][j], kd * v[j]); }
          continue;
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) { S[r][j] = fmaf(f, S[r][j], kd * v[j]); o[j] = fmaf(S[r][j], qd, o[j]); }
      }
    }
    if (!CHAN && warp == 0) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = fmaf(skip, v[j], o[j]);
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
    // the shared rows are rewritten only after every thread has passed the second barrier; red is read before the next token's first barrier
  }
  if (live) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = warp + 8 * r;
      if (d < a.dim) store_cols<VEC>(st + (size_t)d * a.vdim, S[r]);
    }
  }
}

template <typename TI, int KIND>
static int recurrent_step_launch(const RecurrentArgs& a, int n_seqs, cudaStream_t stream) {
  const bool vec = a.vdim % 4 == 0 && a.vdim > 32 && a.dim <= 256 && ((uintptr_t)a.state & 15) == 0;
  const int cols = vec ? 128 : 32;
  const dim3 grid((unsigned)a.heads, (unsigned)((a.vdim + cols - 1) / cols), (unsigned)n_seqs);
#define GB_RS(VECV, RV) launch_k(recurrent_step_kernel<TI, KIND, VECV, RV>, grid, 256, 0, stream, a)
  if (vec) {
    if (a.dim <= 32) GB_RS(4, 4); else if (a.dim <= 64) GB_RS(4, 8); else if (a.dim <= 128) GB_RS(4, 16); else GB_RS(4, 32);
  } else {
    if (a.dim <= 64) GB_RS(1, 8); else if (a.dim <= 256) GB_RS(1, 32); else GB_RS(1, 64);
  }
#undef GB_RS
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// ------------------------------------------------------------------------------------------ mixes with the token in front
struct TokenShiftArgs {
  const void* h; int ld;                                      // [tokens, ld], `width` columns
  const float* mu; int n;                                     // [n, width]
  float* state; int n_slots;                                  // [slots, width]: the row in front of a sequence's next token
  const int* cu_q; const int* seq_slots;
  void* out; long mix_stride; int ld_out;                     // [n][.., ld_out], zero behind `width`
  int width;
};

constexpr int kShiftTile = 8;                                 // tokens per CTA

// V neighbouring columns per thread.  Only a sequence's first tile reads the state, and the same threads write it.
template <typename T, int V>
__global__ void __launch_bounds__(128)
token_shift_kernel(const TokenShiftArgs a) {
  pdl_wait();
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, s = blockIdx.z;
  const int t0 = a.cu_q[s], t1 = a.cu_q[s + 1];
  const int tb = t0 + blockIdx.y * kShiftTile, te = min(t1, tb + kShiftTile);
  const int slot = a.seq_slots[s];
  if (c >= a.ld_out || tb >= t1 || slot < 0 || slot >= a.n_slots) return;
  const bool live = c < a.width;                              // V > 1: width % V == 0
  const T* h = (const T*)a.h + c;
  float prev[V], cur[V];
#pragma unroll
  for (int i = 0; i < V; ++i) prev[i] = cur[i] = 0.f;
  if (live) {
    float* st = a.state + (size_t)slot * a.width + c;
    if (blockIdx.y == 0) {
      float last[V];
      load_cols<V>(st, prev);
      load_cols<V>(h + (size_t)(t1 - 1) * a.ld, last);
      store_cols<V>(st, last);
    } else load_cols<V>(h + (size_t)(tb - 1) * a.ld, prev);
  }
  for (int t = tb; t < te; ++t) {
    if (live) load_cols<V>(h + (size_t)t * a.ld, cur);
    for (int x = 0; x < a.n; ++x) {
      float m[V];
#pragma unroll
      for (int i = 0; i < V; ++i) m[i] = 0.f;
      if (live) {
        load_cols<V>(a.mu + (size_t)x * a.width + c, m);
#pragma unroll
        for (int i = 0; i < V; ++i) m[i] = fmaf(prev[i] - cur[i], m[i], cur[i]);
      }
      store_cols<V>((T*)a.out + (size_t)x * a.mix_stride + (size_t)t * a.ld_out + c, m);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) prev[i] = cur[i];
  }
}

template <typename T>
static int token_shift_launch(const TokenShiftArgs& a, int max_tokens, int n_seqs, cudaStream_t stream) {
  const size_t es = 4 * sizeof(T);
  const bool vec = a.width % 4 == 0 && a.ld % 4 == 0 && a.ld_out % 4 == 0 && a.mix_stride % 4 == 0 && (uintptr_t)a.h % es == 0 && (uintptr_t)a.out % es == 0 &&
                   ((uintptr_t)a.state & 15) == 0 && ((uintptr_t)a.mu & 15) == 0;
  const int cols = vec ? 512 : 128;
  const dim3 grid((unsigned)((a.ld_out + cols - 1) / cols), (unsigned)((max_tokens + kShiftTile - 1) / kShiftTile), (unsigned)n_seqs);
  if (vec) launch_k(token_shift_kernel<T, 4>, grid, 128, 0, stream, a);
  else launch_k(token_shift_kernel<T, 1>, grid, 128, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const TI* __restrict__ z, int n_part, long part_stride, int ld, TO* __restrict__ out, int ld_out, long total, int n) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const long r = i / ld_out;
  const int c = (int)(i - r * ld_out);
  float v = 0.f;
  if (c < n) {
    for (int q = 0; q < n_part; ++q) v += ldv(z + (size_t)q * part_stride + (size_t)r * ld + c);
    v = tanhf(v);
  }
  stv(out + i, v);
}

template <typename TI, typename TO>
static int causal_conv_launch(const CausalConvArgs& a, int max_tokens, int n_seqs, cudaStream_t stream) {
  const bool vec = a.taps <= 4 && a.channels % 4 == 0 && a.ld_x % 4 == 0 && a.part_stride % 4 == 0 && a.ld_out % 4 == 0 && (uintptr_t)a.x % (4 * sizeof(TI)) == 0 &&
                   (uintptr_t)a.out % (4 * sizeof(TO)) == 0 && ((uintptr_t)a.state & 15) == 0;
  const int cols = vec ? 512 : 128;
  const dim3 grid((unsigned)((a.channels + cols - 1) / cols), (unsigned)((max_tokens + kConvTile - 1) / kConvTile), (unsigned)n_seqs);
  if (vec) launch_k(causal_conv_kernel<TI, TO, 4, 4>, grid, 128, 0, stream, a);
  else if (a.taps <= 4) launch_k(causal_conv_kernel<TI, TO, 1, 4>, grid, 128, 0, stream, a);
  else launch_k(causal_conv_kernel<TI, TO, 1, kMaxTaps>, grid, 128, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

// x: channels in the first columns of [n_part][tokens, ld_x]; out [tokens, ld_out] = SiLU(conv + bias); max_tokens: of the longest sequence.
GB_API int gb_causal_conv(const void* x, int x_f32, int n_part, long part_stride, int ld_x, const float* w, const float* b, float* state, int n_slots,
                          const int* cu_q, const int* seq_slots, void* out, int out_f32, int ld_out, int channels, int taps, int max_tokens, int n_seqs,
                          cudaStream_t stream) {
  if (n_seqs <= 0 || max_tokens <= 0) return 0;
  if (channels < 1 || taps < 1 || taps > kMaxTaps || n_part < 1 || ld_x < channels || ld_out < channels) return fail("causal_conv: bad sizes (at most 16 taps)%s");
  if (n_seqs > 65535 || (max_tokens + kConvTile - 1) / kConvTile > 65535) return fail("causal_conv: too many tokens%s");
  CausalConvArgs a;
  a.x = x; a.n_part = n_part; a.part_stride = part_stride; a.ld_x = ld_x; a.w = w; a.b = b; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q;
  a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out; a.channels = channels; a.taps = taps;
  if (x_f32) return out_f32 ? causal_conv_launch<float, float>(a, max_tokens, n_seqs, stream) : causal_conv_launch<float, __nv_bfloat16>(a, max_tokens, n_seqs, stream);
  if (out_f32) return fail("causal_conv: 32-bit results take 32-bit rows%s");
  return causal_conv_launch<__nv_bfloat16, __nv_bfloat16>(a, max_tokens, n_seqs, stream);
}

// See RecurrentArgs.  gla != 0: HGRN2 (groups and d_skip are not used); else Mamba-2.
GB_API int gb_recurrent_step(int gla, const void* in, int in_f32, int n_part, long part_stride, int ld, const float* gate, int g_part, long g_stride, int g_ld,
                             const float* gate_bias, const float* par, const float* d_skip, float* state, int n_slots, const int* cu_q, const int* seq_slots,
                             float* out, int ld_out, int heads, int groups, int dim, int vdim, int q_raw, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || n_part < 1 || g_part < 1 || groups < 1 || heads % groups || ld_out < heads * vdim) return fail("recurrent: bad sizes%s");
  if (gla ? (ld < heads * (dim + vdim) || g_ld < heads * dim) : (ld < heads * vdim + 2 * groups * dim || g_ld < heads || n_part != 1 || d_skip == nullptr))
    return fail("recurrent: rows are too short%s");
  if (dim > 512) return fail("recurrent: a key dimension of at most 512%s");
  if (n_seqs > 65535) return fail("recurrent: too many sequences%s");
  RecurrentArgs a;
  a.in = in; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.gate = gate; a.g_part = g_part; a.g_stride = g_stride; a.g_ld = g_ld;
  a.gate_bias = gate_bias; a.par = par; a.d_skip = d_skip; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out;
  a.ld_out = ld_out; a.heads = heads; a.groups = groups; a.dim = dim; a.vdim = vdim; a.q_raw = q_raw; a.rank = 0; a.w2 = nullptr;
  if (gla) return in_f32 ? recurrent_step_launch<float, kGla>(a, n_seqs, stream) : recurrent_step_launch<__nv_bfloat16, kGla>(a, n_seqs, stream);
  return in_f32 ? recurrent_step_launch<float, kSsd>(a, n_seqs, stream) : recurrent_step_launch<__nv_bfloat16, kSsd>(a, n_seqs, stream);
}

// r, k, v: three blocks [tokens, ld] of one element type, `block_stride` elements apart; z [z_part][tokens, z_ld]: w = exp(-exp(z + w0)), or with rank > 0 (at most
// 256) w = exp(-exp(w2 tanh(z) + w0)), w2 bf16 [heads * dim, rank]; u, w0 [heads * dim].  See RecurrentArgs for the rest.
GB_API int gb_rwkv_step(const void* rkv, int in_f32, long block_stride, int ld, const float* z, int z_part, long z_stride, int z_ld, const void* w2, int rank,
                        const float* w0, const float* u, float* state, int n_slots, const int* cu_q, const int* seq_slots, float* out, int ld_out, int heads, int dim, int vdim, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || z_part < 1 || ld_out < heads * vdim || ld < heads * dim || ld < heads * vdim || z_ld < (rank > 0 ? rank : heads * dim)) return fail("rwkv: bad sizes%s");
  if (rank < 0 || rank > kMaxRank || (rank > 0 && w2 == nullptr) || (rank % 16 == 0 && ((uintptr_t)w2 & 15))) return fail("rwkv: bad low-rank projection%s");
  if (dim > 512) return fail("rwkv: a key dimension of at most 512%s");
  if (n_seqs > 65535) return fail("rwkv: too many sequences%s");
  RecurrentArgs a;
  memset(&a, 0, sizeof(a));
  a.in = rkv; a.n_part = 1; a.part_stride = block_stride; a.ld = ld; a.gate = z; a.g_part = z_part; a.g_stride = z_stride; a.g_ld = z_ld; a.gate_bias = w0; a.par = u;
  a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out; a.heads = heads; a.groups = 1; a.dim = dim; a.vdim = vdim; a.rank = rank; a.w2 = (const __nv_bfloat16*)w2;
  if (rank > 0) return in_f32 ? recurrent_step_launch<float, kRwkvLow>(a, n_seqs, stream) : recurrent_step_launch<__nv_bfloat16, kRwkvLow>(a, n_seqs, stream);
  return in_f32 ? recurrent_step_launch<float, kRwkv>(a, n_seqs, stream) : recurrent_step_launch<__nv_bfloat16, kRwkv>(a, n_seqs, stream);
}

// See TokenShiftArgs.  max_tokens: of the longest sequence.
GB_API int gb_token_shift(const void* h, int h_f32, int ld, int width, const float* mu, int n, float* state, int n_slots, const int* cu_q, const int* seq_slots, void* out,
                          long mix_stride, int ld_out, int max_tokens, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0 || max_tokens <= 0) return 0;
  if (width < 1 || n < 1 || ld < width || ld_out < width) return fail("token_shift: bad sizes%s");
  if (n_seqs > 65535 || (max_tokens + kShiftTile - 1) / kShiftTile > 65535) return fail("token_shift: too many tokens%s");
  TokenShiftArgs a;
  a.h = h; a.ld = ld; a.mu = mu; a.n = n; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.mix_stride = mix_stride;
  a.ld_out = ld_out; a.width = width;
  return h_f32 ? token_shift_launch<float>(a, max_tokens, n_seqs, stream) : token_shift_launch<__nv_bfloat16>(a, max_tokens, n_seqs, stream);
}

// out [rows, ld_out] = tanh of the first n columns of z [n_part][rows, ld], zero behind.
GB_API int gb_tanh_rows(const void* z, int z_f32, int n_part, long part_stride, int ld, void* out, int out_f32, int ld_out, int rows, int n, cudaStream_t stream) {
  const long total = (long)rows * ld_out;
  if (total <= 0) return 0;
  if (n < 1 || n_part < 1 || ld < n || ld_out < n) return fail("tanh_rows: bad sizes%s");
  const unsigned grid = (unsigned)((total + 255) / 256);
  if (z_f32) {
    if (out_f32) launch_k(tanh_rows_kernel<float, float>, grid, 256, 0, stream, (const float*)z, n_part, part_stride, ld, (float*)out, ld_out, total, n);
    else launch_k(tanh_rows_kernel<float, __nv_bfloat16>, grid, 256, 0, stream, (const float*)z, n_part, part_stride, ld, (__nv_bfloat16*)out, ld_out, total, n);
  } else {
    if (out_f32) return fail("tanh_rows: 32-bit results take 32-bit rows%s");
    launch_k(tanh_rows_kernel<__nv_bfloat16, __nv_bfloat16>, grid, 256, 0, stream, (const __nv_bfloat16*)z, n_part, part_stride, ld, (__nv_bfloat16*)out, ld_out, total, n);
  }
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}
