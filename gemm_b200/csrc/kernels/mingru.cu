// minGRU: s_t = (1 - z_t) s_{t-1} + z_t c_t per channel, where the gate z = sigmoid(w_z h + b_z) and the candidate c = g(w_x h + b_x), g(u) = u + 1/2 for u >= 0
// and sigmoid(u) below, read the current token only; the result row is s_t * silu(w_g h).  Both kernels read the projections, form gates and candidates,
// run the recurrence and gate the result in one pass; the state [width] is f32 and lives in a slot per sequence.
//
//   mingru_step   token by token, a thread per channel (or four): decode steps, short portions, the 32-bit format.  K-split partial sums of the
//                 projections are added at the load.
//   mingru_scan   prompts: tokens in parallel.  The recurrence is linear in the state, so a run of tokens is a pair (A, B), s -> A s + B, and runs compose:
//                 every warp forms the pair of its 8 tokens, the warps of a CTA and then the CTAs of a cluster (which split the time axis of the same
//                 channels) exchange pairs through shared memory, and each warp replays its tokens from the state in front of them.  A is a product of factors
//                 in [0, 1]; nothing is divided, so gates that close or open fully are exact.
// Projections wider than the channels, sequences of unequal lengths: one packed batch, cu_q names each sequence's tokens.
#include "sm100.cuh"
#include "host_common.h"
#include "recurrent.cuh"
#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace gb {

struct MinGruArgs {
  const void* xg; int n_part; long part_stride; int ld;        // [n_part][tokens, ld]: x in columns 0 .. n - 1, output gate in n .. 2 n - 1
  const float* z; int z_part; long z_stride; int z_ld;         // [z_part][tokens, z_ld] f32: the gate's logits
  const float* x_bias; const float* z_bias;                    // [n]
  float* state; int n_slots;                                   // [slots, n]
  const int* cu_q; const int* seq_slots;
  void* out; int ld_out;                                       // [tokens, ld_out], zero behind n
  int n;
};

__device__ __forceinline__ float2 pair(float x) { return make_float2(x, x); }

// keep = 1 - z and add = z * candidate of two channels, from the gate's logits and u.  The bound on the logit
// keeps its exponential finite; the candidate is max(u, 0) + sigmoid(min(u, 0)); one reciprocal serves both sigmoids.
__device__ __forceinline__ void gru_gate2(float2 z, float2 u, float2& keep, float2& add) {
  constexpr float kLog2e = 1.4426950408889634f;
  const float2 zs = __fmul2_rn(z, pair(kLog2e)), us = __fmul2_rn(u, pair(kLog2e));
  const float2 ez = make_float2(fast_exp2(fminf(zs.x, 115.f)), fast_exp2(fminf(zs.y, 115.f)));
  const float2 eu = make_float2(fast_exp2(fminf(us.x, 0.f)), fast_exp2(fminf(us.y, 0.f)));
  const float2 nz = __fadd2_rn(ez, pair(1.0f)), nu = __fadd2_rn(eu, pair(1.0f)), d = __fmul2_rn(nz, nu);
  const float2 r = make_float2(fast_rcp(d.x), fast_rcp(d.y));
  const float2 gate = __fmul2_rn(ez, __fmul2_rn(r, nu));
  keep = __ffma2_rn(gate, pair(-1.0f), pair(1.0f));            // exactly 1 behind a gate that is shut: a state may have to hold for very long
  const float2 cand = __ffma2_rn(eu, __fmul2_rn(r, nz), make_float2(fmaxf(u.x, 0.f), fmaxf(u.y, 0.f)));
  add = __fmul2_rn(gate, cand);
}
// One channel, with the full-precision functions (steps).
__device__ __forceinline__ void gru_gate_exact(float z, float u, float& keep, float& add) {
  const float ez = expf(-fabsf(z)), big = 1.0f / (1.0f + ez), small = ez * big;
  keep = z >= 0.f ? small : big;
  const float eu = expf(fminf(u, 0.f));
  add = (z >= 0.f ? big : small) * (u >= 0.f ? u + 0.5f : eu / (1.0f + eu));
}

template <typename TI, typename TO, int V>                     // V neighbouring channels per thread
__global__ void __launch_bounds__(128)
mingru_step_kernel(const MinGruArgs a) {
  pdl_wait();
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, s = blockIdx.y;
  const int t0 = a.cu_q[s], t1 = a.cu_q[s + 1], slot = a.seq_slots[s];
  if (c >= a.ld_out || t1 <= t0 || slot < 0 || slot >= a.n_slots) return;
  TO* out = (TO*)a.out;
  if (c >= a.n) {                                              // padding
    for (int t = t0; t < t1; ++t)
#pragma unroll
      for (int i = 0; i < V; ++i) if (c + i < a.ld_out) stv(out + (size_t)t * a.ld_out + c + i, 0.f);
    return;
  }
  float st[V], xb[V], zb[V];
  float* sp = a.state + (size_t)slot * a.n + c;
  load_cols<V>(sp, st);
  load_cols<V>(a.x_bias + c, xb);
  load_cols<V>(a.z_bias + c, zb);
  auto input = [&](const auto* p, int parts, long stride, float* v) {
    load_cols<V>(p, v);
    for (int q = 1; q < parts; ++q) {
      float y[V];
      load_cols<V>(p + (size_t)q * stride, y);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += y[i];
    }
  };
  for (int t = t0; t < t1; ++t) {
    float x[V], g[V], z[V];
    const TI* row = (const TI*)a.xg + (size_t)t * a.ld + c;
    input(row, a.n_part, a.part_stride, x);
    input(row + a.n, a.n_part, a.part_stride, g);
    input(a.z + (size_t)t * a.z_ld + c, a.z_part, a.z_stride, z);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      float keep, add;
      gru_gate_exact(z[i] + zb[i], x[i] + xb[i], keep, add);
      st[i] = fmaf(keep, st[i], add);
      x[i] = st[i] * g[i] / (1.0f + expf(-g[i]));
    }
    store_cols<V>(out + (size_t)t * a.ld_out + c, x);
  }
  store_cols<V>(sp, st);
}

// ------------------------------------------------------------------------------------------ scan
constexpr int kGruWarps = 16, kGruRun = 8;                     // tokens of a CTA's tile: 16 warps x 8
constexpr int kGruTile = kGruWarps * kGruRun, kGruCols = 64;   // a lane owns two neighbouring channels
constexpr int kGruMaxCluster = 8;

// Two CTAs share an SM: one's loads travel under the other's arithmetic.
__global__ void __launch_bounds__(kGruWarps * 32, 2)
mingru_scan_kernel(const MinGruArgs a, int cluster) {
  __shared__ float2 s_a[kGruWarps][32], s_b[kGruWarps][32];    // the warps' pairs
  __shared__ float2 s_ca[2][kGruMaxCluster][32], s_cb[2][kGruMaxCluster][32];     // the cluster's CTAs' pairs, by parity of the tile
  pdl_wait();
  pdl_trigger();
  cg::cluster_group cl = cg::this_cluster();
  const int rank = cluster > 1 ? (int)cl.block_rank() : 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = (blockIdx.x / cluster) * kGruCols + lane * 2, s = blockIdx.y;
  const int t0 = a.cu_q[s], t1 = a.cu_q[s + 1], slot = a.seq_slots[s];
  if (t1 <= t0 || slot < 0 || slot >= a.n_slots) return;       // the same for every CTA of the cluster
  const bool live = c < a.n;                                   // n is even
  float2 st = make_float2(0.f, 0.f), xb = st, zb = st;
  if (live) {
    st = *reinterpret_cast<const float2*>(a.state + (size_t)slot * a.n + c);
    xb = *reinterpret_cast<const float2*>(a.x_bias + c);
    zb = *reinterpret_cast<const float2*>(a.z_bias + c);
  }
  if (cluster > 1) cl.sync();                                  // all CTAs run, and have read the state
  const __nv_bfloat16* xg = (const __nv_bfloat16*)a.xg;
  __nv_bfloat16* out = (__nv_bfloat16*)a.out;
  const int step = kGruTile * cluster;                         // tokens per round of the cluster
  for (int base = t0, round = 0; base < t1; base += step, ++round) {
    float2 keep[kGruRun], add[kGruRun];
    uint32_t g[kGruRun];
    float2 pa = pair(1.f), pb = pair(0.f);
    const int first = base + rank * kGruTile + warp * kGruRun;
    const int n_tok = live ? max(0, min(kGruRun, t1 - first)) : 0;
    const float* zp = a.z + (size_t)first * a.z_ld + c;
    const __nv_bfloat16* xp = xg + (size_t)first * a.ld + c;
    // all loads in flight at once; keep holds the logits and add holds x for now
    auto fetch = [&](int i) {
      keep[i] = *reinterpret_cast<const float2*>(zp + (size_t)i * a.z_ld);
      add[i].x = __uint_as_float(*reinterpret_cast<const uint32_t*>(xp + (size_t)i * a.ld));
      g[i] = *reinterpret_cast<const uint32_t*>(xp + (size_t)i * a.ld + a.n);
    };
    auto form = [&](int i) {
      const uint32_t u = __float_as_uint(add[i].x);
      gru_gate2(__fadd2_rn(keep[i], zb), __fadd2_rn(make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u)), xb), keep[i], add[i]);
      pa = __fmul2_rn(pa, keep[i]);
      pb = __ffma2_rn(keep[i], pb, add[i]);
    };
    if (n_tok == kGruRun) {
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) fetch(i);
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) form(i);
    } else {
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) { keep[i] = pair(1.f); add[i] = pair(0.f); g[i] = 0; }       // no token: the state stays
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) if (i < n_tok) fetch(i);
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) if (i < n_tok) form(i);
    }
    s_a[warp][lane] = pa; s_b[warp][lane] = pb;
    __syncthreads();
    // the state in front of this CTA, and behind the whole round
    float2 cur = st, end;
    if (cluster > 1) {
      if (warp < cluster) {                                    // warp w hands the CTA's pair to CTA w of the cluster
        float2 ta = pair(1.f), tb = pair(0.f);
#pragma unroll
        for (int w = 0; w < kGruWarps; ++w) {
          const float2 wa = s_a[w][lane];
          ta = __fmul2_rn(ta, wa);
          tb = __ffma2_rn(wa, tb, s_b[w][lane]);
        }
        *cl.map_shared_rank(&s_ca[round & 1][rank][lane], warp) = ta;
        *cl.map_shared_rank(&s_cb[round & 1][rank][lane], warp) = tb;
      }
      cl.sync();
      end = st;
      for (int r = 0; r < cluster; ++r) {
        if (r == rank) cur = end;
        end = __ffma2_rn(s_ca[round & 1][r][lane], end, s_cb[round & 1][r][lane]);
      }
    }
    float2 mine = cur;                                         // in front of this warp
    if (cluster > 1) {
      for (int w = 0; w < warp; ++w) mine = __ffma2_rn(s_a[w][lane], mine, s_b[w][lane]);
    } else {
      end = cur;
#pragma unroll
      for (int w = 0; w < kGruWarps; ++w) {
        if (w == warp) mine = end;
        end = __ffma2_rn(s_a[w][lane], end, s_b[w][lane]);
      }
    }
    st = end;
    __nv_bfloat16* op = out + (size_t)first * a.ld_out + c;
    auto emit = [&](int i) {
      mine = __ffma2_rn(keep[i], mine, add[i]);
      const float2 y = make_float2(__uint_as_float(g[i] << 16), __uint_as_float(g[i] & 0xffff0000u)), e = __fmul2_rn(y, pair(-1.4426950408889634f));
      const float2 d = __fadd2_rn(make_float2(fast_exp2(fminf(e.x, 115.f)), fast_exp2(fminf(e.y, 115.f))), pair(1.0f));
      const float2 o = __fmul2_rn(__fmul2_rn(mine, y), make_float2(fast_rcp(d.x), fast_rcp(d.y)));
      *reinterpret_cast<uint32_t*>(op + (size_t)i * a.ld_out) = pack_bf16x2(o.x, o.y);
    };
    if (n_tok == kGruRun) {
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) emit(i);
    } else {
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) {
        if (i < n_tok) emit(i);
        else if (!live && c < a.ld_out && first + i < t1) *reinterpret_cast<uint32_t*>(op + (size_t)i * a.ld_out) = 0u;     // padding
      }
    }
    __syncthreads();                                           // s_a, s_b are read
  }
  // every warp ends with the state behind the last token (rounds cover all CTAs' tokens)
  if (live && rank == 0 && warp == 0) *reinterpret_cast<float2*>(a.state + (size_t)slot * a.n + c) = st;
}

}  // namespace gb

using namespace gb;

// See MinGruArgs.  in_f32 / out_f32: element types of xg and out.  parallel: long sequences may take the scan.
GB_API int gb_mingru(const void* xg, int in_f32, int n_part, long part_stride, int ld, const float* z, int z_part, long z_stride, int z_ld, const float* x_bias,
                     const float* z_bias, float* state, int n_slots, const int* cu_q, const int* seq_slots, void* out, int out_f32, int ld_out, int n, int max_tokens,
                     int n_seqs, int parallel, cudaStream_t stream) {
  if (n_seqs <= 0 || max_tokens <= 0) return 0;
  if (n < 1 || ld < 2 * n || z_ld < n || ld_out < n || n_part < 1 || z_part < 1) return fail("mingru: bad sizes%s");
  if (!in_f32 && out_f32) return fail("mingru: 32-bit results take 32-bit rows%s");
  MinGruArgs a;
  a.xg = xg; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.z = z; a.z_part = z_part; a.z_stride = z_stride; a.z_ld = z_ld; a.x_bias = x_bias;
  a.z_bias = z_bias; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out; a.n = n;
  const auto al = [](const void* p, size_t b) { return (uintptr_t)p % b == 0; };
  if (parallel && !in_f32 && !out_f32 && n_part == 1 && z_part == 1 && n % 2 == 0 && ld % 2 == 0 && z_ld % 2 == 0 && ld_out % 2 == 0 && al(xg, 4) && al(z, 8) &&
      al(x_bias, 8) && al(z_bias, 8) && al(state, 8) && al(out, 4)) {
    const int blocks = (ld_out + kGruCols - 1) / kGruCols;
    int cluster = 1;                                           // CTAs along the time axis: while they fit the GPU at once and a round is shorter than the longest sequence
    while (cluster < kGruMaxCluster && (long)blocks * n_seqs * cluster * 2 <= 2L * sm_count() && cluster * kGruTile < max_tokens) cluster *= 2;
    const dim3 grid((unsigned)(blocks * cluster), (unsigned)n_seqs);
    GB_CUDA_OK(launch_k_cluster(mingru_scan_kernel, grid, kGruWarps * 32, 0, stream, (unsigned)cluster, a, cluster));
    return 0;
  }
  const bool vec = n % 4 == 0 && ld % 4 == 0 && part_stride % 4 == 0 && z_ld % 4 == 0 && z_stride % 4 == 0 && ld_out % 4 == 0 && al(xg, in_f32 ? 16 : 8) && al(z, 16) &&
                   al(x_bias, 16) && al(z_bias, 16) && al(state, 16) && al(out, out_f32 ? 16 : 8);
#define GB_GRU(TI, TO)                                                                                                                                          \
  do {                                                                                                                                                          \
    if (vec) launch_k(mingru_step_kernel<TI, TO, 4>, dim3((unsigned)((ld_out + 511) / 512), (unsigned)n_seqs), 128, 0, stream, a);                               \
    else launch_k(mingru_step_kernel<TI, TO, 1>, dim3((unsigned)((ld_out + 127) / 128), (unsigned)n_seqs), 128, 0, stream, a);                                   \
  } while (0)
  if (in_f32 && out_f32) GB_GRU(float, float);
  else if (in_f32) GB_GRU(float, __nv_bfloat16);
  else GB_GRU(__nv_bfloat16, __nv_bfloat16);
#undef GB_GRU
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}
