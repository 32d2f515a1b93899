// Paged attention for any head sizes and element types, one warp per (token, query head): the path of the "f32" weight format and
// of head sizes the tcgen05 kernels (flash_attn.cu) are not built for.  Keys and values may differ in size.  A query at position i
// sees j <= i with i - j < window (0 = no limit) or j < keep_first; an optional table adds bias[h][min(i - j, n_bias - 1)] to the
// score, or r1[h] ln(1 + r2[h] (i - j)) is taken off it, a cap c > 0 makes it c tanh(score / c) (q then arrives multiplied by scale / c), and a learned score per head (a sink) may join the sum of the weights.  Q arrives multiplied by scale * log2(e), bias table and sinks by log2(e);
// scores, weights and sums are f32.  Latent attention runs here as one key / value head whose values are the first columns of the keys.
#include "sm100.cuh"
#include "host_common.h"

namespace gb {

struct AttnAnyArgs {
  const void* q; const void* k; const void* v; void* out;      // q [T, hq, dk], caches [slots, hkv, dk] / [slots, hkv, dv], out [T, hq, dv],
  long q_ts, q_hs, k_ss, k_hs, v_ss, v_hs, o_ts, o_hs;         // their strides by token / slot and head, in elements
  const int* tok_seq; const int* tok_kv;                       // sequence (row of the block table) and key count of each token; null: from cu_q, kv_len
  const float* sink;                                           // [hq]; null = none
  const int* cu_q; const int* kv_len; const int* block_table; int max_pages, page_size, n_seqs;
  long num_slots;
  int tokens, hq, hkv, dk, dv, window, keep_first;
  const float* bias; int n_bias, ld_bias;
  float cap;                                                   // softcap * log2(e); 0 = none
  const float* log_bias;                                       // [2][hq]: r1, r2; null = none
};

__device__ __forceinline__ float lda(const float* p) { return *p; }
__device__ __forceinline__ float lda(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void sta(float* p, float v) { *p = v; }
__device__ __forceinline__ void sta(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <typename T, int NV>                       // dv <= 32 * NV
__global__ void __launch_bounds__(128)
attn_any_kernel(const AttnAnyArgs a) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float s_q[];                    // [4 warps][dk]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long item = (long)blockIdx.x * 4 + warp;
  if (item >= (long)a.tokens * a.hq) return;
  const int t = (int)(item / a.hq), h = (int)(item - (long)t * a.hq);
  // the sequence of this token: cu_q is short and ordered
  int seq, i;                                                  // i: position of the token
  if (a.tok_seq != nullptr) { seq = a.tok_seq[t]; i = a.tok_kv[t] - 1; }
  else {
    int lo = 0, hi = a.n_seqs;
    while (hi - lo > 1) { const int mid = (lo + hi) >> 1; if (a.cu_q[mid] <= t) lo = mid; else hi = mid; }
    seq = lo;
    i = a.kv_len[seq] - (a.cu_q[seq + 1] - t);
  }
  const int kvh = h / (a.hq / a.hkv);
  float* q = s_q + warp * a.dk;
  for (int c = lane; c < a.dk; c += 32) q[c] = lda((const T*)a.q + (size_t)t * a.q_ts + (size_t)h * a.q_hs + c);
  __syncwarp();
  const int first = a.window > 0 ? max(0, i - a.window + 1) : 0;
  const int n_keep = min(a.keep_first, first);
  const int n = n_keep + (i - first + 1);           // visible keys: [0, n_keep) and [first, i]
  const int* bt = a.block_table + (size_t)seq * a.max_pages;
  const float r1 = a.log_bias != nullptr ? a.log_bias[h] : 0.f, r2 = a.log_bias != nullptr ? a.log_bias[a.hq + h] : 0.f;
  float m = -INFINITY, l = 0.f, acc[NV];
#pragma unroll
  for (int c = 0; c < NV; ++c) acc[c] = 0.f;
  for (int b = 0; b < n; b += 32) {
    const int x = b + lane;
    const bool live = x < n;
    long slot = 0;
    float sc = -INFINITY;
    if (live) {
      const int j = x < n_keep ? x : first + (x - n_keep);
      slot = (long)bt[j / a.page_size] * a.page_size + j % a.page_size;
      if (slot < 0 || slot >= a.num_slots) slot = 0;
      const T* kr = (const T*)a.k + (size_t)slot * a.k_ss + (size_t)kvh * a.k_hs;
      float s = 0.f;
      for (int c = 0; c < a.dk; ++c) s = fmaf(q[c], lda(kr + c), s);
      if (a.cap > 0.f) s = a.cap * tanhf(s);
      if (a.bias != nullptr) s += a.bias[(size_t)h * a.ld_bias + min(i - j, a.n_bias - 1)];
      if (a.log_bias != nullptr) s = fmaf(-r1, log2f(fmaf(r2, (float)(i - j), 1.0f)), s);
      sc = s;
    }
    const float mn = fmaxf(m, warp_max(sc));
    const float alpha = exp2f(m - mn);
    const float p = live ? exp2f(sc - mn) : 0.f;
    m = mn;
    l = l * alpha + warp_sum(p);
#pragma unroll
    for (int c = 0; c < NV; ++c) acc[c] *= alpha;
    const int cnt = min(32, n - b);
    for (int y = 0; y < cnt; ++y) {
      const float py = __shfl_sync(0xffffffffu, p, y);
      const long sy = __shfl_sync(0xffffffffu, slot, y);
      const T* vr = (const T*)a.v + (size_t)sy * a.v_ss + (size_t)kvh * a.v_hs;
#pragma unroll
      for (int c = 0; c < NV; ++c) { const int e = lane + 32 * c; if (e < a.dv) acc[c] = fmaf(py, lda(vr + e), acc[c]); }
    }
  }
  if (a.sink != nullptr) {                          // counts once, has no value
    const float sk = a.sink[h], mn = fmaxf(m, sk), alpha = exp2f(m - mn);
    l = l * alpha + exp2f(sk - mn);
#pragma unroll
    for (int c = 0; c < NV; ++c) acc[c] *= alpha;
  }
  T* o = (T*)a.out + (size_t)t * a.o_ts + (size_t)h * a.o_hs;
#pragma unroll
  for (int c = 0; c < NV; ++c) { const int e = lane + 32 * c; if (e < a.dv) sta(o + e, l > 0.f ? acc[c] / l : 0.f); }
}

template <typename T>
static int attn_any_launch(const AttnAnyArgs& a, cudaStream_t stream) {
  const unsigned grid = (unsigned)(((long)a.tokens * a.hq + 3) / 4);
  const size_t smem = (size_t)4 * a.dk * sizeof(float);
  if (a.dv <= 64) launch_k(attn_any_kernel<T, 2>, grid, 128, smem, stream, a);
  else if (a.dv <= 128) launch_k(attn_any_kernel<T, 4>, grid, 128, smem, stream, a);
  else if (a.dv <= 256) launch_k(attn_any_kernel<T, 8>, grid, 128, smem, stream, a);
  else if (a.dv <= 512) launch_k(attn_any_kernel<T, 16>, grid, 128, smem, stream, a);
  else launch_k(attn_any_kernel<T, 32>, grid, 128, smem, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

GB_API int gb_attn_any(const void* q, const void* k, const void* v, void* out, int f32, const int* cu_q, const int* kv_len, const int* block_table,
                       int max_pages, int page_size, int n_seqs, long num_slots, int tokens, int hq, int hkv, int dk, int dv, int window, int keep_first,
                       const float* bias, int n_bias, int ld_bias, float softcap, const float* sink, const float* log_bias, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (hq < 1 || hkv < 1 || hq % hkv || dk < 1 || dv < 1 || n_seqs < 1 || page_size < 1) return fail("attn_any: bad sizes%s");
  if (dk > 2048 || dv > 1024) return fail("attn_any: keys of at most 2048 and values of at most 1024 features%s");
  if (bias != nullptr && (n_bias < 1 || ld_bias < n_bias)) return fail("attn_any: bad bias table%s");
  AttnAnyArgs a;
  a.q = q; a.k = k; a.v = v; a.out = out; a.cu_q = cu_q; a.kv_len = kv_len; a.block_table = block_table; a.max_pages = max_pages; a.page_size = page_size;
  a.n_seqs = n_seqs; a.num_slots = num_slots; a.tokens = tokens; a.hq = hq; a.hkv = hkv; a.dk = dk; a.dv = dv; a.window = window; a.keep_first = keep_first;
  a.bias = bias; a.n_bias = n_bias; a.ld_bias = ld_bias;
  a.q_hs = dk; a.q_ts = (long)hq * dk; a.k_hs = dk; a.k_ss = (long)hkv * dk; a.v_hs = dv; a.v_ss = (long)hkv * dv; a.o_hs = dv; a.o_ts = (long)hq * dv;
  a.tok_seq = nullptr; a.tok_kv = nullptr; a.sink = sink; a.cap = softcap > 0.f ? softcap * 1.4426950408889634f : 0.f;
  a.log_bias = log_bias;
  return f32 ? attn_any_launch<float>(a, stream) : attn_any_launch<__nv_bfloat16>(a, stream);
}

// Attention over cached latents: cache rows [slots, ld_c] hold `dk` key columns of which the first `dv` are the values, one for all heads.  q: head h of
// token t at q + t q_ts + h q_hs, out likewise.  tok_seq / tok_kv (null: one token per sequence, key counts kv_len): see AttnAnyArgs.
GB_API int gb_attn_latent_any(const void* q, long q_ts, long q_hs, const void* cache, int ld_c, void* out, long o_ts, long o_hs, int f32, const int* cu_q,
                              const int* kv_len, const int* tok_seq, const int* tok_kv, const int* block_table, int max_pages, int page_size, int n_seqs,
                              long num_slots, int tokens, int heads, int dk, int dv, const float* sink, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (heads < 1 || dk < 1 || dv < 1 || dv > dk || ld_c < dk || n_seqs < 1 || page_size < 1) return fail("attn_latent_any: bad sizes%s");
  if (dk > 2048 || dv > 1024) return fail("attn_latent_any: keys of at most 2048 and latents of at most 1024 features%s");
  if ((tok_seq == nullptr) != (tok_kv == nullptr)) return fail("attn_latent_any: tok_seq and tok_kv come together%s");
  AttnAnyArgs a;
  memset(&a, 0, sizeof(a));
  a.q = q; a.k = cache; a.v = cache; a.out = out; a.q_ts = q_ts; a.q_hs = q_hs; a.k_ss = ld_c; a.v_ss = ld_c; a.o_ts = o_ts; a.o_hs = o_hs;
  a.tok_seq = tok_seq; a.tok_kv = tok_kv; a.sink = sink; a.cu_q = cu_q; a.kv_len = kv_len; a.block_table = block_table; a.max_pages = max_pages;
  a.page_size = page_size; a.n_seqs = n_seqs; a.num_slots = num_slots; a.tokens = tokens; a.hq = heads; a.hkv = 1; a.dk = dk; a.dv = dv;
  return f32 ? attn_any_launch<float>(a, stream) : attn_any_launch<__nv_bfloat16>(a, stream);
}
