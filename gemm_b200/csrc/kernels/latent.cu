// Token-wise kernels of latent attention (keys and values are projections of a cached latent):
//   latent_store    [q latent | kv latent | rotated key part] rows of the first projection -> RMSNorm of the q latent (rows for the next projection),
//                   RMSNorm of the kv latent and rotation of the key part into the token's cache row
//   latent_q        query heads [unrotated | rotated] -> scaled and rotated, laid out for one of the two forms of the attention:
//                   over the latents (head by head, rows of the absorbed product) or over expanded keys (token by token)
//   latent_gather   cache rows of whole sequences, in order, for the expansion to keys and values
// Rotation: neighbours (2i, 2i + 1) turn by position * freq[i]; the angle is formed and reduced in 64-bit floats.
#include "sm100.cuh"
#include "host_common.h"
#include "recurrent.cuh"

namespace gb {

// cos and sin of position * freq, times mag
__device__ __forceinline__ void rotation(int pos, double freq, float mag, float& c, float& s) {
  const double turn = 6.283185307179586476925286766559, inv_turn = 0.15915494309189533576888376337251;
  double a = (double)pos * freq;
  a = fma(-turn, rint(a * inv_turn), a);
  sincosf((float)a, &s, &c);
  c *= mag; s *= mag;
}

struct LatentStoreArgs {
  const void* a; int n_part; long part_stride; int ld;         // [n_part][tokens, ld]: q latent, kv latent, rotated key part
  const int* positions; const int* slots;
  const float* q_norm; const float* kv_norm;                   // kv_norm null: only the q latent; q_rank 0: none
  const double* freq; float mag;
  void* q_out; int ld_q;                                       // [tokens, ld_q], zero behind q_rank
  void* cache; long num_slots; int ld_c;                       // [slots, ld_c], zero behind rank + rot_dim
  int q_rank, rank, rot_dim; float eps;
};

constexpr int kLatKeep = 8;                                    // values per thread kept in registers (ranks up to threads * kLatKeep)

template <typename TI, typename TO, int V, int NT>             // V columns at a time, NT threads per token
__global__ void __launch_bounds__(NT)
latent_store_kernel(const LatentStoreArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][NT / 32];
  constexpr int N = kLatKeep / V;
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5;
  const TI* src = (const TI*)a.a + (size_t)t * a.ld;
  auto values = [&](int c, float* v) {
    load_cols<V>(src + c, v);
    for (int p = 1; p < a.n_part; ++p) {
      float y[V];
      load_cols<V>(src + (size_t)p * a.part_stride + c, y);
#pragma unroll
      for (int x = 0; x < V; ++x) v[x] += y[x];
    }
  };
  const int slot = a.kv_norm != nullptr ? a.slots[t] : -1;
  const bool kv = slot >= 0 && slot < a.num_slots;
  float q[N][V], k[N][V], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (tid + i * NT) * V;
#pragma unroll
    for (int x = 0; x < V; ++x) q[i][x] = k[i][x] = 0.f;
    if (c < a.q_rank) values(c, q[i]);
    if (kv && c < a.rank) values(a.q_rank + c, k[i]);
#pragma unroll
    for (int x = 0; x < V; ++x) { sq += q[i][x] * q[i][x]; sk += k[i][x] * k[i][x]; }
  }
  sq = warp_sum(sq); sk = warp_sum(sk);
  if ((tid & 31) == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  TO* co = (TO*)a.cache + (size_t)(kv ? slot : 0) * a.ld_c;
  if (kv) {
    for (int i = NT - 1 - tid; i < a.rot_dim / 2; i += NT) {     // (the last warps: the first hold the ends of the ranks)
      float c, s, u = 0.f, v = 0.f;
      rotation(a.positions[t], a.freq[i], a.mag, c, s);
      const TI* p0 = src + a.q_rank + a.rank + 2 * i;
      for (int p = 0; p < a.n_part; ++p) { u += ldv(p0 + (size_t)p * a.part_stride); v += ldv(p0 + (size_t)p * a.part_stride + 1); }
      stv(co + a.rank + 2 * i, u * c - v * s);
      stv(co + a.rank + 2 * i + 1, v * c + u * s);
    }
    for (int c = a.rank + a.rot_dim + tid; c < a.ld_c; c += NT) stv(co + c, 0.f);
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float iq = a.q_rank > 0 ? 1.0f / sqrtf(sq / (float)a.q_rank + a.eps) : 0.f, ik = 1.0f / sqrtf(sk / (float)a.rank + a.eps);
  TO* qo = (TO*)a.q_out + (size_t)t * a.ld_q;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (tid + i * NT) * V;
    if (c < a.ld_q) {                                          // zero behind q_rank
      float w[V];
#pragma unroll
      for (int x = 0; x < V; ++x) w[x] = 0.f;
      if (c < a.q_rank) load_cols<V>(a.q_norm + c, w);
#pragma unroll
      for (int x = 0; x < V; ++x) w[x] *= q[i][x] * iq;
      store_cols<V>(qo + c, w);
    }
    if (kv && c < a.rank) {
      float w[V];
      load_cols<V>(a.kv_norm + c, w);
#pragma unroll
      for (int x = 0; x < V; ++x) w[x] *= k[i][x] * ik;
      store_cols<V>(co + c, w);
    }
  }
}

struct LatentQArgs {
  const void* q; int n_part; long part_stride; int ld;         // [n_part][tokens, ld]: per head dim unrotated, rot_dim rotated
  const int* positions; const double* freq; float mag, scale;
  const int* dst;                                              // per token: row r >= 0 of the absorbed form, or -1 - r of the expanded form; null: row t
  void* a_n; long an_ts, an_hs; int an_w;                      // absorbed: unrotated part (an_w columns, zero behind dim) ...
  void* a_r; long ar_ts, ar_hs; int ar_w;                      // ... and rotated part (ar_w columns, zero behind rot_dim)
  void* m_n; long mn_ts, mn_hs; int mn_w;                      // expanded: the same
  void* m_r; long mr_ts, mr_hs; int mr_w;
  int heads, dim, rot_dim;
};

// A CTA: one token, `per` heads; a warp per head, a lane per pair of columns.
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
latent_q_kernel(const LatentQArgs a, int per) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float cs[];                                // cos, sin of the token's pairs
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int half = a.rot_dim / 2;
  for (int i = tid; i < half; i += 256) rotation(a.positions[t], a.freq[i], a.mag * a.scale, cs[i], cs[half + i]);
  __syncthreads();
  const int d = a.dst != nullptr ? a.dst[t] : t;
  const bool ab = d >= 0;
  const size_t row = ab ? (size_t)d : (size_t)(-1 - d);
  const int nw = ab ? a.an_w : a.mn_w, rw = ab ? a.ar_w : a.mr_w, hd = a.dim + a.rot_dim;
  const int h_end = min(a.heads, (int)(blockIdx.y + 1) * per);
  for (int h = blockIdx.y * per + warp; h < h_end; h += 8) {
    TO* on = (TO*)(ab ? a.a_n : a.m_n) + row * (ab ? a.an_ts : a.mn_ts) + h * (ab ? a.an_hs : a.mn_hs);
    TO* orr = (TO*)(ab ? a.a_r : a.m_r) + row * (ab ? a.ar_ts : a.mr_ts) + h * (ab ? a.ar_hs : a.mr_hs);
    const TI* src = (const TI*)a.q + (size_t)t * a.ld + h * hd;
    auto value = [&](int c) {
      float v = ldv(src + c);
      for (int p = 1; p < a.n_part; ++p) v += ldv(src + (size_t)p * a.part_stride + c);
      return v;
    };
    for (int c = lane; c < nw; c += 32) stv(on + c, c < a.dim ? value(c) * a.scale : 0.f);
    for (int i = lane; i < half; i += 32) {
      const float u = value(a.dim + 2 * i), v = value(a.dim + 2 * i + 1), co = cs[i], si = cs[half + i];
      stv(orr + 2 * i, u * co - v * si);
      stv(orr + 2 * i + 1, v * co + u * si);
    }
    for (int c = a.rot_dim + lane; c < rw; c += 32) stv(orr + c, 0.f);
  }
}

// rows of 16-byte vectors: row r belongs to sequence s with kv0[s] <= r < kv0[s + 1], at position r - kv0[s]
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, long num_slots, int vecs, const int* __restrict__ kv0, const int* __restrict__ seq, int n_seqs,
                     const int* __restrict__ block_table, int max_pages, int page_size, uint4* __restrict__ out, int rows) {
  pdl_wait();
  pdl_trigger();
  const long i = (long)blockIdx.x * 256 + threadIdx.x;
  const long r = i / vecs;
  const int c = (int)(i - r * vecs);
  if (r >= rows) return;
  int lo = 0, hi = n_seqs;
  while (hi - lo > 1) { const int mid = (lo + hi) >> 1; if (kv0[mid] <= r) lo = mid; else hi = mid; }
  const int pos = (int)(r - kv0[lo]), pg = pos / page_size;
  if (pg >= max_pages) return;
  const long slot = (long)block_table[(size_t)seq[lo] * max_pages + pg] * page_size + pos % page_size;
  if (slot < 0 || slot >= num_slots) return;
  out[r * vecs + c] = cache[slot * vecs + c];
}

}  // namespace gb

using namespace gb;

// See LatentStoreArgs.  in_f32 / out_f32: element types of the projection rows and of q_out and the cache.
GB_API int gb_latent_store(const void* rows, int in_f32, int n_part, long part_stride, int ld, const int* positions, const int* slots, const float* q_norm,
                           const float* kv_norm, const double* freq, float mag, void* q_out, int ld_q, void* cache, int out_f32, long num_slots, int ld_c, int tokens,
                           int q_rank, int rank, int rot_dim, float eps, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (q_rank < 0 || (q_rank == 0 ? kv_norm == nullptr || ld_q != 0 : q_out == nullptr) || rank < 1 || rot_dim < 0 || rot_dim % 2 || n_part < 1 || ld_q < q_rank || (kv_norm != nullptr && ld_c < rank + rot_dim) ||
      ld < q_rank + (kv_norm != nullptr ? rank + rot_dim : 0)) return fail("latent_store: bad sizes%s");
  if (ld_q > 256 * kLatKeep || rank > 256 * kLatKeep) return fail("latent_store: ranks of at most 2048%s");
  LatentStoreArgs a;
  a.a = rows; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.positions = positions; a.slots = slots; a.q_norm = q_norm; a.kv_norm = kv_norm;
  a.freq = freq; a.mag = mag; a.q_out = q_out; a.ld_q = ld_q; a.cache = cache; a.num_slots = num_slots; a.ld_c = ld_c; a.q_rank = q_rank; a.rank = rank;
  a.rot_dim = rot_dim; a.eps = eps;
  const auto al = [](const void* p, size_t n) { return (uintptr_t)p % n == 0; };
  const size_t ei = in_f32 ? 16 : 8, eo = out_f32 ? 16 : 8;
  const bool vec = q_rank % 4 == 0 && rank % 4 == 0 && ld % 4 == 0 && part_stride % 4 == 0 && ld_q % 4 == 0 && ld_c % 4 == 0 && al(rows, ei) && al(q_out, eo) && al(cache, eo) &&
                   al(q_norm, 16) && al(kv_norm, 16);
  if (!in_f32 && out_f32) return fail("latent_store: a 32-bit cache takes 32-bit rows%s");
  const bool narrow = vec && ld_q <= 64 * kLatKeep && rank <= 64 * kLatKeep;     // short rows: more tokens per SM
#define GB_LAT(TI, TO)                                                                                                                    \
  (narrow ? launch_k(latent_store_kernel<TI, TO, 4, 64>, (unsigned)tokens, 64, 0, stream, a)                                               \
   : vec  ? launch_k(latent_store_kernel<TI, TO, 4, 256>, (unsigned)tokens, 256, 0, stream, a)                                             \
          : launch_k(latent_store_kernel<TI, TO, 1, 256>, (unsigned)tokens, 256, 0, stream, a))
  if (in_f32 && out_f32) GB_LAT(float, float);
  else if (in_f32) GB_LAT(float, __nv_bfloat16);
  else GB_LAT(__nv_bfloat16, __nv_bfloat16);
#undef GB_LAT
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// See LatentQArgs; strides in elements.
GB_API int gb_latent_q(const void* q, int in_f32, int n_part, long part_stride, int ld, const int* positions, const double* freq, float mag, float scale, const int* dst,
                       void* a_n, long an_ts, long an_hs, int an_w, void* a_r, long ar_ts, long ar_hs, int ar_w, void* m_n, long mn_ts, long mn_hs, int mn_w, void* m_r,
                       long mr_ts, long mr_hs, int mr_w, int out_f32, int tokens, int heads, int dim, int rot_dim, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (heads < 1 || dim < 1 || rot_dim < 0 || rot_dim % 2 || rot_dim > 1024 || n_part < 1 || ld < heads * (dim + rot_dim)) return fail("latent_q: bad sizes%s");
  if ((a_n != nullptr && (an_w < dim || ar_w < rot_dim)) || (m_n != nullptr && (mn_w < dim || mr_w < rot_dim))) return fail("latent_q: outputs are too narrow%s");
  LatentQArgs a;
  a.q = q; a.n_part = n_part; a.part_stride = part_stride; a.ld = ld; a.positions = positions; a.freq = freq; a.mag = mag; a.scale = scale; a.dst = dst;
  a.a_n = a_n; a.an_ts = an_ts; a.an_hs = an_hs; a.an_w = an_w; a.a_r = a_r; a.ar_ts = ar_ts; a.ar_hs = ar_hs; a.ar_w = ar_w;
  a.m_n = m_n; a.mn_ts = mn_ts; a.mn_hs = mn_hs; a.mn_w = mn_w; a.m_r = m_r; a.mr_ts = mr_ts; a.mr_hs = mr_hs; a.mr_w = mr_w;
  a.heads = heads; a.dim = dim; a.rot_dim = rot_dim;
  const size_t smem = (size_t)rot_dim * sizeof(float);
  const int per = tokens >= 1024 ? heads : 8;                  // small batches spread a token's heads over CTAs
  const dim3 grid((unsigned)tokens, (unsigned)((heads + per - 1) / per));
  if (in_f32 && out_f32) launch_k(latent_q_kernel<float, float>, grid, 256, smem, stream, a, per);
  else if (in_f32) launch_k(latent_q_kernel<float, __nv_bfloat16>, grid, 256, smem, stream, a, per);
  else if (out_f32) return fail("latent_q: 32-bit results take 32-bit rows%s");
  else launch_k(latent_q_kernel<__nv_bfloat16, __nv_bfloat16>, grid, 256, smem, stream, a, per);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

// Cache rows (row_bytes each, a multiple of 16) of n_seqs whole sequences in order: kv0 [n_seqs + 1] first output row of each, seq [n_seqs] its row of
// the block table.
GB_API int gb_latent_gather(const void* cache, long num_slots, int row_bytes, const int* kv0, const int* seq, int n_seqs, const int* block_table, int max_pages,
                            int page_size, void* out, int rows, cudaStream_t stream) {
  if (rows <= 0 || n_seqs <= 0) return 0;
  if (row_bytes < 16 || row_bytes % 16 || ((uintptr_t)cache & 15) || ((uintptr_t)out & 15) || page_size < 1) return fail("latent_gather: rows of whole 16-byte vectors%s");
  const int vecs = row_bytes / 16;
  launch_k(latent_gather_kernel, (unsigned)(((long)rows * vecs + 255) / 256), 256, 0, stream, (const uint4*)cache, num_slots, vecs, kv0, seq, n_seqs, block_table, max_pages,
           page_size, (uint4*)out, rows);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}
