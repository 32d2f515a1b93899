// Latent attention on tcgen05, in its two forms (see ops/latent.py).
//
// latent_decode_kernel (absorbed form): the cached rows [latent | rotated key part] are keys and values of all query heads at once.  A CTA owns one
// token, a tile of NH heads and a range of its keys.  As in the decode kernel of flash_attn.cu the key POSITIONS are the MMA's M dimension:
//   S^T[positions x NH]   = C_j[positions x width] Q^T       (A = rows as they are cached, K-major; B = the heads' queries)
//   O^T[128 columns x NH] += C_j^T[128 x positions] P_j      (A = the same rows, MN-major, one product per 128 latent columns; B = P^T in shared memory)
// so that every cached byte is fetched once for both products.  A block of 128 positions is a row of boxes of 64 columns (16 KB), a pair of boxes
// sharing a barrier: S starts with the first pair that lands, and O's products free the pairs one by one for the next block.  With 512 + 64 columns
// one block fills shared memory.  Two half-sized blocks in turn were measured 1.2 to 1.5 times slower: what bounds the loop is the chain load -> S ->
// softmax -> O -> load, whose length hardly depends on the block's size.
//
// latent_prefill_kernel (expanded form): keys [expanded part | rotated part shared by the heads] and values of one head.  A CTA owns one head and
// two tiles of 128 tokens, which take turns: while one tile's softmax runs, the tensor core works for the other.  K is double-buffered.
//
// In both a learned score per head (sink) joins the softmax's sum.  Scores arrive in base 2: Q is multiplied by scale * log2 e, sinks by log2 e.
#include "sm100.cuh"
#include "host_common.h"
#include "flash_common.cuh"
#include "recurrent.cuh"

namespace gb {

constexpr int kLdThreads = 224;         // TMA warp, S warp, O warp, 4 softmax warps
constexpr int kLdB = 128;                 // positions per block
constexpr int kLdBox = 16384;             // 128 positions x 64 columns
constexpr int kLdMaxPairs = 24;           // pairs of boxes in shared memory

struct LatentDecodeArgs {
  const int* tok_seq; const int* tok_kv;  // per token: row of the block table, number of keys; null: token i is sequence i, kv_len[i] keys
  const int* kv_len;
  const int* block_table; int max_pages, page_size;
  int tokens, heads, head_tiles, splits;
  int width, rank;                        // key columns, of which the first `rank` are the values
  int boxes, stages;                      // 64-column boxes per block, blocks in shared memory
  __nv_bfloat16* out; int m_rows, ld_out; // [heads][m_rows][ld_out]
  float* part_o; float* part_lse;         // [splits][tokens][heads][rank], [splits][tokens][heads] (splits > 1)
  const float* sink;
  KernelStatus* status;
};

template <int NH>
__device__ __forceinline__ void tmem_ld_heads(uint32_t t, uint32_t* r) { if constexpr (NH == 32) tmem_ld_x32(t, r); else tmem_ld_x16(t, r); }
template <int NH>
__device__ __forceinline__ void tmem_st_heads(uint32_t t, const uint32_t* r) { if constexpr (NH == 32) tmem_st_x32(t, r); else tmem_st_x16(t, r); }

template <int NH>
__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, const LatentDecodeArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  constexpr int kQ = NH * 128;            // bytes of a 64-column box of queries, and of half of P^T
  const int pairs = (a.boxes + 1) >> 1;
  uint8_t* sC = smem;
  uint8_t* sP = sC + a.boxes * a.stages * kLdBox;      // two buffers
  uint8_t* sQ = sP + 4 * kQ;              // (behind the last box at least 16 KB are P and queries: where the number of boxes is odd, O's operand goes on there)
  uint64_t* bars = (uint64_t*)(sQ + max(a.boxes, 4) * kQ);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;            // 2, by block parity
  uint64_t* p_ready = bars + 3;           // 2, 128 arrivals each (two for the reason given in flash_decode_kernel)
  uint64_t* o_ready = bars + 5;           // 2
  uint64_t* t_full = bars + 7;            // per box
  uint64_t* t_empty = t_full + kLdMaxPairs;
  uint32_t* tmem_slot = (uint32_t*)(t_empty + kLdMaxPairs);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
  float* red_max = (float*)(((uintptr_t)(tmem_slot + 2) + 15) & ~(uintptr_t)15);       // [4 warps][NH]
  float* red_sum = red_max + 4 * NH;                                                   // [4][NH]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_ready[i], 128); mbar_init(&o_ready[i], 1); }
    for (int i = 0; i < pairs * a.stages; ++i) { mbar_init(&t_full[i], 1); mbar_init(&t_empty[i], 1); }
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmC);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 256); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 2 * NH;
  pdl_wait();

  const int split = blockIdx.x % a.splits, ht = (blockIdx.x / a.splits) % a.head_tiles, tok = blockIdx.x / (a.splits * a.head_tiles);
  const int h0 = ht * NH, n_heads = min(NH, a.heads - h0);
  const int seq = a.tok_seq != nullptr ? a.tok_seq[tok] : tok;
  const int kv = a.tok_kv != nullptr ? a.tok_kv[tok] : a.kv_len[tok];
  const int n_all = (kv + kLdB - 1) / kLdB, per = (n_all + a.splits - 1) / a.splits;
  const int blk0 = split * per, n_blk = max(0, min(n_all, blk0 + per) - blk0);
  const int m_tiles = (a.rank + 127) >> 7;

  if (warp == 0) {
    if (lane == 0 && n_blk > 0) {
      mbar_expect_tx(q_full, (uint32_t)(a.boxes * kQ));
      for (int b = 0; b < a.boxes; ++b) tma_load_3d(sQ + b * kQ, &tmQ, q_full, b * 64, tok, h0);
      // page sizes are powers of two.  Pages behind the last one are replaced by it: finite rows, masked
      const int shift = __ffs(a.page_size) - 1, last_page = (kv - 1) >> shift;
      const int* bt = a.block_table + (size_t)seq * a.max_pages;
      auto cache_row = [&](int pos) { return (bt[min(pos >> shift, last_page)] << shift) + (pos & (a.page_size - 1)); };
      bool ok = true;
      int st = 0; uint32_t ph = 1;
      if (2 * a.page_size >= kLdB) {             // a block lies in one or two pages; their rows are looked up a block ahead
        const bool halves = a.page_size < kLdB;
        const int half = kLdBox / 2;
        int next0 = cache_row(blk0 * kLdB), next1 = halves ? cache_row(blk0 * kLdB + kLdB / 2) : 0;
        for (int j = 0; j < n_blk && ok; ++j) {
          const int row0 = next0, row1 = next1;
          if (j + 1 < n_blk) { next0 = cache_row((blk0 + j + 1) * kLdB); if (halves) next1 = cache_row((blk0 + j + 1) * kLdB + kLdB / 2); }
          uint8_t* dst = sC + st * a.boxes * kLdBox;
          for (int b = 0; b < a.boxes; b += 2, dst += 2 * kLdBox) {
            const int s = st * pairs + (b >> 1);
            if (!mbar_wait(&t_empty[s], ph, abort_flag, a.status, 800, j)) { ok = false; break; }
            const bool two = b + 1 < a.boxes;
            mbar_expect_tx(&t_full[s], two ? 2 * kLdBox : kLdBox);
            tma_load_2d(dst, &tmC, &t_full[s], b * 64, row0);
            if (two) tma_load_2d(dst + kLdBox, &tmC, &t_full[s], b * 64 + 64, row0);
            if (halves) {
              tma_load_2d(dst + half, &tmC, &t_full[s], b * 64, row1);
              if (two) tma_load_2d(dst + kLdBox + half, &tmC, &t_full[s], b * 64 + 64, row1);
            }
          }
          if (++st == a.stages) { st = 0; ph ^= 1; }
        }
      } else {
        for (int j = 0; j < n_blk && ok; ++j) {
          for (int b = 0; b < a.boxes; b += 2) {
            const int s = st * pairs + (b >> 1);
            if (!mbar_wait(&t_empty[s], ph, abort_flag, a.status, 801, j)) { ok = false; break; }
            const bool two = b + 1 < a.boxes;
            mbar_expect_tx(&t_full[s], two ? 2 * kLdBox : kLdBox);
            for (int x = 0; x < kLdB; x += a.page_size) {
              const int row = cache_row((blk0 + j) * kLdB + x);
              uint8_t* dst = sC + (st * a.boxes + b) * kLdBox + x * 128;
              tma_load_2d(dst, &tmC, &t_full[s], b * 64, row);
              if (two) tma_load_2d(dst + kLdBox, &tmC, &t_full[s], b * 64 + 64, row);
            }
          }
          if (++st == a.stages) { st = 0; ph ^= 1; }
        }
      }
    }
  } else if (warp == 1) {
    // the products are issued by two threads: one needs longer to issue a block's MMAs than its data take to arrive
    if (lane == 0 && n_blk > 0) {
      constexpr uint32_t id_s = make_idesc(128, NH, 1, 1, 0, 0);
      const uint64_t d_q = make_sdesc_sw128(smem_u32(sQ)), d_c = make_sdesc_sw128(smem_u32(sC));
      const int k_steps = (a.width + 15) >> 4;
      bool ok = mbar_wait(q_full, 0, abort_flag, a.status, 810);
      int st = 0; uint32_t ph = 0;
      for (int j = 0; j < n_blk && ok; ++j) {
        // the scores of block j - 2 have been read
        if (j >= 2 && !mbar_wait(&p_ready[j & 1], (uint32_t)((j - 2) >> 1) & 1, abort_flag, a.status, 813, j)) break;
        const uint32_t d = tmem_s + (j & 1) * NH;
        uint64_t dc = sdesc_at(d_c, st * a.boxes * kLdBox), dq = d_q;
        for (int b = 0; b < pairs; ++b) {
          if (!mbar_wait(&t_full[st * pairs + b], ph, abort_flag, a.status, 811, j)) { ok = false; break; }
          tc_fence_after();
          const uint32_t acc = b > 0 ? 1u : 0u;
          if (b * 8 + 8 <= k_steps) {
#pragma unroll
            for (int x = 0; x < 8; ++x)
              mma_f16_ss(d, sdesc_at(dc, (x >> 2) * kLdBox + (x & 3) * 32), sdesc_at(dq, (x >> 2) * kQ + (x & 3) * 32), id_s, x > 0 ? 1u : acc);
          } else {
            for (int x = 0; b * 8 + x < k_steps; ++x)
              mma_f16_ss(d, sdesc_at(dc, (x >> 2) * kLdBox + (x & 3) * 32), sdesc_at(dq, (x >> 2) * kQ + (x & 3) * 32), id_s, x > 0 ? 1u : acc);
          }
          if (b >= m_tiles) tc_commit(&t_empty[st * pairs + b]);        // no values in these boxes
          dc = sdesc_at(dc, 2 * kLdBox); dq = sdesc_at(dq, 2 * kQ);
        }
        if (!ok) break;
        tc_commit(&s_full[j & 1]);
        if (++st == a.stages) { st = 0; ph ^= 1; }
      }
    }
  } else if (warp == 2) {
    if (lane == 0 && n_blk > 0) {
      constexpr uint32_t id_o = make_idesc(128, NH, 1, 1, 1, 0);      // A (latents by position) is MN-major
      const uint64_t d_p = make_sdesc_sw128(smem_u32(sP)), d_v = make_sdesc_sw128_mn(smem_u32(sC), kLdBox);
      int st = 0;
      for (int j = 0; j < n_blk; ++j) {
        // P follows from S, so the block's boxes have landed and S has read them
        if (!mbar_wait(&p_ready[j & 1], (uint32_t)(j >> 1) & 1, abort_flag, a.status, 812, j)) break;
        tc_fence_after();
        uint64_t dv = sdesc_at(d_v, st * a.boxes * kLdBox);
        const uint64_t dp = sdesc_at(d_p, (j & 1) * 2 * kQ);
        const uint32_t acc = j > 0 ? 1u : 0u;
        for (int m = 0; m < m_tiles; ++m) {
#pragma unroll
          for (int ks = 0; ks < 8; ++ks) mma_f16_ss(tmem_o + m * NH, sdesc_at(dv, ks * 2048), sdesc_at(dp, (ks >> 2) * kQ + (ks & 3) * 32), id_o, ks > 0 ? 1u : acc);
          tc_commit(&t_empty[st * pairs + m]);
          dv = sdesc_at(dv, 2 * kLdBox);
        }
        tc_commit(&o_ready[j & 1]);
        if (++st == a.stages) st = 0;
      }
    }
  } else {
    // thread r: position r of the block, column r of each tile of O
    const int q = warp & 3, r = q * 32 + lane;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    float m[NH], l[NH];                                  // reference maximum; this thread's share of the sums
#pragma unroll
    for (int h = 0; h < NH; ++h) { m[h] = -INFINITY; l[h] = 0.f; }
    constexpr float kTau = 8.0f;                         // O and l are rescaled only when a maximum has grown by more than 2^kTau
    bool ok = true, fail_o = false;                      // fail_o: a wait for O ran out; it is put to the vote at the next barrier
    for (int j = 0; j < n_blk && ok; ++j) {
      const bool got = warp_wait(&s_full[j & 1], (uint32_t)(j >> 1) & 1, abort_flag, a.status, 820, j);
      tc_fence_after();
      float sv[NH];
      bool grow = false;
      tmem_ld_heads<NH>(tmem_s + (j & 1) * NH + lane_off, reinterpret_cast<uint32_t*>(sv));
      tc_wait_ld();
      const bool live = (blk0 + j) * kLdB + r < kv;
#pragma unroll
      for (int h = 0; h < NH; ++h) {
        if (!live || h >= n_heads) sv[h] = -INFINITY;
        grow |= sv[h] > m[h] + kTau;                     // also the first finite score
      }
      bool got_o = true;
      if (!bar128_and(got && !fail_o && !grow)) {        // rare: some score has outgrown its reference, or a wait ran out
        if (!bar128_and(got && !fail_o)) { ok = false; break; }         // all 128 threads leave together
#pragma unroll
        for (int x = 0; x < NH; x += 16) {
          const float v = warp_reduce16_max(sv + x, lane);
          if ((lane & 1) == 0) red_max[q * NH + x + (lane >> 1)] = v;
        }
        bar128_and(true);
        // every earlier product is in O before it is rescaled
        if (j > 0) got_o = warp_wait(&o_ready[(j - 1) & 1], (uint32_t)((j - 1) >> 1) & 1, abort_flag, a.status, 821, j);
        tc_fence_after();
        float al[NH];
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          const float mn = fmaxf(m[h], fmaxf(fmaxf(red_max[h], red_max[NH + h]), fmaxf(red_max[2 * NH + h], red_max[3 * NH + h])));
          al[h] = mn == -INFINITY ? 1.0f : fast_exp2(m[h] - mn);
          m[h] = mn; l[h] *= al[h];
        }
        bar128_and(true);                                // red_max may be written again
        if (j > 0 && got_o)
          for (int t = 0; t < m_tiles; ++t) {
            uint32_t o[NH];
            tmem_ld_heads<NH>(tmem_o + t * NH + lane_off, o);
            tc_wait_ld();
#pragma unroll
            for (int h = 0; h < NH; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * al[h]);
            tmem_st_heads<NH>(tmem_o + t * NH + lane_off, o);
            tc_wait_st();
          }
      }
      // the P buffer of this parity was read by the product of block j - 2
      if (got_o && j >= 2) got_o = warp_wait(&o_ready[j & 1], (uint32_t)((j - 2) >> 1) & 1, abort_flag, a.status, 822, j);
      if (got_o) {
        uint8_t* pb = sP + ((j & 1) * 2 + (r >> 6)) * kQ + (r & 7) * 2;
        const int chunk = (r & 63) >> 3;
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          const float p = h < n_heads ? fast_exp2(sv[h] - m[h]) : 0.f;
          l[h] += p;
          *reinterpret_cast<__nv_bfloat16*>(pb + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16(p);
        }
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(&p_ready[j & 1]);
      }
      fail_o |= !got_o;
    }
    if (ok && !fail_o && n_blk > 0) ok = warp_wait(&o_ready[(n_blk - 1) & 1], (uint32_t)((n_blk - 1) >> 1) & 1, abort_flag, a.status, 823, 0);
#pragma unroll
    for (int x = 0; x < NH; x += 16) {
      const float v = warp_reduce16_sum(l + x, lane);
      if ((lane & 1) == 0) red_sum[q * NH + x + (lane >> 1)] = v;
    }
    ok = bar128_and(ok && !fail_o);
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int h = 0; h < NH; ++h) l[h] = red_sum[h] + red_sum[NH + h] + red_sum[2 * NH + h] + red_sum[3 * NH + h];
      float inv[NH];
#pragma unroll
      for (int h = 0; h < NH; ++h) {
        float den = l[h];
        if (a.splits == 1 && a.sink != nullptr && h < n_heads) den += fast_exp2(a.sink[h0 + h] - (m[h] == -INFINITY ? 0.f : m[h]));
        inv[h] = den > 0.f ? 1.0f / den : 0.f;
      }
      for (int t = 0; t < m_tiles; ++t) {
        uint32_t o[NH];
        if (n_blk > 0) { tmem_ld_heads<NH>(tmem_o + t * NH + lane_off, o); tc_wait_ld(); }
        else {
#pragma unroll
          for (int h = 0; h < NH; ++h) o[h] = 0u;
        }
        const int c = t * 128 + r;
        if (c < a.rank) {
#pragma unroll
          for (int h = 0; h < NH; ++h) {
            if (h >= n_heads) continue;
            const float v = __uint_as_float(o[h]) * inv[h];
            if (a.splits == 1) a.out[((size_t)(h0 + h) * a.m_rows + tok) * a.ld_out + c] = __float2bfloat16(v);
            else a.part_o[(((size_t)split * a.tokens + tok) * a.heads + h0 + h) * a.rank + c] = v;
          }
        }
      }
      if (a.splits > 1 && r == 0) {
#pragma unroll
        for (int h = 0; h < NH; ++h)
          if (h < n_heads) a.part_lse[((size_t)split * a.tokens + tok) * a.heads + h0 + h] = l[h] > 0.f ? m[h] + log2f(l[h]) : -INFINITY;
      }
    }
  }

  pdl_trigger();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_s, 256); }
}

// Merge of the key ranges, and the sink: out[h][tok] = sum_s 2^(lse_s) O_s / (sum_s 2^(lse_s) + 2^(sink)).  One CTA per (token, head) and 128 columns.
constexpr int kLdMaxSplits = 64;
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse, const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, int splits,
                      int tokens, int heads, int rank, int m_rows, int ld_out) {
  pdl_wait();
  pdl_trigger();
  __shared__ float w[kLdMaxSplits];
  const int h = blockIdx.x % heads, tok = blockIdx.x / heads, c = blockIdx.y * 128 + threadIdx.x;
  const size_t row = (size_t)tok * heads + h, rows = (size_t)tokens * heads;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const float sk = sink != nullptr ? sink[h] : -INFINITY;
    float l[kLdMaxSplits / 32], mx = sk, den = 0.f;
#pragma unroll
    for (int i = 0; i < kLdMaxSplits / 32; ++i) { const int s = lane + 32 * i; l[i] = s < splits ? part_lse[s * rows + row] : -INFINITY; mx = fmaxf(mx, l[i]); }
    mx = warp_max(mx);
#pragma unroll
    for (int i = 0; i < kLdMaxSplits / 32; ++i) { l[i] = l[i] > -INFINITY ? exp2f(l[i] - mx) : 0.f; den += l[i]; }
    den = warp_sum(den) + (sk > -INFINITY ? exp2f(sk - mx) : 0.f);
#pragma unroll
    for (int i = 0; i < kLdMaxSplits / 32; ++i) w[lane + 32 * i] = den > 0.f ? l[i] / den : 0.f;
  }
  __syncthreads();
  if (c >= rank) return;
  float v = 0.f;
#pragma unroll 8
  for (int s = 0; s < splits; ++s) v = fmaf(w[s], part_o[(s * rows + row) * rank + c], v);
  out[((size_t)h * m_rows + tok) * ld_out + c] = __float2bfloat16(v);
}

// ------------------------------------------------------------------------------------------ expanded form
constexpr int kLpThreads = 320;
constexpr int kLpSmem = 2 * 49152 + 2 * 49152 + 32768 + 256 + 1024;     // two Q tiles, two K blocks (each 32 KB + 16 KB), one V block

struct LatentPrefillArgs {
  const int* tiles; int n_tiles;          // [n_tiles, 2] {sequence, first token of the 256}
  const int* q0; const int* kv0;          // [S + 1] first query row / first key row of each sequence; the queries are the last of its keys
  const int* tok;                         // output token of each query row
  __nv_bfloat16* out;                     // [T][heads][dv]
  int heads, dn, dr, dv;                  // key columns (expanded, rotated) and value columns, multiples of 8
  const float* sink;
  KernelStatus* status;
};

__global__ void __launch_bounds__(kLpThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQn, const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmKn,
                      const __grid_constant__ CUtensorMap tmKr, const __grid_constant__ CUtensorMap tmV, const LatentPrefillArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  uint8_t* sQ = smem;                      // tile t at t * 49152: two halves of 64 expanded columns, then the rotated ones
  uint8_t* sK = smem + 2 * 49152;          // block j & 1, same layout
  uint8_t* sV = sK + 2 * 49152;
  uint64_t* bars = (uint64_t*)(sV + 32768);
  uint64_t* q_full = bars;                 // 2: per tile
  uint64_t* k_full = bars + 2;             // 2
  uint64_t* k_empty = bars + 4;            // 2
  uint64_t* v_full = bars + 6;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 8;             // 2: per tile
  uint64_t* p_ready = bars + 10;           // 2: per tile, 128 arrivals
  uint64_t* o_ready = bars + 12;           // 2
  uint32_t* tmem_slot = (uint32_t*)(bars + 14);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&q_full[i], 1); mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&s_full[i], 1); mbar_init(&p_ready[i], 128); mbar_init(&o_ready[i], 1);
    }
    mbar_init(v_full, 1); mbar_init(v_empty, 1);
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQn); tma_prefetch_desc(&tmQr); tma_prefetch_desc(&tmKn); tma_prefetch_desc(&tmKr); tma_prefetch_desc(&tmV);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;        // S / P of tile t at 128 t, O of tile t at 256 + 128 t
  pdl_wait();

  const int h = blockIdx.x % a.heads, ti = blockIdx.x / a.heads;
  const int seq = a.tiles[2 * ti], x0 = a.tiles[2 * ti + 1];
  const int qb = a.q0[seq], q_len = a.q0[seq + 1] - qb, kb = a.kv0[seq], kv_len = a.kv0[seq + 1] - kb;
  int n_tok[2], pos0[2], n_blk[2];         // tokens, first position and key blocks of the two tiles
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    n_tok[t] = max(0, min(128, q_len - x0 - 128 * t));
    pos0[t] = kv_len - q_len + x0 + 128 * t;
    n_blk[t] = n_tok[t] > 0 ? (pos0[t] + n_tok[t] - 1) / 128 + 1 : 0;
  }
  const int n_max = max(n_blk[0], n_blk[1]);
  const bool n2 = a.dn > 64, v2 = a.dv > 64;

  if (warp == 0) {
    if (lane == 0) {
      const uint32_t kbytes = 16384u * ((n2 ? 2 : 1) + 1);
      for (int t = 0; t < 2; ++t) {
        if (n_blk[t] == 0) continue;
        mbar_expect_tx(&q_full[t], kbytes);
        const int row = qb + x0 + 128 * t;
        tma_load_3d(sQ + t * 49152, &tmQn, &q_full[t], 0, h, row);
        if (n2) tma_load_3d(sQ + t * 49152 + 16384, &tmQn, &q_full[t], 64, h, row);
        tma_load_3d(sQ + t * 49152 + 32768, &tmQr, &q_full[t], 0, h, row);
      }
      for (int j = 0; j < n_max; ++j) {
        const int b = j & 1, row = kb + j * 128;
        uint8_t* k = sK + b * 49152;
        if (!mbar_wait(&k_empty[b], ((uint32_t)(j >> 1) & 1) ^ 1, abort_flag, a.status, 830, j)) break;
        mbar_expect_tx(&k_full[b], kbytes);
        tma_load_3d(k, &tmKn, &k_full[b], 0, h, row);
        if (n2) tma_load_3d(k + 16384, &tmKn, &k_full[b], 64, h, row);
        tma_load_2d(k + 32768, &tmKr, &k_full[b], 0, row);
        if (!mbar_wait(v_empty, (uint32_t)(j & 1) ^ 1, abort_flag, a.status, 831, j)) break;
        mbar_expect_tx(v_full, v2 ? 32768u : 16384u);
        tma_load_3d(sV, &tmV, v_full, 0, h, row);
        if (v2) tma_load_3d(sV + 16384, &tmV, v_full, 64, h, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t id_s = make_idesc(128, 128, 1, 1, 0, 0);
      const uint32_t id_o = v2 ? make_idesc(128, 128, 1, 1, 0, 1) : make_idesc(128, 64, 1, 1, 0, 1);
      const uint64_t d_q = make_sdesc_sw128(smem_u32(sQ)), d_k = make_sdesc_sw128(smem_u32(sK)), d_v = make_sdesc_sw128_mn(smem_u32(sV), 16384);
      const int kn = (a.dn + 15) >> 4, kr = (a.dr + 15) >> 4;
      auto issue_s = [&](int t, int j) {
        const uint64_t q = sdesc_at(d_q, t * 49152), k = sdesc_at(d_k, (j & 1) * 49152);
        const uint32_t d = tmem + 128 * t;
        for (int ks = 0; ks < kn; ++ks) {
          const uint32_t off = (ks >> 2) * 16384 + (ks & 3) * 32;
          mma_f16_ss(d, sdesc_at(q, off), sdesc_at(k, off), id_s, ks > 0 ? 1u : 0u);
        }
        for (int ks = 0; ks < kr; ++ks) mma_f16_ss(d, sdesc_at(q, 32768 + ks * 32), sdesc_at(k, 32768 + ks * 32), id_s, 1u);
        tc_commit(&s_full[t]);
      };
      bool ok = true;
      for (int t = 0; t < 2 && ok; ++t) if (n_blk[t] > 0) ok = mbar_wait(&q_full[t], 0, abort_flag, a.status, 840, t);
      if (ok && n_max > 0) ok = mbar_wait(&k_full[0], 0, abort_flag, a.status, 841, 0);
      if (ok && n_max > 0) {
        tc_fence_after();
        for (int t = 0; t < 2; ++t) if (n_blk[t] > 0) issue_s(t, 0);
        tc_commit(&k_empty[0]);
      }
      for (int j = 0; j < n_max && ok; ++j) {
        if (!mbar_wait(v_full, j & 1, abort_flag, a.status, 842, j)) { ok = false; break; }
        if (j + 1 < n_max && !mbar_wait(&k_full[(j + 1) & 1], (uint32_t)((j + 1) >> 1) & 1, abort_flag, a.status, 843, j)) { ok = false; break; }
        for (int t = 0; t < 2 && ok; ++t) {
          if (j >= n_blk[t]) continue;
          if (!mbar_wait(&p_ready[t], j & 1, abort_flag, a.status, 844, j)) { ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int ks = 0; ks < 8; ++ks)
            mma_f16_ts(tmem + 256 + 128 * t, tmem + 128 * t + ks * 8, sdesc_at(d_v, ks * 2048), id_o, (j > 0 || ks > 0) ? 1u : 0u);
          if (j + 1 < n_blk[t]) issue_s(t, j + 1);          // in order behind the product that reads P from the same columns
          else tc_commit(&o_ready[t]);
        }
        if (!ok) break;
        tc_commit(v_empty);
        if (j + 1 < n_max) tc_commit(&k_empty[(j + 1) & 1]);
      }
    }
  } else {
    const int t = (warp - 2) >> 2, q = warp & 3, r = q * 32 + lane;       // tile, row
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    const uint32_t s_t = tmem + 128 * t + lane_off, o_t = tmem + 256 + 128 * t + lane_off;
    const int nt = t == 0 ? n_tok[0] : n_tok[1], nb = t == 0 ? n_blk[0] : n_blk[1];
    const int qpos = (t == 0 ? pos0[0] : pos0[1]) + min(r, max(nt - 1, 0));
    constexpr float kTau = 8.0f;
    const int o_chunks = v2 ? 4 : 2;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nb; ++j) {
      if (!warp_wait(&s_full[t], j & 1, abort_flag, a.status, 850, j)) { ok = false; break; }
      tc_fence_after();
      const int kv0 = j * 128;
      const bool edge = kv0 + 127 > qpos;
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float sv[32];
        tmem_ld_x32(s_t + c * 32, reinterpret_cast<uint32_t*>(sv));
        tc_wait_ld();
        if (edge) {
#pragma unroll
          for (int i = 0; i < 32; ++i) if (kv0 + c * 32 + i > qpos) sv[i] = -INFINITY;
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) mx = fmaxf(mx, sv[i]);
      }
      float alpha = 1.0f;
      const bool grow = mx > m + kTau || (m == -INFINITY && mx > -INFINITY);
      if (grow) { alpha = fast_exp2(m - mx); m = mx; }
      const float m_use = m == -INFINITY ? 0.f : m;
      if (j > 0 && __any_sync(0xffffffffu, grow)) {        // O holds every product up to block j - 1 (see s_full)
        for (int c = 0; c < o_chunks; ++c) {
          uint32_t o[32];
          tmem_ld_x32(o_t + c * 32, o);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
          tmem_st_x32(o_t + c * 32, o);
        }
      }
      float rs = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float sv[32];
        tmem_ld_x32(s_t + c * 32, reinterpret_cast<uint32_t*>(sv));
        tc_wait_ld();
        if (edge) {
#pragma unroll
          for (int i = 0; i < 32; ++i) if (kv0 + c * 32 + i > qpos) sv[i] = -INFINITY;
        }
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float p0 = fast_exp2(sv[2 * i] - m_use), p1 = fast_exp2(sv[2 * i + 1] - m_use);
          rs += p0 + p1;
          pk[i] = pack_bf16x2(p0, p1);
        }
        tmem_st_x16(s_t + c * 16, pk);
      }
      l = l * alpha + rs;
      tc_wait_st();
      tc_fence_before();
      mbar_arrive(&p_ready[t]);
    }
    if (ok && nb > 0) ok = warp_wait(&o_ready[t], 0, abort_flag, a.status, 851, 0);
    if (ok && nb > 0) {
      tc_fence_after();
      if (a.sink != nullptr) l += fast_exp2(a.sink[h] - m);
      const float inv = l > 0.f ? 1.0f / l : 0.f;
      __nv_bfloat16* dst = r < nt ? a.out + ((size_t)a.tok[qb + x0 + 128 * t + r] * a.heads + h) * a.dv : nullptr;
      for (int c = 0; c < o_chunks; ++c) {
        uint32_t o[32];
        tmem_ld_x32(o_t + c * 32, o);
        tc_wait_ld();
        if (dst != nullptr) {
#pragma unroll
          for (int v = 0; v < 4; ++v) {
            if (c * 32 + v * 8 >= a.dv) continue;
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(o[v * 8 + 0]) * inv, __uint_as_float(o[v * 8 + 1]) * inv);
            w.y = pack_bf16x2(__uint_as_float(o[v * 8 + 2]) * inv, __uint_as_float(o[v * 8 + 3]) * inv);
            w.z = pack_bf16x2(__uint_as_float(o[v * 8 + 4]) * inv, __uint_as_float(o[v * 8 + 5]) * inv);
            w.w = pack_bf16x2(__uint_as_float(o[v * 8 + 6]) * inv, __uint_as_float(o[v * 8 + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + v * 8) = w;
          }
        }
      }
    }
  }

  pdl_trigger();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem, 512); }
}

// Shared memory of the decode kernel with `boxes` boxes per block and `stages` blocks.
static int latent_decode_smem(int boxes, int stages, int nh) {
  return boxes * stages * kLdBox + ((boxes > 4 ? boxes : 4) + 4) * nh * 128 + (7 + 2 * kLdMaxPairs) * 8 + 32 + 8 * nh * 4 + 1024;
}

struct LatentDecodeShape { int nh, boxes, stages; };

// nh = 0: sizes the kernel is not built for.
static LatentDecodeShape latent_decode_shape(int heads, int width, int rank) {
  LatentDecodeShape s = {heads <= 16 ? 16 : 32, (width + 63) / 64, 4};
  auto fits = [&]() { return (s.boxes + 1) / 2 * s.stages <= kLdMaxPairs && latent_decode_smem(s.boxes, s.stages, s.nh) <= 227 * 1024; };
  while (s.stages > 1 && !fits()) --s.stages;
  if (!fits() || ((rank + 127) / 128 + 2) * s.nh > 256) s.nh = 0;
  return s;
}

}  // namespace gb

using namespace gb;

// Whether gb_latent_decode takes these sizes; heads per CTA (0 = no).
GB_API int gb_latent_decode_heads(int heads, int width, int rank, int page_size) {
  if (heads < 1 || width < 1 || rank < 1 || rank > width || page_size < 8 || page_size % 8 || 128 % page_size) return 0;
  return latent_decode_shape(heads, width, rank).nh;
}

// q bf16 [heads][m_rows][ld_c], cache bf16 [num_slots][ld_c], out bf16 [heads][m_rows][ld_out]; see LatentDecodeArgs.
GB_API int gb_latent_decode(const void* q, const void* cache, int ld_c, long num_slots, const int* tok_seq, const int* tok_kv, const int* kv_len, const int* block_table,
                            int max_pages, int page_size, int tokens, int heads, int width, int rank, int splits, void* out, int m_rows, int ld_out, float* part_o,
                            float* part_lse, const float* sink, void* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (gb_latent_decode_heads(heads, width, rank, page_size) == 0) return fail("latent_decode: unsupported sizes%s");
  if (ld_c % 8 || ld_c < width || ld_out < rank || m_rows < tokens || ((uintptr_t)q & 15) || ((uintptr_t)cache & 15)) return fail("latent_decode: bad rows%s");
  if (splits < 1 || splits > kLdMaxSplits || (splits > 1 && (part_o == nullptr || part_lse == nullptr))) return fail("latent_decode: bad splits%s");
  if ((tok_seq == nullptr) != (tok_kv == nullptr)) return fail("latent_decode: tok_seq and tok_kv come together%s");
  const LatentDecodeShape sh = latent_decode_shape(heads, width, rank);
  CUtensorMap tmQ, tmC;
  uint64_t dq[3] = {(uint64_t)ld_c, (uint64_t)m_rows, (uint64_t)heads}, sq[2] = {(uint64_t)ld_c * 2, (uint64_t)m_rows * ld_c * 2};
  uint32_t bq[3] = {64, 1, (uint32_t)sh.nh};
  if (make_tmap(&tmQ, q, TM_BF16, 3, dq, sq, bq, TM_SW_128)) return -1;
  if (make_tmap_2d(&tmC, cache, TM_BF16, (uint64_t)ld_c, (uint64_t)num_slots, (uint64_t)ld_c * 2, 64, (uint32_t)(page_size < kLdB ? page_size : kLdB), TM_SW_128)) return -1;
  LatentDecodeArgs a;
  a.tok_seq = tok_seq; a.tok_kv = tok_kv; a.kv_len = kv_len; a.block_table = block_table; a.max_pages = max_pages; a.page_size = page_size; a.tokens = tokens;
  a.heads = heads; a.head_tiles = (heads + sh.nh - 1) / sh.nh; a.splits = splits; a.width = width; a.rank = rank; a.boxes = sh.boxes; a.stages = sh.stages;
  a.out = (__nv_bfloat16*)out; a.m_rows = m_rows; a.ld_out = ld_out; a.part_o = part_o; a.part_lse = part_lse; a.sink = sink; a.status = (KernelStatus*)status;
  const int smem = latent_decode_smem(sh.boxes, sh.stages, sh.nh);
  static bool attr_set = false;
  if (!attr_set) {
    GB_CUDA_OK(cudaFuncSetAttribute(latent_decode_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    GB_CUDA_OK(cudaFuncSetAttribute(latent_decode_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    attr_set = true;
  }
  const unsigned grid = (unsigned)((long)tokens * a.head_tiles * splits);
  if (sh.nh == 16) launch_k(latent_decode_kernel<16>, grid, kLdThreads, smem, stream, tmQ, tmC, a);
  else launch_k(latent_decode_kernel<32>, grid, kLdThreads, smem, stream, tmQ, tmC, a);
  GB_CUDA_OK(cudaGetLastError());
  if (splits > 1) {
    launch_k(latent_combine_kernel, dim3((unsigned)((long)tokens * heads), (unsigned)((rank + 127) / 128)), 128, 0, stream, (const float*)part_o, (const float*)part_lse, sink, (__nv_bfloat16*)out, splits, tokens,
             heads, rank, m_rows, ld_out);
    GB_CUDA_OK(cudaGetLastError());
  }
  return 0;
}

// q_n bf16 [n_q][heads][dn], q_r [n_q][heads][dr]; k_n and v: columns [heads x dn] and [heads x dv] of rows of pitch ld_kv; k_r: dr columns of rows of
// pitch ld_r; n_kv key rows.  out bf16 [T][heads][dv].  See LatentPrefillArgs.
GB_API int gb_latent_prefill(const void* q_n, const void* q_r, const void* k_n, const void* k_r, const void* v, int ld_kv, int ld_r, int n_q, int n_kv, const int* tiles,
                             int n_tiles, const int* q0, const int* kv0, const int* tok, void* out, int heads, int dn, int dr, int dv, const float* sink, void* status,
                             cudaStream_t stream) {
  if (n_tiles <= 0) return 0;
  if (heads < 1 || dn < 8 || dn > 128 || dn % 8 || dr < 8 || dr > 64 || dr % 8 || dv < 8 || dv > 128 || dv % 8) return fail("latent_prefill: unsupported head sizes%s");
  if (ld_kv % 8 || ld_r % 8 || ((uintptr_t)q_n & 15) || ((uintptr_t)q_r & 15) || ((uintptr_t)k_n & 15) || ((uintptr_t)k_r & 15) || ((uintptr_t)v & 15) || ((uintptr_t)out & 15))
    return fail("latent_prefill: misaligned rows%s");
  CUtensorMap tmQn, tmQr, tmKn, tmKr, tmV;
  uint32_t box[3] = {64, 1, 128};
  auto map3 = [&](CUtensorMap* m, const void* p, int d, int rows, long pitch) {
    uint64_t dims[3] = {(uint64_t)d, (uint64_t)heads, (uint64_t)rows}, st[2] = {(uint64_t)d * 2, (uint64_t)pitch * 2};
    return make_tmap(m, p, TM_BF16, 3, dims, st, box, TM_SW_128);
  };
  if (map3(&tmQn, q_n, dn, n_q, (long)heads * dn) || map3(&tmQr, q_r, dr, n_q, (long)heads * dr) || map3(&tmKn, k_n, dn, n_kv, ld_kv) || map3(&tmV, v, dv, n_kv, ld_kv)) return -1;
  if (make_tmap_2d(&tmKr, k_r, TM_BF16, (uint64_t)dr, (uint64_t)n_kv, (uint64_t)ld_r * 2, 64, 128, TM_SW_128)) return -1;
  LatentPrefillArgs a;
  a.tiles = tiles; a.n_tiles = n_tiles; a.q0 = q0; a.kv0 = kv0; a.tok = tok; a.out = (__nv_bfloat16*)out; a.heads = heads; a.dn = dn; a.dr = dr; a.dv = dv; a.sink = sink;
  a.status = (KernelStatus*)status;
  static bool attr_set = false;
  if (!attr_set) {
    GB_CUDA_OK(cudaFuncSetAttribute(latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kLpSmem));
    attr_set = true;
  }
  launch_k(latent_prefill_kernel, (unsigned)((long)n_tiles * heads), kLpThreads, kLpSmem, stream, tmQn, tmQr, tmKn, tmKr, tmV, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}
