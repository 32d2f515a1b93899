// Chunked scan of lightning (decayed linear) attention for prefill, on tcgen05 (the token-by-token form is in lightning.cu).
//
// Over a chunk of C = 128 tokens with the state S0 in front of it and the scalar decay g of the head:
//   O_i   = g^(i+1) (q_i S0) + sum_{j <= i} g^(i-j) (q_i . k_j) v_j
//   S_end = g^n S0 + sum_j k_j (g^(n-1-j) v_j)^T                       (n tokens in the chunk)
// One CTA walks the chunks of one (sequence, head, slice of 64 value columns).  Q, K, V are bf16 rows of the mixer's input projection
// with the activation applied (the projection's GEMM does it), fetched by TMA; the state is f32 in registers, one key row per thread.
//   TMA warp    : Q, K, V of chunk j + 1 land while chunk j is computed
//   MMA thread  : S1 = Q K^T;  dS = K^T (w V);  O1 = Q S;  O2 = P V         (A of O2 is P in TMEM; S and w V are written to smem)
//   P warps     : S1 row -> times g^(i-j), lower triangle -> P in TMEM;  g^(i+1) O1 + O2 -> global f32 (TMA)
//   state warps : V -> w V in smem;  S <- g^n S + dS;  S -> smem for the next chunk's O1
// The SSD form (Mamba-2) is the same scan with a decay per token: with L_i the sum of a dt log2(e) up to token i, g^(i-j) becomes
// 2^(L_i - L_j) dt_j (one exponential of L_i - (L_j - log2 dt_j)), w of a token 2^(L_(n-1) - L_j) dt_j, and D x_i joins P's diagonal.  q and k are C
// and B of the head's group.  Every warp of the two groups sums the chunk's step sizes itself, so they need no exchange.
// Every f32 factor that goes through the tensor cores (P, w V, S) is the sum of two bf16 operands (hi + lo, 16 bits of mantissa), so
// decays and state keep 32-bit accuracy; only q, k and v themselves are bf16.
#include "sm100.cuh"
#include "host_common.h"
#include "recurrent.cuh"

namespace gb {

constexpr int kLcC = 128;                  // tokens per chunk
constexpr int kLcV = 64;                   // value columns per CTA
constexpr int kLcThreads = 320;            // TMA warp, MMA warp, 4 P warps, 4 state warps
constexpr int kLcQ = 32768, kLcVt = 16384; // bytes of a Q / K tile (two halves of 64 columns), of a tile of 64 columns
constexpr int kLcStage = 2 * kLcQ + kLcVt;
constexpr int kLcSmem = 2 * kLcStage + 4 * kLcVt + 256 + 257 * 4 + 1024;

struct LightningChunkArgs {
  const float* decay;           // [heads]
  float* state;                 // [slots, heads, dim, vdim]
  int n_slots;
  const int* cu_q; const int* seq_slots;
  float* out; int ld_out;       // [tokens, heads * vdim] f32
  int heads, dim, vdim;
  KernelStatus* status;
  // SSD
  const float* gate; int g_part; long g_stride; int g_ld;       // step sizes before bias and softplus, [g_part][tokens, g_ld], column = head
  const float* gate_bias; const float* d_skip; int groups;      // `decay` holds a (negative)
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Step sizes of a chunk, of token 32 b + lane for b = 0 .. 3, before bias and softplus.
__device__ __forceinline__ void ssd_load(const LightningChunkArgs& a, int t0, int n, int h, int lane, float* raw) {
#pragma unroll
  for (int b = 0; b < 4; ++b) {
    raw[b] = 0.f;
    if (32 * b + lane < n) {
      const float* p = a.gate + (size_t)(t0 + 32 * b + lane) * a.g_ld + h;
      for (int i = 0; i < a.g_part; ++i) raw[b] += p[(size_t)i * a.g_stride];
    }
  }
}

// Of the logarithmic decays (base 2): the sum L over block q of 32 tokens up to token 32 q + lane, the sums S of the four blocks, and the token's step
// size.  Sums that go on over the whole chunk would lose the small decays between neighbours behind large ones; so a pair in one block takes the
// difference of its L, and only pairs further apart add block sums.
__device__ __forceinline__ void ssd_scan(const float* raw, int n, float bias, float a2, int q, int lane, float& L, float& dt, float* S) {
  float own = 0.f;
  dt = 0.f;
#pragma unroll
  for (int b = 0; b < 4; ++b) {
    const float d = 32 * b + lane < n ? softplus_exact(raw[b] + bias) : 0.f;
    const float l = a2 * d;
    if (b == q) { dt = d; own = l; }
    S[b] = warp_sum(l);
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, own, o); if (lane >= o) own += v; }
  L = own;
}

template <int DP, bool SSD>                // DP: key size padded, 64 or 128
__global__ void __launch_bounds__(kLcThreads, 1)
lightning_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                       const __grid_constant__ CUtensorMap tmO, const LightningChunkArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);      // an offset, so that accesses stay shared-memory ones
  // stage b at b * kLcStage: Q, K, V
  uint8_t* sWV = smem + 2 * kLcStage;                       // hi, lo
  uint8_t* sS = sWV + 2 * kLcVt;                            // hi, lo
  uint64_t* bars = (uint64_t*)(sS + 2 * kLcVt);
  uint64_t* qk_full = bars;          // 2
  uint64_t* v_full = bars + 2;       // 2
  uint64_t* t_empty = bars + 4;      // 2: the chunk's last MMA, and the output tile (staged over Q) has been read
  uint64_t* s1_full = bars + 6;
  uint64_t* p_ready = bars + 7;      // 128 arrivals
  uint64_t* wv_ready = bars + 8;     // 128
  uint64_t* s_ready = bars + 9;      // 128
  uint64_t* ds_full = bars + 10;
  uint64_t* o_full = bars + 11;
  uint64_t* o_free = bars + 12;      // 128
  uint64_t* o1_done = bars + 13;
  uint32_t* tmem_slot = (uint32_t*)(bars + 14);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
  float* pz = (float*)(bars + 32);                          // 128 zeros, then g^0 .. g^128

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) { mbar_init(&qk_full[i], 1); mbar_init(&v_full[i], 1); mbar_init(&t_empty[i], 2); }
    mbar_init(s1_full, 1); mbar_init(p_ready, 128); mbar_init(wv_ready, 128); mbar_init(s_ready, 128); mbar_init(ds_full, 1); mbar_init(o_full, 1); mbar_init(o_free, 128); mbar_init(o1_done, 1);
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV); tma_prefetch_desc(&tmO);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  pdl_wait();
  const int h = blockIdx.x, e0 = blockIdx.y * kLcV, seq = blockIdx.z;
  const float g = a.decay[h];
  if constexpr (!SSD) { for (int i = threadIdx.x; i < 257; i += kLcThreads) pz[i] = i < 128 ? 0.f : i == 128 ? 1.f : powf(g, (float)(i - 128)); }
  const int hk = SSD ? h / (a.heads / a.groups) : h;            // head of q and k
  const float a2 = SSD ? g * 1.4426950408889634f : 0.f, dt_bias = SSD ? a.gate_bias[h] : 0.f;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t t_s1 = tmem_base, t_o1 = tmem_base + 128, t_o2 = tmem_base + 192, t_ds = tmem_base + 256, t_plo = tmem_base + 320;

  const int t_begin = a.cu_q[seq], t_end = a.cu_q[seq + 1], slot = a.seq_slots[seq];
  const bool run = t_end > t_begin && slot >= 0 && slot < a.n_slots;
  const int n_chunks = run ? (t_end - t_begin + kLcC - 1) / kLcC : 0;

  if (warp == 0) {
    if (lane == 0) {
      for (int j = 0; j < n_chunks; ++j) {
        const int b = j & 1, t0 = t_begin + j * kLcC;
        uint8_t* st = smem + b * kLcStage;
        if (!mbar_wait(&t_empty[b], ((uint32_t)(j >> 1) & 1) ^ 1, abort_flag, a.status, 700, j)) break;
        mbar_expect_tx(&qk_full[b], 4u * kLcC * DP);
        tma_load_3d(st, &tmQ, &qk_full[b], 0, hk, t0);
        tma_load_3d(st + kLcQ, &tmK, &qk_full[b], 0, hk, t0);
        if constexpr (DP > 64) {
          tma_load_3d(st + 16384, &tmQ, &qk_full[b], 64, hk, t0);
          tma_load_3d(st + kLcQ + 16384, &tmK, &qk_full[b], 64, hk, t0);
        }
        mbar_expect_tx(&v_full[b], 2u * kLcC * kLcV);
        tma_load_3d(st + 2 * kLcQ, &tmV, &v_full[b], e0, h, t0);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t id_s1 = make_idesc(128, 128, 1, 1, 0, 0);
      constexpr uint32_t id_ds = make_idesc(128, kLcV, 1, 1, 1, 1);       // K^T and w V, both stored token by token
      constexpr uint32_t id_o = make_idesc(128, kLcV, 1, 1, 0, 1);        // S and V stored row by row of the inner index
      const uint32_t wv = smem_u32(sWV), sst = smem_u32(sS);
      for (int j = 0; j < n_chunks; ++j) {
        const int b = j & 1;
        const uint32_t ph = j & 1, ph2 = (uint32_t)(j >> 1) & 1;
        const uint32_t q_addr = smem_u32(smem + b * kLcStage), k_addr = q_addr + kLcQ, v_addr = k_addr + kLcQ;
        if (!mbar_wait(&qk_full[b], ph2, abort_flag, a.status, 710, j)) break;
        tc_fence_after();
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
          const uint32_t off = (ks >> 2) * 16384 + (ks & 3) * 32;
          mma_f16_ss(t_s1, make_sdesc_sw128(q_addr + off), make_sdesc_sw128(k_addr + off), id_s1, ks > 0 ? 1u : 0u);
        }
        tc_commit(s1_full);
        // DP = 64: rows 64 .. 127 of dS are products of whatever the second half of the K tile holds; nobody reads them
        if (!mbar_wait(wv_ready, ph, abort_flag, a.status, 711, j)) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int ks = 0; ks < 8; ++ks)
            mma_f16_ss(t_ds, make_sdesc_sw128_mn(k_addr + ks * 2048, 16384), make_sdesc_sw128_mn(wv + part * kLcVt + ks * 2048, 16384), id_ds,
                       (part > 0 || ks > 0) ? 1u : 0u);
        tc_commit(ds_full);
        if (!mbar_wait(s_ready, ph, abort_flag, a.status, 712, j)) break;
        if (j > 0 && !mbar_wait(o_free, ph ^ 1, abort_flag, a.status, 715, j)) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int ks = 0; ks < DP / 16; ++ks)
            mma_f16_ss(t_o1, make_sdesc_sw128(q_addr + (ks >> 2) * 16384 + (ks & 3) * 32), make_sdesc_sw128_mn(sst + part * kLcVt + ks * 2048, 16384), id_o,
                       (part > 0 || ks > 0) ? 1u : 0u);
        tc_commit(o1_done);
        if (!mbar_wait(p_ready, ph, abort_flag, a.status, 713, j)) break;
        if (!mbar_wait(&v_full[b], ph2, abort_flag, a.status, 714, j)) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int ks = 0; ks < 8; ++ks)
            mma_f16_ts(t_o2, (part ? t_plo : t_s1) + ks * 8, make_sdesc_sw128_mn(v_addr + ks * 2048, 16384), id_o, (part > 0 || ks > 0) ? 1u : 0u);
        tc_commit(o_full);
        tc_commit(&t_empty[b]);
      }
    }
  } else if (warp < 6) {
    // ---------------------------------------------------------------- P and output: thread = token row i of the chunk
    const int q = warp & 3, i = q * 32 + lane;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    const float* pw = pz + 128;
    float gi = SSD ? 0.f : pw[i + 1];
    const float skip = SSD ? a.d_skip[h] : 0.f;
    float raw[4];
    if (SSD && n_chunks > 0) ssd_load(a, t_begin, min(kLcC, t_end - t_begin), h, lane, raw);
    bool staged = false;                    // the output tile of the previous chunk is on its way out of stage (j - 1) & 1
    for (int j = 0; j < n_chunks; ++j) {
      const uint32_t ph = j & 1;
      const int b = j & 1, t0 = t_begin + j * kLcC;
      float Li = 0.f, S[4] = {0.f, 0.f, 0.f, 0.f};
      if constexpr (SSD) {
        float dt;
        ssd_scan(raw, min(kLcC, t_end - t0), dt_bias, a2, q, lane, Li, dt, S);
        pz[i] = Li - log2f(dt);             // (read by everyone below; the barrier at the end of the chunk lets the next one overwrite it)
        gi = Li;
#pragma unroll
        for (int c = 2; c >= 0; --c) if (c < q) gi += S[c];
        gi = ex2(gi);
        if (j + 1 < n_chunks) ssd_load(a, t0 + kLcC, min(kLcC, t_end - t0 - kLcC), h, lane, raw);
        bar128_and(true);
      }
      bool ok = warp_wait(s1_full, ph, abort_flag, a.status, 720, j);
      tc_fence_after();
      if (ok) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t hi[16], lo[16];
          if (c <= q) {                     // columns up to the warp's own rows; the rest of P is zero
            float s[32];
            tmem_ld_x32(t_s1 + lane_off + c * 32, reinterpret_cast<uint32_t*>(s));
            float w[32];                    // zero above the diagonal
#pragma unroll
            for (int x = 0; x < 32; ++x) {
              if constexpr (SSD) w[x] = pz[c * 32 + x];
              else { w[x] = (pw + (i - c * 32))[-x]; asm volatile("" : "+f"(w[x])); }
            }
            if constexpr (SSD) {
              float L = Li;                     // to the start of block c (its own sums count from there)
#pragma unroll
              for (int y = 2; y >= 0; --y) if (y < q && y >= c) L += S[y];
#pragma unroll
              for (int x = 0; x < 32; ++x) w[x] = ex2(L - w[x]);        // above the diagonal anything, cleared below
            }
            tc_wait_ld();
#pragma unroll
            for (int x = 0; x < 32; ++x) s[x] *= w[x];
            if (c == q) {
#pragma unroll
              for (int x = 0; x < 32; ++x) s[x] = x < lane ? s[x] : x == lane ? (SSD ? s[x] + skip : s[x]) : 0.f;
            }
#pragma unroll
            for (int x = 0; x < 16; ++x) split_bf16x2(s[2 * x], s[2 * x + 1], hi[x], lo[x]);
          } else {
#pragma unroll
            for (int x = 0; x < 16; ++x) hi[x] = lo[x] = 0u;
          }
          tmem_st_x16(t_s1 + lane_off + c * 16, hi);        // over columns that are already read
          tmem_st_x16(t_plo + lane_off + c * 16, lo);
        }
        tc_wait_st();
        tc_fence_before();
        mbar_arrive(p_ready);
      }
      if (staged && threadIdx.x == 64) { tma_store_wait_read(); mbar_arrive(&t_empty[b ^ 1]); }
      if (ok) ok = warp_wait(o_full, ph, abort_flag, a.status, 721, j);
      tc_fence_after();
      const bool full = t0 + kLcC <= t_end;         // a whole tile leaves through shared memory (over the chunk's Q) and TMA
      uint8_t* so = smem + b * kLcStage;
      if (ok) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          float o1[32], o2[32];
          tmem_ld_x32(t_o1 + lane_off + c * 32, reinterpret_cast<uint32_t*>(o1));
          tmem_ld_x32(t_o2 + lane_off + c * 32, reinterpret_cast<uint32_t*>(o2));
          tc_wait_ld();
          float* dst = a.out + (size_t)(t0 + i) * a.ld_out + (size_t)h * a.vdim + e0 + c * 32;
#pragma unroll
          for (int x = 0; x < 8; ++x) {
            const float4 v = make_float4(fmaf(gi, o1[4 * x], o2[4 * x]), fmaf(gi, o1[4 * x + 1], o2[4 * x + 1]), fmaf(gi, o1[4 * x + 2], o2[4 * x + 2]),
                                         fmaf(gi, o1[4 * x + 3], o2[4 * x + 3]));
            if (full) *reinterpret_cast<float4*>(so + c * 16384 + i * 128 + ((x ^ (i & 7)) << 4)) = v;
            else if (t0 + i < t_end && e0 + c * 32 + x * 4 < a.vdim) *reinterpret_cast<float4*>(dst + x * 4) = v;
          }
        }
        tc_fence_before();
        mbar_arrive(o_free);
        fence_proxy_async_smem();
      }
      if (!bar128_and(ok)) break;
      staged = full;
      if (full && threadIdx.x == 64) {
        tma_store_3d(&tmO, so, e0, h, t0);
        if (e0 + 32 < a.vdim) tma_store_3d(&tmO, so + 16384, e0 + 32, h, t0);
        tma_store_commit();
      }
    }
    if (threadIdx.x == 64) tma_store_wait_read();
  } else {
    // ---------------------------------------------------------------- state: thread = key row d; for w V: thread = token row
    const int q = warp & 3, d = q * 32 + lane;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    const float* pw = pz + 128;
    const bool row = d < a.dim;
    float* st = a.state + (((size_t)(run ? slot : 0) * a.heads + h) * a.dim + (row ? d : 0)) * a.vdim + e0;
    float S[kLcV];
#pragma unroll
    for (int x = 0; x < kLcV / 4; ++x) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (run && row && e0 + 4 * x < a.vdim) v = *reinterpret_cast<const float4*>(st + 4 * x);
      S[4 * x] = v.x; S[4 * x + 1] = v.y; S[4 * x + 2] = v.z; S[4 * x + 3] = v.w;
    }
    auto publish = [&]() {                  // S -> smem rows [d][64], 128-byte swizzle, hi and lo
      if (d < DP) {
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          uint4 hi, lo;
          split_bf16x2(S[8 * c], S[8 * c + 1], hi.x, lo.x); split_bf16x2(S[8 * c + 2], S[8 * c + 3], hi.y, lo.y);
          split_bf16x2(S[8 * c + 4], S[8 * c + 5], hi.z, lo.z); split_bf16x2(S[8 * c + 6], S[8 * c + 7], hi.w, lo.w);
          const int off = d * 128 + ((c ^ (d & 7)) << 4);
          *reinterpret_cast<uint4*>(sS + off) = hi;
          *reinterpret_cast<uint4*>(sS + kLcVt + off) = lo;
        }
      }
      fence_proxy_async_smem();
      mbar_arrive(s_ready);
    };
    bool ok = true;
    float raw[4];
    if (SSD && n_chunks > 0) ssd_load(a, t_begin, min(kLcC, t_end - t_begin), h, lane, raw);
    if (n_chunks > 0) publish();
    for (int j = 0; j < n_chunks; ++j) {
      const uint32_t ph = j & 1;
      const int b = j & 1, n = min(kLcC, t_end - (t_begin + j * kLcC));
      float after = 0.f, dt = 0.f, total = 0.f;
      if constexpr (SSD) {
        float L, B[4];
        ssd_scan(raw, n, dt_bias, a2, q, lane, L, dt, B);
        total = ((B[0] + B[1]) + B[2]) + B[3];
#pragma unroll
        for (int c = 0; c < 4; ++c) if (c == q) after = B[c] - L;
#pragma unroll
        for (int c = 1; c < 4; ++c) if (c > q) after += B[c];
        if (j + 1 < n_chunks) ssd_load(a, t_begin + (j + 1) * kLcC, min(kLcC, t_end - t_begin - (j + 1) * kLcC), h, lane, raw);
      }
      // w V: a token's values times what its contribution still decays by until the end of the chunk
      if (!warp_wait(&v_full[b], (uint32_t)(j >> 1) & 1, abort_flag, a.status, 730, j)) { ok = false; break; }
      {
        const uint8_t* sV = smem + b * kLcStage + 2 * kLcQ;
        const bool live = d < n;
        const float w = !live ? 0.f : SSD ? ex2(after) * dt : pw[n - 1 - d];
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const int off = d * 128 + ((c ^ (d & 7)) << 4);
          uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
          if (live) {
            const uint4 v = *reinterpret_cast<const uint4*>(sV + off);
            const __nv_bfloat162* vb = reinterpret_cast<const __nv_bfloat162*>(&v);
            uint32_t* hp = &hi.x; uint32_t* lp = &lo.x;
#pragma unroll
            for (int x = 0; x < 4; ++x) { const float2 f = __bfloat1622float2(vb[x]); split_bf16x2(f.x * w, f.y * w, hp[x], lp[x]); }
          }
          *reinterpret_cast<uint4*>(sWV + off) = hi;
          *reinterpret_cast<uint4*>(sWV + kLcVt + off) = lo;
        }
        fence_proxy_async_smem();
        mbar_arrive(wv_ready);
      }
      if (!warp_wait(ds_full, ph, abort_flag, a.status, 731, j)) { ok = false; break; }
      tc_fence_after();
      const float gn = SSD ? ex2(total) : pw[n];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float x[32];
        tmem_ld_x32(t_ds + lane_off + c * 32, reinterpret_cast<uint32_t*>(x));
        tc_wait_ld();
#pragma unroll
        for (int y = 0; y < 32; ++y) S[c * 32 + y] = row ? fmaf(gn, S[c * 32 + y], x[y]) : 0.f;
      }
      tc_fence_before();
      if (j + 1 < n_chunks) {
        // the chunk's O1 has read the state in shared memory
        if (!warp_wait(o1_done, ph, abort_flag, a.status, 732, j)) { ok = false; break; }
        publish();
      }
    }
    if (ok && run && row) {
#pragma unroll
      for (int x = 0; x < kLcV / 4; ++x)
        if (e0 + 4 * x < a.vdim) *reinterpret_cast<float4*>(st + 4 * x) = make_float4(S[4 * x], S[4 * x + 1], S[4 * x + 2], S[4 * x + 3]);
    }
  }

  pdl_trigger();
  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, 512); }
}

template <int DP, bool SSD>
static int lightning_chunk_launch(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV, const CUtensorMap& tmO, const LightningChunkArgs& a, int n_seqs,
                                  cudaStream_t stream) {
  static bool attr_set = false;
  if (!attr_set) {
    GB_CUDA_OK(cudaFuncSetAttribute(lightning_chunk_kernel<DP, SSD>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLcSmem));
    attr_set = true;
  }
  const dim3 grid((unsigned)a.heads, (unsigned)((a.vdim + kLcV - 1) / kLcV), (unsigned)n_seqs);
  launch_k(lightning_chunk_kernel<DP, SSD>, grid, kLcThreads, kLcSmem, stream, tmQ, tmK, tmV, tmO, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

// Tensor maps and launch: q, k [tokens, qk_heads, dim] and v [tokens, heads, vdim] inside bf16 rows of pitch ld.
template <bool SSD>
static int chunk_launch(const void* q, const void* k, const void* v, int ld, int tokens, int qk_heads, LightningChunkArgs& a, int n_seqs, cudaStream_t stream) {
  if (a.heads < 1 || a.dim < 8 || a.dim > 128 || a.dim % 8 || a.vdim < 8 || a.vdim % 8) return fail("lightning_chunk: dim <= 128, dim and vdim multiples of 8%s");
  if (ld % 8 || a.ld_out < a.heads * a.vdim || a.ld_out % 4) return fail("lightning_chunk: bad row pitch%s");
  if (((uintptr_t)q & 15) || ((uintptr_t)k & 15) || ((uintptr_t)v & 15) || ((uintptr_t)a.state & 15) || ((uintptr_t)a.out & 15)) return fail("lightning_chunk: misaligned rows%s");
  if (n_seqs > 65535 || (a.vdim + kLcV - 1) / kLcV > 65535) return fail("lightning_chunk: too many sequences%s");
  const int dim = a.dim, vdim = a.vdim;
  CUtensorMap tmQ, tmK, tmV, tmO;
  uint32_t box[3] = {64, 1, (uint32_t)kLcC};
  uint64_t dk[3] = {(uint64_t)dim, (uint64_t)qk_heads, (uint64_t)tokens}, dv[3] = {(uint64_t)vdim, (uint64_t)a.heads, (uint64_t)tokens};
  uint64_t sk[2] = {(uint64_t)dim * 2, (uint64_t)ld * 2}, sv[2] = {(uint64_t)vdim * 2, (uint64_t)ld * 2};
  if (make_tmap(&tmQ, q, TM_BF16, 3, dk, sk, box, TM_SW_128)) return -1;
  if (make_tmap(&tmK, k, TM_BF16, 3, dk, sk, box, TM_SW_128)) return -1;
  if (make_tmap(&tmV, v, TM_BF16, 3, dv, sv, box, TM_SW_128)) return -1;
  uint32_t obox[3] = {32, 1, (uint32_t)kLcC};
  uint64_t so[2] = {(uint64_t)vdim * 4, (uint64_t)a.ld_out * 4};
  if (make_tmap(&tmO, a.out, TM_F32, 3, dv, so, obox, TM_SW_128)) return -1;
  return dim <= 64 ? lightning_chunk_launch<64, SSD>(tmQ, tmK, tmV, tmO, a, n_seqs, stream) : lightning_chunk_launch<128, SSD>(tmQ, tmK, tmV, tmO, a, n_seqs, stream);
}

// proj: bf16 rows [tokens, ld] with columns [q heads x dim | k heads x dim | v heads x vdim | ...], SiLU applied; dim <= 128, dim and vdim
// multiples of 8.  state and out as in gb_lightning_step.
GB_API int gb_lightning_chunk(const void* proj, int ld, int tokens, const float* decay, float* state, int n_slots, const int* cu_q, const int* seq_slots,
                              float* out, int ld_out, int heads, int dim, int vdim, int n_seqs, void* status, cudaStream_t stream) {
  if (n_seqs <= 0 || tokens <= 0) return 0;
  if (ld < 2 * heads * dim + heads * vdim) return fail("lightning_chunk: bad row pitch%s");
  const __nv_bfloat16* p = (const __nv_bfloat16*)proj;
  LightningChunkArgs a;
  memset(&a, 0, sizeof(a));
  a.decay = decay; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out;
  a.heads = heads; a.dim = dim; a.vdim = vdim; a.status = (KernelStatus*)status;
  return chunk_launch<false>(p, p + (size_t)heads * dim, p + (size_t)2 * heads * dim, ld, tokens, heads, a, n_seqs, stream);
}

// xbc: bf16 rows [tokens, ld] with columns [x heads x vdim | B groups x dim | C groups x dim | ...]; the other arguments as in gb_recurrent_step.
GB_API int gb_ssd_chunk(const void* xbc, int ld, int tokens, const float* gate, int g_part, long g_stride, int g_ld, const float* gate_bias, const float* par,
                        const float* d_skip, float* state, int n_slots, const int* cu_q, const int* seq_slots, float* out, int ld_out, int heads, int groups, int dim,
                        int vdim, int n_seqs, void* status, cudaStream_t stream) {
  if (n_seqs <= 0 || tokens <= 0) return 0;
  if (groups < 1 || heads % groups || g_part < 1 || g_ld < heads || ld < heads * vdim + 2 * groups * dim) return fail("ssd_chunk: bad sizes%s");
  const __nv_bfloat16* p = (const __nv_bfloat16*)xbc;
  LightningChunkArgs a;
  memset(&a, 0, sizeof(a));
  a.decay = par; a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out;
  a.heads = heads; a.dim = dim; a.vdim = vdim; a.status = (KernelStatus*)status;
  a.gate = gate; a.g_part = g_part; a.g_stride = g_stride; a.g_ld = g_ld; a.gate_bias = gate_bias; a.d_skip = d_skip; a.groups = groups;
  const __nv_bfloat16* bm = p + (size_t)heads * vdim;
  return chunk_launch<true>(bm + (size_t)groups * dim, bm, p, ld, tokens, groups, a, n_seqs, stream);
}
