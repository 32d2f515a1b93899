// Prefill scan of linear attention with a decay per key channel (HGRN2, RWKV; the token-by-token forms are in recurrent.cu), in two kernels:
//
//   S_t = diag(f_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t,  k = 1 - f                    (HGRN2)
//   S_t = diag(f_t) S_{t-1} + k_t v_t^T,  o_t = (S_{t-1} + diag(u) k_t v_t^T)^T q_t      (RWKV; f = exp(-exp(z)))
//
// Over a block of 16 tokens with the state S0 in front of it, c_i = f_0 ... f_i, r_j = f_{j+1} ... f_15 and b = c_15 (per channel):
//   O_i   = (q_i c_i) S0 + sum_{j <= i} P_ij v_j,   P_ij = sum_d q_i k_j f_{j+1} ... f_i
//   S_end = diag(b) S0 + sum_j (k_j r_j) v_j^T
// RWKV's output reads the state in front of the token: c_i = f_0 ... f_{i-1}, P_ij = sum_d q_i k_j f_{j+1} ... f_{i-1} for j < i, P_ii = sum_d q_i u k_i.
// All decays are products of gates, never quotients or differences of logarithms, so gates of any size (down to 0) are exact.
//
// gla_prep_kernel, parallel over blocks and heads: gates, q c, k r, P and b.  It writes a record per (block, head) that is the image of the scan's
// operand tiles in shared memory.
// gla_scan_kernel, one CTA per (sequence, head, 128 value columns), walks the blocks.  The transposed state [value columns x channels] is f32 in
// registers and goes to tensor memory as the A operand of the output's product:
//   producer    : records (bulk copies) and V (TMA), several blocks ahead
//   MMA thread  : dS^T = V^T (k r);  O^T = S^T (q c)^T + V^T P^T
//   state warps : S <- S diag(b) + dS;  S -> tensor memory
//   output warps: O^T -> global f32
// Every f32 factor of a product (q c, k r, P, S) is the sum of two bf16 operands (hi + lo, 16 bits of mantissa); q and v themselves are bf16.
#include "sm100.cuh"
#include "host_common.h"
#include "recurrent.cuh"

namespace gb {

constexpr int kGlB = 16;                   // tokens per block

// Layout of a record (bytes), channels padded to DP: q c (DP / 64 tiles of 16 hi rows, then 16 lo rows, of 128 bytes); k r hi, then lo (each DP / 64
// tiles of 16 rows x 128 bytes); P (16 rows x 128 bytes: 16 hi, 16 lo); b (f32).  128-byte swizzle.
template <int DP> struct GlaRecord {
  static constexpr int kTile = DP / 64 * 2048;
  static constexpr int kQ = 0, kK = 2 * kTile, kP = 4 * kTile, kB = kP + 2048, kBytes = kB + DP * 4;
};

// First block of a sequence in the workspace: sequences have ceil(n / 16) blocks each.
__device__ __forceinline__ int gla_first_block(int t0, int seq) { return t0 / kGlB + seq; }

struct GlaArgs {
  const __nv_bfloat16* qv; int ld;           // [tokens, ld]: q heads x dim (HGRN2: SiLU applied)
  const __nv_bfloat16* k;                    // RWKV: [tokens, ld]: k heads x dim
  const float* u;                            // RWKV: [heads x dim]
  const float* gate; int g_part; long g_stride; int g_ld;      // forget gates before bias and sigmoid
  const float* gate_bias; const float* lower;
  float* state; int n_slots;
  const int* cu_q; const int* seq_slots;
  float* out; int ld_out;
  int heads, dim, vdim;
  uint8_t* ws;                               // [blocks][heads] records
  KernelStatus* status;
};

template <int DP, bool RWKV>
__global__ void __launch_bounds__(256)
gla_prep_kernel(const GlaArgs a) {
  using R = GlaRecord<DP>;
  __shared__ __align__(16) float sf[kGlB][DP], sk[kGlB][DP], sq[kGlB][DP];
  __shared__ float part[8][kGlB][kGlB];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int t_begin = a.cu_q[s], t0 = t_begin + blockIdx.x * kGlB, n = min(kGlB, a.cu_q[s + 1] - t0);
  if (n <= 0) return;
  uint8_t* rec = a.ws + ((size_t)(gla_first_block(t_begin, s) + blockIdx.x) * a.heads + h) * R::kBytes;
  for (int x = tid; x < kGlB * DP; x += 256) {
    const int i = x / DP, c = x % DP;
    float f = 1.f, k = 0.f, q = 0.f;
    if (i < n && c < a.dim) {
      const int col = h * a.dim + c;
      const float* g = a.gate + (size_t)(t0 + i) * a.g_ld + col;
      float z = *g;
      for (int p = 1; p < a.g_part; ++p) z += g[(size_t)p * a.g_stride];
      if constexpr (RWKV) {
        f = expf(-expf(z + a.gate_bias[col]));
        k = __bfloat162float(a.k[(size_t)(t0 + i) * a.ld + col]);
      } else f = forget_gate(z + a.gate_bias[col], a.lower[col], k);
      q = __bfloat162float(a.qv[(size_t)(t0 + i) * a.ld + col]);
    }
    sf[i][c] = f; sk[i][c] = k; sq[i][c] = q;
  }
  __syncthreads();
  // running products, two channels per thread: the first DP / 2 threads q c, the next k r and b
  const int role = tid / (DP / 2), c2 = (tid % (DP / 2)) * 2;
  const int tile = (c2 >> 6) * 2048, chunk = (c2 & 63) >> 3, in = (c2 & 7) * 2;
  if (role == 0) {
    float p0 = 1.f, p1 = 1.f;
#pragma unroll
    for (int i = 0; i < kGlB; ++i) {
      const float2 f = *reinterpret_cast<const float2*>(&sf[i][c2]), q = *reinterpret_cast<const float2*>(&sq[i][c2]);
      if constexpr (!RWKV) { p0 *= f.x; p1 *= f.y; }
      uint32_t hi, lo;
      split_bf16x2(q.x * p0, q.y * p1, hi, lo);
      if constexpr (RWKV) { p0 *= f.x; p1 *= f.y; }
      uint8_t* dst = rec + R::kQ + 2 * tile + i * 128 + ((chunk ^ (i & 7)) << 4) + in;
      *reinterpret_cast<uint32_t*>(dst) = hi;
      *reinterpret_cast<uint32_t*>(dst + 2048) = lo;
    }
  } else if (role == 1) {
    float p0 = 1.f, p1 = 1.f;
#pragma unroll
    for (int i = kGlB - 1; i >= 0; --i) {
      const float2 f = *reinterpret_cast<const float2*>(&sf[i][c2]), k = *reinterpret_cast<const float2*>(&sk[i][c2]);
      uint32_t hi, lo;
      split_bf16x2(k.x * p0, k.y * p1, hi, lo);
      uint8_t* dst = rec + R::kK + tile + i * 128 + ((chunk ^ (i & 7)) << 4) + in;
      *reinterpret_cast<uint32_t*>(dst) = hi;
      *reinterpret_cast<uint32_t*>(dst + R::kTile) = lo;
      p0 *= f.x; p1 *= f.y;
    }
    *reinterpret_cast<float2*>(rec + R::kB + c2 * 4) = make_float2(p0, p1);
  }
  // P: a lane follows the decayed key of token j through the block, in CH channels; warps and half-warps share the channels
  {
    constexpr int CH = DP / 16;
    const int warp = tid >> 5, lane = tid & 31, j = lane & 15, c0 = warp * (DP / 8) + (lane >> 4) * CH;
    float w[CH], k[CH], uk[RWKV ? CH : 1], fl[RWKV ? CH : 1];    // fl: the gates of the token in front
#pragma unroll
    for (int x = 0; x < CH; ++x) {
      w[x] = 0.f; k[x] = sk[j][c0 + x];
      if constexpr (RWKV) { uk[x] = c0 + x < a.dim ? k[x] * a.u[h * a.dim + c0 + x] : 0.f; fl[x] = 1.f; }
    }
#pragma unroll
    for (int i = 0; i < kGlB; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int x = 0; x < CH; x += 4) {
        const float4 f = *reinterpret_cast<const float4*>(&sf[i][c0 + x]), q = *reinterpret_cast<const float4*>(&sq[i][c0 + x]);
        const float fv[4] = {f.x, f.y, f.z, f.w}, qv[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
        for (int y = 0; y < 4; ++y) {
          if constexpr (RWKV) {
            w[x + y] = i == j + 1 ? k[x + y] : w[x + y] * fl[x + y];
            fl[x + y] = fv[y];
            acc = fmaf(qv[y], i == j ? uk[x + y] : w[x + y], acc);
          } else {
            w[x + y] = i == j ? k[x + y] : w[x + y] * fv[y];
            acc = fmaf(qv[y], w[x + y], acc);
          }
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 16);
      if (lane < 16) part[warp][i][j] = acc;
    }
  }
  __syncthreads();
  {
    const int i = tid >> 4, j = tid & 15;
    float p = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) p += part[w][i][j];
    const __nv_bfloat16 hi = __float2bfloat16(p), lo = __float2bfloat16(p - __bfloat162float(hi));
    uint8_t* dst = rec + R::kP + i * 128 + (j & 7) * 2;
    *reinterpret_cast<__nv_bfloat16*>(dst + (((j >> 3) ^ (i & 7)) << 4)) = hi;
    *reinterpret_cast<__nv_bfloat16*>(dst + (((2 + (j >> 3)) ^ (i & 7)) << 4)) = lo;
  }
}

constexpr int kGlStages = 8;
template <int DP> constexpr int gla_stage() { return (4096 + GlaRecord<DP>::kBytes + 1023) / 1024 * 1024; }        // V (two tiles), record
template <int DP> constexpr int gla_smem() { return kGlStages * gla_stage<DP>() + 512 + 1024; }
template <int DP> constexpr int gla_threads() { return 32 * (8 + DP / 16); }      // producer, two MMA warps, one idle, 4 output, state warps

template <int DP>
__global__ void __launch_bounds__(32 * (8 + DP / 16), 1)
gla_scan_kernel(const __grid_constant__ CUtensorMap tmV, const GlaArgs a) {
  using R = GlaRecord<DP>;
  constexpr int kStage = gla_stage<DP>(), kStateWarps = DP / 16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  uint64_t* full = (uint64_t*)(smem + kGlStages * kStage);
  uint64_t* empty = full + kGlStages;      // both products, and the state warps (b has been read)
  uint64_t* ds_full = empty + kGlStages;
  uint64_t* ds_free = ds_full + 1;         // state warps
  uint64_t* s_ready = ds_full + 2;         // 2, by block parity; state warps
  uint64_t* o_full = ds_full + 4;          // 2
  uint64_t* o_free = ds_full + 6;          // 2; output warps
  uint32_t* tmem_slot = (uint32_t*)(ds_full + 8);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kGlStages; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 2 + kStateWarps); }
    mbar_init(ds_full, 1); mbar_init(ds_free, kStateWarps);
    for (int i = 0; i < 2; ++i) { mbar_init(&s_ready[i], kStateWarps); mbar_init(&o_full[i], 1); mbar_init(&o_free[i], 4); }
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t t_ds = tmem, t_s = tmem + 128, t_o = tmem + 384;       // dS: DP columns; S: two buffers of (hi 64, lo 64); O: two of 32
  pdl_wait();

  const int h = blockIdx.x, e0 = blockIdx.y * 128, seq = blockIdx.z;
  const int t_begin = a.cu_q[seq], t_end = a.cu_q[seq + 1], slot = a.seq_slots[seq];
  const bool run = t_end > t_begin && slot >= 0 && slot < a.n_slots;
  const int n_blk = run ? (t_end - t_begin + kGlB - 1) / kGlB : 0;

  if (warp == 0) {
    if (lane == 0) {
      const bool two = e0 + 64 < a.vdim;
      const uint8_t* rec = a.ws + ((size_t)gla_first_block(t_begin, seq) * a.heads + h) * R::kBytes;
      for (int b = 0; b < n_blk; ++b) {
        const int st = b % kGlStages;
        uint8_t* p = smem + st * kStage;
        if (!mbar_wait(&empty[st], ((uint32_t)(b / kGlStages) & 1) ^ 1, abort_flag, a.status, 900, b)) break;
        mbar_expect_tx(&full[st], (uint32_t)R::kBytes + (two ? 4096u : 2048u));
        bulk_load(p + 4096, rec + (size_t)b * a.heads * R::kBytes, R::kBytes, &full[st]);
        tma_load_3d(p, &tmV, &full[st], e0, h, t_begin + b * kGlB);
        if (two) tma_load_3d(p + 2048, &tmV, &full[st], e0 + 64, h, t_begin + b * kGlB);
      }
    }
  } else if (warp == 1) {
    // dS is on the chain from block to block, O is not: two threads issue them
    if (lane == 0) {
      constexpr uint32_t id_ds = make_idesc(128, DP, 1, 1, 1, 1);
      const uint64_t d_mn = make_sdesc_sw128_mn(smem_u32(smem), 2048);      // of stage 0's start
      int st = 0; uint32_t ph = 0;
      for (int b = 0; b < n_blk; ++b) {
        if (!mbar_wait(&full[st], ph, abort_flag, a.status, 910, b)) break;
        if (b > 0 && !mbar_wait(ds_free, (uint32_t)(b - 1) & 1, abort_flag, a.status, 911, b)) break;
        tc_fence_after();
        // vdim <= 64: rows 64 .. 127 of the products come from whatever the second V tile holds; nobody reads them
        const uint64_t v = sdesc_at(d_mn, st * kStage), k = sdesc_at(v, 4096 + R::kK);
        mma_f16_ss(t_ds, v, k, id_ds, 0u);
        mma_f16_ss(t_ds, v, sdesc_at(k, R::kTile), id_ds, 1u);
        tc_commit(ds_full);
        tc_commit(&empty[st]);
        if (++st == kGlStages) { st = 0; ph ^= 1; }
      }
    }
  } else if (warp == 2) {
    if (lane == 0) {
      // S_hi meets [q c hi; q c lo] in one product of 32 columns, which the output warps add
      constexpr uint32_t id_hi = make_idesc(128, 2 * kGlB, 1, 1, 0, 0), id_lo = make_idesc(128, kGlB, 1, 1, 0, 0), id_p = make_idesc(128, kGlB, 1, 1, 1, 0);
      const uint64_t d_k = make_sdesc_sw128(smem_u32(smem)), d_mn = make_sdesc_sw128_mn(smem_u32(smem), 2048);
      int st = 0; uint32_t ph = 0;
      for (int b = 0; b < n_blk; ++b) {
        if (!mbar_wait(&full[st], ph, abort_flag, a.status, 915, b)) break;
        if (!mbar_wait(&s_ready[b & 1], (uint32_t)(b >> 1) & 1, abort_flag, a.status, 912, b)) break;
        if (b >= 2 && !mbar_wait(&o_free[b & 1], ((uint32_t)(b >> 1) & 1) ^ 1, abort_flag, a.status, 913, b)) break;
        tc_fence_after();
        const uint64_t v = sdesc_at(d_mn, st * kStage), q = sdesc_at(d_k, st * kStage + 4096 + R::kQ), p = sdesc_at(d_k, st * kStage + 4096 + R::kP);
        const uint32_t s_hi = t_s + (b & 1) * 128, s_lo = s_hi + 64, o = t_o + (b & 1) * 2 * kGlB;
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) mma_f16_ts(o, s_hi + ks * 8, sdesc_at(q, (ks >> 2) * 4096 + (ks & 3) * 32), id_hi, ks > 0 ? 1u : 0u);
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) mma_f16_ts(o, s_lo + ks * 8, sdesc_at(q, (ks >> 2) * 4096 + (ks & 3) * 32), id_lo, 1u);
        mma_f16_ss(o, v, p, id_p, 1u);
        mma_f16_ss(o, v, sdesc_at(p, 32), id_p, 1u);
        tc_commit(&o_full[b & 1]);
        tc_commit(&empty[st]);
        if (++st == kGlStages) { st = 0; ph ^= 1; }
      }
    }
  } else if (warp >= 4 && warp < 8) {
    // ---------------------------------------------------------------- output: lane = value column
    const int q = warp & 3, v = e0 + q * 32 + lane;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    for (int b = 0; b < n_blk; ++b) {
      if (!warp_wait(&o_full[b & 1], (uint32_t)(b >> 1) & 1, abort_flag, a.status, 920, b)) break;
      tc_fence_after();
      float o[2 * kGlB];
      tmem_ld_x32(t_o + (b & 1) * 2 * kGlB + lane_off, reinterpret_cast<uint32_t*>(o));
      tc_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&o_free[b & 1]);
      const int t0 = t_begin + b * kGlB, n = t_end - t0;
      if (v < a.vdim) {
        float* dst = a.out + (size_t)t0 * a.ld_out + (size_t)h * a.vdim + v;
#pragma unroll
        for (int i = 0; i < kGlB; ++i) if (i < n) dst[(size_t)i * a.ld_out] = o[i] + o[kGlB + i];
      }
    }
  } else if (warp >= 8) {
    // ---------------------------------------------------------------- state: lane = value column, 64 channels per warp
    const int q = warp & 3, g = (warp - 8) >> 2, v = e0 + q * 32 + lane;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    const bool live = v < a.vdim;
    float* st = a.state + ((size_t)(run ? slot : 0) * a.heads + h) * a.dim * a.vdim + (live ? v : 0);
    float S[64];
#pragma unroll
    for (int c = 0; c < 64; ++c) S[c] = run && live && g * 64 + c < a.dim ? st[(size_t)(g * 64 + c) * a.vdim] : 0.f;
    auto publish = [&](int b) {                // S in front of block b
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int y = 0; y < 16; ++y) split_bf16x2(S[x * 32 + 2 * y], S[x * 32 + 2 * y + 1], hi[y], lo[y]);
        const uint32_t t = t_s + (b & 1) * 128 + g * 32 + x * 16 + lane_off;
        tmem_st_x16(t, hi);
        tmem_st_x16(t + 64, lo);
      }
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_ready[b & 1]);
    };
    bool ok = true;
    if (n_blk > 0) publish(0);
    for (int b = 0; b < n_blk; ++b) {
      const int sg = b % kGlStages;
      if (!warp_wait(ds_full, b & 1, abort_flag, a.status, 930, b)) { ok = false; break; }
      tc_fence_after();
      if (!warp_wait(&full[sg], (uint32_t)(b / kGlStages) & 1, abort_flag, a.status, 931, b)) { ok = false; break; }
      const float4* dec = reinterpret_cast<const float4*>(smem + sg * kStage + 4096 + R::kB) + g * 16;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        float d[32];
        tmem_ld_x32(t_ds + g * 64 + x * 32 + lane_off, reinterpret_cast<uint32_t*>(d));
        tc_wait_ld();
#pragma unroll
        for (int y = 0; y < 8; ++y) {
          const float4 f = dec[x * 8 + y];
          S[x * 32 + 4 * y] = fmaf(f.x, S[x * 32 + 4 * y], d[4 * y]);
          S[x * 32 + 4 * y + 1] = fmaf(f.y, S[x * 32 + 4 * y + 1], d[4 * y + 1]);
          S[x * 32 + 4 * y + 2] = fmaf(f.z, S[x * 32 + 4 * y + 2], d[4 * y + 2]);
          S[x * 32 + 4 * y + 3] = fmaf(f.w, S[x * 32 + 4 * y + 3], d[4 * y + 3]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) { mbar_arrive(ds_free); mbar_arrive(&empty[sg]); }
      if (b + 1 < n_blk) {
        // the buffer held S in front of block b - 1: its output is done (so a phase of s_ready cannot end unseen either)
        if (b >= 1 && !warp_wait(&o_full[(b - 1) & 1], (uint32_t)((b - 1) >> 1) & 1, abort_flag, a.status, 932, b)) { ok = false; break; }
        tc_fence_after();
        publish(b + 1);
      }
    }
    if (ok && run && live) {
#pragma unroll
      for (int c = 0; c < 64; ++c) if (g * 64 + c < a.dim) st[(size_t)(g * 64 + c) * a.vdim] = S[c];
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

template <int DP, bool RWKV>
static int gla_chunk_launch(const CUtensorMap& tmV, const GlaArgs& a, int max_tokens, int n_seqs, cudaStream_t stream) {
  static bool attr_set = false;
  if (!attr_set) {
    GB_CUDA_OK(cudaFuncSetAttribute(gla_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, gla_smem<DP>()));
    attr_set = true;
  }
  launch_k(gla_prep_kernel<DP, RWKV>, dim3((unsigned)((max_tokens + kGlB - 1) / kGlB), (unsigned)a.heads, (unsigned)n_seqs), 256, 0, stream, a);
  GB_CUDA_OK(cudaGetLastError());
  launch_k(gla_scan_kernel<DP>, dim3((unsigned)a.heads, (unsigned)((a.vdim + 127) / 128), (unsigned)n_seqs), gla_threads<DP>(), gla_smem<DP>(), stream, tmV, a);
  GB_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace gb

using namespace gb;

// Bytes of workspace gb_gla_chunk needs.
GB_API long gb_gla_chunk_workspace(long tokens, int n_seqs, int heads, int dim) {
  return (tokens / kGlB + n_seqs + 1) * heads * (long)(dim <= 64 ? GlaRecord<64>::kBytes : GlaRecord<128>::kBytes);
}

// qv: bf16 rows [tokens, ld] with columns [q heads x dim (SiLU applied) | v heads x vdim | ...], dim <= 128, dim and vdim multiples of 8; the other
// arguments as in gb_recurrent_step.
GB_API int gb_gla_chunk(const void* qv, int ld, int tokens, const float* gate, int g_part, long g_stride, int g_ld, const float* gate_bias, const float* lower,
                        float* state, int n_slots, const int* cu_q, const int* seq_slots, float* out, int ld_out, int heads, int dim, int vdim, int max_tokens,
                        int n_seqs, void* ws, long ws_bytes, void* status, cudaStream_t stream) {
  if (n_seqs <= 0 || tokens <= 0 || max_tokens <= 0) return 0;
  if (heads < 1 || dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim % 8 || g_part < 1) return fail("gla_chunk: dim <= 128, dim and vdim multiples of 8%s");
  if (ld % 8 || ld < heads * (dim + vdim) || g_ld < heads * dim || ld_out < heads * vdim || ((uintptr_t)qv & 15) || ((uintptr_t)ws & 15)) return fail("gla_chunk: bad rows%s");
  if (ws_bytes < gb_gla_chunk_workspace(tokens, n_seqs, heads, dim)) return fail("gla_chunk: workspace too small%s");
  if (n_seqs > 65535 || heads > 65535) return fail("gla_chunk: too many sequences%s");
  CUtensorMap tmV;
  uint32_t box[3] = {64, 1, kGlB};
  uint64_t dv[3] = {(uint64_t)vdim, (uint64_t)heads, (uint64_t)tokens}, sv[2] = {(uint64_t)vdim * 2, (uint64_t)ld * 2};
  if (make_tmap(&tmV, (const __nv_bfloat16*)qv + (size_t)heads * dim, TM_BF16, 3, dv, sv, box, TM_SW_128)) return -1;
  GlaArgs a;
  a.k = nullptr; a.u = nullptr;
  a.qv = (const __nv_bfloat16*)qv; a.ld = ld; a.gate = gate; a.g_part = g_part; a.g_stride = g_stride; a.g_ld = g_ld; a.gate_bias = gate_bias; a.lower = lower;
  a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out; a.heads = heads; a.dim = dim; a.vdim = vdim;
  a.ws = (uint8_t*)ws; a.status = (KernelStatus*)status;
  return dim <= 64 ? gla_chunk_launch<64, false>(tmV, a, max_tokens, n_seqs, stream) : gla_chunk_launch<128, false>(tmV, a, max_tokens, n_seqs, stream);
}

// The RWKV form: rkv holds r, k and v as three blocks of bf16 rows [tokens, ld], `block_stride` elements apart; the other arguments as in gb_rwkv_step and
// gb_gla_chunk.
GB_API int gb_rwkv_chunk(const void* rkv, long block_stride, int ld, int tokens, const float* z, int z_part, long z_stride, int z_ld, const float* w0, const float* u,
                         float* state, int n_slots, const int* cu_q, const int* seq_slots, float* out, int ld_out, int heads, int dim, int vdim, int max_tokens, int n_seqs,
                         void* ws, long ws_bytes, void* status, cudaStream_t stream) {
  if (n_seqs <= 0 || tokens <= 0 || max_tokens <= 0) return 0;
  if (heads < 1 || dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim % 8 || z_part < 1) return fail("rwkv_chunk: dim <= 128, dim and vdim multiples of 8%s");
  if (ld % 8 || block_stride % 8 || ld < heads * dim || ld < heads * vdim || z_ld < heads * dim || ld_out < heads * vdim || ((uintptr_t)rkv & 15) || ((uintptr_t)ws & 15))
    return fail("rwkv_chunk: bad rows%s");
  if (ws_bytes < gb_gla_chunk_workspace(tokens, n_seqs, heads, dim)) return fail("rwkv_chunk: workspace too small%s");
  if (n_seqs > 65535 || heads > 65535) return fail("rwkv_chunk: too many sequences%s");
  const __nv_bfloat16* r = (const __nv_bfloat16*)rkv;
  CUtensorMap tmV;
  uint32_t box[3] = {64, 1, kGlB};
  uint64_t dv[3] = {(uint64_t)vdim, (uint64_t)heads, (uint64_t)tokens}, sv[2] = {(uint64_t)vdim * 2, (uint64_t)ld * 2};
  if (make_tmap(&tmV, r + 2 * block_stride, TM_BF16, 3, dv, sv, box, TM_SW_128)) return -1;
  GlaArgs a;
  memset(&a, 0, sizeof(a));
  a.qv = r; a.k = r + block_stride; a.ld = ld; a.u = u; a.gate = z; a.g_part = z_part; a.g_stride = z_stride; a.g_ld = z_ld; a.gate_bias = w0;
  a.state = state; a.n_slots = n_slots; a.cu_q = cu_q; a.seq_slots = seq_slots; a.out = out; a.ld_out = ld_out; a.heads = heads; a.dim = dim; a.vdim = vdim;
  a.ws = (uint8_t*)ws; a.status = (KernelStatus*)status;
  return dim <= 64 ? gla_chunk_launch<64, true>(tmV, a, max_tokens, n_seqs, stream) : gla_chunk_launch<128, true>(tmV, a, max_tokens, n_seqs, stream);
}
