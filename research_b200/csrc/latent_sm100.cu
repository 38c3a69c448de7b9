// Attention over a shared latent ("latent attention") on a paged cache, for sm_100a.
//
// A token keeps one row in the cache, shared by all heads: the normalised latent c (kv_rank channels) and one rotated
// key part. Per layer: [num_blocks, 16, CW], a row = c | zeros to a multiple of 16 | rotated part | zeros, CW a
// multiple of 32. Head h's key is (W_uk[h] c, rotated part) and its value W_uv[h] c.
//
// Two evaluations of the same attention:
//   absorbed : q_lat = W_uk[h]^T q, scores = q_lat . c + q_rot . k_rot, output W_uv[h] (sum_j p_j c_j). The cached rows are
//              read as they are, once for all heads. Decoding and short portions of a prompt.
//   expanded : keys and values of the visible rows are multiplied out and the tensor cores run ordinary
//              multi-head attention on them (flash_sm100.cu). Long portions of a prompt.
//
// This file: the steps between the projections and the attention (norms, rotation, cache append), the absorbed
// attention (bf16 on the 5th-generation tensor cores; fp32 for the exact mode), the merge of its pieces, and the gather of
// cached rows for the expanded form.
//
// All heads of a token form rows of one score tile: row r of a sequence is (token r / H, head r % H). The mask is a
// causal sliding window; the softmax denominator also contains exp(sink[h]); every head's output is multiplied by a gate.
#include "common.cuh"
#include "tma_host.h"

#include <math.h>

namespace rb {

constexpr int LAT_BLOCK = 16;     // tokens per cache block

template <typename TA> __device__ __forceinline__ TA lat_cast(float v);
template <> __device__ __forceinline__ float lat_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 lat_cast<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float lat_f(float v) { return v; }
__device__ __forceinline__ float lat_f(__nv_bfloat16 v) { return __bfloat162float(v); }

// Sums of two values over the CTA in one round; every thread receives both.
__device__ __forceinline__ float2 lat_block_sum2(float a, float b, float2* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = make_float2(a, b);
  __syncthreads();
  const float2 t = lane < nw ? red[lane] : make_float2(0.f, 0.f);
  return make_float2(warp_sum(t.x), warp_sum(t.y));
}

// ------------------------------------------------------------------------------------------
// After the joint down projection (fp32 row: query latent | kv latent | rotated key part | gate logits): RMS norms of both
// latents, rotation of the shared key part, cache append at `slots` (negative: skipped), sigmoid of the gates.
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void latent_append_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ qn_w,
                                     const float* __restrict__ kn_w, float eps, const int* __restrict__ positions,
                                     const int* __restrict__ slots, const float2* __restrict__ table, int max_pos, int rot_pairs,
                                     TA* __restrict__ cache, long long num_slots, int CW, int rot_off, TA* __restrict__ cq,
                                     long long ldq, float* __restrict__ gate, int q_rank, int kv_rank, int rot_dim, int H,
                                     int* status) {
  __shared__ float2 red[32];
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int slot = slots[t], pos = positions[t];
  const float* p = proj + t * ldp;
  const float* pc = p + q_rank;
  const float* pr = pc + kv_rank;
  float sq = 0.f, sc = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) sq = fmaf(p[i], p[i], sq);
#pragma unroll 2
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) sc = fmaf(pc[i], pc[i], sc);
  const float2 sums = lat_block_sum2(sq, sc, red);
  const float rq = 1.f / sqrtf(sums.x / (float)q_rank + eps), rc = 1.f / sqrtf(sums.y / (float)kv_rank + eps);
#pragma unroll 4
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) cq[t * ldq + i] = lat_cast<TA>(p[i] * rq * qn_w[i]);
  for (int h = threadIdx.x; h < H; h += blockDim.x) gate[t * H + h] = 1.f / (1.f + expf(-pr[rot_dim + h]));
  if (slot < 0) return;
  if (slot >= num_slots || pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX);
    return;
  }
  TA* row = cache + (long long)slot * CW;
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) row[i] = lat_cast<TA>(pc[i] * rc * kn_w[i]);
  for (int i = threadIdx.x; i < rot_dim; i += blockDim.x) {
    float v = pr[i];
    if (i < 2 * rot_pairs) {
      const int k = i < rot_pairs ? i : i - rot_pairs;
      const float2 cs = table[(long long)pos * rot_pairs + k];
      v = i < rot_pairs ? pr[k] * cs.x - pr[k + rot_pairs] * cs.y : pr[k + rot_pairs] * cs.x + pr[k] * cs.y;
    }
    row[rot_off + i] = lat_cast<TA>(v);
  }
}

// ------------------------------------------------------------------------------------------
// Queries q [T, H, DP + RP] (unrotated part padded to DP, rotated part to RP columns).
//   tokens < n_light : unrotated part -> qn [H][S][DP], rotated part -> qa [H][S][CW] at column rot_off (for the absorbed form)
//   the others       : rotated in place (expanded form)
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void latent_query_kernel(TA* __restrict__ q, const int* __restrict__ positions, const float2* __restrict__ table,
                                    int max_pos, int rot_pairs, int n_light, TA* __restrict__ qn, TA* __restrict__ qa, long long S,
                                    int H, int DP, int RP, int rot_dim, int CW, int rot_off, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  int pos = positions[t];
  if (pos < 0 || pos >= max_pos) { if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX); pos = 0; }
  const float2* tab = table + (long long)pos * rot_pairs;
  TA* qt = q + t * (long long)H * (DP + RP);
  const bool light = t < n_light;
  if (light) {
    constexpr int V = 16 / (int)sizeof(TA);
    const int per = DP / V;
    for (int i = threadIdx.x; i < H * per; i += blockDim.x) {
      const int h = i / per, c = (i - h * per) * V;
      *reinterpret_cast<uint4*>(qn + ((long long)h * S + t) * DP + c) = *reinterpret_cast<const uint4*>(qt + h * (DP + RP) + c);
    }
    const int rest = rot_dim - 2 * rot_pairs;      // channels the rotation leaves alone
    for (int i = threadIdx.x; i < H * rest; i += blockDim.x) {
      const int h = i / rest, c = 2 * rot_pairs + i - h * rest;
      qa[((long long)h * S + t) * CW + rot_off + c] = qt[h * (DP + RP) + DP + c];
    }
  }
  for (int i = threadIdx.x; i < H * rot_pairs; i += blockDim.x) {
    const int h = i / rot_pairs, k = i - h * rot_pairs;
    TA* src = qt + h * (DP + RP) + DP;
    const float a = lat_f(src[k]), b = lat_f(src[k + rot_pairs]);
    const float2 cs = tab[k];
    TA* dst = light ? qa + ((long long)h * S + t) * CW + rot_off : src;
    dst[k] = lat_cast<TA>(a * cs.x - b * cs.y);
    dst[k + rot_pairs] = lat_cast<TA>(b * cs.x + a * cs.y);
  }
}

// ------------------------------------------------------------------------------------------
// Absorbed attention, bf16, on the 5th-generation tensor cores.
//
// Work is a list of key tiles (KT keys) over all units; a unit is NH (16 or 32) rows of one sequence. Every CTA takes an equal
// share of the list, so ragged batches and short ones fill the machine alike; a unit cut by a CTA boundary leaves partial
// results that latent_merge_kernel combines. The prefix sums of the units' tile counts come from latent_plan_kernel, once
// per step and kind of layer.
//
// A tile of cached rows is brought into shared memory once (TMA, 16-row blocks, 128-byte swizzle) and is the operand of two
// products:
//   S   [rows, KT]      = Q C^T    : A = Q (K-major), B = the tile (K-major, all CW channels)
//   O^T [channels, NH] += C^T P^T  : A = the tile read MN-major in blocks of 128 channels, B = P (K-major)
// With the output transposed the few rows of a unit are the N side, so the accumulators take NH columns per 128 channels.
// S has M = 64 although only NH rows are queries: the A descriptor runs on into the shared memory behind them, and those
// rows of S are never read.
//
// Warps: 0 TMA producer, 1 MMA issuer + TMEM owner, 2-3 load the queries of the next unit, 4 (and 5) softmax, one row
// per lane, 4-7 rescale and store O^T. The running maximum is refreshed only when it grew by more than 2^8. A wait that runs out sets
// the status and an abort flag that ends all other waits; the steps still run through, so that every barrier is met.
// ------------------------------------------------------------------------------------------
constexpr int LAT_THREADS = 256;
constexpr int LAT_MIN_TILES = 2;                 // least share of a CTA
constexpr int LAT_MAX_STAGES = 6;
constexpr float LAT_RESCALE = 8.f;               // log2 units

struct LatentAttnParams {
  CUtensorMap map;         // cache rows [num_blocks * 16, CW], box 64 x 16
  CUtensorMap q_map;       // one new token per sequence: qa as [H, S, CW], box 64 channels x 1 token x NH heads
  const void* qa;          // [H][S][CW]
  const void* cache;       // [num_blocks, 16, CW]
  const int* block_tables; // [B, max_blocks]
  const int* cu_q;         // [B+1] rows of every sequence, or null: sequence b is row b
  const int* seq_lens;     // [B] keys per sequence, this step's tokens included
  const float* sink;       // [H]
  const float* gate;       // [T, H]
  void* out;               // [H][S][OW] gate * sum_j p_j c_j
  const int* plan;         // [B * row_tiles + 1] prefix sums of the units' tiles
  float* part_o;           // [2 * grid][RW][rows]
  float* part_ml;          // [2 * grid][rows][2]
  long long S;
  int B, H, CW, RW, OW, row_tiles;       // RW: latent columns (a multiple of 16) that are summed
  int max_blocks, num_blocks, window, stages, q_tma;
  float scale;
  int* status;
};

// Keys visible to the tokens [tok_lo, tok_hi] of a sequence with L keys of which the last q_len are new.
__device__ __forceinline__ void latent_key_range(int L, int q_len, int tok_lo, int tok_hi, int window, int& lo, int& hi) {
  const int off = L - q_len;
  lo = off + tok_lo - window + 1;
  lo = lo < 0 ? 0 : lo;
  hi = off + tok_hi + 1;
}

// Rows, first key (on a block boundary) and end of the keys of unit u.
struct LatentUnit { int b, t0, q_len, L, r0, n_rows, lo, hi; };
__device__ __forceinline__ LatentUnit latent_unit(const int* cu_q, const int* seq_lens, int u, int row_tiles, int rows, int H, int window) {
  LatentUnit w;
  w.b = u / row_tiles;
  w.t0 = cu_q != nullptr ? cu_q[w.b] : w.b;
  w.q_len = cu_q != nullptr ? cu_q[w.b + 1] - w.t0 : 1;
  w.L = seq_lens[w.b];
  w.r0 = (u - w.b * row_tiles) * rows;
  w.n_rows = min(rows, w.q_len * H - w.r0);
  w.lo = w.hi = 0;
  if (w.n_rows > 0 && w.L > 0) {
    latent_key_range(w.L, w.q_len, w.r0 / H, (w.r0 + w.n_rows - 1) / H, window, w.lo, w.hi);
    w.lo &= ~(LAT_BLOCK - 1);
  }
  return w;
}

// One CTA: prefix sums of the tile counts of all units.
__global__ void __launch_bounds__(1024) latent_plan_kernel(const int* __restrict__ cu_q, const int* __restrict__ seq_lens, int B, int H,
                                                           int rows, int row_tiles, int window, int keys, int* __restrict__ plan) {
  __shared__ int warp_tot[32];
  __shared__ int carry;
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, units = B * row_tiles;
  if (threadIdx.x == 0) { carry = 0; plan[0] = 0; }
  __syncthreads();
  for (int u0 = 0; u0 < units; u0 += 1024) {
    const int u = u0 + threadIdx.x;
    int n = 0;
    if (u < units) {
      const LatentUnit w = latent_unit(cu_q, seq_lens, u, row_tiles, rows, H, window);
      n = (w.hi - w.lo + keys - 1) / keys;
    }
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, n, o);
      if (lane >= o) n += v;
    }
    if (lane == 31) warp_tot[warp] = n;
    __syncthreads();
    int before = carry;
    for (int i = 0; i < warp; ++i) before += warp_tot[i];
    if (u < units) plan[u + 1] = before + n;
    __syncthreads();
    if (threadIdx.x == 1023) carry = before + n;
    __syncthreads();
  }
}

// The unit that holds `tile` (plan[u] <= tile < plan[u + 1]), found by all threads of a CTA at once.
__device__ __forceinline__ int latent_find_cta(const int* __restrict__ plan, int units, int tile, int* shared) {
  for (int u = threadIdx.x; u < units; u += blockDim.x)
    if (plan[u] <= tile && tile < plan[u + 1]) *shared = u;
  __syncthreads();
  return *shared;
}
__device__ __forceinline__ int latent_share(int total, int ctas) { return max((total + ctas - 1) / ctas, LAT_MIN_TILES); }

__device__ __forceinline__ bool mbar_test(uint32_t bar, uint32_t parity) {     // one look, never waits
  uint32_t done;
  asm volatile(
      "{\n\t.reg .pred P;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 P, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, P;\n\t}"
      : "=r"(done)
      : "r"(bar), "r"(parity)
      : "memory");
  return done != 0;
}
__device__ __forceinline__ float lat_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void lat_bar(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

template <int NH, int KT>
__global__ void __launch_bounds__(LAT_THREADS, 1) latent_attn_kernel(const __grid_constant__ LatentAttnParams p) {
  constexpr int CHUNK = KT * 128;                // bytes of 64 channels of a tile
  constexpr int PAGES = KT / LAT_BLOCK;
  constexpr int SB = 3;                          // score, weight and alpha buffers
  constexpr int SW = NH / 16;                    // softmax warps
  constexpr uint32_t O_COL = SB * 64;            // TMEM: S at columns 0, 64, 128, O^T behind
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t kv_full[LAT_MAX_STAGES], kv_empty[LAT_MAX_STAGES];
  __shared__ __align__(8) uint64_t q_full, q_empty, s_full[SB], a_full[SB], p_full[SB], o_done[SB], o_free;
  __shared__ float s_alpha[SB][NH], s_scale[NH];
  __shared__ int s_flag[SB][SW];
  __shared__ long long s_row[NH];
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag, u_shared;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nch = (p.CW + 63) / 64, nblk = (p.RW + 127) / 128, tile_bytes = max(nch, 2 * nblk) * CHUNK;
  pdl_launch_dependents();
  pdl_wait();
  const int units = p.B * p.row_tiles, total = p.plan[units];
  const int share = latent_share(total, gridDim.x);
  const int t_begin = min((int)blockIdx.x * share, total), t_end = min(t_begin + share, total);
  if (t_begin >= t_end) return;                  // uniform per CTA, before any set-up
  const int u_first = latent_find_cta(p.plan, units, t_begin, &u_shared);

  const uint32_t q_s = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* q_ptr = smem_raw + (q_s - smem_u32(smem_raw));
  const uint32_t p_s = q_s + nch * NH * 128, kv_s = p_s + SB * NH * 128;
  uint8_t* p_ptr = q_ptr + nch * NH * 128;
  if (threadIdx.x == 0) {
    abort_flag = 0;
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(smem_u32(&kv_full[i]), 1);
      mbar_init(smem_u32(&kv_empty[i]), 1);
    }
    mbar_init(smem_u32(&q_full), p.q_tma ? 1 : 2);
    mbar_init(smem_u32(&q_empty), 1);
    for (int i = 0; i < SB; ++i) {
      mbar_init(smem_u32(&s_full[i]), 1);
      mbar_init(smem_u32(&a_full[i]), SW);
      mbar_init(smem_u32(&p_full[i]), 4);
      mbar_init(smem_u32(&o_done[i]), 1);
    }
    mbar_init(smem_u32(&o_free), 4);
    fence_mbar_init();
  }
  const uint32_t tmem_cols = O_COL + (nblk * NH + 31) / 32 * 32 <= 256 ? 256 : 512;
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_smem), tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_smem, tmem_o = tmem_base + O_COL;
  volatile int* abortp = &abort_flag;

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer: lane i loads boxes i, i + 32, ...
    uint32_t it = 0;
    bool ok = true;
    const int boxes = PAGES * nch;
    for (int u = u_first, t = t_begin; t < t_end && ok; ++u) {
      const int u_end = min(p.plan[u + 1], t_end);
      if (u_end <= t) continue;
      const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, NH, p.H, p.window);
      const int* bt = p.block_tables + (long long)w.b * p.max_blocks;
      const int n_pages = (w.hi + LAT_BLOCK - 1) / LAT_BLOCK;
      for (int k0 = w.lo + (t - p.plan[u]) * KT; t < u_end && ok; ++t, k0 += KT, ++it) {
        const uint32_t s = it % p.stages;
        ok = mbar_wait_bounded(smem_u32(&kv_empty[s]), ((it / p.stages) & 1u) ^ 1u, abortp, p.status, ST_TIMEOUT_SMEM_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        const uint32_t bar = smem_u32(&kv_full[s]), dst = kv_s + s * tile_bytes;
        if (lane == 0) mbar_expect_tx(bar, boxes * 2048);
        __syncwarp();
        for (int i = lane; i < boxes; i += 32) {
          const int pg = i / nch, c = i - pg * nch;
          int blk = p.num_blocks;                 // past the sequence's end: the copy fills zeros
          if (k0 / LAT_BLOCK + pg < n_pages) {
            blk = bt[k0 / LAT_BLOCK + pg];
            if (blk < 0 || blk >= p.num_blocks) { set_status(p.status, ST_BAD_INDEX); blk = p.num_blocks; }
          }
          tma_load_2d(dst + c * CHUNK + pg * 2048, &p.map, bar, c * 64, blk * LAT_BLOCK);
        }
      }
    }
    if (!ok && lane == 0) {   // drain: no bulk copy may land after the CTA has gone
      for (uint32_t j = it > (uint32_t)p.stages ? it - p.stages : 0; j < it; ++j) {
        const uint64_t c0 = globaltimer_ns();
        while (!mbar_try_wait(smem_u32(&kv_full[j % p.stages]), (j / p.stages) & 1u))
          if (globaltimer_ns() - c0 > 50000000ull) break;
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (elect_one_sync()) {
      constexpr uint32_t idesc_s = make_idesc_bf16(64, KT, 0, 0);
      constexpr uint32_t idesc_o = make_idesc_bf16(128, NH, 1, 0);
      const int n = t_end - t_begin, ksteps = p.CW / 16;
      int uq = 0, u_s = u_first, u_o = u_first;      // units started by the scores / being summed
      uint32_t o_units = 0;
      auto new_unit = [&](int t) {                   // moves u_s to the unit of tile t
        while (p.plan[u_s + 1] <= t) ++u_s;
        return t == t_begin || t == p.plan[u_s];
      };
      // the operands of tile j's scores are in shared memory
      auto s_ready = [&](int j) {
        if (new_unit(t_begin + j) && !mbar_test(smem_u32(&q_full), (uint32_t)uq & 1u)) return false;
        return mbar_test(smem_u32(&kv_full[j % p.stages]), (j / p.stages) & 1u);
      };
      auto issue_s = [&](int j) {
        const int t = t_begin + j;
        if (new_unit(t))                             // its queries
          mbar_wait_bounded(smem_u32(&q_full), (uint32_t)(uq++) & 1u, abortp, p.status, ST_TIMEOUT_SMEM_FULL);
        const uint32_t s = j % p.stages;
        mbar_wait_bounded(smem_u32(&kv_full[s]), (j / p.stages) & 1u, abortp, p.status, ST_TIMEOUT_SMEM_FULL);
        tc_fence_after();
        const uint32_t tile = kv_s + s * tile_bytes;
        // descriptors advance by plain additions (addresses in 16-byte units): one thread issues all of this
        uint64_t ad = make_smem_desc_sw128(q_s, 16, 1024), bd = make_smem_desc_sw128(tile, 16, 1024);
        const uint32_t d = tmem_base + (j % SB) * 64;
        umma_bf16(d, ad, bd, idesc_s, 0u);
        umma_bf16(d, ad + 2, bd + 2, idesc_s, 1u);
        if (ksteps > 2) {
          umma_bf16(d, ad + 4, bd + 4, idesc_s, 1u);
          umma_bf16(d, ad + 6, bd + 6, idesc_s, 1u);
        }
#pragma unroll 2
        for (int c = 1; c < nch; ++c) {
          ad += (NH * 128) >> 4;
          bd += CHUNK >> 4;
          umma_bf16(d, ad, bd, idesc_s, 1u);
          umma_bf16(d, ad + 2, bd + 2, idesc_s, 1u);
          if (c * 4 + 2 < ksteps) {              // CW is a multiple of 32: the last chunk may be half
            umma_bf16(d, ad + 4, bd + 4, idesc_s, 1u);
            umma_bf16(d, ad + 6, bd + 6, idesc_s, 1u);
          }
        }
        umma_commit(smem_u32(&s_full[j % SB]));
        if (t + 1 == t_end || t + 1 == p.plan[u_s + 1]) umma_commit(smem_u32(&q_empty));   // the unit's last scores
      };
      const int ahead = min(SB - 1, p.stages - 1);   // scores of later tiles overlap this tile's softmax, as far as stages allow
      int js = 0;
      for (int j = 0; j < n; ++j) {
        const int t = t_begin + j;
        while (p.plan[u_o + 1] <= t) ++u_o;
        const bool first = t == t_begin || t == p.plan[u_o];
        if (js == j) issue_s(js++);
        const uint32_t pb = smem_u32(&p_full[j % SB]), pph = (j / SB) & 1u;
        const uint64_t c0 = globaltimer_ns();
        for (uint32_t spins = 0; !mbar_test(pb, pph);) {
          if (js < n && js <= j + ahead && s_ready(js)) { issue_s(js++); continue; }
          if ((++spins & 0x3f) == 0) {
            if (*abortp != 0) break;
            if (globaltimer_ns() - c0 > RB_WAIT_BUDGET_NS) {
              *abortp = 1;
              set_status(p.status, ST_TIMEOUT_TMEM_FULL);
              break;
            }
          }
        }
        if (first && o_units++ > 0)                 // the previous unit's sums have left TMEM
          mbar_wait_bounded(smem_u32(&o_free), (o_units - 2) & 1u, abortp, p.status, ST_TIMEOUT_TMEM_EMPTY);
        tc_fence_after();
        const uint32_t s = j % p.stages, tile = kv_s + s * tile_bytes;
        uint64_t ad = make_smem_desc_sw128(tile, CHUNK, 1024);
        const uint64_t bd = make_smem_desc_sw128(p_s + (j % SB) * (NH * 128), 16, 1024);
#pragma unroll 2
        for (int m = 0; m < nblk; ++m, ad += (2 * CHUNK) >> 4)
#pragma unroll
          for (int k = 0; k < KT / 16; ++k)
            umma_bf16(tmem_o + m * NH, ad + k * (2048 >> 4), bd + 2 * k, idesc_o, (!first || k > 0) ? 1u : 0u);
        umma_commit(smem_u32(&kv_empty[s]));
        umma_commit(smem_u32(&o_done[j % SB]));
      }
      // nothing of this CTA is in flight when it frees its TMEM
      mbar_wait_bounded(smem_u32(&o_done[(n - 1) % SB]), ((n - 1) / SB) & 1u, abortp, p.status, ST_TIMEOUT_TMEM_FULL);
    }
  } else if (warp < 4) {
    // ---------------------------------------------------------------- query rows of every unit
    int uq = 0;
    const int per_row = nch * 8, tid = threadIdx.x - 64;
    const bool q_tma = p.q_tma != 0;
    for (int u = u_first, t = t_begin; t < t_end; ++u) {
      const int u_end = min(p.plan[u + 1], t_end);
      if (u_end <= t) continue;
      t = u_end;
      const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, NH, p.H, p.window);
      if (uq > 0) mbar_wait_bounded(smem_u32(&q_empty), (uint32_t)(uq - 1) & 1u, abortp, p.status, ST_TIMEOUT_SMEM_EMPTY);
      if (q_tma) {                                  // the unit's rows are heads r0.. of one token
        if (warp == 2 && lane == 0) {
          mbar_expect_tx(smem_u32(&q_full), nch * NH * 128);
          for (int c = 0; c < nch; ++c) tma_load_3d(q_s + c * (NH * 128), &p.q_map, smem_u32(&q_full), c * 64, w.t0, w.r0);
        }
        ++uq;
        continue;
      }
#pragma unroll 4
      for (int i = tid; i < NH * per_row; i += 64) {
        const int r = i / per_row, c = i - r * per_row;      // 16-byte unit c of row r
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < w.n_rows && c * 8 < p.CW) {
          const int tok = (w.r0 + r) / p.H, h = (w.r0 + r) - tok * p.H;
          v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.qa) + ((long long)h * p.S + w.t0 + tok) * p.CW + c * 8);
        }
        *reinterpret_cast<uint4*>(q_ptr + (c >> 3) * (NH * 128) + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&q_full));
      ++uq;
    }
  } else {
    // ---------------------------------------------------------------- softmax (warps 4..), O^T (warps 4-7)
    // S has M = 64: rows 16q .. 16q+15 lie in lanes 0-15 of TMEM quarter q, so warp 4 + q owns rows 16q + lane.
    const int qd = warp - 4, row = qd * 16 + lane;
    const bool soft = qd < SW, mine = soft && lane < 16;
    const uint32_t lane_addr = (uint32_t)(qd * 32) << 16;
    const float log2e = 1.4426950408889634f, scale_log2 = p.scale * log2e;
    // The sums of tile j have been added. One barrier per buffer: its phase before the awaited one is over by then (a tile's
    // scores are complete only after the sums of three tiles ago), which a single barrier would not guarantee.
    auto o_wait = [&](int j) {
      mbar_wait_bounded(smem_u32(&o_done[j % SB]), (j / SB) & 1u, abortp, p.status, ST_TIMEOUT_TMEM_FULL);
    };
    int j = 0;
    for (int u = u_first, t = t_begin; t < t_end; ++u) {
      const int u_begin = p.plan[u], u_stop = p.plan[u + 1], u_end = min(u_stop, t_end);
      if (u_end <= t) continue;
      const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, NH, p.H, p.window);
      const bool has_first = t == u_begin, whole = has_first && u_end == u_stop, row_ok = mine && row < w.n_rows;
      const int tok = (w.r0 + (row_ok ? row : 0)) / p.H, head = (w.r0 + (row_ok ? row : 0)) - tok * p.H;
      const int pos = w.L - w.q_len + tok;
      const int pos_min = w.L - w.q_len + w.r0 / p.H, pos_max = w.L - w.q_len + (w.r0 + w.n_rows - 1) / p.H;
      float m_used = -INFINITY, l = 0.f, sink = 0.f, gate = 0.f;
      if (row_ok) {
        sink = p.sink[head] * log2e;
        gate = p.gate[(long long)(w.t0 + tok) * p.H + head];
      }
      const int t_piece = t;
      for (int k0 = w.lo + (t - u_begin) * KT; t < u_end; ++t, k0 += KT, ++j) {
        const int b = j % SB;
        const uint32_t ph = (j / SB) & 1u;
        if (soft) {
          mbar_wait_bounded(smem_u32(&s_full[b]), ph, abortp, p.status, ST_TIMEOUT_TMEM_FULL);
          __syncwarp();
          tc_fence_after();
          uint32_t v[KT];
          tmem_ld_32x32(tmem_base + lane_addr + b * 64, *reinterpret_cast<uint32_t(*)[32]>(&v[0]));
          if constexpr (KT == 48) tmem_ld_32x16(tmem_base + lane_addr + b * 64 + 32, *reinterpret_cast<uint32_t(*)[16]>(&v[32]));
          tmem_ld_wait();
          tc_fence_before();
          if (k0 + KT - 1 > pos_min || k0 <= pos_max - p.window) {
#pragma unroll
            for (int i = 0; i < KT; ++i)
              if (k0 + i > pos || k0 + i <= pos - p.window) v[i] = 0xff800000u;   // -inf
          }
          float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
          for (int i = 0; i < KT; ++i) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(v[i]));
          const float m_new = fmaxf(m_used, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * scale_log2);
          const bool need = row_ok && (m_new > m_used + LAT_RESCALE || (m_used == -INFINITY && m_new != -INFINITY));
          const float alpha = need && m_used != -INFINITY ? lat_exp2(m_used - m_new) : 1.f;
          const int any = __any_sync(0xffffffffu, need && t > t_piece);
          if (need) { m_used = m_new; l *= alpha; }
          if (mine) s_alpha[b][row] = alpha;
          if (lane == 0) s_flag[b][qd] = any;
          const float mref = m_used == -INFINITY ? 0.f : m_used;
          float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
          for (int i = 0; i < KT; ++i) {
            const float x = lat_exp2(fmaf(__uint_as_float(v[i]), scale_log2, -mref));
            ls[i & 3] += x;
            v[i] = __float_as_uint(x);
          }
          l += (ls[0] + ls[1]) + (ls[2] + ls[3]);
          if (mine) {
            uint8_t* prow = p_ptr + b * (NH * 128) + row * 128;
#pragma unroll
            for (int i = 0; i < KT / 8; ++i) {
              uint4 o;
              o.x = pack_bf16x2(__uint_as_float(v[i * 8]), __uint_as_float(v[i * 8 + 1]));
              o.y = pack_bf16x2(__uint_as_float(v[i * 8 + 2]), __uint_as_float(v[i * 8 + 3]));
              o.z = pack_bf16x2(__uint_as_float(v[i * 8 + 4]), __uint_as_float(v[i * 8 + 5]));
              o.w = pack_bf16x2(__uint_as_float(v[i * 8 + 6]), __uint_as_float(v[i * 8 + 7]));
              if (!row_ok) o = make_uint4(0, 0, 0, 0);
              *reinterpret_cast<uint4*>(prow + ((i ^ (row & 7)) << 4)) = o;
            }
          }
          fence_proxy_async_smem();
          __syncwarp();
          if (lane == 0) mbar_arrive(smem_u32(&a_full[b]));
        }
        mbar_wait_bounded(smem_u32(&a_full[b]), ph, abortp, p.status, ST_TIMEOUT_TMEM_FULL);
        __syncwarp();
        int flag = 0;
#pragma unroll
        for (int i = 0; i < SW; ++i) flag |= *(volatile int*)&s_flag[b][i];
        if (flag) {                                 // O^T holds the tiles before this one
          o_wait(j - 1);
          __syncwarp();
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < nblk * NH; c += 32) {
            uint32_t o[32];
            tmem_ld_32x32(tmem_o + lane_addr + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_alpha[b][i & (NH - 1)]);
            tmem_st_32x32(tmem_o + lane_addr + c, o);
          }
          tmem_st_wait();
          tc_fence_before();
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&p_full[b]));
      }
      // ---- the piece is complete ----
      const long long slot = 2ll * blockIdx.x + (u_begin > t_begin ? 1 : 0);
      if (mine) {
        float m = m_used, f = 1.f;
        if (has_first) {                            // the sink: in the denominator once, no value
          m = fmaxf(m_used, sink);
          f = lat_exp2(m_used - m);
          l = l * f + lat_exp2(sink - m);
        }
        if (whole) f = l > 0.f ? f * gate / l : 0.f;
        s_scale[row] = f;
        s_row[row] = ((long long)head * p.S + w.t0 + tok) * p.OW;
        if (!whole && row_ok) {
          p.part_ml[(slot * NH + row) * 2] = m;
          p.part_ml[(slot * NH + row) * 2 + 1] = l;
        }
      }
      o_wait(j - 1);
      lat_bar(1, 128);
      tc_fence_after();
#pragma unroll 1
      for (int c = 0; c < nblk * NH; c += 32) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_o + lane_addr + c, o);
        tmem_ld_wait();
        if (whole) {
          // a lane holds one channel of 32 rows; neighbours trade, so that each stores two channels of every other row
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const int r = i & (NH - 1), ch = (c + i) / NH * 128 + qd * 32 + (lane & ~1);
            const float x = __uint_as_float(o[i]) * s_scale[r], y = __uint_as_float(o[i + 1]) * s_scale[r + 1];
            const float got = __shfl_xor_sync(0xffffffffu, (lane & 1) ? x : y, 1);
            const int ro = r + (lane & 1);
            if (ro < w.n_rows && ch < p.RW)
              *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + s_row[ro] + ch) =
                  (lane & 1) ? pack_bf16x2(got, y) : pack_bf16x2(x, got);
          }
        } else {
          // pieces are kept transposed, [channel][row]: contiguous for a lane
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const int r = i & (NH - 1), ch = (c + i) / NH * 128 + qd * 32 + lane;
            if (ch < p.RW)
              *reinterpret_cast<float4*>(p.part_o + (slot * p.RW + ch) * NH + r) =
                  make_float4(__uint_as_float(o[i]) * s_scale[r], __uint_as_float(o[i + 1]) * s_scale[r + 1],
                              __uint_as_float(o[i + 2]) * s_scale[r + 2], __uint_as_float(o[i + 3]) * s_scale[r + 3]);
          }
        }
      }
      tc_fence_before();
      lat_bar(1, 128);                              // the row tables are rewritten by the next unit
      if (lane == 0) mbar_arrive(smem_u32(&o_free));
    }
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, tmem_cols);
  }
}

// Combine the pieces of units that a CTA boundary cuts: blockIdx.x is the boundary (the first one inside such a unit acts),
// blockIdx.y a range of 128 channels. The pieces' weights are worked out once per row; almost always there are two pieces.
constexpr int LAT_MERGE_MAX = 160;               // pieces of one unit: at most one per CTA
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatentAttnParams p, int ctas, int rows) {
  __shared__ int u_shared;
  __shared__ float wgt[LAT_MERGE_MAX][32];
  __shared__ long long dst[32];
  pdl_launch_dependents();
  pdl_wait();
  const int units = p.B * p.row_tiles, total = p.plan[units], share = latent_share(total, ctas);
  const long long cut = (long long)(blockIdx.x + 1) * share;
  if (cut >= total) return;
  const int u = latent_find_cta(p.plan, units, (int)cut, &u_shared), u_begin = p.plan[u], u_stop = p.plan[u + 1];
  if (u_begin == cut || cut - share > u_begin) return;            // no cut, or an earlier boundary has it
  const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, rows, p.H, p.window);
  const int c_first = blockIdx.x, n = min((u_stop - 1) / share - c_first + 1, LAT_MERGE_MAX);
  auto slot = [&](int i) { return 2ll * (c_first + i) + ((long long)u_begin > (long long)(c_first + i) * share ? 1 : 0); };
  if (threadIdx.x < 32) {
    const int r = threadIdx.x;
    if (r < w.n_rows) {
      const int tok = (w.r0 + r) / p.H, h = (w.r0 + r) - tok * p.H;
      float m = -INFINITY, l = 0.f;
      for (int i = 0; i < n; ++i) m = fmaxf(m, p.part_ml[(slot(i) * rows + r) * 2]);
      const float base = m == -INFINITY ? 0.f : m;
      for (int i = 0; i < n; ++i) {
        const float e = exp2f(p.part_ml[(slot(i) * rows + r) * 2] - base);
        l += p.part_ml[(slot(i) * rows + r) * 2 + 1] * e;
        wgt[i][r] = e;
      }
      const float f = l > 0.f ? p.gate[(long long)(w.t0 + tok) * p.H + h] / l : 0.f;
      for (int i = 0; i < n; ++i) wgt[i][r] *= f;
      dst[r] = ((long long)h * p.S + w.t0 + tok) * p.OW;
    }
  }
  __syncthreads();
  // a thread takes four rows of one channel; a warp's lanes are neighbouring channels
  for (int k = threadIdx.x; k < 128 * (rows / 4); k += blockDim.x) {
    const int ch = blockIdx.y * 128 + (k & 127), r = (k >> 7) * 4;
    if (ch >= p.RW) continue;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = 0; i < n; ++i) {
      const float4 v = __ldcg(reinterpret_cast<const float4*>(p.part_o + (slot(i) * p.RW + ch) * rows + r));
      acc.x = fmaf(wgt[i][r], v.x, acc.x);
      acc.y = fmaf(wgt[i][r + 1], v.y, acc.y);
      acc.z = fmaf(wgt[i][r + 2], v.z, acc.z);
      acc.w = fmaf(wgt[i][r + 3], v.w, acc.w);
    }
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + ch;
    if (r < w.n_rows) out[dst[r]] = __float2bfloat16_rn(acc.x);
    if (r + 1 < w.n_rows) out[dst[r + 1]] = __float2bfloat16_rn(acc.y);
    if (r + 2 < w.n_rows) out[dst[r + 2]] = __float2bfloat16_rn(acc.z);
    if (r + 3 < w.n_rows) out[dst[r + 3]] = __float2bfloat16_rn(acc.w);
  }
}

// Exact mode: one warp per row, all in fp32, keys in order.
constexpr int LAT_F32_MAX = 36;   // columns per lane: CW <= 1152
__global__ void __launch_bounds__(128) latent_attn_f32_kernel(const LatentAttnParams p, int total_rows, int B) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (row >= total_rows * p.H) return;
  const int t = row / p.H, h = row - t * p.H;
  int b = t, tok = 0, q_len = 1;
  if (p.cu_q != nullptr) {
    b = 0;
    while (b + 1 < B && p.cu_q[b + 1] <= t) ++b;
    tok = t - p.cu_q[b];
    q_len = p.cu_q[b + 1] - p.cu_q[b];
  }
  const int L = p.seq_lens[b];
  int lo, hi;
  latent_key_range(L, q_len, tok, tok, p.window, lo, hi);
  const float* q = reinterpret_cast<const float*>(p.qa) + ((long long)h * p.S + t) * p.CW;
  float qv[LAT_F32_MAX], o[LAT_F32_MAX];
#pragma unroll
  for (int i = 0; i < LAT_F32_MAX; ++i) {
    qv[i] = lane + 32 * i < p.CW ? q[lane + 32 * i] : 0.f;
    o[i] = 0.f;
  }
  float m = p.sink[h], l = 1.f;
  for (int key = lo; key < hi; ++key) {
    const int blk = p.block_tables[(long long)b * p.max_blocks + key / LAT_BLOCK];
    if (blk < 0 || blk >= p.num_blocks) { set_status(p.status, ST_BAD_INDEX); continue; }
    const float* c = reinterpret_cast<const float*>(p.cache) + ((long long)blk * LAT_BLOCK + (key & (LAT_BLOCK - 1))) * p.CW;
    float kv[LAT_F32_MAX];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < LAT_F32_MAX; ++i) {
      kv[i] = lane + 32 * i < p.CW ? c[lane + 32 * i] : 0.f;
      s = fmaf(qv[i], kv[i], s);
    }
    s = warp_sum(s) * p.scale;
    const float m_new = fmaxf(m, s);
    const float alpha = expf(m - m_new), e = expf(s - m_new);
    l = l * alpha + e;
    m = m_new;
#pragma unroll
    for (int i = 0; i < LAT_F32_MAX; ++i) o[i] = o[i] * alpha + e * kv[i];
  }
  const float f = L > 0 ? p.gate[(long long)t * p.H + h] / l : 0.f;
  float* dst = reinterpret_cast<float*>(p.out) + ((long long)h * p.S + t) * p.OW;
#pragma unroll
  for (int i = 0; i < LAT_F32_MAX; ++i)
    if (lane + 32 * i < p.RW) dst[lane + 32 * i] = o[i] * f;
}

// Cached rows [k_lo[b], k_lo[b] + cu_k[b+1] - cu_k[b]) of every sequence, packed: latent part [n, RW], rotated part [n, RP].
__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_tables, int bt_row0,
                                     int max_blocks, int num_blocks, const int* __restrict__ cu_k, const int* __restrict__ k_lo,
                                     int B, __nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ rot, int CW, int RW,
                                     int RP, int rot_off, int rot_cols, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= cu_k[B]) return;
  int b = 0;
  while (b + 1 < B && cu_k[b + 1] <= row) ++b;
  const int key = k_lo[b] + row - cu_k[b];
  const int blk = block_tables[(long long)(bt_row0 + b) * max_blocks + key / LAT_BLOCK];
  if (blk < 0 || blk >= num_blocks) { if (lane == 0) set_status(status, ST_BAD_INDEX); return; }
  const __nv_bfloat16* src = cache + ((long long)blk * LAT_BLOCK + (key & (LAT_BLOCK - 1))) * CW;
  for (int c = lane; c < RW / 8; c += 32)
    *reinterpret_cast<uint4*>(lat + (long long)row * RW + c * 8) = *reinterpret_cast<const uint4*>(src + c * 8);
  for (int c = lane; c < RP / 8; c += 32)
    *reinterpret_cast<uint4*>(rot + (long long)row * RP + c * 8) =
        c * 8 < rot_cols ? *reinterpret_cast<const uint4*>(src + rot_off + c * 8) : make_uint4(0, 0, 0, 0);
}

static int latent_sms() {
  static int n = 0;
  if (n == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
  }
  return n;
}

// Rows of a unit, keys of a tile and stages of the ring for a batch and a row width.
struct LatentShape { int rows, row_tiles, keys, stages, smem; };
static LatentShape latent_shape(int max_q, int H, int CW, int RW) {
  constexpr int limit = 224 * 1024;
  LatentShape s;
  s.rows = max_q * H > 16 ? 32 : 16;
  s.row_tiles = (max_q * H + s.rows - 1) / s.rows;
  const int nch = (CW + 63) / 64, nblk = (RW + 127) / 128, fixed = 1024 + nch * s.rows * 128 + 3 * s.rows * 128;
  const int chunks = nch > 2 * nblk ? nch : 2 * nblk;
  s.keys = fixed + 3 * chunks * 48 * 128 <= limit ? 48 : 32;
  s.stages = (limit - fixed) / (chunks * s.keys * 128);
  if (s.stages > LAT_MAX_STAGES) s.stages = LAT_MAX_STAGES;
  s.smem = fixed + s.stages * chunks * s.keys * 128;
  return s;
}

// qa [H][S][CW] as a 3-D map with boxes of 64 channels x 1 token x `heads` heads (heads past the end read as zero).
static int latent_q_map(CUtensorMap* out, const void* qa, int H, long long S, int CW, int heads) {
  EncodeTiledFnT fn = tma_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(qa) & 15) != 0 || CW % 8 != 0) return -2;
  cuuint64_t dims[3] = {(cuuint64_t)CW, (cuuint64_t)S, (cuuint64_t)H};
  cuuint64_t strides[2] = {(cuuint64_t)CW * 2, (cuuint64_t)S * CW * 2};
  cuuint32_t box[3] = {64, 1, (cuuint32_t)heads};
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(qa), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

template <int NH, int KT>
static int launch_latent(const LatentAttnParams& p, int smem, int ctas, cudaStream_t stream) {
  auto kern = latent_attn_kernel<NH, KT>;
  static bool attr_dev[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (!attr_dev[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024) != cudaSuccess) return -10;
    attr_dev[dev] = true;
  }
  return launch_kernel(kern, dim3(ctas), dim3(LAT_THREADS), (size_t)smem, stream, p) == cudaSuccess ? 0 : -11;
}

}  // namespace rb

using namespace rb;

extern "C" void rb_latent_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

// dtype: 0 bf16, 1 fp32
extern "C" int rb_latent_append(const float* proj, long long ldp, const float* qn_w, const float* kn_w, float eps,
                                const int* positions, const int* slots, const float* table, int max_pos, int rot_pairs,
                                void* cache, long long num_slots, int CW, int rot_off, void* cq, long long ldq, float* gate,
                                int q_rank, int kv_rank, int rot_dim, int H, int T, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || rot_off < kv_rank || rot_off + rot_dim > CW || 2 * rot_pairs > rot_dim || ldq < q_rank) return -1;
  if (ldp < (long long)q_rank + kv_rank + rot_dim + H) return -1;
  const int threads = q_rank + kv_rank <= 512 ? 128 : (T <= 512 && q_rank > 1024 ? 512 : 256);
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(latent_append_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, proj, ldp, qn_w, kn_w, eps, positions,
                      slots, (const float2*)table, max_pos, rot_pairs, (__nv_bfloat16*)cache, num_slots, CW, rot_off,
                      (__nv_bfloat16*)cq, ldq, gate, q_rank, kv_rank, rot_dim, H, status);
  else
    e = launch_kernel(latent_append_kernel<float>, dim3(T), dim3(threads), 0, stream, proj, ldp, qn_w, kn_w, eps, positions, slots,
                      (const float2*)table, max_pos, rot_pairs, (float*)cache, num_slots, CW, rot_off, (float*)cq, ldq, gate,
                      q_rank, kv_rank, rot_dim, H, status);
  return e == cudaSuccess ? 0 : -11;
}

extern "C" int rb_latent_query(void* q, const int* positions, const float* table, int max_pos, int rot_pairs, int n_light,
                               void* qn, void* qa, long long S, int H, int DP, int RP, int rot_dim, int CW, int rot_off, int T,
                               int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || n_light < 0 || n_light > T || n_light > S || DP % 8 != 0 || RP % 8 != 0 || rot_dim > RP || rot_off + rot_dim > CW)
    return -1;
  const int threads = H * DP >= 2048 ? 256 : 128;
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(latent_query_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (__nv_bfloat16*)q, positions,
                      (const float2*)table, max_pos, rot_pairs, n_light, (__nv_bfloat16*)qn, (__nv_bfloat16*)qa, S, H, DP, RP,
                      rot_dim, CW, rot_off, status);
  else
    e = launch_kernel(latent_query_kernel<float>, dim3(T), dim3(threads), 0, stream, (float*)q, positions, (const float2*)table,
                      max_pos, rot_pairs, n_light, (float*)qn, (float*)qa, S, H, DP, RP, rot_dim, CW, rot_off, status);
  return e == cudaSuccess ? 0 : -11;
}

// plan: [B * row tiles + 1] ints; CW and RW as in rb_latent_attn.
extern "C" int rb_latent_plan(const int* cu_q, const int* seq_lens, int B, int H, int max_q, int window, int CW, int RW, int* plan,
                              cudaStream_t stream) {
  if (B <= 0 || H <= 0 || max_q <= 0 || window < 1) return -1;
  const LatentShape s = latent_shape(max_q, H, CW, RW);
  return launch_kernel(latent_plan_kernel, dim3(1), dim3(1024), 0, stream, cu_q, seq_lens, B, H, s.rows, s.row_tiles, window, s.keys,
                       plan) == cudaSuccess ? 0 : -11;
}

// T rows of B sequences (cu_q null: one row per sequence). max_q: most rows of any sequence. bf16: `plan` from rb_latent_plan
// for the same batch; part_o [2 * CTAs][RW][rows of a unit] and part_ml [2 * CTAs][rows][2] hold the pieces of cut units.
extern "C" int rb_latent_attn(const void* qa, const void* cache, const int* block_tables, const int* cu_q, const int* seq_lens,
                              const float* sink, const float* gate, void* out, const int* plan, float* part_o, float* part_ml,
                              long long S, int H, int CW, int RW, int OW, int max_blocks, int num_blocks, int window,
                              float scale, int B, int T, int max_q, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || H <= 0 || window < 1 || RW > OW || RW > CW || CW % 32 != 0 || max_q <= 0) return -1;
  const LatentShape s = latent_shape(max_q, H, CW, RW);
  LatentAttnParams p;
  p.qa = qa; p.cache = cache; p.block_tables = block_tables; p.cu_q = cu_q; p.seq_lens = seq_lens; p.sink = sink; p.gate = gate;
  p.out = out; p.plan = plan; p.part_o = part_o; p.part_ml = part_ml; p.S = S; p.B = B; p.H = H; p.CW = CW; p.RW = RW; p.OW = OW;
  p.row_tiles = s.row_tiles; p.max_blocks = max_blocks; p.num_blocks = num_blocks; p.window = window; p.stages = s.stages;
  p.scale = scale; p.status = status;
  if (dtype == 1) {
    if (CW > 32 * LAT_F32_MAX) return -1;
    return launch_kernel(latent_attn_f32_kernel, dim3((unsigned)(((long long)T * H + 3) / 4)), dim3(128), 0, stream, p, T, B) ==
                   cudaSuccess ? 0 : -11;
  }
  if (plan == nullptr || part_o == nullptr || part_ml == nullptr || RW % 16 != 0 || OW % 8 != 0 || RW > 1024 || s.stages < 2) return -1;
  if (tma_map_2d_bf16(&p.map, cache, (unsigned long long)num_blocks * LAT_BLOCK, CW, CW, LAT_BLOCK) != 0) return -20;
  p.q_tma = max_q == 1 ? 1 : 0;
  if (p.q_tma && latent_q_map(&p.q_map, qa, H, S, CW, s.rows) != 0) return -21;
  const int ctas = latent_sms() < LAT_MERGE_MAX ? latent_sms() : LAT_MERGE_MAX;
  int rc;
  if (s.keys == 48) rc = s.rows == 32 ? launch_latent<32, 48>(p, s.smem, ctas, stream) : launch_latent<16, 48>(p, s.smem, ctas, stream);
  else rc = s.rows == 32 ? launch_latent<32, 32>(p, s.smem, ctas, stream) : launch_latent<16, 32>(p, s.smem, ctas, stream);
  if (rc != 0) return rc;
  return launch_kernel(latent_merge_kernel, dim3(ctas - 1, (RW + 127) / 128), dim3(256), 0, stream, p, ctas, s.rows) == cudaSuccess ? 0 : -11;
}

extern "C" int rb_latent_gather(const void* cache, const int* block_tables, int bt_row0, int max_blocks, int num_blocks,
                                const int* cu_k, const int* k_lo, int B, int n_rows, void* lat, void* rot, int CW, int RW, int RP,
                                int rot_off, int rot_cols, int* status, cudaStream_t stream) {
  if (n_rows <= 0 || B <= 0 || RW % 8 != 0 || RP % 8 != 0 || rot_off % 8 != 0) return -1;
  return launch_kernel(latent_gather_kernel, dim3((n_rows + 7) / 8), dim3(256), 0, stream, (const __nv_bfloat16*)cache, block_tables,
                       bt_row0, max_blocks, num_blocks, cu_k, k_lo, B, (__nv_bfloat16*)lat, (__nv_bfloat16*)rot, CW, RW, RP, rot_off,
                       rot_cols, status) == cudaSuccess ? 0 : -11;
}
