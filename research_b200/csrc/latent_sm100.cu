// Attention over a shared latent ("latent attention") on a paged cache, for sm_100a.
//
// A token keeps one row in the cache, shared by all heads: the normalised latent c (kv_rank channels) and one rotated
// key part. Per layer: [num_blocks, 16, CS], a row = c | zeros to a multiple of 16 | rotated part | zeros to CW, a
// multiple of 32 | 8 unused channels (CS = CW + 8). Head h's key is (W_uk[h] c, rotated part) and its value W_uv[h] c.
//
// Two evaluations of the same attention:
//   absorbed : q_lat = W_uk[h]^T q, scores = q_lat . c + q_rot . k_rot, output W_uv[h] (sum_j p_j c_j). The cached rows are
//              read as they are, once for all heads. Decoding and short portions of a prompt.
//   expanded : keys and values of the visible rows are multiplied out and the tensor cores run ordinary
//              multi-head attention on them (flash_sm100.cu). Long portions of a prompt.
//
// This file: the steps between the projections and the attention (norms, rotation, cache append), the absorbed
// attention (bf16 on mma.sync: one pass over the cached rows is bound by HBM, not by the tensor pipe; fp32 for the exact
// mode), the merge of its splits, and the gather of cached rows for the expanded form.
//
// All heads of a token form rows of one score tile: row r of a sequence is (token r / H, head r % H). The mask is a
// causal sliding window; the softmax denominator also contains exp(sink[h]); every head's output is multiplied by a gate.
#include "common.cuh"

#include <math.h>

namespace rb {

constexpr int LAT_BLOCK = 16;     // tokens per cache block

template <typename TA> __device__ __forceinline__ TA lat_cast(float v);
template <> __device__ __forceinline__ float lat_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 lat_cast<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float lat_f(float v) { return v; }
__device__ __forceinline__ float lat_f(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float lat_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

// ------------------------------------------------------------------------------------------
// After the joint down projection (fp32 row: query latent | kv latent | rotated key part | gate logits): RMS norms of both
// latents, rotation of the shared key part, cache append at `slots` (negative: skipped), sigmoid of the gates.
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void latent_append_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ qn_w,
                                     const float* __restrict__ kn_w, float eps, const int* __restrict__ positions,
                                     const int* __restrict__ slots, const float2* __restrict__ table, int max_pos, int rot_pairs,
                                     TA* __restrict__ cache, long long num_slots, int CS, int rot_off, TA* __restrict__ cq,
                                     long long ldq, float* __restrict__ gate, int q_rank, int kv_rank, int rot_dim, int H,
                                     int* status) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const float* p = proj + t * ldp;
  float ss = 0.f;
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) ss = fmaf(p[i], p[i], ss);
  const float rq = 1.f / sqrtf(lat_block_sum(ss, red) / (float)q_rank + eps);
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) cq[t * ldq + i] = lat_cast<TA>(p[i] * rq * qn_w[i]);
  const float* pc = p + q_rank;
  ss = 0.f;
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) ss = fmaf(pc[i], pc[i], ss);
  const float rc = 1.f / sqrtf(lat_block_sum(ss, red) / (float)kv_rank + eps);
  const float* pr = pc + kv_rank;
  for (int h = threadIdx.x; h < H; h += blockDim.x) gate[t * H + h] = 1.f / (1.f + expf(-pr[rot_dim + h]));
  const int slot = slots[t];
  if (slot < 0) return;
  int pos = positions[t];
  if (slot >= num_slots || pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX);
    return;
  }
  TA* row = cache + (long long)slot * CS;
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
// Absorbed attention, bf16.
//
// Work is a list of key tiles (32 keys) over all units; a unit is one row tile (16 or 32 rows) of one sequence. Every CTA
// takes an equal share of the list, so ragged batches and short ones fill the machine alike; a unit cut by a CTA boundary
// leaves partial results that latent_merge_kernel combines. The prefix sums of the units' tile counts come from
// latent_plan_kernel, once per step and window.
//
// A CTA is a producer warp, which streams whole cache blocks (16 rows, one contiguous run) through a ring of shared-memory
// stages, and two groups of four warps. In a group, warp w multiplies a quarter of the row's channels (its query fragments stay
// in registers), the four partial scores meet in shared memory, every warp forms the same weights and sums a quarter of the
// latent columns. With 16-row units the groups take alternate tiles and merge at the unit's end; with 32-row units each takes
// half the rows and both read every tile. Cache rows carry 8 channels of padding, which keeps ldmatrix free of bank conflicts.
// ------------------------------------------------------------------------------------------
constexpr int LAT_KT = 32;                       // keys per tile
constexpr int LAT_THREADS = 9 * 32;
constexpr int LAT_MIN_TILES = 2;                 // least share of a CTA
constexpr int LAT_MAX_STAGES = 6;

struct LatentAttnParams {
  const void* qa;          // [H][S][CW]
  const void* cache;       // [num_blocks, 16, CS]
  const int* block_tables; // [B, max_blocks]
  const int* cu_q;         // [B+1] rows of every sequence, or null: sequence b is row b
  const int* seq_lens;     // [B] keys per sequence, this step's tokens included
  const float* sink;       // [H]
  const float* gate;       // [T, H]
  void* out;               // [H][S][OW] gate * sum_j p_j c_j
  const int* plan;         // [B * row_tiles + 1] prefix sums of the units' tiles
  float* part_o;           // [2 * grid][rows][RW]
  float* part_ml;          // [2 * grid][rows][2]
  long long S;
  int B, H, CW, CS, RW, OW, row_tiles;   // RW: latent columns (a multiple of 16) that are summed
  int max_blocks, num_blocks, window, stages;
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
                                                           int rows, int row_tiles, int window, int* __restrict__ plan) {
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
      n = (w.hi - w.lo + LAT_KT - 1) / LAT_KT;
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

// First unit whose tiles reach past `tile` (prefix[u] <= tile < prefix[u+1]).
__device__ __forceinline__ int latent_find(const int* __restrict__ plan, int units, int tile) {
  int lo = 0, hi = units;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (plan[mid] <= tile) lo = mid; else hi = mid;
  }
  return lo;
}
__device__ __forceinline__ int latent_share(int total, int ctas) { return max((total + ctas - 1) / ctas, LAT_MIN_TILES); }

__device__ __forceinline__ void lat_bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
__device__ __forceinline__ void lat_bar(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void lat_ldsm4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void lat_ldsm4t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void lat_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int NT, int KW, bool WIDE>
__global__ void __launch_bounds__(LAT_THREADS, 1) latent_attn_kernel(const LatentAttnParams p) {
  constexpr int ROWS = WIDE ? 32 : 16;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ __align__(8) uint64_t full[LAT_MAX_STAGES], empty[LAT_MAX_STAGES];
  __shared__ int abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile_bytes = LAT_KT * p.CS * 2, page_bytes = LAT_BLOCK * p.CS * 2;
  const uint32_t ring = smem_u32(smem);
  uint8_t* exch = smem + p.stages * tile_bytes;         // partial scores of both groups, or a group's sums at a unit's end
  if (threadIdx.x == 0) {
    abort_flag = 0;
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(smem_u32(&full[i]), 1);
      mbar_init(smem_u32(&empty[i]), WIDE ? 8 : 4);
    }
    fence_mbar_init();
  }
  pdl_launch_dependents();
  __syncthreads();
  pdl_wait();
  volatile int* abortp = &abort_flag;
  const int units = p.B * p.row_tiles, total = p.plan[units];
  const int share = latent_share(total, gridDim.x);
  const int t_begin = min((int)blockIdx.x * share, total), t_end = min(t_begin + share, total);
  if (t_begin >= t_end) return;                         // uniform per CTA
  const int u_first = latent_find(p.plan, units, t_begin);

  if (warp == 8) {
    // ---------------------------------------------------------------- producer
    if (lane == 0) {
      uint32_t it = 0;
      bool ok = true;
      for (int u = u_first, t = t_begin; t < t_end; ++u) {
        const int u_end = min(p.plan[u + 1], t_end);
        if (u_end <= t) continue;
        const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, ROWS, p.H, p.window);
        const int* bt = p.block_tables + (long long)w.b * p.max_blocks;
        const int last_page = (w.hi - 1) / LAT_BLOCK;
        for (int k0 = w.lo + (t - p.plan[u]) * LAT_KT; t < u_end; ++t, k0 += LAT_KT, ++it) {
          const uint32_t s = it % p.stages;
          if (ok) ok = mbar_wait_bounded(smem_u32(&empty[s]), ((it / p.stages) & 1u) ^ 1u, abortp, p.status, ST_TIMEOUT_SMEM_EMPTY);
          if (!ok) break;                               // the consumers' waits end with the abort flag
          const uint32_t bar = smem_u32(&full[s]);
          mbar_expect_tx(bar, 2 * page_bytes);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            // past the last page the tile repeats it: those keys are masked, and their values are finite
            int blk = bt[min(k0 / LAT_BLOCK + i, last_page)];
            if (blk < 0 || blk >= p.num_blocks) { set_status(p.status, ST_BAD_INDEX); blk = 0; }
            lat_bulk_load(ring + s * tile_bytes + i * page_bytes,
                          reinterpret_cast<const __nv_bfloat16*>(p.cache) + (long long)blk * LAT_BLOCK * p.CS, page_bytes, bar);
          }
        }
        if (!ok) break;
      }
      if (!ok) {   // drain: no bulk copy may land after the CTA has gone
        for (uint32_t j = it > (uint32_t)p.stages ? it - p.stages : 0; j < it; ++j) {
          const uint64_t c0 = globaltimer_ns();
          while (!mbar_try_wait(smem_u32(&full[j % p.stages]), (j / p.stages) & 1u))
            if (globaltimer_ns() - c0 > 50000000ull) break;
        }
      }
    }
    return;
  }

  // ------------------------------------------------------------------ consumers
  const int group = warp >> 2, wg = warp & 3, g = lane >> 2, tq = lane & 3;
  const int ksteps = p.CW / 16, k_per = (ksteps + 3) / 4, k_lo = wg * k_per, k_n = max(0, min(k_per, ksteps - k_lo));
  const int n16 = p.RW / 16, n_per = (n16 + 3) / 4, col0 = wg * n_per * 16, n_n = max(0, min(n_per, n16 - wg * n_per));   // 16-column pairs
  const float log2e = 1.4426950408889634f, scale_log2 = p.scale * log2e;
  float2* my_exch = reinterpret_cast<float2*>(exch + group * (2 * 4 * 8 * 32 * 8));   // [2 buffers][4 warps][8][32 lanes]
  const int row_bytes = p.CS * 2;
  uint32_t it = 0, local = 0;
  for (int u = u_first, t = t_begin; t < t_end; ++u) {
    const int u_begin = p.plan[u], u_stop = p.plan[u + 1], u_end = min(u_stop, t_end);
    if (u_end <= t) continue;
    const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, ROWS, p.H, p.window);
    const int rg = WIDE ? group * 16 : 0;               // this group's rows: rg + g and rg + g + 8
    // query fragments of this warp's channels, and the positions of this lane's two rows
    uint32_t qf[KW][4];
    int pos[2];
    float m[2], l[2];
    {
      const __nv_bfloat16* src[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = rg + g + i * 8;
        const bool ok = r < w.n_rows;
        const int tok = (w.r0 + (ok ? r : 0)) / p.H, h = (w.r0 + (ok ? r : 0)) - tok * p.H;
        src[i] = ok ? reinterpret_cast<const __nv_bfloat16*>(p.qa) + ((long long)h * p.S + w.t0 + tok) * p.CW : nullptr;
        pos[i] = w.L - w.q_len + tok;
        // the sink enters the running maximum and the sum once, with the unit's first tile
        const bool sink = t == u_begin && (WIDE || group == 0);
        m[i] = sink ? p.sink[h] * log2e : -INFINITY;
        l[i] = sink ? 1.f : 0.f;
      }
#pragma unroll
      for (int k = 0; k < KW; ++k) {
        const int c = (k_lo + k) * 16 + 2 * tq;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const bool ok = k < k_n && src[i] != nullptr;
          qf[k][i] = ok ? *reinterpret_cast<const uint32_t*>(src[i] + c) : 0u;
          qf[k][i + 2] = ok ? *reinterpret_cast<const uint32_t*>(src[i] + c + 8) : 0u;
        }
      }
    }
    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    const int t_unit = t;
    for (int k0 = w.lo + (t - u_begin) * LAT_KT; t < u_end; ++t, k0 += LAT_KT, ++it) {
      if (!WIDE && (int)(it & 1u) != group) continue;
      const uint32_t s = it % p.stages;
      // a wait that runs out sets the status and the abort flag; the remaining (meaningless) steps run through so that every
      // barrier is met
      mbar_wait_bounded(smem_u32(&full[s]), (it / p.stages) & 1u, abortp, p.status, ST_TIMEOUT_SMEM_FULL);
      const uint32_t tile = ring + s * tile_bytes;
      float acc[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
      {
        const uint32_t ka = tile + (uint32_t)(((lane >> 4) * 8 + (lane & 7)) * row_bytes + (k_lo * 16 + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          if (k < k_n) {
            uint32_t b0, b1, b2, b3;
            lat_ldsm4(ka + k * 32, b0, b1, b2, b3);
            lat_mma(acc[0], qf[k], b0, b1);
            lat_mma(acc[1], qf[k], b2, b3);
            lat_ldsm4(ka + 16 * row_bytes + k * 32, b0, b1, b2, b3);
            lat_mma(acc[2], qf[k], b0, b1);
            lat_mma(acc[3], qf[k], b2, b3);
          }
        }
      }
      // sum the four quarters: every lane reads its own fragment positions of all warps, in the same order everywhere
      float2* ex = my_exch + (local & 1u) * (4 * 8 * 32);
      ++local;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        ex[(wg * 8 + 2 * n) * 32 + lane] = make_float2(acc[n][0], acc[n][1]);
        ex[(wg * 8 + 2 * n + 1) * 32 + lane] = make_float2(acc[n][2], acc[n][3]);
      }
      lat_bar(1 + group, 128);
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        float2 a = ex[n * 32 + lane];
#pragma unroll
        for (int i = 1; i < 4; ++i) {
          const float2 b = ex[(i * 8 + n) * 32 + lane];
          a.x += b.x;
          a.y += b.y;
        }
        acc[n >> 1][(n & 1) * 2] = a.x;
        acc[n >> 1][(n & 1) * 2 + 1] = a.y;
      }
      // mask, online softmax; row i of the lane has columns 8n + 2tq, +1
      float alpha[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        float mx = -INFINITY;
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int key = k0 + n * 8 + 2 * tq + j;
            float v = acc[n][i * 2 + j] * scale_log2;
            if (key > pos[i] || key <= pos[i] - p.window) v = -INFINITY;
            acc[n][i * 2 + j] = v;
            mx = fmaxf(mx, v);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m[i], mx), base = m_new == -INFINITY ? 0.f : m_new;
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const float e = exp2f(acc[n][i * 2 + j] - base);
            acc[n][i * 2 + j] = e;
            sum += e;
          }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        alpha[i] = exp2f(m[i] - base);
        l[i] = l[i] * alpha[i] + sum;
        m[i] = m_new;
      }
      if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[n][0] *= alpha[0]; o[n][1] *= alpha[0]; o[n][2] *= alpha[1]; o[n][3] *= alpha[1]; }
      }
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        const uint32_t a[4] = {pack_bf16x2(acc[2 * ks][0], acc[2 * ks][1]), pack_bf16x2(acc[2 * ks][2], acc[2 * ks][3]),
                               pack_bf16x2(acc[2 * ks + 1][0], acc[2 * ks + 1][1]), pack_bf16x2(acc[2 * ks + 1][2], acc[2 * ks + 1][3])};
        const uint32_t va = tile + (uint32_t)((ks * 16 + (lane & 15)) * row_bytes + (col0 + (lane >> 4) * 8) * 2);
#pragma unroll
        for (int n = 0; n < NT / 2; ++n) {
          if (n < n_n) {
            uint32_t b0, b1, b2, b3;
            lat_ldsm4t(va + n * 32, b0, b1, b2, b3);
            lat_mma(o[2 * n], a, b0, b1);
            lat_mma(o[2 * n + 1], a, b2, b3);
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&empty[s]));
    }

    if (!WIDE) {
      // the groups' sums over alternate tiles meet: group 1 leaves its own in shared memory, group 0 adds them
      float4* mo = reinterpret_cast<float4*>(exch);               // [4 warps][NT][32 lanes]
      float4* mml = mo + 4 * NT * 32;                             // [32 lanes] (m, m', l, l')
      lat_bar(3, 256);                                            // both groups are done with the partial scores
      if (group == 1) {
#pragma unroll
        for (int n = 0; n < NT; ++n) mo[(wg * NT + n) * 32 + lane] = make_float4(o[n][0], o[n][1], o[n][2], o[n][3]);
        if (wg == 0) mml[lane] = make_float4(m[0], m[1], l[0], l[1]);
      }
      lat_bar(3, 256);
      if (group == 0) {
        const float4 q4 = mml[lane];
        float fa[2], fb[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float mb = i ? q4.y : q4.x, lb = i ? q4.w : q4.z;
          const float mn = fmaxf(m[i], mb), base = mn == -INFINITY ? 0.f : mn;
          fa[i] = exp2f(m[i] - base);
          fb[i] = exp2f(mb - base);
          l[i] = l[i] * fa[i] + lb * fb[i];
          m[i] = mn;
        }
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const float4 v = mo[(wg * NT + n) * 32 + lane];
          o[n][0] = o[n][0] * fa[0] + v.x * fb[0];
          o[n][1] = o[n][1] * fa[0] + v.y * fb[0];
          o[n][2] = o[n][2] * fa[1] + v.z * fb[1];
          o[n][3] = o[n][3] * fa[1] + v.w * fb[1];
        }
      }
      lat_bar(3, 256);
    }
    if (WIDE || group == 0) {
      const bool whole = t_unit == u_begin && u_end == u_stop;
      const long long slot = 2ll * blockIdx.x + (u_begin > t_begin ? 1 : 0);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = rg + g + i * 8;
        if (r >= w.n_rows) continue;
        if (whole) {
          const int tok = (w.r0 + r) / p.H, h = (w.r0 + r) - tok * p.H;
          const float f = l[i] > 0.f ? p.gate[(long long)(w.t0 + tok) * p.H + h] / l[i] : 0.f;
          __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + ((long long)h * p.S + w.t0 + tok) * p.OW + col0 + 2 * tq;
#pragma unroll
          for (int n = 0; n < NT; ++n)
            if (n < 2 * n_n) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16x2(o[n][2 * i] * f, o[n][2 * i + 1] * f);
        } else {
          float* dst = p.part_o + (slot * ROWS + r) * p.RW + col0 + 2 * tq;
#pragma unroll
          for (int n = 0; n < NT; ++n)
            if (n < 2 * n_n) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
          if (wg == 0 && tq == 0) {
            p.part_ml[(slot * ROWS + r) * 2] = m[i];
            p.part_ml[(slot * ROWS + r) * 2 + 1] = l[i];
          }
        }
      }
    }
  }
}

// Combine the pieces of units that a CTA boundary cuts: CTA (row, boundary), for the first boundary inside each such unit.
__global__ void latent_merge_kernel(const LatentAttnParams p, int ctas, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int units = p.B * p.row_tiles, total = p.plan[units], share = latent_share(total, ctas);
  const long long cut = (long long)(blockIdx.y + 1) * share;
  if (cut >= total) return;
  const int u = latent_find(p.plan, units, (int)cut), u_begin = p.plan[u], u_stop = p.plan[u + 1];
  if (u_begin == cut || cut - share > u_begin) return;            // no cut, or an earlier boundary has it
  const LatentUnit w = latent_unit(p.cu_q, p.seq_lens, u, p.row_tiles, rows, p.H, p.window);
  const int r = blockIdx.x;
  if (r >= w.n_rows) return;
  const int tok = (w.r0 + r) / p.H, h = (w.r0 + r) - tok * p.H;
  const int c_first = blockIdx.y, c_last = (u_stop - 1) / share;
  auto slot = [&](int c) { return (2ll * c + ((long long)u_begin > (long long)c * share ? 1 : 0)) * rows + r; };
  float m = -INFINITY;
  for (int c = c_first; c <= c_last; ++c) m = fmaxf(m, p.part_ml[slot(c) * 2]);
  const float base = m == -INFINITY ? 0.f : m;
  float l = 0.f;
  for (int c = c_first; c <= c_last; ++c) l += p.part_ml[slot(c) * 2 + 1] * exp2f(p.part_ml[slot(c) * 2] - base);
  const float f = l > 0.f ? p.gate[(long long)(w.t0 + tok) * p.H + h] / l : 0.f;
  __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + ((long long)h * p.S + w.t0 + tok) * p.OW;
  for (int col = 2 * threadIdx.x; col < p.RW; col += 2 * blockDim.x) {
    float x = 0.f, y = 0.f;
    for (int c = c_first; c <= c_last; ++c) {
      const float wgt = exp2f(p.part_ml[slot(c) * 2] - base);
      const float2 v = *reinterpret_cast<const float2*>(p.part_o + slot(c) * p.RW + col);
      x = fmaf(wgt, v.x, x);
      y = fmaf(wgt, v.y, y);
    }
    *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(x * f, y * f);
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
    const float* c = reinterpret_cast<const float*>(p.cache) + ((long long)blk * LAT_BLOCK + (key & (LAT_BLOCK - 1))) * p.CS;
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
                                     int B, __nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ rot, int CS, int RW,
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
  const __nv_bfloat16* src = cache + ((long long)blk * LAT_BLOCK + (key & (LAT_BLOCK - 1))) * CS;
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

template <int NT, bool WIDE>
static int launch_latent(LatentAttnParams p, int ctas, cudaStream_t stream) {
  constexpr int KW = NT / 2 + 1;
  auto kern = latent_attn_kernel<NT, KW, WIDE>;
  const int tile = LAT_KT * p.CS * 2, limit = 226 * 1024;
  const int exch = NT * 2048 + 512 > 32768 ? NT * 2048 + 512 : 32768;
  p.stages = (limit - exch) / tile;
  if (p.stages > LAT_MAX_STAGES) p.stages = LAT_MAX_STAGES;
  if (p.stages < 2) return -14;
  static bool attr_dev[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (!attr_dev[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, limit) != cudaSuccess) return -10;
    attr_dev[dev] = true;
  }
  return launch_kernel(kern, dim3(ctas), dim3(LAT_THREADS), (size_t)(p.stages * tile + exch), stream, p) == cudaSuccess ? 0 : -11;
}

}  // namespace rb

using namespace rb;

extern "C" void rb_latent_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

// dtype: 0 bf16, 1 fp32
extern "C" int rb_latent_append(const float* proj, long long ldp, const float* qn_w, const float* kn_w, float eps,
                                const int* positions, const int* slots, const float* table, int max_pos, int rot_pairs,
                                void* cache, long long num_slots, int CS, int rot_off, void* cq, long long ldq, float* gate,
                                int q_rank, int kv_rank, int rot_dim, int H, int T, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || rot_off < kv_rank || rot_off + rot_dim > CS || 2 * rot_pairs > rot_dim || ldq < q_rank) return -1;
  if (ldp < (long long)q_rank + kv_rank + rot_dim + H) return -1;
  const int threads = q_rank + kv_rank <= 512 ? 128 : 256;
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(latent_append_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, proj, ldp, qn_w, kn_w, eps, positions,
                      slots, (const float2*)table, max_pos, rot_pairs, (__nv_bfloat16*)cache, num_slots, CS, rot_off,
                      (__nv_bfloat16*)cq, ldq, gate, q_rank, kv_rank, rot_dim, H, status);
  else
    e = launch_kernel(latent_append_kernel<float>, dim3(T), dim3(threads), 0, stream, proj, ldp, qn_w, kn_w, eps, positions, slots,
                      (const float2*)table, max_pos, rot_pairs, (float*)cache, num_slots, CS, rot_off, (float*)cq, ldq, gate,
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

// Rows of one unit and row tiles per sequence for batches whose longest sequence has max_q new rows.
static int latent_rows(int max_q, int H) { return max_q * H > 16 ? 32 : 16; }
extern "C" int rb_latent_units(int B, int H, int max_q) { return B * ((max_q * H + latent_rows(max_q, H) - 1) / latent_rows(max_q, H)); }
extern "C" int rb_latent_ctas() { return latent_sms(); }

// plan: [units + 1] ints (rb_latent_units).
extern "C" int rb_latent_plan(const int* cu_q, const int* seq_lens, int B, int H, int max_q, int window, int* plan, cudaStream_t stream) {
  if (B <= 0 || H <= 0 || max_q <= 0 || window < 1) return -1;
  const int rows = latent_rows(max_q, H);
  return launch_kernel(latent_plan_kernel, dim3(1), dim3(1024), 0, stream, cu_q, seq_lens, B, H, rows, (max_q * H + rows - 1) / rows,
                       window, plan) == cudaSuccess ? 0 : -11;
}

// T rows of B sequences (cu_q null: one row per sequence). max_q: most rows of any sequence. bf16: `plan` from rb_latent_plan
// for the same batch; part_o [2 * ctas][rows of a unit][RW] and part_ml [.., 2] hold the pieces of cut units.
extern "C" int rb_latent_attn(const void* qa, const void* cache, const int* block_tables, const int* cu_q, const int* seq_lens,
                              const float* sink, const float* gate, void* out, const int* plan, float* part_o, float* part_ml,
                              long long S, int H, int CW, int CS, int RW, int OW, int max_blocks, int num_blocks, int window,
                              float scale, int B, int T, int max_q, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || H <= 0 || window < 1 || RW > OW || RW > CW || CW % 32 != 0 || CS < CW || max_q <= 0) return -1;
  const int rows = latent_rows(max_q, H);
  LatentAttnParams p = {qa, cache, block_tables, cu_q, seq_lens, sink, gate, out, plan, part_o, part_ml, S, B, H, CW, CS, RW, OW,
                        (max_q * H + rows - 1) / rows, max_blocks, num_blocks, window, 2, scale, status};
  if (dtype == 1) {
    if (CW > 32 * LAT_F32_MAX) return -1;
    return launch_kernel(latent_attn_f32_kernel, dim3((unsigned)(((long long)T * H + 3) / 4)), dim3(128), 0, stream, p, T, B) ==
                   cudaSuccess ? 0 : -11;
  }
  if (plan == nullptr || part_o == nullptr || part_ml == nullptr || RW % 16 != 0 || OW % 8 != 0 || CS != CW + 8) return -1;
  const int ctas = latent_sms();
  int rc = -1;
#define LAT_GO(NT) rc = rows == 32 ? launch_latent<NT, true>(p, ctas, stream) : launch_latent<NT, false>(p, ctas, stream)
  if (RW <= 128 && CW <= 192) LAT_GO(4);
  else if (RW <= 256 && CW <= 320) LAT_GO(8);
  else if (RW <= 512 && CW <= 576) LAT_GO(16);
  else if (RW <= 1024 && CW <= 1088) LAT_GO(32);
#undef LAT_GO
  if (rc != 0) return rc;
  return launch_kernel(latent_merge_kernel, dim3(rows, ctas - 1), dim3(RW >= 256 ? 128 : 64), 0, stream, p, ctas, rows) == cudaSuccess
             ? 0 : -11;
}

extern "C" int rb_latent_gather(const void* cache, const int* block_tables, int bt_row0, int max_blocks, int num_blocks,
                                const int* cu_k, const int* k_lo, int B, int n_rows, void* lat, void* rot, int CS, int RW, int RP,
                                int rot_off, int rot_cols, int* status, cudaStream_t stream) {
  if (n_rows <= 0 || B <= 0 || RW % 8 != 0 || RP % 8 != 0 || rot_off % 8 != 0) return -1;
  return launch_kernel(latent_gather_kernel, dim3((n_rows + 7) / 8), dim3(256), 0, stream, (const __nv_bfloat16*)cache, block_tables,
                       bt_row0, max_blocks, num_blocks, cu_k, k_lo, B, (__nv_bfloat16*)lat, (__nv_bfloat16*)rot, CS, RW, RP, rot_off,
                       rot_cols, status) == cudaSuccess ? 0 : -11;
}
