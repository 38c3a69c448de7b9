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
// attention (bf16 on mma.sync: one pass over the cached rows is bound by HBM, not by the tensor pipe; fp32 for the exact
// mode), the merge of its splits, and the gather of cached rows for the expanded form.
//
// All heads of a token form rows of one score tile: row r of a sequence is (token r / H, head r % H). The mask is a
// causal sliding window; the softmax denominator also contains exp(sink[h]); every head's output is multiplied by a gate.
#include "common.cuh"

#include <math.h>

namespace rb {

constexpr int LAT_BLOCK = 16;     // tokens per cache block
constexpr int LAT_KT = 64;        // keys per tile
constexpr int LAT_WARPS = 8;

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
                                     TA* __restrict__ cache, long long num_slots, int CW, int rot_off, TA* __restrict__ cq,
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

struct LatentAttnParams {
  const void* qa;          // [H][S][CW]
  const void* cache;       // [num_blocks, 16, CW]
  const int* block_tables; // [B, max_blocks]
  const int* cu_q;         // [B+1] rows of every sequence, or null: sequence b is row b
  const int* seq_lens;     // [B] keys per sequence, this step's tokens included
  const float* sink;       // [H]
  const float* gate;       // [T, H]
  void* out;               // [H][S][OW] gate * sum_j p_j c_j
  float* part_o;           // splits > 1: [T, H, splits, RW]
  float* part_ml;          //             [T, H, splits, 2]
  long long S;
  int H, CW, RW, OW, rot_off; // RW: latent columns (multiple of 16) that are summed
  int max_blocks, num_blocks, splits, window, stages;
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

__device__ __forceinline__ void lat_cp16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
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

// One CTA: 16*MT rows of one sequence against one split of their keys, 64 keys at a time. A tile of cached rows is loaded
// once and used as keys (all CW columns) and as values (the first RW columns). Warp w scores keys 8w..8w+7; for the sum
// it owns latent columns [8*NT*w, 8*NT*(w+1)). Shared rows are padded by 16 bytes: conflict-free ldmatrix.
template <int NT, int MT>
__global__ void __launch_bounds__(LAT_WARPS * 32) latent_attn_kernel(const LatentAttnParams p) {
  constexpr int ROWS = 16 * MT;
  constexpr int SS = LAT_KT + 4;    // fp32 score row
  constexpr int PS = LAT_KT + 8;    // bf16 weight row
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, split = blockIdx.x;
  const int t0 = p.cu_q != nullptr ? p.cu_q[b] : b;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - t0 : 1;
  const int L = p.seq_lens[b];
  const int r0 = blockIdx.y * ROWS, n_rows = q_len * p.H;
  if (r0 >= n_rows) return;
  const int r_last = min(r0 + ROWS, n_rows) - 1;
  int lo, hi;
  latent_key_range(L, q_len, r0 / p.H, r_last / p.H, p.window, lo, hi);
  lo &= ~(LAT_BLOCK - 1);
  const int n_tiles_all = hi > lo ? (hi - lo + LAT_KT - 1) / LAT_KT : 0;
  const int per = (n_tiles_all + p.splits - 1) / p.splits;
  const int tile_begin = min(split * per, n_tiles_all), tile_end = min(tile_begin + per, n_tiles_all);

  const int KS = p.CW + 8;                                   // bf16 elements per shared row
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* sk = sq + ROWS * KS;
  float* ss = reinterpret_cast<float*>(sk + p.stages * LAT_KT * KS);
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(ss + ROWS * SS);
  float* s_m = reinterpret_cast<float*>(sp + ROWS * PS);
  float* s_l = s_m + ROWS;
  float* s_a = s_l + ROWS;

  const int chunks = p.CW / 8;
  auto load_tile = [&](int tile, int stage) {
    const int k0 = lo + tile * LAT_KT;
    const uint32_t dst = smem_u32(sk + stage * LAT_KT * KS);
    for (int i = threadIdx.x; i < LAT_KT * chunks; i += LAT_WARPS * 32) {
      const int r = i / chunks, c = i - r * chunks;
      const int key = k0 + r;
      int bytes = 0;
      const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.cache);
      if (key < hi) {
        const int blk = p.block_tables[(long long)b * p.max_blocks + key / LAT_BLOCK];
        if (blk < 0 || blk >= p.num_blocks) {
          set_status(p.status, ST_BAD_INDEX);
        } else {
          src += ((long long)blk * LAT_BLOCK + (key & (LAT_BLOCK - 1))) * p.CW + c * 8;
          bytes = 16;
        }
      }
      lat_cp16(dst + (uint32_t)(r * KS + c * 8) * 2, src, bytes);   // bytes 0: the copy fills zeros
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  if (tile_begin < tile_end) load_tile(tile_begin, 0);
  // query rows (rows past the end are zero)
  for (int i = threadIdx.x; i < ROWS * chunks; i += LAT_WARPS * 32) {
    const int r = i / chunks, c = i - r * chunks;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r0 + r < n_rows) {
      const int tok = (r0 + r) / p.H, h = (r0 + r) - tok * p.H;
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.qa) + ((long long)h * p.S + t0 + tok) * p.CW + c * 8);
    }
    *reinterpret_cast<uint4*>(sq + r * KS + c * 8) = v;
  }
  const float log2e = 1.4426950408889634f;
  for (int r = threadIdx.x; r < ROWS; r += LAT_WARPS * 32) {
    // the sink enters the running maximum and the sum once, with the first split
    const int h = (r0 + r) % p.H;
    s_m[r] = split == 0 ? p.sink[h] * log2e : -INFINITY;
    s_l[r] = split == 0 ? 1.f : 0.f;
    s_a[r] = 1.f;
  }

  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;

  const int g = lane >> 2, tq = lane & 3;
  const int col_warp = warp * NT * 8;
  const float scale_log2 = p.scale * log2e;
  const uint32_t sq_u = smem_u32(sq), sp_u = smem_u32(sp);
  for (int tile = tile_begin; tile < tile_end; ++tile) {
    const int stage = p.stages == 2 ? (tile - tile_begin) & 1 : 0;
    if (p.stages == 2 && tile + 1 < tile_end) {
      load_tile(tile + 1, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const uint32_t sk_u = smem_u32(sk + stage * LAT_KT * KS);
    // ---- scores of this warp's 8 keys ----
    {
      float acc[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) acc[m][0] = acc[m][1] = acc[m][2] = acc[m][3] = 0.f;
      const uint32_t kaddr = sk_u + (uint32_t)((warp * 8 + (lane & 7)) * KS + (lane >> 3) * 8) * 2;
      const uint32_t qaddr = sq_u + (uint32_t)((lane & 15) * KS + (lane >> 4) * 8) * 2;
#pragma unroll 2
      for (int kk = 0; kk < p.CW; kk += 32) {
        uint32_t b0, b1, b2, b3;
        lat_ldsm4(kaddr + kk * 2, b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a[4];
          lat_ldsm4(qaddr + (uint32_t)(m * 16 * KS + kk) * 2, a[0], a[1], a[2], a[3]);
          lat_mma(acc[m], a, b0, b1);
          lat_ldsm4(qaddr + (uint32_t)(m * 16 * KS + kk + 16) * 2, a[0], a[1], a[2], a[3]);
          lat_mma(acc[m], a, b2, b3);
        }
      }
      const int key = lo + tile * LAT_KT + warp * 8 + 2 * tq;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = m * 16 + half * 8 + g;
          const int pos = L - q_len + (r0 + r) / p.H;
          float x = acc[m][half * 2] * scale_log2, y = acc[m][half * 2 + 1] * scale_log2;
          if (key > pos || key <= pos - p.window) x = -INFINITY;
          if (key + 1 > pos || key + 1 <= pos - p.window) y = -INFINITY;
          *reinterpret_cast<float2*>(ss + r * SS + warp * 8 + 2 * tq) = make_float2(x, y);
        }
    }
    __syncthreads();
    // ---- online softmax, 2*MT rows per warp ----
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
      const int r = warp * 2 * MT + i;
      const float2 s2 = *reinterpret_cast<const float2*>(ss + r * SS + 2 * lane);
      const float m_old = s_m[r];
      const float m_new = fmaxf(m_old, warp_max(fmaxf(s2.x, s2.y)));
      const float base = m_new == -INFINITY ? 0.f : m_new;
      const float e0 = exp2f(s2.x - base), e1 = exp2f(s2.y - base);
      const float sum = warp_sum(e0 + e1);
      *reinterpret_cast<uint32_t*>(sp + r * PS + 2 * lane) = pack_bf16x2(e0, e1);
      __syncwarp();
      if (lane == 0) {
        const float alpha = exp2f(m_old - base);
        s_a[r] = alpha;
        s_l[r] = s_l[r] * alpha + sum;
        s_m[r] = m_new;
      }
    }
    __syncthreads();
    // ---- weighted sum of the latent rows ----
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a0 = s_a[m * 16 + g], a1 = s_a[m * 16 + 8 + g];
#pragma unroll
      for (int n = 0; n < NT; ++n) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
    }
    if (col_warp < p.RW) {
#pragma unroll
      for (int ks = 0; ks < LAT_KT / 16; ++ks) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          lat_ldsm4(sp_u + (uint32_t)((m * 16 + (lane & 15)) * PS + ks * 16 + (lane >> 4) * 8) * 2, a[m][0], a[m][1], a[m][2], a[m][3]);
        const uint32_t vaddr = sk_u + (uint32_t)((ks * 16 + (lane & 15)) * KS + col_warp + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          if (col_warp + n * 8 < p.RW) {
            uint32_t b0, b1, b2, b3;
            lat_ldsm4t(vaddr + n * 16, b0, b1, b2, b3);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              lat_mma(o[m][n], a[m], b0, b1);
              lat_mma(o[m][n + 1], a[m], b2, b3);
            }
          }
        }
      }
    }
    __syncthreads();     // the stage, the scores and the weights are reused
    if (p.stages == 1 && tile + 1 < tile_end) load_tile(tile + 1, 0);
  }
  __syncthreads();

#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + half * 8 + g;
      if (r0 + r >= n_rows) continue;
      const int tok = (r0 + r) / p.H, h = (r0 + r) - tok * p.H;
      const long long th = (long long)(t0 + tok) * p.H + h;
      if (p.splits == 1) {
        const float l = s_l[r];
        const float f = (L > 0 && l > 0.f) ? p.gate[th] / l : 0.f;
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + ((long long)h * p.S + t0 + tok) * p.OW;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int c = col_warp + n * 8 + 2 * tq;
          if (c < p.RW) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(o[m][n][half * 2] * f, o[m][n][half * 2 + 1] * f);
        }
      } else {
        float* dst = p.part_o + (th * p.splits + split) * p.RW;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int c = col_warp + n * 8 + 2 * tq;
          if (c < p.RW) *reinterpret_cast<float2*>(dst + c) = make_float2(o[m][n][half * 2], o[m][n][half * 2 + 1]);
        }
        if (warp == 0 && tq == 0) {
          p.part_ml[(th * p.splits + split) * 2] = s_m[r];
          p.part_ml[(th * p.splits + split) * 2 + 1] = s_l[r];
        }
      }
    }
}

// Combine the splits of one (token, head): CTA (h, t).
__global__ void latent_merge_kernel(const LatentAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x;
  const long long t = blockIdx.y, th = t * p.H + h;
  const float* ml = p.part_ml + th * p.splits * 2;
  float m = -INFINITY;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[2 * s]);
  const float base = m == -INFINITY ? 0.f : m;
  float l = 0.f;
  for (int s = 0; s < p.splits; ++s) l += ml[2 * s + 1] * exp2f(ml[2 * s] - base);
  const float f = l > 0.f ? p.gate[th] / l : 0.f;
  const float* po = p.part_o + th * p.splits * p.RW;
  __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + ((long long)h * p.S + t) * p.OW;
  for (int c = 2 * threadIdx.x; c < p.RW; c += 2 * blockDim.x) {
    float x = 0.f, y = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float w = exp2f(ml[2 * s] - base);
      const float2 v = *reinterpret_cast<const float2*>(po + (long long)s * p.RW + c);
      x = fmaf(w, v.x, x);
      y = fmaf(w, v.y, y);
    }
    *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(x * f, y * f);
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

template <int NT, int MT>
static int launch_latent(LatentAttnParams p, int B, int max_q, cudaStream_t stream) {
  constexpr int ROWS = 16 * MT;
  auto kern = latent_attn_kernel<NT, MT>;
  const int KS = p.CW + 8;
  const int fixed = ROWS * KS * 2 + ROWS * (LAT_KT + 4) * 4 + ROWS * (LAT_KT + 8) * 2 + ROWS * 12;
  const int tile = LAT_KT * KS * 2;
  const int limit = 227 * 1024;
  p.stages = fixed + 2 * tile <= limit ? 2 : 1;
  const int smem = fixed + p.stages * tile;
  if (smem > limit) return -14;
  static bool attr_dev[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (!attr_dev[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, limit) != cudaSuccess) return -10;
    attr_dev[dev] = true;
  }
  const dim3 grid(p.splits, (max_q * p.H + ROWS - 1) / ROWS, B);
  return launch_kernel(kern, grid, dim3(LAT_WARPS * 32), smem, stream, p) == cudaSuccess ? 0 : -11;
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
  const int threads = q_rank + kv_rank <= 512 ? 128 : 256;
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

// T rows of B sequences (cu_q null: one row per sequence). max_q: most rows of any sequence.
extern "C" int rb_latent_attn(const void* qa, const void* cache, const int* block_tables, const int* cu_q, const int* seq_lens,
                              const float* sink, const float* gate, void* out, float* part_o, float* part_ml, long long S, int H,
                              int CW, int RW, int OW, int rot_off, int max_blocks, int num_blocks, int splits, int window,
                              float scale, int B, int T, int max_q, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || B > 65535 || H <= 0 || splits < 1 || window < 1 || RW > OW || RW > rot_off || CW % 32 != 0) return -1;
  LatentAttnParams p = {qa, cache, block_tables, cu_q, seq_lens, sink, gate, out, part_o, part_ml, S, H, CW, RW, OW, rot_off,
                        max_blocks, num_blocks, splits, window, 2, scale, status};
  if (dtype == 1) {
    if (CW > 32 * LAT_F32_MAX || splits != 1) return -1;
    return launch_kernel(latent_attn_f32_kernel, dim3((unsigned)(((long long)T * H + 3) / 4)), dim3(128), 0, stream, p, T, B) ==
                   cudaSuccess ? 0 : -11;
  }
  if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return -1;
  if (RW % 16 != 0 || OW % 8 != 0 || RW > 1024) return -1;
  const bool wide = max_q * H > 16;
  int rc = -1;
#define LAT_GO(NT) rc = wide ? launch_latent<NT, 2>(p, B, max_q, stream) : launch_latent<NT, 1>(p, B, max_q, stream)
  if (RW <= 128) LAT_GO(2);
  else if (RW <= 256) LAT_GO(4);
  else if (RW <= 512) LAT_GO(8);
  else LAT_GO(16);
#undef LAT_GO
  if (rc != 0 || splits == 1) return rc;
  return launch_kernel(latent_merge_kernel, dim3(H, T), dim3(RW >= 256 ? 128 : 64), 0, stream, p) == cudaSuccess ? 0 : -11;
}

extern "C" int rb_latent_gather(const void* cache, const int* block_tables, int bt_row0, int max_blocks, int num_blocks,
                                const int* cu_k, const int* k_lo, int B, int n_rows, void* lat, void* rot, int CW, int RW, int RP,
                                int rot_off, int rot_cols, int* status, cudaStream_t stream) {
  if (n_rows <= 0 || B <= 0 || RW % 8 != 0 || RP % 8 != 0 || rot_off % 8 != 0) return -1;
  return launch_kernel(latent_gather_kernel, dim3((n_rows + 7) / 8), dim3(256), 0, stream, (const __nv_bfloat16*)cache, block_tables,
                       bt_row0, max_blocks, num_blocks, cu_k, k_lo, B, (__nv_bfloat16*)lat, (__nv_bfloat16*)rot, CW, RW, RP, rot_off,
                       rot_cols, status) == cudaSuccess ? 0 : -11;
}
