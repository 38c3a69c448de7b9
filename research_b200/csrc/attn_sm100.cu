// Paged-KV attention for sm_100a.
//
// KV cache layout (per layer): [num_blocks, Hkv, 16, D] bf16, so the 16 tokens of one block
// of one KV head are one contiguous 2 KB (D=64) / 4 KB (D=128) run: a block is the unit the
// kernels stream with 16-byte asynchronous copies. Sequences that share a prefix through the
// radix tree simply list the same physical block ids in their block tables.
//
//   decode  : one CTA per (sequence, KV head, split). All G = Hq/Hkv query heads of the group
//             are rows of one MMA tile, so K/V are read from HBM once per group (no
//             materialised GQA repeat). Each warp streams its own blocks through a 4-stage
//             cp.async ring, keeps an online-softmax state, and the warps (and splits) are
//             merged at the end. The op is HBM-bound: what matters is bytes in flight.
//   prefill : varlen causal attention of new tokens against cached prefix + themselves; one
//             CTA per (sequence, query head, 64-query tile), K/V tiles double-buffered.
//
// Behaviour replaced: rollouts/inference/attention/flex_backend.py:144-279 (SDPA prefill and
// the host-loop gather decode). Numerics oracle: qwen_functional.py:173-248.
#include "common.cuh"
#include "history.cuh"
#include "tma_host.h"

#include <stdlib.h>

namespace rb {

constexpr int KV_BLOCK = 16;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                          uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Byte offset of 16-byte chunk `c` of row `r` in a tile whose rows hold D bf16, with the low
// three chunk bits XOR-swizzled by the row so ldmatrix reads are bank-conflict free.
template <int D>
__device__ __forceinline__ uint32_t swz(int r, int c) {
  return (uint32_t)(r * (D * 2) + ((c ^ (r & 7)) << 4));
}

// S(16 x 16 keys) += Q(16 x D) K^T for keys [key0, key0+16) of a swizzled K tile.
template <int D>
__device__ __forceinline__ void qk_16x16(float (&s0)[4], float (&s1)[4], const uint32_t (&qf)[D / 16][4],
                                         uint32_t k_smem, int key0, int lane) {
  const int mat = lane >> 3, r = lane & 7;
#pragma unroll
  for (int ks = 0; ks < D / 16; ++ks) {
    uint32_t b0, b1, b2, b3;
    ldsm_x4(k_smem + swz<D>(key0 + (mat >> 1) * 8 + r, 2 * ks + (mat & 1)), b0, b1, b2, b3);
    mma_16816(s0, qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b0, b1);
    mma_16816(s1, qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b2, b3);
  }
}

// O(16 x D) += P(16 x 16 keys) V for keys [key0, key0+16) of a swizzled V tile.
template <int D>
__device__ __forceinline__ void pv_16x16(float (&o)[D / 8][4], uint32_t p0, uint32_t p1, uint32_t p2, uint32_t p3,
                                         uint32_t v_smem, int key0, int lane) {
  const int mat = lane >> 3, r = lane & 7;
#pragma unroll
  for (int dp = 0; dp < D / 16; ++dp) {
    uint32_t b0, b1, b2, b3;
    ldsm_x4_t(v_smem + swz<D>(key0 + (mat & 1) * 8 + r, 2 * dp + (mat >> 1)), b0, b1, b2, b3);
    mma_16816(o[2 * dp], p0, p1, p2, p3, b0, b1);
    mma_16816(o[2 * dp + 1], p0, p1, p2, p3, b2, b3);
  }
}

// Online-softmax update of one 16x16 score tile held as two C fragments. Rows g (c0,c1) and
// g+8 (c2,c3). `valid0/valid1` give, per fragment, which of this thread's two columns are
// inside the sequence / causal range.
struct RowState { float m0, m1, l0, l1; };

template <int D>
__device__ __forceinline__ void softmax_update(float (&s0)[4], float (&s1)[4], RowState& st, float (&o)[D / 8][4],
                                               float scale_log2, uint32_t& p0, uint32_t& p1, uint32_t& p2,
                                               uint32_t& p3) {
  // scores are already masked with -inf where invalid; work in base-2
#pragma unroll
  for (int j = 0; j < 4; ++j) { s0[j] *= scale_log2; s1[j] *= scale_log2; }
  float mx0 = fmaxf(fmaxf(s0[0], s0[1]), fmaxf(s1[0], s1[1]));
  float mx1 = fmaxf(fmaxf(s0[2], s0[3]), fmaxf(s1[2], s1[3]));
  mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
  mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
  mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
  mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
  const float mn0 = fmaxf(st.m0, mx0), mn1 = fmaxf(st.m1, mx1);
  // a row with nothing valid so far keeps m = -inf; use 0 as the subtraction base then
  const float base0 = (mn0 == -INFINITY) ? 0.f : mn0;
  const float base1 = (mn1 == -INFINITY) ? 0.f : mn1;
  const float corr0 = exp2f(st.m0 - base0), corr1 = exp2f(st.m1 - base1);
  float e00 = exp2f(s0[0] - base0), e01 = exp2f(s0[1] - base0), e10 = exp2f(s1[0] - base0), e11 = exp2f(s1[1] - base0);
  float f00 = exp2f(s0[2] - base1), f01 = exp2f(s0[3] - base1), f10 = exp2f(s1[2] - base1), f11 = exp2f(s1[3] - base1);
  float rs0 = e00 + e01 + e10 + e11;
  float rs1 = f00 + f01 + f10 + f11;
  rs0 += __shfl_xor_sync(0xffffffffu, rs0, 1);
  rs0 += __shfl_xor_sync(0xffffffffu, rs0, 2);
  rs1 += __shfl_xor_sync(0xffffffffu, rs1, 1);
  rs1 += __shfl_xor_sync(0xffffffffu, rs1, 2);
  st.l0 = st.l0 * corr0 + rs0;
  st.l1 = st.l1 * corr1 + rs1;
  st.m0 = mn0;
  st.m1 = mn1;
#pragma unroll
  for (int n = 0; n < D / 8; ++n) {
    o[n][0] *= corr0; o[n][1] *= corr0;
    o[n][2] *= corr1; o[n][3] *= corr1;
  }
  // C fragments of two adjacent 8-key tiles form the A fragment of one 16-key step
  p0 = pack_bf16x2(e00, e01);
  p1 = pack_bf16x2(f00, f01);
  p2 = pack_bf16x2(e10, e11);
  p3 = pack_bf16x2(f10, f11);
}

// ------------------------------------------------------------------------------------------
// Decode
// ------------------------------------------------------------------------------------------
constexpr int DEC_WARPS = 4;
constexpr int DEC_STAGES = 3;  // 50 KB (D=64) / 100 KB (D=128) per CTA -> 4 / 2 CTAs per SM

template <int D>
__global__ void __launch_bounds__(DEC_WARPS * 32)
paged_decode_kernel(const __nv_bfloat16* __restrict__ q,         // [B, Hq, D]
                    const __nv_bfloat16* __restrict__ k_cache,   // [num_blocks, Hkv, 16, D]
                    const __nv_bfloat16* __restrict__ v_cache,
                    const int* __restrict__ block_tables,        // [B, max_blocks]
                    const int* __restrict__ seq_lens,            // [B]
                    __nv_bfloat16* __restrict__ out,             // [B, Hq, D]
                    float* __restrict__ part_o,                  // [B, Hq, S, D]   (S > 1)
                    float* __restrict__ part_ml,                 // [B, Hq, S, 2]
                    int Hq, int Hkv, int max_blocks, int num_blocks, int num_splits, float scale,
                    int* status) {
  constexpr int CH = D / 8;                 // 16-byte chunks per row
  constexpr int TILE_BYTES = KV_BLOCK * D * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int split = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = Hq / Hkv;
  const int L = seq_lens[b];
  const int n_chunks = (L + KV_BLOCK - 1) / KV_BLOCK;
  const int per = (n_chunks + num_splits - 1) / num_splits;
  const int c_begin = split * per;
  const int c_end = min(n_chunks, c_begin + per);

  // shared memory: Q tile [16][D] then per warp DEC_STAGES x (K tile, V tile)
  const uint32_t q_smem = smem_u32(smem);
  const uint32_t kv_smem = q_smem + 16 * D * 2 + warp * (DEC_STAGES * 2 * TILE_BYTES);

  // stage Q (rows >= G zero)
  for (int i = threadIdx.x; i < 16 * CH; i += blockDim.x) {
    const int r = i / CH, c = i % CH;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < G) v = *reinterpret_cast<const uint4*>(q + ((long long)b * Hq + kvh * G + r) * D + c * 8);
    *reinterpret_cast<uint4*>(smem + swz<D>(r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[D / 16][4];
  {
    const int mat = lane >> 3, r = lane & 7;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
      ldsm_x4(q_smem + swz<D>((mat & 1) * 8 + r, 2 * ks + (mat >> 1)), qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
  }

  float o[D / 8][4];
#pragma unroll
  for (int n = 0; n < D / 8; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
  RowState st = {-INFINITY, -INFINITY, 0.f, 0.f};
  const float scale_log2 = scale * 1.4426950408889634f;

  auto issue = [&](int chunk, int stage) {
    if (chunk < c_end) {
      int blk = block_tables[(long long)b * max_blocks + chunk];
      if (blk < 0 || blk >= num_blocks) { set_status(status, ST_BAD_INDEX); blk = 0; }
      const __nv_bfloat16* ksrc = k_cache + ((long long)blk * Hkv + kvh) * KV_BLOCK * D;
      const __nv_bfloat16* vsrc = v_cache + ((long long)blk * Hkv + kvh) * KV_BLOCK * D;
      const uint32_t ks = kv_smem + stage * 2 * TILE_BYTES, vs = ks + TILE_BYTES;
#pragma unroll
      for (int i = lane; i < KV_BLOCK * CH; i += 32) {
        const int r = i / CH, c = i % CH;
        cp_async16(ks + swz<D>(r, c), ksrc + r * D + c * 8);
        cp_async16(vs + swz<D>(r, c), vsrc + r * D + c * 8);
      }
    }
    cp_async_commit();
  };

  int my = c_begin + warp;
#pragma unroll
  for (int s = 0; s < DEC_STAGES - 1; ++s) issue(my + s * DEC_WARPS, s);
  int stage = 0;
  for (int chunk = my; chunk < c_end; chunk += DEC_WARPS) {
    issue(chunk + (DEC_STAGES - 1) * DEC_WARPS, (stage + DEC_STAGES - 1) % DEC_STAGES);
    cp_async_wait<DEC_STAGES - 1>();
    __syncwarp();
    const uint32_t ks = kv_smem + stage * 2 * TILE_BYTES, vs = ks + TILE_BYTES;
    float s0[4] = {0, 0, 0, 0}, s1[4] = {0, 0, 0, 0};
    qk_16x16<D>(s0, s1, qf, ks, 0, lane);
    const int tok0 = chunk * KV_BLOCK + 2 * (lane & 3);
    if (tok0 >= L) { s0[0] = s0[2] = -INFINITY; }
    if (tok0 + 1 >= L) { s0[1] = s0[3] = -INFINITY; }
    if (tok0 + 8 >= L) { s1[0] = s1[2] = -INFINITY; }
    if (tok0 + 9 >= L) { s1[1] = s1[3] = -INFINITY; }
    uint32_t p0, p1, p2, p3;
    softmax_update<D>(s0, s1, st, o, scale_log2, p0, p1, p2, p3);
    pv_16x16<D>(o, p0, p1, p2, p3, vs, 0, lane);
    __syncwarp();
    stage = (stage + 1) % DEC_STAGES;
  }
  cp_async_wait<0>();
  __syncthreads();

  // ---- merge the warps through shared memory (re-using the KV ring) ----
  float* mo = reinterpret_cast<float*>(smem + 16 * D * 2);          // [DEC_WARPS][8][D]
  float* mml = mo + DEC_WARPS * 8 * D;                              // [DEC_WARPS][8][2]
  const int g = lane >> 2, t = lane & 3;
  if (g < 8) {
#pragma unroll
    for (int n = 0; n < D / 8; ++n) {
      mo[(warp * 8 + g) * D + n * 8 + 2 * t] = o[n][0];
      mo[(warp * 8 + g) * D + n * 8 + 2 * t + 1] = o[n][1];
    }
    if (t == 0) { mml[(warp * 8 + g) * 2] = st.m0; mml[(warp * 8 + g) * 2 + 1] = st.l0; }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < G * D; i += blockDim.x) {
    const int r = i / D, d = i % D;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < DEC_WARPS; ++w) M = fmaxf(M, mml[(w * 8 + r) * 2]);
    float acc = 0.f, l = 0.f;
    if (M != -INFINITY) {
#pragma unroll
      for (int w = 0; w < DEC_WARPS; ++w) {
        const float e = exp2f(mml[(w * 8 + r) * 2] - M);
        acc += e * mo[(w * 8 + r) * D + d];
        l += e * mml[(w * 8 + r) * 2 + 1];
      }
    }
    const int h = kvh * G + r;
    if (num_splits == 1) {
      out[((long long)b * Hq + h) * D + d] = __float2bfloat16_rn(l > 0.f ? acc / l : 0.f);
    } else {
      const long long pi = ((long long)b * Hq + h) * num_splits + split;
      part_o[pi * D + d] = acc;
      if (d == 0) { part_ml[pi * 2] = M; part_ml[pi * 2 + 1] = l; }
    }
  }
}

// ------------------------------------------------------------------------------------------
// Decode, TMA variant (default): every 16-token block of one KV head is a contiguous [16, D]
// tile, fetched with ONE tile copy per 128 bytes of row (1 for D=64, 2 for D=128) instead of 128
// sixteen-byte requests. The 128-byte swizzle of the copy is exactly the XOR layout ldmatrix
// needs. Each warp owns a ring of 3-4 (K,V) tiles with one mbarrier per stage; an
// out-of-range block id lands on an out-of-bounds coordinate, which TMA fills with zeros.
// ------------------------------------------------------------------------------------------
template <int D>
__host__ __device__ constexpr int dec_tma_stages() { return 3; }   // 52 KB (D=64: 4 CTAs/SM) or 103 KB (D=128: 2 CTAs/SM)

// 16-byte chunk c of row r inside a [16, D] tile loaded as D/64 swizzled [16][128 B] half tiles
template <int D>
__device__ __forceinline__ uint32_t swz_tma(int r, int c) {
  return (uint32_t)((c >> 3) * (KV_BLOCK * 128) + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}

template <int D>
__global__ void __launch_bounds__(DEC_WARPS * 32)
paged_decode_tma_kernel(const __nv_bfloat16* __restrict__ q, const __grid_constant__ CUtensorMap k_map,
                        const __grid_constant__ CUtensorMap v_map, const int* __restrict__ block_tables,
                        const int* __restrict__ seq_lens, __nv_bfloat16* __restrict__ out,
                        float* __restrict__ part_o, float* __restrict__ part_ml, int Hq, int Hkv, int max_blocks,
                        int num_blocks, int num_splits, float scale, int* status) {
  constexpr int CH = D / 8;
  constexpr int TILE_BYTES = KV_BLOCK * D * 2;
  constexpr int ST = dec_tma_stages<D>();
  extern __shared__ __align__(128) uint8_t smem[];   // the ring is aligned to 1024 bytes by hand below
  __shared__ __align__(8) uint64_t bars[DEC_WARPS][ST];
  __shared__ int abort_flag;
  pdl_launch_dependents();
  const int split = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = Hq / Hkv;
  // layout: [ring: DEC_WARPS x ST x (K tile, V tile)] (1024-byte aligned) then the Q tile
  const uint32_t ring0 = (smem_u32(smem) + 1023u) & ~1023u;
  uint8_t* ring_ptr = smem + (ring0 - smem_u32(smem));
  const uint32_t kv_smem = ring0 + warp * (ST * 2 * TILE_BYTES);
  uint8_t* q_ptr = ring_ptr + DEC_WARPS * ST * 2 * TILE_BYTES;
  const uint32_t q_smem = smem_u32(q_ptr);
  if (threadIdx.x == 0) {
    abort_flag = 0;
    for (int w = 0; w < DEC_WARPS; ++w)
      for (int s2 = 0; s2 < ST; ++s2) mbar_init(smem_u32(&bars[w][s2]), 1);
    fence_mbar_init();
  }
  pdl_wait();
  const int L = seq_lens[b];
  const int n_chunks = (L + KV_BLOCK - 1) / KV_BLOCK;
  const int per = (n_chunks + num_splits - 1) / num_splits;
  const int c_begin = split * per;
  const int c_end = min(n_chunks, c_begin + per);
  for (int i = threadIdx.x; i < 16 * CH; i += blockDim.x) {
    const int r = i / CH, c = i % CH;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < G) v = *reinterpret_cast<const uint4*>(q + ((long long)b * Hq + kvh * G + r) * D + c * 8);
    *reinterpret_cast<uint4*>(q_ptr + swz<D>(r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[D / 16][4];
  {
    const int mat = lane >> 3, r = lane & 7;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
      ldsm_x4(q_smem + swz<D>((mat & 1) * 8 + r, 2 * ks + (mat >> 1)), qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
  }
  float o[D / 8][4];
#pragma unroll
  for (int n = 0; n < D / 8; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
  RowState st = {-INFINITY, -INFINITY, 0.f, 0.f};
  const float scale_log2 = scale * 1.4426950408889634f;
  volatile int* abortp = &abort_flag;

  const int first = c_begin + warp;
  const int n_my = first < c_end ? (c_end - first + DEC_WARPS - 1) / DEC_WARPS : 0;
  // Block ids of this warp's chunks are fetched 32 at a time (lane j holds chunk round*32+j) so the
  // table lookup is off the critical path of every copy.
  const int* bt_row = block_tables + (long long)b * max_blocks;
  auto load_ids = [&](int round) {
    const int j = round * 32 + lane;
    return j < n_my ? __ldg(bt_row + first + j * DEC_WARPS) : 0;
  };
  int ids_round = 0, ids = load_ids(0), ids_next = load_ids(1);
  auto blk_of = [&](int i) {   // all lanes, i uniform and non-decreasing
    if ((i >> 5) > ids_round) { ids = ids_next; ids_round = i >> 5; ids_next = load_ids(ids_round + 1); }
    return __shfl_sync(0xffffffffu, ids, i & 31);
  };
  auto issue = [&](int i, int blk) {   // lane 0 only
    const int stage = i % ST;
    if (blk < 0 || blk >= num_blocks) { set_status(status, ST_BAD_INDEX); blk = num_blocks; }  // OOB -> zeros
    const int y = (blk * Hkv + kvh) * KV_BLOCK;
    const uint32_t bar = smem_u32(&bars[warp][stage]);
    const uint32_t ks = kv_smem + stage * 2 * TILE_BYTES, vs = ks + TILE_BYTES;
    mbar_expect_tx(bar, 2 * TILE_BYTES);
#pragma unroll
    for (int hx = 0; hx < D / 64; ++hx) {
      tma_load_2d(ks + hx * (KV_BLOCK * 128), &k_map, bar, hx * 64, y);
      tma_load_2d(vs + hx * (KV_BLOCK * 128), &v_map, bar, hx * 64, y);
    }
  };
  int issued = 0;
  for (; issued < ST - 1 && issued < n_my; ++issued) {
    const int blk = blk_of(issued);
    if (lane == 0) issue(issued, blk);
  }
  bool ok = true;
  const int mat = lane >> 3, rr = lane & 7;
  for (int i = 0; i < n_my; ++i) {
    if (issued < n_my) {
      const int blk = blk_of(issued);
      if (lane == 0) issue(issued, blk);
      ++issued;
    }
    const int stage = i % ST;
    ok = mbar_wait_bounded(smem_u32(&bars[warp][stage]), (uint32_t)((i / ST) & 1), abortp, status, ST_TIMEOUT_SMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) break;
    const uint32_t ks = kv_smem + stage * 2 * TILE_BYTES, vs = ks + TILE_BYTES;
    float s0[4] = {0, 0, 0, 0}, s1[4] = {0, 0, 0, 0};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4(ks + swz_tma<D>((mat >> 1) * 8 + rr, 2 * kk + (mat & 1)), b0, b1, b2, b3);
      mma_16816(s0, qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b0, b1);
      mma_16816(s1, qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b2, b3);
    }
    const int tok0 = (first + i * DEC_WARPS) * KV_BLOCK + 2 * (lane & 3);
    if (tok0 >= L) { s0[0] = s0[2] = -INFINITY; }
    if (tok0 + 1 >= L) { s0[1] = s0[3] = -INFINITY; }
    if (tok0 + 8 >= L) { s1[0] = s1[2] = -INFINITY; }
    if (tok0 + 9 >= L) { s1[1] = s1[3] = -INFINITY; }
    uint32_t p0, p1, p2, p3;
    softmax_update<D>(s0, s1, st, o, scale_log2, p0, p1, p2, p3);
#pragma unroll
    for (int dp = 0; dp < D / 16; ++dp) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4_t(vs + swz_tma<D>((mat & 1) * 8 + rr, 2 * dp + (mat >> 1)), b0, b1, b2, b3);
      mma_16816(o[2 * dp], p0, p1, p2, p3, b0, b1);
      mma_16816(o[2 * dp + 1], p0, p1, p2, p3, b2, b3);
    }
    __syncwarp();   // every lane is done with this stage before lane 0 refills it
  }
  if (!ok && lane == 0) {
    // drain: wait (bounded) for copies already issued so none lands after the CTA has exited
    for (int j = max(0, issued - ST); j < issued; ++j) {   // the latest phase of every stage
      const uint64_t t0 = globaltimer_ns();
      while (!mbar_try_wait(smem_u32(&bars[warp][j % ST]), (uint32_t)((j / ST) & 1)))
        if (globaltimer_ns() - t0 > 50000000ull) break;
    }
  }
  __syncthreads();

  float* mo = reinterpret_cast<float*>(ring_ptr);                   // [DEC_WARPS][8][D]
  float* mml = mo + DEC_WARPS * 8 * D;                              // [DEC_WARPS][8][2]
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int n = 0; n < D / 8; ++n) {
    mo[(warp * 8 + g) * D + n * 8 + 2 * t] = o[n][0];
    mo[(warp * 8 + g) * D + n * 8 + 2 * t + 1] = o[n][1];
  }
  if (t == 0) { mml[(warp * 8 + g) * 2] = st.m0; mml[(warp * 8 + g) * 2 + 1] = st.l0; }
  __syncthreads();
  for (int i = threadIdx.x; i < G * D; i += blockDim.x) {
    const int r = i / D, d = i % D;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < DEC_WARPS; ++w) M = fmaxf(M, mml[(w * 8 + r) * 2]);
    float acc = 0.f, l = 0.f;
    if (M != -INFINITY) {
#pragma unroll
      for (int w = 0; w < DEC_WARPS; ++w) {
        const float e = exp2f(mml[(w * 8 + r) * 2] - M);
        acc += e * mo[(w * 8 + r) * D + d];
        l += e * mml[(w * 8 + r) * 2 + 1];
      }
    }
    const int h = kvh * G + r;
    if (num_splits == 1) {
      out[((long long)b * Hq + h) * D + d] = __float2bfloat16_rn(l > 0.f ? acc / l : 0.f);
    } else {
      const long long pi = ((long long)b * Hq + h) * num_splits + split;
      part_o[pi * D + d] = acc;
      if (d == 0) { part_ml[pi * 2] = M; part_ml[pi * 2 + 1] = l; }
    }
  }
}

template <int D>
__global__ void decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                    __nv_bfloat16* __restrict__ out, int num_splits) {
  pdl_launch_dependents();
  pdl_wait();
  const long long bh = blockIdx.x;
  const int d = threadIdx.x;
  if (d >= D) return;
  float M = -INFINITY;
  for (int s = 0; s < num_splits; ++s) M = fmaxf(M, part_ml[(bh * num_splits + s) * 2]);
  float acc = 0.f, l = 0.f;
  if (M != -INFINITY) {
    for (int s = 0; s < num_splits; ++s) {
      const float e = exp2f(part_ml[(bh * num_splits + s) * 2] - M);
      acc += e * part_o[(bh * num_splits + s) * D + d];
      l += e * part_ml[(bh * num_splits + s) * 2 + 1];
    }
  }
  out[bh * D + d] = __float2bfloat16_rn(l > 0.f ? acc / l : 0.f);
}

// ------------------------------------------------------------------------------------------
// Prefill (varlen, causal, prefix-aware, optional sliding window)
// ------------------------------------------------------------------------------------------
constexpr int PF_WARPS = 4;
constexpr int PF_BM = 64;
constexpr int PF_BN = 64;

template <int D>
__global__ void __launch_bounds__(PF_WARPS * 32)
paged_prefill_kernel(const __nv_bfloat16* __restrict__ q,        // [T, Hq, D] packed new tokens
                     const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
                     const int* __restrict__ block_tables,       // [B, max_blocks]
                     const int* __restrict__ cu_q,               // [B+1] offsets of new tokens
                     const int* __restrict__ seq_lens,           // [B] total context (prefix + new)
                     __nv_bfloat16* __restrict__ out,            // [T, Hq, D]
                     float* __restrict__ lse,                    // [T, Hq] natural-log LSE or null
                     int Hq, int Hkv, int max_blocks, int num_blocks, float scale, int window,
                     int* status) {
  constexpr int CH = D / 8;
  constexpr int KTILE_BYTES = PF_BN * D * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  const int qt = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int q_begin = cu_q[b], q_end = cu_q[b + 1];
  const int n_new = q_end - q_begin;
  if (qt * PF_BM >= n_new) return;
  const int L = seq_lens[b];
  const int prefix = L - n_new;                 // tokens already cached before this call
  const int kvh = h / (Hq / Hkv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t q_smem = smem_u32(smem);
  const uint32_t k_smem0 = q_smem + PF_BM * D * 2;          // 2 stages of K then 2 stages of V
  const uint32_t v_smem0 = k_smem0 + 2 * KTILE_BYTES;

  for (int i = threadIdx.x; i < PF_BM * CH; i += blockDim.x) {
    const int r = i / CH, c = i % CH;
    const int tq = qt * PF_BM + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (tq < n_new) v = *reinterpret_cast<const uint4*>(q + ((long long)(q_begin + tq) * Hq + h) * D + c * 8);
    *reinterpret_cast<uint4*>(smem + swz<D>(r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[D / 16][4];
  {
    const int mat = lane >> 3, r = lane & 7;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
      ldsm_x4(q_smem + swz<D>(warp * 16 + (mat & 1) * 8 + r, 2 * ks + (mat >> 1)), qf[ks][0], qf[ks][1], qf[ks][2],
              qf[ks][3]);
  }

  // absolute positions of this thread's two query rows
  const int g = lane >> 2, t4 = lane & 3;
  const int row0 = qt * PF_BM + warp * 16 + g, row1 = row0 + 8;
  const int pos0 = prefix + row0, pos1 = prefix + row1;
  // keys needed by this CTA: [k_lo, k_hi)
  const int last_q = min(n_new, (qt + 1) * PF_BM) - 1;
  const int k_hi = min(L, prefix + last_q + 1);
  int k_lo = 0;
  if (window > 0) k_lo = max(0, prefix + qt * PF_BM - window + 1);
  const int tile_lo = k_lo / PF_BN, tile_hi = (k_hi + PF_BN - 1) / PF_BN;

  auto issue = [&](int tile, int stage) {
    if (tile < tile_hi) {
      const uint32_t ks = k_smem0 + stage * KTILE_BYTES, vs = v_smem0 + stage * KTILE_BYTES;
      for (int i = threadIdx.x; i < PF_BN * CH; i += blockDim.x) {
        const int r = i / CH, c = i % CH;
        const int key = tile * PF_BN + r;
        if (key < L) {
          int blk = block_tables[(long long)b * max_blocks + key / KV_BLOCK];
          if (blk < 0 || blk >= num_blocks) { set_status(status, ST_BAD_INDEX); blk = 0; }
          const long long off = (((long long)blk * Hkv + kvh) * KV_BLOCK + (key % KV_BLOCK)) * D + c * 8;
          cp_async16(ks + swz<D>(r, c), k_cache + off);
          cp_async16(vs + swz<D>(r, c), v_cache + off);
        } else {
          // rows past the sequence end are masked below, but V must not hold NaN garbage
          *reinterpret_cast<uint4*>(smem + (vs - q_smem) + swz<D>(r, c)) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(smem + (ks - q_smem) + swz<D>(r, c)) = make_uint4(0, 0, 0, 0);
        }
      }
    }
    cp_async_commit();
  };

  float o[D / 8][4];
#pragma unroll
  for (int n = 0; n < D / 8; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
  RowState st = {-INFINITY, -INFINITY, 0.f, 0.f};
  const float scale_log2 = scale * 1.4426950408889634f;

  issue(tile_lo, 0);
  int stage = 0;
  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    issue(tile + 1, stage ^ 1);
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t ks = k_smem0 + stage * KTILE_BYTES, vs = v_smem0 + stage * KTILE_BYTES;
#pragma unroll
    for (int kk = 0; kk < PF_BN / 16; ++kk) {
      const int key_base = tile * PF_BN + kk * 16;
      // skip 16-key steps that are entirely in this warp's causal future
      if (key_base > prefix + qt * PF_BM + warp * 16 + 15) continue;
      float s0[4] = {0, 0, 0, 0}, s1[4] = {0, 0, 0, 0};
      qk_16x16<D>(s0, s1, qf, ks, kk * 16, lane);
      const int c0 = key_base + 2 * t4;
      auto dead = [&](int key, int pos) {
        return key > pos || key >= L || (window > 0 && key <= pos - window);
      };
      if (dead(c0, pos0)) s0[0] = -INFINITY;
      if (dead(c0 + 1, pos0)) s0[1] = -INFINITY;
      if (dead(c0, pos1)) s0[2] = -INFINITY;
      if (dead(c0 + 1, pos1)) s0[3] = -INFINITY;
      if (dead(c0 + 8, pos0)) s1[0] = -INFINITY;
      if (dead(c0 + 9, pos0)) s1[1] = -INFINITY;
      if (dead(c0 + 8, pos1)) s1[2] = -INFINITY;
      if (dead(c0 + 9, pos1)) s1[3] = -INFINITY;
      uint32_t p0, p1, p2, p3;
      softmax_update<D>(s0, s1, st, o, scale_log2, p0, p1, p2, p3);
      pv_16x16<D>(o, p0, p1, p2, p3, vs, kk * 16, lane);
    }
    __syncthreads();
    stage ^= 1;
  }
  cp_async_wait<0>();

  const float inv0 = st.l0 > 0.f ? 1.f / st.l0 : 0.f;
  const float inv1 = st.l1 > 0.f ? 1.f / st.l1 : 0.f;
  if (row0 < n_new) {
    __nv_bfloat16* dst = out + ((long long)(q_begin + row0) * Hq + h) * D;
#pragma unroll
    for (int n = 0; n < D / 8; ++n)
      *reinterpret_cast<uint32_t*>(dst + n * 8 + 2 * t4) = pack_bf16x2(o[n][0] * inv0, o[n][1] * inv0);
    if (lse != nullptr && t4 == 0)
      lse[(long long)(q_begin + row0) * Hq + h] = (st.m0 + log2f(st.l0)) * 0.6931471805599453f;
  }
  if (row1 < n_new) {
    __nv_bfloat16* dst = out + ((long long)(q_begin + row1) * Hq + h) * D;
#pragma unroll
    for (int n = 0; n < D / 8; ++n)
      *reinterpret_cast<uint32_t*>(dst + n * 8 + 2 * t4) = pack_bf16x2(o[n][2] * inv1, o[n][3] * inv1);
    if (lse != nullptr && t4 == 0)
      lse[(long long)(q_begin + row1) * Hq + h] = (st.m1 + log2f(st.l1)) * 0.6931471805599453f;
  }
}

template <int D>
constexpr int decode_smem_bytes() {
  return 16 * D * 2 + DEC_WARPS * DEC_STAGES * 2 * KV_BLOCK * D * 2;
}
template <int D>
constexpr int decode_tma_smem_bytes() {
  return 1024 + DEC_WARPS * dec_tma_stages<D>() * 2 * KV_BLOCK * D * 2 + 16 * D * 2;
}
template <int D>
constexpr int prefill_smem_bytes() {
  return PF_BM * D * 2 + 4 * PF_BN * D * 2;
}

}  // namespace rb

using namespace rb;

extern "C" void rb_attn_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

// Function attributes (the dynamic shared-memory opt-in) belong to a device, so the "already set" flags of the
// launchers below are kept per device: a process that drives several GPUs sets them on each.
#define RB_MAX_DEVICES 64
static int current_device_index() {
  int dev = -1;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= RB_MAX_DEVICES) return -1;
  return dev;
}

// Scratch needed by rb_paged_decode when num_splits > 1, in floats.
extern "C" long long rb_paged_decode_workspace_floats(int B, int Hq, int D, int num_splits) {
  if (num_splits <= 1) return 0;
  return (long long)B * Hq * num_splits * (D + 2);
}

extern "C" int rb_paged_decode(const void* q, const void* k_cache, const void* v_cache, const int* block_tables,
                               const int* seq_lens, void* out, float* workspace, int B, int Hq, int Hkv, int D,
                               int max_blocks, int num_blocks, int block_size, int num_splits, float scale,
                               int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (block_size != KV_BLOCK || Hq % Hkv != 0 || Hq / Hkv > 8 || num_splits < 1) return -1;
  if (num_splits > 1 && workspace == nullptr) return -1;
  float* part_o = workspace;
  float* part_ml = workspace ? workspace + (long long)B * Hq * num_splits * D : nullptr;
  dim3 grid(num_splits, Hkv, B);
  static const bool use_cpasync = getenv("RB_DECODE_CPASYNC") != nullptr;
  if (!use_cpasync) {
    CUtensorMap kmap, vmap;
    const unsigned long long rows = (unsigned long long)num_blocks * Hkv * KV_BLOCK;
    if (tma_map_2d_bf16(&kmap, k_cache, rows, D, D, KV_BLOCK) != 0) return -20;
    if (tma_map_2d_bf16(&vmap, v_cache, rows, D, D, KV_BLOCK) != 0) return -21;
#define LAUNCH_DEC_TMA(DD)                                                                                    \
  do {                                                                                                        \
    static bool attr[RB_MAX_DEVICES] = {};   /* the opt-in above 48 KB is a per-device function attribute */  \
    const int dev_ = current_device_index();                                                                  \
    if (dev_ < 0) return -10;                                                                                 \
    if (!attr[dev_]) {                                                                                        \
      if (cudaFuncSetAttribute(paged_decode_tma_kernel<DD>, cudaFuncAttributeMaxDynamicSharedMemorySize,      \
                               decode_tma_smem_bytes<DD>()) != cudaSuccess) return -10;                       \
      attr[dev_] = true;                                                                                      \
    }                                                                                                         \
    launch_kernel(paged_decode_tma_kernel<DD>, grid, dim3(DEC_WARPS * 32), decode_tma_smem_bytes<DD>(), stream, \
        (const __nv_bfloat16*)q, kmap, vmap, block_tables, seq_lens, (__nv_bfloat16*)out, part_o, part_ml, Hq, \
        Hkv, max_blocks, num_blocks, num_splits, scale, status);                                              \
    if (num_splits > 1)                                                                                       \
      launch_kernel(decode_merge_kernel<DD>, dim3(B * Hq), dim3(DD), 0, stream, (const float*)part_o,         \
                    (const float*)part_ml, (__nv_bfloat16*)out, num_splits);                                  \
  } while (0)
    if (D == 64) LAUNCH_DEC_TMA(64);
    else if (D == 128) LAUNCH_DEC_TMA(128);
    else return -1;
#undef LAUNCH_DEC_TMA
    return cudaGetLastError() == cudaSuccess ? 0 : -11;
  }
#define LAUNCH_DEC(DD)                                                                                        \
  do {                                                                                                        \
    static bool attr[RB_MAX_DEVICES] = {};                                                                    \
    const int dev_ = current_device_index();                                                                  \
    if (dev_ < 0) return -10;                                                                                 \
    if (!attr[dev_]) {                                                                                        \
      if (cudaFuncSetAttribute(paged_decode_kernel<DD>, cudaFuncAttributeMaxDynamicSharedMemorySize,          \
                               decode_smem_bytes<DD>()) != cudaSuccess) return -10;                           \
      attr[dev_] = true;                                                                                      \
    }                                                                                                         \
    launch_kernel(paged_decode_kernel<DD>, grid, dim3(DEC_WARPS * 32), decode_smem_bytes<DD>(), stream,        \
        (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, block_tables,  \
        seq_lens, (__nv_bfloat16*)out, part_o, part_ml, Hq, Hkv, max_blocks, num_blocks, num_splits, scale,   \
        status);                                                                                              \
    if (num_splits > 1)                                                                                       \
      launch_kernel(decode_merge_kernel<DD>, dim3(B * Hq), dim3(DD), 0, stream, (const float*)part_o,         \
                    (const float*)part_ml, (__nv_bfloat16*)out, num_splits);                                  \
  } while (0)
  if (D == 64) LAUNCH_DEC(64);
  else if (D == 128) LAUNCH_DEC(128);
  else return -1;
#undef LAUNCH_DEC
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

extern "C" int rb_paged_prefill(const void* q, const void* k_cache, const void* v_cache, const int* block_tables,
                                const int* cu_q, const int* seq_lens, void* out, float* lse, int B, int max_new,
                                int Hq, int Hkv, int D, int max_blocks, int num_blocks, int block_size, float scale,
                                int window, int* status, cudaStream_t stream) {
  if (B <= 0 || max_new <= 0) return 0;
  if (block_size != KV_BLOCK || Hq % Hkv != 0) return -1;
  dim3 grid((max_new + PF_BM - 1) / PF_BM, Hq, B);
#define LAUNCH_PF(DD)                                                                                         \
  do {                                                                                                        \
    static bool attr[RB_MAX_DEVICES] = {};                                                                    \
    const int dev_ = current_device_index();                                                                  \
    if (dev_ < 0) return -10;                                                                                 \
    if (!attr[dev_]) {                                                                                        \
      if (cudaFuncSetAttribute(paged_prefill_kernel<DD>, cudaFuncAttributeMaxDynamicSharedMemorySize,         \
                               prefill_smem_bytes<DD>()) != cudaSuccess) return -10;                          \
      attr[dev_] = true;                                                                                      \
    }                                                                                                         \
    paged_prefill_kernel<DD><<<grid, PF_WARPS * 32, prefill_smem_bytes<DD>(), stream>>>(                       \
        (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, block_tables,  \
        cu_q, seq_lens, (__nv_bfloat16*)out, lse, Hq, Hkv, max_blocks, num_blocks, scale, window, status);    \
  } while (0)
  if (D == 64) LAUNCH_PF(64);
  else if (D == 128) LAUNCH_PF(128);
  else return -1;
#undef LAUNCH_PF
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

// ------------------------------------------------------------------------------------------
// Attention whose values are its keys (ops/keyvalue.py): one cached row per token and kv head, [num_blocks, G, 16, D]. The joint
// projection of a token is q [H, D] | k [G, D] | gate [H, D]; the softmax denominator also holds exp(sink[h]), and the
// output is multiplied by sigmoid(gate) element by element.
// ------------------------------------------------------------------------------------------
namespace rb {

__device__ __forceinline__ float kv_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float kv_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float kv_to_f(float v) { return v; }
__device__ __forceinline__ float kv_to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void kv_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void kv_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Queries times 1 + coef ln(floor((p + 1) / every) + 1) in place, keys into the cache. One CTA per token, 16 bytes at a time.
template <typename T>
__global__ void kv_append_kernel(T* __restrict__ proj, long long ld, const int* __restrict__ positions, const int* __restrict__ slots, float coef,
                                 int every, T* __restrict__ cache, int num_blocks, int H, int G, int D, int* status) {
  constexpr int V = 16 / sizeof(T);
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  T* row = proj + t * ld;
  const int slot = slots[t];
  const float f = 1.f + coef * logf((float)((positions[t] + 1) / every) + 1.f);
  if (f != 1.f)
    for (int i = threadIdx.x * V; i < H * D; i += blockDim.x * V) {
      union { uint4 u; T e[V]; } x;
      x.u = *reinterpret_cast<const uint4*>(row + i);
#pragma unroll
      for (int j = 0; j < V; ++j) kv_store(&x.e[j], kv_to_f(x.e[j]) * f);
      *reinterpret_cast<uint4*>(row + i) = x.u;
    }
  if (slot < 0) return;
  const int blk = slot / KV_BLOCK;
  if (blk >= num_blocks) { if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX); return; }
  for (int i = threadIdx.x * V; i < G * D; i += blockDim.x * V)
    *reinterpret_cast<uint4*>(cache + (((long long)blk * G + i / D) * KV_BLOCK + slot % KV_BLOCK) * D + i % D) =
        *reinterpret_cast<const uint4*>(row + H * D + i);
}

// Which keys j <= i a query at position i sees: all, the last `size` (window), or those of its own chunk of `size` positions.
struct KeySpan {
  int window, chunk;       // 0: none
};
__device__ __forceinline__ int first_key(const KeySpan& s, int position) {
  if (s.window > 0) return max(0, position - s.window + 1);
  return s.chunk > 0 ? position - position % s.chunk : 0;
}

// What multiplies a head's output: the sigmoid of one number per channel (activation type) or per head (fp32), or nothing;
// times a constant.
struct OutputGate {
  const void* channels;    // [T, ld_channels], H * D of a row
  long long ld_channels;
  const float* heads;      // [T, ld_heads], H of a row
  long long ld_heads;
  float scale;
};
template <typename T>
__device__ __forceinline__ float output_gate(const OutputGate& g, long long t, int h, int D, int d) {
  if (g.channels != nullptr) return g.scale * kv_sigmoid(kv_to_f(reinterpret_cast<const T*>(g.channels)[t * g.ld_channels + h * D + d]));
  return g.heads != nullptr ? g.scale * kv_sigmoid(g.heads[t * g.ld_heads + h]) : g.scale;
}

// Weight of the softmax sink relative to the maximum M (base 2); no sink: none.
__device__ __forceinline__ float sink_weight(const float* sink, int h, float M) {
  return sink != nullptr ? exp2f(sink[h] * 1.4426950408889634f - M) : 0.f;
}

// Decode: the structure of paged_decode_tma_kernel for up to 16 query heads per CTA (blockIdx.y = kv head x chunk of 16 query
// heads). SHARED: values are keys, one tile serves as both, two blocks (32 keys) per stage; otherwise a stage is a block of
// keys and one of values. The sums of weights stay per thread until the end, and the accumulators are rescaled only when a
// row's maximum moves.
template <int D, bool SHARED>
__host__ __device__ constexpr int kv_dec_stages() { return SHARED && D == 64 ? 4 : 3; }      // 64 / 96 KB of ring per CTA, 48 / 96 KB
constexpr int KV_MERGE_LD_PAD = 4;

template <int D, bool SHARED>
__global__ void __launch_bounds__(DEC_WARPS * 32)
kv_decode_kernel(const __nv_bfloat16* __restrict__ q, long long ld, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                 const int* __restrict__ block_tables, const int* __restrict__ seq_lens, const float* __restrict__ sink, const OutputGate gate,
                 __nv_bfloat16* __restrict__ out, long long ldo, float* __restrict__ part_o, float* __restrict__ part_ml, int H, int Hkv,
                 int bt_stride, int num_blocks, int num_splits, const KeySpan span, float scale, int* status) {
  constexpr int CH = D / 8;
  constexpr int NB = SHARED ? 2 : 1;                               // blocks of keys in a stage
  constexpr int BLK_BYTES = KV_BLOCK * D * 2, TILE_BYTES = 2 * BLK_BYTES;
  constexpr int ST = kv_dec_stages<D, SHARED>();
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ __align__(8) uint64_t bars[DEC_WARPS][ST];
  __shared__ int abort_flag;
  pdl_launch_dependents();
  const int G = H / Hkv, chunks = (G + 15) / 16;
  const int split = blockIdx.x, kvh = blockIdx.y / chunks, b = blockIdx.z;
  const int h0 = kvh * G + (blockIdx.y % chunks) * 16;      // first query head of this CTA
  const int rows = min(16, kvh * G + G - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t ring0 = (smem_u32(smem) + 1023u) & ~1023u;
  uint8_t* ring_ptr = smem + (ring0 - smem_u32(smem));
  const uint32_t k_smem = ring0 + warp * (ST * TILE_BYTES);
  uint8_t* q_ptr = ring_ptr + DEC_WARPS * ST * TILE_BYTES;
  const uint32_t q_smem = smem_u32(q_ptr);
  if (threadIdx.x == 0) {
    abort_flag = 0;
    for (int w = 0; w < DEC_WARPS; ++w)
      for (int s2 = 0; s2 < ST; ++s2) mbar_init(smem_u32(&bars[w][s2]), 1);
    fence_mbar_init();
  }
  pdl_wait();
  const int L = seq_lens[b];
  const int n_blocks = (L + KV_BLOCK - 1) / KV_BLOCK, n_chunks = (n_blocks + NB - 1) / NB;
  const int key0 = L > 0 ? first_key(span, L - 1) : 0, c_first = key0 / (NB * KV_BLOCK);
  const int per = (n_chunks - c_first + num_splits - 1) / num_splits;
  const int c_begin = c_first + split * per;
  const int c_end = min(n_chunks, c_begin + per);
  for (int i = threadIdx.x; i < 16 * CH; i += blockDim.x) {
    const int r = i / CH, c = i % CH;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < rows) v = *reinterpret_cast<const uint4*>(q + b * ld + (h0 + r) * D + c * 8);
    *reinterpret_cast<uint4*>(q_ptr + swz<D>(r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[D / 16][4];
  {
    const int mat = lane >> 3, r = lane & 7;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
      ldsm_x4(q_smem + swz<D>((mat & 1) * 8 + r, 2 * ks + (mat >> 1)), qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
  }
  float o[D / 8][4];
#pragma unroll
  for (int n = 0; n < D / 8; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
  RowState st = {-INFINITY, -INFINITY, 0.f, 0.f};
  const float scale_log2 = scale * 1.4426950408889634f;
  volatile int* abortp = &abort_flag;
  const int first = c_begin + warp;
  const int n_my = first < c_end ? (c_end - first + DEC_WARPS - 1) / DEC_WARPS : 0;
  const int* bt_row = block_tables + (long long)b * bt_stride;
  auto load_ids = [&](int round) {
    const int j = round * 32 + lane, blk = NB * (first + (j / NB) * DEC_WARPS) + j % NB;
    return j / NB < n_my && blk < n_blocks ? __ldg(bt_row + blk) : num_blocks;     // past the end: out of bounds, zeros
  };
  int ids_round = 0, ids = load_ids(0), ids_next = load_ids(1);
  auto blocks_of = [&](int i) {   // all lanes, i uniform and non-decreasing
    if (i / (32 / NB) > ids_round) { ids = ids_next; ids_round = i / (32 / NB); ids_next = load_ids(ids_round + 1); }
    return make_int2(__shfl_sync(0xffffffffu, ids, (NB * i) & 31), __shfl_sync(0xffffffffu, ids, (NB * i + NB - 1) & 31));
  };
  auto issue = [&](int i, int2 blk) {   // lane 0 only
    const int stage = i % ST;
    if (blk.x < 0 || blk.x > num_blocks || blk.y < 0 || blk.y > num_blocks) { set_status(status, ST_BAD_INDEX); blk.x = blk.y = num_blocks; }
    const uint32_t bar = smem_u32(&bars[warp][stage]), ks = k_smem + stage * TILE_BYTES;
    mbar_expect_tx(bar, TILE_BYTES);
#pragma unroll
    for (int hx = 0; hx < D / 64; ++hx) {
      tma_load_2d(ks + hx * (KV_BLOCK * 128), &k_map, bar, hx * 64, (blk.x * Hkv + kvh) * KV_BLOCK);
      tma_load_2d(ks + BLK_BYTES + hx * (KV_BLOCK * 128), SHARED ? &k_map : &v_map, bar, hx * 64, (blk.y * Hkv + kvh) * KV_BLOCK);
    }
  };
  int issued = 0;
  for (; issued < ST - 1 && issued < n_my; ++issued) {
    const int2 blk = blocks_of(issued);
    if (lane == 0) issue(issued, blk);
  }
  bool ok = true;
  const int mat = lane >> 3, rr = lane & 7;
  for (int i = 0; i < n_my; ++i) {
    if (issued < n_my) {
      const int2 blk = blocks_of(issued);
      if (lane == 0) issue(issued, blk);
      ++issued;
    }
    const int stage = i % ST;
    ok = mbar_wait_bounded(smem_u32(&bars[warp][stage]), (uint32_t)((i / ST) & 1), abortp, status, ST_TIMEOUT_SMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) break;
    const uint32_t ks = k_smem + stage * TILE_BYTES, vs = SHARED ? ks : ks + BLK_BYTES;
    float sc[2 * NB][4] = {};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
      for (int half = 0; half < NB; ++half) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4(ks + half * BLK_BYTES + swz_tma<D>((mat >> 1) * 8 + rr, 2 * kk + (mat & 1)), b0, b1, b2, b3);
        mma_16816(sc[2 * half], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b0, b1);
        mma_16816(sc[2 * half + 1], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b2, b3);
      }
    const int tile0 = (first + i * DEC_WARPS) * NB * KV_BLOCK, tok0 = tile0 + 2 * (lane & 3);
    if (tile0 + NB * KV_BLOCK > L || tile0 < key0) {
#pragma unroll
      for (int n8 = 0; n8 < 2 * NB; ++n8) {
        if (tok0 + 8 * n8 >= L || tok0 + 8 * n8 < key0) sc[n8][0] = sc[n8][2] = -INFINITY;
        if (tok0 + 8 * n8 + 1 >= L || tok0 + 8 * n8 + 1 < key0) sc[n8][1] = sc[n8][3] = -INFINITY;
      }
    }
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int n8 = 0; n8 < 2 * NB; ++n8) {
      mx0 = fmaxf(mx0, fmaxf(sc[n8][0], sc[n8][1]));
      mx1 = fmaxf(mx1, fmaxf(sc[n8][2], sc[n8][3]));
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2)) * scale_log2;
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2)) * scale_log2;
    if (__any_sync(0xffffffffu, mx0 > st.m0 || mx1 > st.m1)) {      // (every tile has a visible key: the maximum is finite)
      const float n0 = fmaxf(st.m0, mx0), n1 = fmaxf(st.m1, mx1);
      const float c0 = exp2f(st.m0 - n0), c1 = exp2f(st.m1 - n1);
      st.m0 = n0; st.m1 = n1;
      st.l0 *= c0; st.l1 *= c1;
#pragma unroll
      for (int n8 = 0; n8 < D / 8; ++n8) { o[n8][0] *= c0; o[n8][1] *= c0; o[n8][2] *= c1; o[n8][3] *= c1; }
    }
    uint32_t pk[2 * NB][2];
#pragma unroll
    for (int n8 = 0; n8 < 2 * NB; ++n8) {
      const float e0 = kv_exp2(fmaf(sc[n8][0], scale_log2, -st.m0)), e1 = kv_exp2(fmaf(sc[n8][1], scale_log2, -st.m0));
      const float f0 = kv_exp2(fmaf(sc[n8][2], scale_log2, -st.m1)), f1 = kv_exp2(fmaf(sc[n8][3], scale_log2, -st.m1));
      st.l0 += e0 + e1;
      st.l1 += f0 + f1;
      pk[n8][0] = pack_bf16x2(e0, e1);
      pk[n8][1] = pack_bf16x2(f0, f1);
    }
#pragma unroll
    for (int dp = 0; dp < D / 16; ++dp)
#pragma unroll
      for (int half = 0; half < NB; ++half) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(vs + half * BLK_BYTES + swz_tma<D>((mat & 1) * 8 + rr, 2 * dp + (mat >> 1)), b0, b1, b2, b3);
        mma_16816(o[2 * dp], pk[2 * half][0], pk[2 * half][1], pk[2 * half + 1][0], pk[2 * half + 1][1], b0, b1);
        mma_16816(o[2 * dp + 1], pk[2 * half][0], pk[2 * half][1], pk[2 * half + 1][0], pk[2 * half + 1][1], b2, b3);
      }
    __syncwarp();   // every lane is done with this stage before lane 0 refills it
  }
  if (!ok && lane == 0) {
    for (int j = max(0, issued - ST); j < issued; ++j) {   // no copy may land after the CTA has gone
      const uint64_t t0 = globaltimer_ns();
      while (!mbar_try_wait(smem_u32(&bars[warp][j % ST]), (uint32_t)((j / ST) & 1)))
        if (globaltimer_ns() - t0 > 50000000ull) break;
    }
  }
  __syncthreads();

  constexpr int LD = D + KV_MERGE_LD_PAD;
  float* mo = reinterpret_cast<float*>(ring_ptr);                   // [DEC_WARPS][16][LD]
  float* mml = mo + DEC_WARPS * 16 * LD;                            // [DEC_WARPS][16][2]
  const int g = lane >> 2, tq = lane & 3;
  st.l0 += __shfl_xor_sync(0xffffffffu, st.l0, 1);
  st.l1 += __shfl_xor_sync(0xffffffffu, st.l1, 1);
  st.l0 += __shfl_xor_sync(0xffffffffu, st.l0, 2);
  st.l1 += __shfl_xor_sync(0xffffffffu, st.l1, 2);
#pragma unroll
  for (int n = 0; n < D / 8; ++n) {
    *reinterpret_cast<float2*>(mo + (warp * 16 + g) * LD + n * 8 + 2 * tq) = make_float2(o[n][0], o[n][1]);
    *reinterpret_cast<float2*>(mo + (warp * 16 + g + 8) * LD + n * 8 + 2 * tq) = make_float2(o[n][2], o[n][3]);
  }
  if (tq == 0) {
    mml[(warp * 16 + g) * 2] = st.m0;
    mml[(warp * 16 + g) * 2 + 1] = st.l0;
    mml[(warp * 16 + g + 8) * 2] = st.m1;
    mml[(warp * 16 + g + 8) * 2 + 1] = st.l1;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < rows * D; i += blockDim.x) {
    const int r = i / D, d = i % D, h = h0 + r;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < DEC_WARPS; ++w) M = fmaxf(M, mml[(w * 16 + r) * 2]);
    float acc = 0.f, l = 0.f;
    if (M != -INFINITY) {
#pragma unroll
      for (int w = 0; w < DEC_WARPS; ++w) {
        const float e = exp2f(mml[(w * 16 + r) * 2] - M);
        acc += e * mo[(w * 16 + r) * LD + d];
        l += e * mml[(w * 16 + r) * 2 + 1];
      }
    }
    if (num_splits == 1) {
      float y = 0.f;
      if (l > 0.f) y = acc / (l + sink_weight(sink, h, M)) * output_gate<__nv_bfloat16>(gate, b, h, D, d);
      out[b * ldo + h * D + d] = __float2bfloat16_rn(y);
    } else {
      const long long pi = ((long long)b * H + h) * num_splits + split;
      part_o[pi * D + d] = acc;
      if (d == 0) { part_ml[pi * 2] = M; part_ml[pi * 2 + 1] = l; }
    }
  }
}

template <int D>
__global__ void kv_decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const OutputGate gate,
                                       const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, long long ldo, int H, int num_splits) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, d = threadIdx.x;
  const long long b = blockIdx.y, bh = b * H + h;
  float M = -INFINITY;
  for (int s = 0; s < num_splits; ++s) M = fmaxf(M, part_ml[(bh * num_splits + s) * 2]);
  float acc = 0.f, l = 0.f, y = 0.f;
  if (M != -INFINITY) {
    for (int s = 0; s < num_splits; ++s) {
      const float e = exp2f(part_ml[(bh * num_splits + s) * 2] - M);
      acc += e * part_o[(bh * num_splits + s) * D + d];
      l += e * part_ml[(bh * num_splits + s) * 2 + 1];
    }
    y = acc / (l + sink_weight(sink, h, M)) * output_gate<__nv_bfloat16>(gate, b, h, D, d);
  }
  out[b * ldo + h * D + d] = __float2bfloat16_rn(y);
}

// Any head size up to 512 and either number format, a warp per (token, query head): the exact mode and sizes without a
// tensor-core kernel. Lanes take one key each for the scores and 1/32 of the channels for the sums.
constexpr int KVS_WARPS = 4, KVS_MAX_D = 512;

template <typename T>
__global__ void __launch_bounds__(KVS_WARPS * 32)
kv_simple_kernel(const T* __restrict__ qrows, long long ld, const T* __restrict__ keys, const T* __restrict__ values,
                 const int* __restrict__ block_tables, const int* __restrict__ cu_q, const int* __restrict__ seq_lens, const float* __restrict__ sink,
                 const OutputGate gate, T* __restrict__ out, long long ldo, int H, int G, int D, int bt_stride, int num_blocks, int rows,
                 const KeySpan span, float scale, int* status) {
  extern __shared__ float kvs_q[];       // [KVS_WARPS][D]
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z, kvh = h / (H / G);
  pdl_wait();
  int t0 = b, t1 = b + 1;
  if (cu_q != nullptr) { t0 = cu_q[b]; t1 = cu_q[b + 1]; }
  const int t = t0 + blockIdx.x * KVS_WARPS + warp;
  if (t >= t1) return;                                     // (no CTA-wide synchronisation below)
  if (t >= rows) { if (lane == 0) set_status(status, ST_BAD_INDEX); return; }
  const int n_keys = seq_lens[b] - (t1 - 1 - t);           // keys this token sees
  T* dst = out + t * ldo + h * D;
  if (n_keys <= 0) {
    for (int d = lane; d < D; d += 32) kv_store(dst + d, 0.f);
    return;
  }
  float* q = kvs_q + warp * D;
  for (int d = lane; d < D; d += 32) q[d] = kv_to_f(qrows[t * ld + h * D + d]) * scale;
  __syncwarp();
  float o[KVS_MAX_D / 32];
#pragma unroll
  for (int i = 0; i < KVS_MAX_D / 32; ++i) o[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  if (sink != nullptr) { m = sink[h]; l = 1.f; }           // the sink: a key of weight exp(sink) without a value
  for (int k0 = first_key(span, n_keys - 1); k0 < n_keys; k0 += 32) {
    const int j = k0 + lane;
    float s = -INFINITY;
    long long row = 0;
    if (j < n_keys) {
      int blk = block_tables[(long long)b * bt_stride + j / KV_BLOCK];
      if (blk < 0 || blk >= num_blocks) { set_status(status, ST_BAD_INDEX); blk = 0; }
      row = (((long long)blk * G + kvh) * KV_BLOCK + j % KV_BLOCK) * D;
      s = 0.f;
      for (int d = 0; d < D; ++d) s = fmaf(q[d], kv_to_f(keys[row + d]), s);
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float c = expf(m - m_new), p = j < n_keys ? expf(s - m_new) : 0.f;
    l = l * c + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < KVS_MAX_D / 32; ++i) o[i] *= c;
    const int n = min(32, n_keys - k0);
    for (int u = 0; u < n; ++u) {
      const float pu = __shfl_sync(0xffffffffu, p, u);
      const long long ru = __shfl_sync(0xffffffffu, row, u);
#pragma unroll
      for (int i = 0; i < KVS_MAX_D / 32; ++i)
        if (lane + 32 * i < D) o[i] = fmaf(pu, kv_to_f(values[ru + lane + 32 * i]), o[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < KVS_MAX_D / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < D) kv_store(dst + d, o[i] / l * output_gate<T>(gate, t, h, D, d));
  }
}

// out *= sigmoid(gate) * exp(lse) / (exp(lse) + exp(sink)) for token rows [row0, row0 + n): what the plain softmax of the
// long-portion kernel lacks.
__global__ void kv_gate_kernel(__nv_bfloat16* __restrict__ out, const float* __restrict__ lse, const float* __restrict__ sink,
                               const __nv_bfloat16* __restrict__ gate, long long ld, int H, int D, int row0, int n, int Tq) {
  pdl_launch_dependents();
  pdl_wait();
  const int vpr = H * D / 8;
  const long long total = (long long)n * vpr;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = row0 + i / vpr;
    const int c = (int)(i % vpr) * 8, h = c / D;
    const float f = kv_sigmoid(lse[(long long)h * Tq + t] - sink[h]);
    uint4* po = reinterpret_cast<uint4*>(out + t * H * D + c);
    const uint4 g = *reinterpret_cast<const uint4*>(gate + t * ld + c);
    uint4 v = *po;
    auto one = [&](uint32_t x, uint32_t y) {
      const float2 a = unpack_bf16x2(x), z = unpack_bf16x2(y);
      return pack_bf16x2(a.x * f * kv_sigmoid(z.x), a.y * f * kv_sigmoid(z.y));
    };
    v.x = one(v.x, g.x); v.y = one(v.y, g.y); v.z = one(v.z, g.z); v.w = one(v.w, g.w);
    *po = v;
  }
}

// ------------------------------------------------------------------------------------------
// Grouped attention with cached keys and values: everything between the joint projection and the attention.
// Every projected channel goes through its causal convolution (if there is one), queries and keys through the norm and the rotation;
// queries land in a buffer with heads padded to DP channels, keys and values in the cache. Look back: history.cuh, over the raw
// projected values.
// ------------------------------------------------------------------------------------------
constexpr int GA_THREADS = 256, GA_MAX_DP = 512;
enum { GA_NORM_NONE = 0, GA_NORM_PROJECTION = 1, GA_NORM_HEAD = 2 };

struct GroupedAppend {
  const void* proj;        // [T, ld]: q at 0, k at k_col, v at v_col (multiples of 8); `channels` columns in all
  long long ld;
  int k_col, v_col, channels;
  const float* conv;       // [taps, channels] or null
  int taps;
  void* hist;              // [slots, taps - 1, channels]
  History rows;
  const int* slots;        // [T] places in the cache, negative: not stored
  const float* q_norm;     // [H * dim], projection norm
  const float* k_norm;     // [G * dim]
  const float* q_factor;   // [H] of the queries, or null
  int norm;
  float eps;
  const float* table;      // [positions, half, 2] cos, sin
  int half, interleaved, max_pos;
  void* q;                 // [T, H * DP]
  void* keys;              // [num_blocks, G, 16, DP]
  void* values;
  int num_blocks, H, G, dim, vdim, DP, T;
  int* status;
};

__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(a, b); }
__device__ __forceinline__ void store8(float* p, const float (&x)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(x[0], x[1], x[2], x[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(x[4], x[5], x[6], x[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&x)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
}

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&x)[8]) {
  constexpr int V = 16 / sizeof(T);
#pragma unroll
  for (int i = 0; i < 8 / V; ++i) {
    union { uint4 u; T e[V]; } a;
    a.u = reinterpret_cast<const uint4*>(p)[i];
#pragma unroll
    for (int j = 0; j < V; ++j) x[i * V + j] = kv_to_f(a.e[j]);
  }
}

// TOK rows per CTA (the convolution's weights are loaded once for them); STEPS: 64 channels of a padded head each; WHOLE: heads of
// queries, keys and values have DP channels, none of them padding.
template <typename T, int TOK, int STEPS, bool WHOLE>
__global__ void __launch_bounds__(GA_THREADS, 4) grouped_append_kernel(const GroupedAppend p) {
  extern __shared__ float ga_rows[];                      // [TOK][v_col] q and k channels, laid out as in the projection
  __shared__ float red[TOK][2][GA_THREADS / 32];
  __shared__ RowPlace places[TOK];
  __shared__ int dests[TOK];
  __shared__ long long caches[TOK];                       // element of the row in the caches, + head * 16 * DP
  const int DP = WHOLE ? STEPS * 64 : p.DP, dim = WHOLE ? DP : p.dim, vdim = WHOLE ? DP : p.vdim;
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * TOK, n_tok = min(TOK, p.T - t0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* rows = reinterpret_cast<const T*>(p.proj);
  T* hist = reinterpret_cast<T*>(p.hist);
  if (threadIdx.x < TOK) {
    RowPlace place{0, 0, -1};
    int slot = -1;
    if (threadIdx.x < n_tok) {
      const int t = t0 + threadIdx.x;
      place.position = p.rows.positions[t];
      if (p.taps > 1) place = row_place(p.rows, t, p.status);
      slot = p.slots[t];
      if (slot >= 0 && slot / KV_BLOCK >= p.num_blocks) { set_status(p.status, ST_BAD_INDEX); slot = -1; }
      if (place.position < 0 || place.position >= p.max_pos) { set_status(p.status, ST_BAD_INDEX); place.position = 0; }
    }
    places[threadIdx.x] = place;
    dests[threadIdx.x] = slot;
    caches[threadIdx.x] = slot < 0 ? 0 : ((long long)(slot / KV_BLOCK) * p.G * KV_BLOCK + slot % KV_BLOCK) * DP;
  }
  __syncthreads();
  bool near = true;                                       // every row's look back lies in the batch
#pragma unroll
  for (int i = 0; i < TOK; ++i) near = near && (i >= n_tok || places[i].offset >= p.taps - 1);
  float ssq[TOK], ssk[TOK];
#pragma unroll
  for (int i = 0; i < TOK; ++i) ssq[i] = ssk[i] = 0.f;
  const int nq = p.H * dim, nk = p.G * dim, nv = p.G * vdim;
  for (int c = threadIdx.x * 8; c < p.channels; c += GA_THREADS * 8) {
    float x[TOK][8], u[8];
    const T* first = rows + (long long)t0 * p.ld + c;
#pragma unroll
    for (int i = 0; i < TOK; ++i)
      if (i < n_tok) load8(first + i * p.ld, x[i]);
    if (p.conv != nullptr) {
      if (TOK == 1)
#pragma unroll
        for (int j = 0; j < 8; ++j) u[j] = x[0][j];
      const float* taps = p.conv + (long long)(p.taps - 1) * p.channels + c;
      float w[8];
      load8(taps, w);
#pragma unroll
      for (int i = 0; i < TOK; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) x[i][j] *= w[j];
      for (int d = 1; d < p.taps; ++d) {
        taps -= p.channels;
        load8(taps, w);
#pragma unroll
        for (int i = 0; i < TOK; ++i) {
          if (i >= n_tok) continue;
          const T* back = near ? first + (i - d) * p.ld : row_before(places[i], d, rows + c, p.ld, t0 + i, (const T*)hist + c, p.taps - 1, p.channels);
          if (near || back != nullptr) {
            float y[8];
            load8(back, y);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[i][j] = fmaf(w[j], y[j], x[i][j]);
          }
        }
      }
      if (TOK == 1 && p.taps > 1 && p.rows.cu_q == nullptr && places[0].slot >= 0) {    // one row per sequence: this thread moves its own channels on
        T* mine = hist + (long long)places[0].slot * (p.taps - 1) * p.channels + c;
        for (int d = p.taps - 2; d >= 1; --d)
#pragma unroll
          for (int i = 0; i < (int)(8 * sizeof(T) / 16); ++i)
            reinterpret_cast<uint4*>(mine + (long long)d * p.channels)[i] = reinterpret_cast<const uint4*>(mine + (long long)(d - 1) * p.channels)[i];
        store8(mine, u);
      }
    }
    if (c >= p.v_col) {
      const int v0 = c - p.v_col;
      if (WHOLE || vdim % 8 == 0) {
        const int at = v0 / vdim * KV_BLOCK * DP + v0 % vdim;
        if (v0 < nv)
#pragma unroll
          for (int i = 0; i < TOK; ++i)
            if (dests[i] >= 0) store8(reinterpret_cast<T*>(p.values) + caches[i] + at, x[i]);
      } else {
#pragma unroll 1
        for (int i = 0; i < TOK; ++i)
          for (int j = 0; j < 8; ++j)
            if (dests[i] >= 0 && v0 + j < nv) {
              float one = 0.f;
#pragma unroll
              for (int k = 0; k < TOK * 8; ++k)
                if (k == i * 8 + j) one = x[k >> 3][k & 7];
              kv_store(reinterpret_cast<T*>(p.values) + caches[i] + (v0 + j) / vdim * KV_BLOCK * DP + (v0 + j) % vdim, one);
            }
      }
    } else {
      const bool is_k = c >= p.k_col;
      const int n = is_k ? nk : nq, c0 = c - (is_k ? p.k_col : 0);
#pragma unroll
      for (int i = 0; i < TOK; ++i) {
        float4* dst = reinterpret_cast<float4*>(ga_rows + i * p.v_col + c);
        dst[0] = make_float4(x[i][0], x[i][1], x[i][2], x[i][3]);
        dst[1] = make_float4(x[i][4], x[i][5], x[i][6], x[i][7]);
        if (p.norm == GA_NORM_PROJECTION) {
          float s = 0.f;
#pragma unroll
          for (int j = 0; j < 8; ++j)
            if (WHOLE || c0 + j < n) s = fmaf(x[i][j], x[i][j], s);
          if (is_k) ssk[i] += s; else ssq[i] += s;
        }
      }
    }
  }
  if (p.norm == GA_NORM_PROJECTION)
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      const float q = warp_sum(ssq[i]), k = warp_sum(ssk[i]);
      if (lane == 0) { red[i][0][warp] = q; red[i][1][warp] = k; }
    }
  __syncthreads();
  if (p.norm == GA_NORM_PROJECTION) {                     // sums -> factors, a thread each
    if (threadIdx.x < 2 * TOK) {
      const int i = threadIdx.x >> 1, is_k = threadIdx.x & 1;
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < GA_THREADS / 32; ++w) s += red[i][is_k][w];
      red[i][is_k][0] = 1.f / sqrtf(s / (float)(is_k ? nk : nq) + p.eps);
    }
    __syncthreads();
  }
  // A warp per head: lane e takes a pair of channels that the rotation turns, (2e, 2e + 1) or (e, e + half), or two that pass.
  const int heads = p.H + p.G, half = p.half;
  int i = 0, hd = warp;
  while (hd >= heads) { hd -= heads; ++i; }
  while (i < n_tok) {
    const bool is_k = hd >= p.H;
    const int head = is_k ? hd - p.H : hd;
    if (!is_k || dests[i] >= 0) {
      const float* src = ga_rows + i * p.v_col + (is_k ? p.k_col : 0) + head * dim;
      const float* w = p.norm == GA_NORM_PROJECTION ? (is_k ? p.k_norm : p.q_norm) + head * dim : nullptr;
      const float r = w != nullptr ? red[i][is_k][0] : 1.f;
      const float2* table = reinterpret_cast<const float2*>(p.table) + (long long)places[i].position * half;
      T* dst = is_k ? reinterpret_cast<T*>(p.keys) + caches[i] + head * KV_BLOCK * DP : reinterpret_cast<T*>(p.q) + ((long long)(t0 + i) * p.H + head) * DP;
      float y[STEPS][2], ss = 0.f;
#pragma unroll
      for (int j = 0; j < STEPS; ++j) {
        const int e = lane + j * 32;
        const bool turned = e < half;
        float a, b;
        if (turned && !p.interleaved) {
          a = src[e];
          b = src[e + half];
          if (w != nullptr) { a *= r * w[e]; b *= r * w[e + half]; }
        } else if (WHOLE) {
          const float2 v = *reinterpret_cast<const float2*>(src + 2 * e);
          a = v.x;
          b = v.y;
          if (w != nullptr) {
            const float2 f = *reinterpret_cast<const float2*>(w + 2 * e);
            a *= r * f.x;
            b *= r * f.y;
          }
        } else {
          a = 2 * e < dim ? src[2 * e] : 0.f;
          b = 2 * e + 1 < dim ? src[2 * e + 1] : 0.f;
          if (w != nullptr) {
            if (2 * e < dim) a *= r * w[2 * e];
            if (2 * e + 1 < dim) b *= r * w[2 * e + 1];
          }
        }
        if (turned) {
          const float2 cs = table[e];
          const float a0 = a;
          a = a0 * cs.x - b * cs.y;
          b = b * cs.x + a0 * cs.y;
        }
        y[j][0] = a;
        y[j][1] = b;
        ss = fmaf(a, a, fmaf(b, b, ss));
      }
      float f = 1.f;
      if (p.norm == GA_NORM_HEAD) f = 1.f / sqrtf(warp_sum(ss) / (float)dim + p.eps);
      if (!is_k && p.q_factor != nullptr) f *= p.q_factor[head];
#pragma unroll
      for (int j = 0; j < STEPS; ++j) {
        const int e = lane + j * 32;
        if (!WHOLE && 2 * e >= DP) continue;
        if (e < half && !p.interleaved) {
          kv_store(dst + e, y[j][0] * f);
          kv_store(dst + e + half, y[j][1] * f);
        } else {
          store2(dst + 2 * e, y[j][0] * f, y[j][1] * f);
        }
      }
    }
    hd += GA_THREADS / 32;
    while (hd >= heads) { hd -= heads; ++i; }
  }
}

template <typename T>
static cudaError_t launch_grouped_append(const GroupedAppend& p, cudaStream_t stream) {
  const int dev = current_device_index();
  if (dev < 0) return cudaErrorInvalidDevice;
  const size_t row = (size_t)p.v_col * 4;
  const bool several = p.rows.cu_q != nullptr && p.T >= 592 && 2 * row <= 100 * 1024;      // (rows of one sequence lie together)
  const bool whole = p.dim == p.DP && p.vdim == p.DP && p.H * p.dim == p.k_col;
#define RB_APPEND(TOK, STEPS, WHOLE)                                                                                           \
  do {                                                                                                                         \
    static bool attr[RB_MAX_DEVICES] = {};                                                                                     \
    if (!attr[dev]) {                                                                                                          \
      const cudaError_t e = cudaFuncSetAttribute(grouped_append_kernel<T, TOK, STEPS, WHOLE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
      if (e != cudaSuccess) return e;                                                                                          \
      attr[dev] = true;                                                                                                        \
    }                                                                                                                          \
    return launch_kernel(grouped_append_kernel<T, TOK, STEPS, WHOLE>, dim3((p.T + TOK - 1) / TOK), dim3(GA_THREADS), TOK * row, stream, p); \
  } while (0)
#define RB_APPEND_SIZE(STEPS, WHOLE)                                                                                           \
  do {                                                                                                                         \
    if (several) RB_APPEND(2, STEPS, WHOLE);                                                                                   \
    RB_APPEND(1, STEPS, WHOLE);                                                                                                \
  } while (0)
  if (p.DP == 64 && whole) RB_APPEND_SIZE(1, true);
  if (p.DP == 64) RB_APPEND_SIZE(1, false);
  if (p.DP == 128 && whole) RB_APPEND_SIZE(2, true);
  if (p.DP == 128) RB_APPEND_SIZE(2, false);
  RB_APPEND_SIZE(GA_MAX_DP / 64, false);
#undef RB_APPEND_SIZE
#undef RB_APPEND
}

template <int D, bool SHARED>
constexpr int kv_decode_smem_bytes() {
  const int ring = DEC_WARPS * kv_dec_stages<D, SHARED>() * 2 * KV_BLOCK * D * 2 + 16 * D * 2;
  const int merge = DEC_WARPS * 16 * (D + KV_MERGE_LD_PAD + 2) * 4;
  return 1024 + (ring > merge ? ring : merge);
}

}  // namespace rb

struct GroupedAppendArgs {       // mirrored by ops/grouped.py
  const void* proj; const float* conv; void* hist; const int* cu_q; const int* positions; const int* state_slots; const int* slots;
  const float* q_norm; const float* k_norm; const float* q_factor; const float* table; void* q; void* keys; void* values; int* status;
  long long ld;
  int k_col, v_col, channels, taps, B, num_state_slots, norm, half, interleaved, max_pos, num_blocks, H, G, dim, vdim, DP, T, dtype;
  float eps;
};

// Norm, rotation, convolution and cache append of a batch; with cu_q also moves the convolution's histories on (a second launch).
extern "C" int rb_grouped_append(const GroupedAppendArgs* a, cudaStream_t stream) {
  if (a->T <= 0) return 0;
  if (a->DP > GA_MAX_DP || a->DP % 64 != 0 || a->dim > a->DP || a->vdim > a->DP || a->G <= 0 || a->H % a->G != 0 || a->taps < 1) return -1;
  if (a->taps > 1 && (a->conv == nullptr || a->hist == nullptr || a->state_slots == nullptr)) return -1;
  if (a->k_col % 8 != 0 || a->v_col % 8 != 0 || a->channels % 8 != 0 || a->ld % 8 != 0 || 2 * a->half > a->dim) return -1;
  if ((size_t)a->v_col * 4 > 200 * 1024) return -1;
  GroupedAppend p;
  p.proj = a->proj; p.ld = a->ld; p.k_col = a->k_col; p.v_col = a->v_col; p.channels = a->channels;
  p.conv = a->conv; p.taps = a->taps; p.hist = a->hist;
  p.rows = History{a->cu_q, a->positions, a->state_slots, a->B, a->taps - 1, a->num_state_slots};
  p.slots = a->slots; p.q_norm = a->q_norm; p.k_norm = a->k_norm; p.q_factor = a->q_factor; p.norm = a->norm; p.eps = a->eps;
  p.table = a->table; p.half = a->half; p.interleaved = a->interleaved; p.max_pos = a->max_pos;
  p.q = a->q; p.keys = a->keys; p.values = a->values; p.num_blocks = a->num_blocks;
  p.H = a->H; p.G = a->G; p.dim = a->dim; p.vdim = a->vdim; p.DP = a->DP; p.T = a->T; p.status = a->status;
  cudaError_t e = a->dtype == 0 ? launch_grouped_append<__nv_bfloat16>(p, stream) : launch_grouped_append<float>(p, stream);
  if (e == cudaSuccess && a->cu_q != nullptr && a->taps > 1)
    e = a->dtype == 0 ? launch_history_update((const __nv_bfloat16*)a->proj, a->ld, p.rows, (__nv_bfloat16*)a->hist, a->channels, stream)
                      : launch_history_update((const float*)a->proj, a->ld, p.rows, (float*)a->hist, a->channels, stream);
  return e == cudaSuccess ? 0 : -11;
}

extern "C" int rb_kv_append(void* proj, long long ld, const int* positions, const int* slots, float coef, int every, void* cache, int num_blocks,
                            int H, int G, int D, int T, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (every <= 0 || H <= 0 || G <= 0 || D <= 0 || D % 8 != 0 || ld % 8 != 0) return -1;
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(kv_append_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, stream, (__nv_bfloat16*)proj, ld, positions, slots, coef, every,
                      (__nv_bfloat16*)cache, num_blocks, H, G, D, status);
  else
    e = launch_kernel(kv_append_kernel<float>, dim3(T), dim3(256), 0, stream, (float*)proj, ld, positions, slots, coef, every, (float*)cache,
                      num_blocks, H, G, D, status);
  return e == cudaSuccess ? 0 : -11;
}

// Gates of rb_kv_decode / rb_kv_simple: gate_channels (activation type, H * D per row) or gate_heads (fp32, H per row), or neither;
// sink may be null. values null (or equal to keys): values are keys. window / chunk: see KeySpan.
extern "C" int rb_kv_decode(const void* q, long long ld, const void* keys, const void* values, const int* block_tables, const int* seq_lens,
                            const float* sink, const void* gate_channels, long long ld_gate_channels, const float* gate_heads, long long ld_gate_heads,
                            float gate_scale, void* out, long long ldo, float* workspace, int B, int H, int G, int D, int bt_stride, int num_blocks,
                            int block_size, int num_splits, int window, int chunk, float scale, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (block_size != KV_BLOCK || G <= 0 || H % G != 0 || num_splits < 1 || (num_splits > 1 && workspace == nullptr) || B > 65535) return -1;
  CUtensorMap kmap, vmap;
  const bool shared = values == nullptr || values == keys;
  const unsigned long long rows = (unsigned long long)num_blocks * G * KV_BLOCK;
  if (tma_map_2d_bf16(&kmap, keys, rows, D, D, KV_BLOCK) != 0) return -20;
  if (tma_map_2d_bf16(&vmap, shared ? keys : values, rows, D, D, KV_BLOCK) != 0) return -20;
  float* part_ml = workspace != nullptr ? workspace + (long long)B * H * num_splits * D : nullptr;
  const dim3 grid(num_splits, G * ((H / G + 15) / 16), B);
  const OutputGate gate{gate_channels, ld_gate_channels, gate_heads, ld_gate_heads, gate_scale};
  const KeySpan span{window, chunk};
#define LAUNCH_KV(DD, SH)                                                                                      \
  do {                                                                                                         \
    static bool attr[RB_MAX_DEVICES] = {};                                                                     \
    const int dev_ = current_device_index();                                                                   \
    if (dev_ < 0) return -10;                                                                                  \
    if (!attr[dev_]) {                                                                                         \
      if (cudaFuncSetAttribute(kv_decode_kernel<DD, SH>, cudaFuncAttributeMaxDynamicSharedMemorySize,          \
                               kv_decode_smem_bytes<DD, SH>()) != cudaSuccess) return -10;                     \
      attr[dev_] = true;                                                                                       \
    }                                                                                                          \
    launch_kernel(kv_decode_kernel<DD, SH>, grid, dim3(DEC_WARPS * 32), kv_decode_smem_bytes<DD, SH>(), stream, \
                  (const __nv_bfloat16*)q, ld, kmap, vmap, block_tables, seq_lens, sink, gate,                 \
                  (__nv_bfloat16*)out, ldo, workspace, part_ml, H, G, bt_stride, num_blocks, num_splits, span, scale, status); \
    if (num_splits > 1)                                                                                        \
      launch_kernel(kv_decode_merge_kernel<DD>, dim3(H, B), dim3(DD), 0, stream, (const float*)workspace,      \
                    (const float*)part_ml, gate, sink, (__nv_bfloat16*)out, ldo, H, num_splits);               \
  } while (0)
  if (D == 64 && shared) LAUNCH_KV(64, true);
  else if (D == 128 && shared) LAUNCH_KV(128, true);
  else if (D == 64) LAUNCH_KV(64, false);
  else if (D == 128) LAUNCH_KV(128, false);
  else return -1;
#undef LAUNCH_KV
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

extern "C" int rb_kv_simple(const void* q, long long ld, const void* keys, const void* values, const int* block_tables, const int* cu_q,
                            const int* seq_lens, const float* sink, const void* gate_channels, long long ld_gate_channels, const float* gate_heads,
                            long long ld_gate_heads, float gate_scale, void* out, long long ldo, int H, int G, int D, int bt_stride, int num_blocks,
                            int B, int rows, int max_q, int window, int chunk, int dtype, float scale, int* status, cudaStream_t stream) {
  if (B <= 0 || rows <= 0) return 0;
  if (D > KVS_MAX_D || G <= 0 || H % G != 0 || H > 65535 || B > 65535) return -1;
  const dim3 grid((max_q + KVS_WARPS - 1) / KVS_WARPS, H, B);
  const size_t smem = (size_t)KVS_WARPS * D * 4;
  const OutputGate gate{gate_channels, ld_gate_channels, gate_heads, ld_gate_heads, gate_scale};
  const KeySpan span{window, chunk};
  if (values == nullptr) values = keys;
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(kv_simple_kernel<__nv_bfloat16>, grid, dim3(KVS_WARPS * 32), smem, stream, (const __nv_bfloat16*)q, ld,
                      (const __nv_bfloat16*)keys, (const __nv_bfloat16*)values, block_tables, cu_q, seq_lens, sink, gate, (__nv_bfloat16*)out, ldo, H, G,
                      D, bt_stride, num_blocks, rows, span, scale, status);
  else
    e = launch_kernel(kv_simple_kernel<float>, grid, dim3(KVS_WARPS * 32), smem, stream, (const float*)q, ld, (const float*)keys, (const float*)values,
                      block_tables, cu_q, seq_lens, sink, gate, (float*)out, ldo, H, G, D, bt_stride, num_blocks, rows, span, scale, status);
  return e == cudaSuccess ? 0 : -11;
}

extern "C" int rb_kv_gate(void* out, const float* lse, const float* sink, const void* gate, long long ld, int H, int D, int row0, int n, int Tq,
                          cudaStream_t stream) {
  if (n <= 0) return 0;
  if (D % 8 != 0 || ld % 8 != 0) return -1;
  long long grid = ((long long)n * (H * D / 8) + 255) / 256;
  if (grid > 148 * 16) grid = 148 * 16;
  return launch_kernel(kv_gate_kernel, dim3((unsigned)grid), dim3(256), 0, stream, (__nv_bfloat16*)out, lse, sink, (const __nv_bfloat16*)gate, ld,
                       H, D, row0, n, Tq) == cudaSuccess ? 0 : -11;
}

// ------------------------------------------------------------------------------------------
// Allocation-free variant (see attn_noalloc.h for the contract and for who needs it).
// ------------------------------------------------------------------------------------------
#include "attn_noalloc.h"

#include <mutex>

// Per-split partial outputs and (max, sum) pairs. In host code this name is only a handle for
// the runtime, not a device address: the address is fetched with cudaGetSymbolAddress below.
static __device__ __align__(256) float rb_decode_noalloc_scratch[RB_DECODE_NOALLOC_MAX_FLOATS];

namespace {
constexpr int kMaxDevices = RB_MAX_DEVICES;
float* g_noalloc_ptr[kMaxDevices] = {};
std::mutex g_noalloc_mutex;

// Device address of the scratch array on the current device, looked up once per device.
int noalloc_scratch_for_current_device(float** out) {
  int dev = -1;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= kMaxDevices) return RB_NOALLOC_SYMBOL_LOOKUP_FAILED;
  std::lock_guard<std::mutex> lock(g_noalloc_mutex);
  if (g_noalloc_ptr[dev] == nullptr) {
    float* p = nullptr;
    const cudaError_t e = cudaGetSymbolAddress(reinterpret_cast<void**>(&p), rb_decode_noalloc_scratch);
    if (e != cudaSuccess || p == nullptr) return RB_NOALLOC_SYMBOL_LOOKUP_FAILED;
    g_noalloc_ptr[dev] = p;
  }
  *out = g_noalloc_ptr[dev];
  return 0;
}
}  // namespace

extern "C" long long rb_paged_decode_noalloc_required_floats(int B, int Hq, int D, int num_splits) {
  // one split writes the output directly: nothing of the array is touched, whatever the batch
  if (B <= 0 || Hq <= 0 || D <= 0 || num_splits <= 1) return 0;
  return (long long)B * Hq * num_splits * (D + 2);
}

extern "C" int rb_paged_decode_noalloc(const void* q, const void* k_cache, const void* v_cache,
                                       const int* block_tables, const int* seq_lens, void* out, int B, int Hq,
                                       int Hkv, int D, int max_blocks, int num_blocks, int block_size, int num_splits,
                                       float scale, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (num_splits < 1) return -1;
  if (rb_paged_decode_noalloc_required_floats(B, Hq, D, num_splits) > (long long)RB_DECODE_NOALLOC_MAX_FLOATS)
    return RB_NOALLOC_TOO_LARGE;
  float* scratch = nullptr;
  if (num_splits > 1) {   // a single split needs no workspace, so no lookup either
    const int rc = noalloc_scratch_for_current_device(&scratch);
    if (rc != 0) return rc;
  }
  // Same kernels and launch logic as the regular entry point, with the library's own workspace.
  return rb_paged_decode(q, k_cache, v_cache, block_tables, seq_lens, out, scratch, B, Hq, Hkv, D, max_blocks,
                         num_blocks, block_size, num_splits, scale, status, stream);
}
