// Gated delta rule: what stands around its recurrence, and its chunked form. Part of recurrent_sm100.cu.
//
//   S <- g_t S,  u_t = beta_t (v_t - S^T k_t),  S <- S + k_t u_t^T,  o_t = S^T q_t
//
// Queries, keys and values come out of a short causal convolution and SiLU in the activation type; queries and keys are unit
// vectors per head, kept as those activations and an fp32 factor, so that products of them on the tensor cores lose nothing.
#pragma once

namespace rb {

// ------------------------------------------------------------------------------------------
// Rows: convolution over q | k | v (heads padded to KP, KP and VP channels), SiLU, the factors of queries and keys, and the
// recurrence's logarithm of the decay and step size. A warp takes a head of `run` rows and keeps its look back in registers.
// ------------------------------------------------------------------------------------------
struct DeltaRows {
  const void* proj;        // [T, ld] q | k | v
  long long ld;
  const float* conv;       // [taps, channels], latest last
  int taps;
  void* hist;              // [slots, taps - 1, channels]
  History rows;
  void* out;               // [T, ldo]
  long long ldo;
  const float* small;      // [T, ld_small] logits of the step size [H], then of the decay [H]
  long long ld_small;
  const float* rate;       // [H] exp(A_log)
  const float* dt_bias;    // [H]
  float* units;            // [T, 2 G]
  float* steps;            // [T, 2 H]
  int G, H, KP, VP, T, run;
  int* status;
};

template <typename T, int N>
__device__ __forceinline__ void lane_load(const T* p, float (&x)[N]) {
  constexpr int BYTES = N * sizeof(T), STEP = BYTES < 16 ? BYTES : 16, PER = STEP / sizeof(T);
#pragma unroll
  for (int i = 0; i < N / PER; ++i) {
    union { uint32_t w[4]; T e[16 / sizeof(T)]; } a;
    if constexpr (STEP == 4) a.w[0] = *reinterpret_cast<const uint32_t*>(p + i * PER);
    else if constexpr (STEP == 8) *reinterpret_cast<uint2*>(a.w) = *reinterpret_cast<const uint2*>(p + i * PER);
    else *reinterpret_cast<uint4*>(a.w) = *reinterpret_cast<const uint4*>(p + i * PER);
#pragma unroll
    for (int j = 0; j < PER; ++j) x[i * PER + j] = to_f<T>(a.e[j]);
  }
}
// Stores x rounded to T, and leaves the rounded values in x.
template <typename T, int N>
__device__ __forceinline__ void lane_store(T* p, float (&x)[N]) {
  constexpr int BYTES = N * sizeof(T), STEP = BYTES < 16 ? BYTES : 16, PER = STEP / sizeof(T);
#pragma unroll
  for (int i = 0; i < N / PER; ++i) {
    union { uint32_t w[4]; T e[16 / sizeof(T)]; } a;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      if constexpr (sizeof(T) == 4) a.e[j] = x[i * PER + j];
      else a.e[j] = __float2bfloat16_rn(x[i * PER + j]);
      x[i * PER + j] = to_f<T>(a.e[j]);
    }
    if constexpr (STEP == 4) *reinterpret_cast<uint32_t*>(p + i * PER) = a.w[0];
    else if constexpr (STEP == 8) *reinterpret_cast<uint2*>(p + i * PER) = *reinterpret_cast<const uint2*>(a.w);
    else *reinterpret_cast<uint4*>(p + i * PER) = *reinterpret_cast<const uint4*>(a.w);
  }
}

constexpr int DR_THREADS = 256;

// CPL: channels per lane (a head has at most 32 CPL); TAPS: most taps
template <typename T, int CPL, int TAPS>
__global__ void __launch_bounds__(DR_THREADS) delta_rows_kernel(const DeltaRows p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, n_units = 2 * p.G + p.H + 1;
  const long long w = (long long)blockIdx.x * (DR_THREADS / 32) + (threadIdx.x >> 5);
  const int unit = (int)(w % n_units), t0 = (int)(w / n_units) * p.run, t1 = min(t0 + p.run, p.T);
  if (t0 >= p.T) return;
  if (unit == n_units - 1) {
    for (int i = lane; i < (t1 - t0) * p.H; i += 32) {
      const long long t = t0 + i / p.H;
      const int h = i % p.H;
      const float z = p.small[t * p.ld_small + p.H + h] + p.dt_bias[h];
      p.steps[t * 2 * p.H + h] = -p.rate[h] * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
      p.steps[t * 2 * p.H + p.H + h] = sigmoid_f(p.small[t * p.ld_small + h]);
    }
    return;
  }
  const bool is_v = unit >= 2 * p.G;
  const int width = is_v ? p.VP : p.KP, c = (is_v ? 2 * p.G * p.KP + (unit - 2 * p.G) * p.VP : unit * p.KP) + lane * CPL;
  const int channels = 2 * p.G * p.KP + p.H * p.VP, depth = p.taps - 1;
  const bool active = lane * CPL < width;
  const T* rows = reinterpret_cast<const T*>(p.proj) + c;
  T* hist = reinterpret_cast<T*>(p.hist) + c;
  float weight[TAPS][CPL], back[TAPS][CPL];            // of the row d places before;  back[d - 1]: that row
#pragma unroll
  for (int d = 0; d < TAPS; ++d)
#pragma unroll
    for (int j = 0; j < CPL; ++j) weight[d][j] = active && d < p.taps ? p.conv[(long long)(p.taps - 1 - d) * channels + c + j] : 0.f;
  int end = t0;                                        // of the sequence the rows are in
  RowPlace place{0, 0, -1};
  for (int t = t0; t < t1; ++t) {
    if (t >= end) {
      place = row_place(p.rows, t, p.status);
      end = p.rows.cu_q == nullptr ? t + 1 : p.rows.cu_q[sequence_of(p.rows.cu_q, p.rows.B, t) + 1];
#pragma unroll
      for (int d = 1; d < TAPS; ++d) {
#pragma unroll
        for (int j = 0; j < CPL; ++j) back[d - 1][j] = 0.f;
        if (active && d < p.taps) {
          const T* src = row_before(place, d, rows, p.ld, t, (const T*)hist, depth, channels);
          if (src != nullptr) lane_load<T, CPL>(src, back[d - 1]);
        }
      }
    }
    float x[CPL], y[CPL], ss = 0.f;
#pragma unroll
    for (int j = 0; j < CPL; ++j) x[j] = 0.f;
    if (active) lane_load<T, CPL>(rows + (long long)t * p.ld, x);
#pragma unroll
    for (int j = 0; j < CPL; ++j) {
      float s = weight[0][j] * x[j];
#pragma unroll
      for (int d = 1; d < TAPS; ++d) s = fmaf(weight[d][j], back[d - 1][j], s);
      y[j] = sizeof(T) == 4 ? s * sigmoid_f(s) : silu_fast(s);
    }
    if (active) lane_store<T, CPL>(reinterpret_cast<T*>(p.out) + (long long)t * p.ldo + c, y);
    if (!is_v) {
#pragma unroll
      for (int j = 0; j < CPL; ++j) ss = fmaf(y[j], y[j], ss);
      ss = warp_sum(ss);
      if (lane == 0) p.units[(long long)t * 2 * p.G + unit] = 1.f / sqrtf(ss + 1e-6f);
    }
#pragma unroll
    for (int d = TAPS - 1; d >= 1; --d)
#pragma unroll
      for (int j = 0; j < CPL; ++j) back[d - 1][j] = d == 1 ? x[j] : back[d >= 2 ? d - 2 : 0][j];
    if (p.rows.cu_q == nullptr && depth > 0 && place.slot >= 0 && active) {      // one row per sequence: its history moves on here
#pragma unroll
      for (int d = 1; d < TAPS; ++d)
        if (d < p.taps) lane_store<T, CPL>(hist + ((long long)place.slot * depth + d - 1) * channels, back[d - 1]);
    }
  }
}

template <typename T, int CPL>
static cudaError_t launch_delta_rows_taps(const DeltaRows& p, cudaStream_t stream) {
  const long long warps = (long long)((p.T + p.run - 1) / p.run) * (2 * p.G + p.H + 1);
  const dim3 grid((unsigned)((warps + DR_THREADS / 32 - 1) / (DR_THREADS / 32)));
  if (p.taps <= 4) return launch_kernel(delta_rows_kernel<T, CPL, 4>, grid, dim3(DR_THREADS), 0, stream, p);
  if (p.taps <= 8) return launch_kernel(delta_rows_kernel<T, CPL, 8>, grid, dim3(DR_THREADS), 0, stream, p);
  return launch_kernel(delta_rows_kernel<T, CPL, 16>, grid, dim3(DR_THREADS), 0, stream, p);
}

template <typename T>
static cudaError_t launch_delta_rows(const DeltaRows& p, cudaStream_t stream) {
  const int most = p.KP > p.VP ? p.KP : p.VP;
  if (most <= 64) return launch_delta_rows_taps<T, 2>(p, stream);
  if (most <= 128) return launch_delta_rows_taps<T, 4>(p, stream);
  if (most <= 256) return launch_delta_rows_taps<T, 8>(p, stream);
  return launch_delta_rows_taps<T, 16>(p, stream);
}

// ------------------------------------------------------------------------------------------
// Chunks of up to CH tokens. With F_t the summed log decays up to and including token t and S the state in front of the chunk,
//
//   (I + L) U = diag(beta) (V - diag(e^F) K S),    L_tj = beta_t e^(F_t - F_j) k_t . k_j  for j < t
//   O = diag(e^F) Q S + P U,   P_tj = e^(F_t - F_j) q_t . k_j  for j <= t,    S' = e^(F_C) S + sum_j e^(F_C - F_j) k_j u_j^T
//
// T = (I + L)^-1 does not depend on the state: one launch makes W = T diag(beta e^F) K and T diag(beta) V for all chunks at once, a
// second one goes over a sequence's chunks with U = T diag(beta) V - W S, and the outputs are recurrent_chunk_out_kernel's with U for
// the values. All factors of the keys are applied in fp32 outside the products; T, W, U and S go in as two bf16 parts each.
//
// The inverse X: its eight 16 x 16 blocks on the diagonal by substitution in fp32, the others by mma.sync with operands in two parts.
// Warp j makes column j of blocks, transposed, X_ij^T = -(sum_(j <= k < i) X_kj^T L_ik^T) X_ii^T, and leaves it in fp32 where L has nothing:
// L fills the blocks below the diagonal of one square, X^T the others.
// ------------------------------------------------------------------------------------------
struct DeltaParams {
  ChunkParams c;
  const float* units;      // [T, 2 G]
  const float* steps;      // [T, 2 H]
  __nv_bfloat16* w_hi;     // [chunks, H, KP / 64, CH, 64], tiles as they lie in shared memory (chunk_addr)
  __nv_bfloat16* w_lo;
  __nv_bfloat16* keys;     // [chunks, G, KP / 64, CH, 64], so too
  float* uv;               // [chunks, H, VP / 64, 16, CH, 4]
  __nv_bfloat16* values;   // [chunks, H, VP / 64, 8, CH, 8] U
};

// Place of L[t][j]: groups of eight exchanged by the row's low bits, so that four rows of a fragment meet no bank twice.
__device__ __forceinline__ int inverse_at(int t, int j) { return t * CH + (j ^ ((t & 3) << 3)); }

template <int DK>
struct DeltaSolveCfg {
  static constexpr int kKBytes = CH * DK * 2;                      // K, then tiles of V
  static constexpr int kLBytes = CH * CH * 4;                      // L, then the inverse's two parts
  static constexpr int kSmem = 1024 + kKBytes + kLBytes;
  static constexpr int kCols = 256;
};

// A 16 x 16 block as first operand of mma.sync, in two parts, from pairs (row g, columns c, c + 1), (g + 8, ..), (g, c + 8 ..), (g + 8, c + 8 ..).
struct Block16 {
  uint32_t hi[4], lo[4];
  __device__ __forceinline__ void set(int e, float x, float y) { split_bf16x2(x, y, hi[e], lo[e]); }
};

// acc += a m^T for a block m of fp32 rows, the two halves of the columns and the three products of parts apart: column n of the product goes
// with row n of m. `m(row, column)` is the address of two elements.
template <typename Block>
__device__ __forceinline__ void block_product(float (&acc)[2][3][4], const Block16& a, Block m, int lane) {
  const int g = lane >> 2, c = 2 * (lane & 3);
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const float2 x = *reinterpret_cast<const float2*>(m(8 * q + g, c)), y = *reinterpret_cast<const float2*>(m(8 * q + g, c + 8));
    uint32_t h0, l0, h1, l1;
    split_bf16x2(x.x, x.y, h0, l0);
    split_bf16x2(y.x, y.y, h1, l1);
    mma_16816_bf16(acc[q][0], a.hi[0], a.hi[1], a.hi[2], a.hi[3], h0, h1);
    mma_16816_bf16(acc[q][1], a.lo[0], a.lo[1], a.lo[2], a.lo[3], h0, h1);
    mma_16816_bf16(acc[q][2], a.hi[0], a.hi[1], a.hi[2], a.hi[3], l0, l1);
  }
}

template <int DK>
__global__ void __launch_bounds__(CHT, 2) delta_solve_kernel(const DeltaParams p) {
  using Cfg = DeltaSolveCfg<DK>;
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ float Fs[CH], betas[CH], rks[CH], sums[4];
  __shared__ __align__(8) float diag[8][16][18];
  __shared__ __align__(8) uint64_t done;
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag;
  const ChunkParams& c = p.c;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t k_s = base, t_s = base + Cfg::kKBytes;
  uint8_t* t_p = smem_raw + (base - smem_u32(smem_raw)) + Cfg::kKBytes;
  float* L = reinterpret_cast<float*>(t_p);
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(smem_u32(&done), 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_smem), Cfg::kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_smem;
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.x / c.H, h = blockIdx.x % c.H, G = c.H / c.ratio, hk = h / c.ratio;
  const int4 ck = c.chunks[chunk];
  const int row0 = ck.x, n = ck.y;
  const long long ch = (long long)chunk * c.H + h;
  const __nv_bfloat16* rows = c.proj + (long long)row0 * c.ld;
  chunk_load<DK>(k_s, rows + c.k_col + hk * c.KP, c.ld, n);
  float run = 0.f, q_factor = 0.f, k_factor = 0.f, step = 0.f;       // a token per thread of the first four warps: F, step sizes, factors
  if (tid < CH) {
    if (tid < n) {
      const long long r = row0 + tid;
      run = fmaxf(p.steps[r * 2 * c.H + h] * LOG2E, -MIX_MOST);
      step = p.steps[r * 2 * c.H + c.H + h];
      q_factor = p.units[r * 2 * G + hk];
      k_factor = p.units[r * 2 * G + G + hk];
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += y;
    }
    if (lane == 31) sums[warp] = run;
  }
  __syncthreads();
  if (tid < CH) {
    for (int w = 0; w < warp; ++w) run += sums[w];
    Fs[tid] = run;
    betas[tid] = step;
    rks[tid] = k_factor;
    float* gates = c.gates + ch * 3 * CH + tid;          // log2 of a key's factor, the row's reference, the query's factor
    gates[0] = tid < n ? log2f(k_factor) - run : -INFINITY;
    gates[CH] = -run;
    gates[2 * CH] = q_factor;
    if (tid == CH - 1) c.um[ch] = make_float2(run, 0.f);
  }
  cp_async_wait_all();
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 0 && elect_one_sync()) {                   // K K^T
    constexpr uint32_t idesc = make_idesc_bf16(CH, CH, 0, 0);
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      const uint64_t a = make_smem_desc_sw128(k_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
      umma_bf16(tmem, a, a, idesc, kk ? 1u : 0u);
    }
    umma_commit(smem_u32(&done));
  }
  __syncwarp();
  if (tid == 32 && h % c.ratio == 0) bulk_store(p.keys + ((long long)chunk * G + hk) * DK * CH, k_s, Cfg::kKBytes);
  const int qd = warp & 3, half = warp >> 2, t = qd * 32 + lane;
  const uint32_t lane_addr = (uint32_t)(qd * 32) << 16;
  int phase = 0;
  bool ok = mbar_wait_bounded(smem_u32(&done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  tc_fence_after();
  if (ok) {
    const float F = Fs[t], f = betas[t] * rks[t];
#pragma unroll
    for (int cc = 0; cc < 2; ++cc) {
      const int j0 = half * 64 + cc * 32;
      if (j0 > qd * 32 + 31) continue;                   // (uniform per warp: above the diagonal, never read)
      uint32_t v[32];
      tmem_ld_32x32(tmem + j0 + lane_addr, v);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; i += 4) {
        float y[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = j0 + i + e;
          y[e] = j < t ? f * rks[j] * chunk_exp2(F - Fs[j]) * __uint_as_float(v[i + e]) : 0.f;
        }
        *reinterpret_cast<float4*>(L + inverse_at(t, j0 + i)) = make_float4(y[0], y[1], y[2], y[3]);
      }
    }
    tc_fence_before();
  }
  ok = __syncthreads_and(ok);
  if (ok) {
    auto at = [&](int row, int col) { return L + inverse_at(row, col); };
    const int j16 = warp * 16;
    {                                                    // the warp's diagonal block, a column per lane
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < i; j += 4) {
          const float4 l = *reinterpret_cast<const float4*>(at(j16 + i, j16 + j));
          s = fmaf(l.x, x[j], s);
          if (j + 1 < i) s = fmaf(l.y, x[j + 1 < i ? j + 1 : 0], s);
          if (j + 2 < i) s = fmaf(l.z, x[j + 2 < i ? j + 2 : 0], s);
          if (j + 3 < i) s = fmaf(l.w, x[j + 3 < i ? j + 3 : 0], s);
        }
        x[i] = (i == (lane & 15) ? 1.f : 0.f) - s;
      }
      __syncwarp();
      if (lane < 16) {
#pragma unroll
        for (int i = 0; i < 16; ++i) diag[warp][i][lane] = x[i];
#pragma unroll
        for (int i = 0; i < 16; i += 4) *reinterpret_cast<float4*>(at(j16 + lane, j16 + i)) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
      }
    }
    __syncthreads();
    const int g = lane >> 2, cq = 2 * (lane & 3);
#pragma unroll 1
    for (int i16 = j16 + 16; i16 < CH; i16 += 16) {
      float acc[2][3][4] = {};
#pragma unroll 2
      for (int k16 = j16; k16 < i16; k16 += 16) {
        Block16 a;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v = *reinterpret_cast<const float2*>(at(j16 + g + (e & 1) * 8, k16 + cq + (e >> 1) * 8));
          a.set(e, v.x, v.y);
        }
        block_product(acc, a, [&](int row, int col) { return at(i16 + row, k16 + col); }, lane);
      }
      Block16 sum;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int q = e >> 1, h2 = (e & 1) * 2;
        sum.set(e, -(acc[q][0][h2] + acc[q][1][h2] + acc[q][2][h2]), -(acc[q][0][h2 + 1] + acc[q][1][h2 + 1] + acc[q][2][h2 + 1]));
      }
      float x[2][3][4] = {};
      block_product(x, sum, [&](int row, int col) { return &diag[i16 >> 4][row][col]; }, lane);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int q = e >> 1, h2 = (e & 1) * 2;
        *reinterpret_cast<float2*>(at(j16 + g + (e & 1) * 8, i16 + cq + q * 8)) =
            make_float2(x[q][0][h2] + x[q][1][h2] + x[q][2][h2], x[q][0][h2 + 1] + x[q][1][h2 + 1] + x[q][2][h2 + 1]);
      }
      __syncwarp();
    }
    __syncthreads();
    // X^T with its rows (columns of the inverse) scaled, in two parts, [CH, CH] as two tiles of 64 columns each: the square it comes from is
    // overwritten, so every thread keeps its eight pieces of eight columns (row 16 k + tid / 16, piece tid % 16).
    float X[8][8];
    const int piece = tid & 15;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const int row = k * 16 + (tid >> 4);
#pragma unroll
      for (int e = 0; e < 8; e += 4) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (piece >> 1 >= k) v = *reinterpret_cast<const float4*>(at(row, piece * 8 + e));
        X[k][e] = v.x; X[k][e + 1] = v.y; X[k][e + 2] = v.z; X[k][e + 3] = v.w;
      }
    }
    __syncthreads();
    auto store_inverse = [&](bool keys) {                // for the product with the keys, or with the values
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int row = k * 16 + (tid >> 4);
        const float f = keys ? betas[row] * rks[row] * chunk_exp2(Fs[row]) : betas[row];
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_bf16x2(X[k][2 * e] * f, X[k][2 * e + 1] * f, hi[e], lo[e]);
        uint8_t* dst = t_p + (piece >> 3) * CH_CHUNK + chunk_addr(row, piece & 7);
        *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(dst + 2 * CH_CHUNK) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    };
    store_inverse(true);
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    constexpr uint32_t idesc = make_idesc_bf16(CH, 64, 1, 1);
    auto product = [&](uint32_t dst, int tiles) {        // T times the tiles of 64 columns at k_s
#pragma unroll
      for (int z = 0; z < DK / 64; ++z) {
        if (z >= tiles) break;
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < CH / 16; ++kk) {
            const uint64_t a = make_smem_desc_sw128(t_s + part * 2 * CH_CHUNK + kk * 2048, CH_CHUNK, 1024);
            const uint64_t b = make_smem_desc_sw128(k_s + z * CH_CHUNK + kk * 2048, CH_CHUNK, 1024);
            umma_bf16(dst + z * 64, a, b, idesc, (part | kk) ? 1u : 0u);
          }
      }
      umma_commit(smem_u32(&done));
    };
    if (warp == 0 && elect_one_sync()) product(tmem, DK / 64);
    __syncwarp();
    phase ^= 1;
    ok = mbar_wait_bounded(smem_u32(&done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
    if (tid == 32) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
    ok = __syncthreads_and(ok);                          // K and the inverse have been read
    if (ok) {
      const __nv_bfloat16* v = rows + c.v_col + h * c.VP;
      const int tiles = c.VP / 64;
      auto load_values = [&](int z0) {
        for (int z = z0; z < min(z0 + DK / 64, tiles); ++z) chunk_load<64>(k_s + (z - z0) * CH_CHUNK, v + z * 64, c.ld, n);
      };
      load_values(0);
      tc_fence_after();
#pragma unroll
      for (int z = 0; z < DK / 64; ++z) {                // W, over the inverse, and from there to global memory as it lies
        uint32_t w[32];
        tmem_ld_32x32(tmem + z * 64 + half * 32 + lane_addr, w);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) split_bf16x2(__uint_as_float(w[8 * i + 2 * e]), __uint_as_float(w[8 * i + 2 * e + 1]), hi[e], lo[e]);
          uint8_t* dst = t_p + z * CH_CHUNK + chunk_addr(t, half * 4 + i);
          *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(dst + Cfg::kKBytes) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      fence_proxy_async_smem();
      __syncthreads();
      if (tid == 32) {
        bulk_store(p.w_hi + ch * DK * CH, t_s, Cfg::kKBytes);
        bulk_store(p.w_lo + ch * DK * CH, t_s + Cfg::kKBytes, Cfg::kKBytes);
        asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
      }
      __syncthreads();
      store_inverse(false);
      for (int z0 = 0; ok && z0 < tiles; z0 += DK / 64) {
        const int have = min(DK / 64, tiles - z0);
        cp_async_wait_all();
        fence_proxy_async_smem();
        tc_fence_before();
        __syncthreads();
        tc_fence_after();
        if (warp == 0 && elect_one_sync()) product(tmem + 128, have);
        __syncwarp();
        phase ^= 1;
        ok = mbar_wait_bounded(smem_u32(&done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
        ok = __syncthreads_and(ok);
        tc_fence_after();
        if (!ok) break;
        if (z0 + have < tiles) load_values(z0 + have);
        for (int z = 0; z < have; ++z) {
          uint32_t u[32];
          tmem_ld_32x32(tmem + 128 + z * 64 + half * 32 + lane_addr, u);
          tmem_ld_wait();
          float4* dst = reinterpret_cast<float4*>(p.uv) + ((ch * tiles + z0 + z) * 16 + half * 8) * CH + t;
#pragma unroll
          for (int i = 0; i < 8; ++i)
            dst[i * CH] = make_float4(__uint_as_float(u[4 * i]), __uint_as_float(u[4 * i + 1]), __uint_as_float(u[4 * i + 2]), __uint_as_float(u[4 * i + 3]));
        }
      }
      tc_fence_before();
    }
  }
  cp_async_wait_all();
  if (tid == 32) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kCols);
  }
}

// The chunks of a sequence one after the other, 64 value channels of a head per CTA; the state in registers. A chunk is two products one
// behind the other (W S, then K^T U), each with both parts of its second operand side by side; what is written to global memory, and
// the next chunk's vectors, pass while the products run.
constexpr int DC_THREADS = 512, DC_COLS = 64 / (DC_THREADS / 128);     // value channels of a thread's row

template <int DK>
struct DeltaChainCfg {
  static constexpr int kWBytes = CH * DK * 2;                      // one part of W; K
  static constexpr int kSBytes = DK * CH_ROWB;                     // one part of the state
  static constexpr int kSmem = 1024 + 3 * kWBytes + 2 * kSBytes + 2 * CH_CHUNK;
  static constexpr int kCols = 256;                                // W S, K^T U: with the first and the second part of S, U
};

template <int DK>
__global__ void __launch_bounds__(DC_THREADS) delta_chain_kernel(const DeltaParams p) {
  using Cfg = DeltaChainCfg<DK>;
  static_assert(DC_COLS == 16, "a thread's row is one TMEM load");
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t u_done, s_done, w_full, k_full;
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag;
  const ChunkParams& c = p.c;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t w_s = base, k_s = w_s + 2 * Cfg::kWBytes, s_s = k_s + Cfg::kWBytes, u_s = s_s + 2 * Cfg::kSBytes;
  uint8_t* s_p = smem_raw + (s_s - smem_u32(smem_raw));
  uint8_t* u_p = smem_raw + (u_s - smem_u32(smem_raw));
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(smem_u32(&u_done), 1);
    mbar_init(smem_u32(&s_done), 1);
    mbar_init(smem_u32(&w_full), 1);
    mbar_init(smem_u32(&k_full), 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_smem), Cfg::kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_smem;
  pdl_launch_dependents();
  pdl_wait();
  const int z = blockIdx.x, h = blockIdx.y, b = blockIdx.z, hk = h / c.ratio;
  const int qd = warp & 3, col = (warp >> 2) * DC_COLS, t = qd * 32 + lane;
  const uint32_t lane_addr = (uint32_t)(qd * 32) << 16;
  const int slot = c.slots[b];
  if (slot >= 0 && slot < c.num_slots) {
    const bool fresh = c.seq_lens[b] == c.cu_q[b + 1] - c.cu_q[b];
    const int c0 = c.seq_chunks[b], c1 = c.seq_chunks[b + 1];
    // key row of this thread's value channels (a 64-row product: row 16 q + lane in 16 lanes)
    const int r = DK == 128 ? t : qd * 16 + lane;
    const bool holds = DK == 128 || lane < 16, live = holds && r < c.dk;
    float4* st = reinterpret_cast<float4*>(c.s + ((((long long)slot * c.H + h) * (c.VP / SC_COLS) + z * 2 + col / SC_COLS) * c.KP + (holds ? r : 0)) * SC_COLS +
                                           col % SC_COLS);
    float S[DC_COLS];
#pragma unroll
    for (int i = 0; i < DC_COLS / 4; ++i) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !fresh) v = st[i];
      S[4 * i] = v.x; S[4 * i + 1] = v.y; S[4 * i + 2] = v.z; S[4 * i + 3] = v.w;
    }
    int w_loads = 0, k_loads = 0;                        // thread 0: copies on their way or landed
    auto load_w = [&](int k) {
      const long long at = ((long long)k * c.H + h) * DK * CH;
      const uint32_t bar = smem_u32(&w_full);
      mbar_expect_tx(bar, 2 * Cfg::kWBytes);
      bulk_load(w_s, p.w_hi + at, Cfg::kWBytes, bar);
      bulk_load(w_s + Cfg::kWBytes, p.w_lo + at, Cfg::kWBytes, bar);
      ++w_loads;
    };
    auto load_k = [&](int k) {
      const uint32_t bar = smem_u32(&k_full);
      mbar_expect_tx(bar, Cfg::kWBytes);
      bulk_load(k_s, p.keys + ((long long)k * (c.H / c.ratio) + hk) * DK * CH, Cfg::kWBytes, bar);
      ++k_loads;
    };
    // what a thread needs of a chunk besides: its row of T diag(beta) V, the factor of its key, the chunk's decay
    float4 uv[DC_COLS / 4];
    float factor = 0.f, decay = 0.f;
    auto fetch = [&](int k) {
      const long long ch = (long long)k * c.H + h;
      const float4* src = reinterpret_cast<const float4*>(p.uv) + ((ch * (c.VP / 64) + z) * 16 + col / 4) * CH + t;
#pragma unroll
      for (int i = 0; i < DC_COLS / 4; ++i) uv[i] = src[i * CH];
      decay = c.um[ch].x;
      factor = c.gates[ch * 3 * CH + t];
    };
    if (c0 < c1) {
      if (tid == 0) { load_w(c0); load_k(c0); }
      fetch(c0);
    }
    bool ok = true;
    constexpr int MOVER = DC_THREADS - 32;               // the thread that stores the state's parts
    for (int k = c0; k < c1; ++k) {
      const uint32_t phase = (uint32_t)((k - c0) & 1);
      const long long ch = (long long)k * c.H + h;
      uint4 hi[2], lo[2];
      auto split8 = [](const float (&x)[DC_COLS], int i, uint4& a, uint4& d) {
        split_bf16x2(x[i], x[i + 1], a.x, d.x);
        split_bf16x2(x[i + 2], x[i + 3], a.y, d.y);
        split_bf16x2(x[i + 4], x[i + 5], a.z, d.z);
        split_bf16x2(x[i + 6], x[i + 7], a.w, d.w);
      };
      if (holds) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          split8(S, i * 8, hi[i], lo[i]);
          const uint32_t o = chunk_addr(r, col / 8 + i);
          *reinterpret_cast<uint4*>(s_p + o) = hi[i];
          *reinterpret_cast<uint4*>(s_p + Cfg::kSBytes + o) = lo[i];
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      if (warp == 0 && ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(smem_u32(&w_full), phase, &abort_flag, c.status, ST_TIMEOUT_SMEM_FULL));
      ok = __syncthreads_and(ok);
      if (!ok) break;
      tc_fence_after();
      if (warp == 0 && elect_one_sync()) {                         // W S without the product of the two small parts
        constexpr uint32_t both = make_idesc_bf16(CH, 128, 0, 1), one = make_idesc_bf16(CH, 64, 0, 1);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < DK / 16; ++kk) {
            const uint64_t a = make_smem_desc_sw128(w_s + part * Cfg::kWBytes + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
            const uint64_t d = make_smem_desc_sw128(s_s + kk * 2048, Cfg::kSBytes, 1024);
            umma_bf16(tmem, a, d, part ? one : both, (part | kk) ? 1u : 0u);
          }
        umma_commit(smem_u32(&u_done));
      }
      __syncwarp();
      const long long tile = ch * (c.VP / 64) + z;
      if (tid == MOVER) {                                          // the state in front of the chunk, for the outputs
        bulk_store(c.s_hi + tile * c.KP * 64, s_s, Cfg::kSBytes);
        bulk_store(c.s_lo + tile * c.KP * 64, s_s + Cfg::kSBytes, Cfg::kSBytes);
        asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
      }
      __syncwarp();
      const float weight = chunk_exp2(decay + factor), keep = chunk_exp2(decay);
      ok = mbar_wait_bounded(smem_u32(&u_done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      uint4 row[2];                                                // U in the activation type
      if (ok) {
        if (tid == 0 && k + 1 < c1) load_w(k + 1);                 // W has been read
        uint32_t a[DC_COLS], d[DC_COLS];
        tmem_ld_32x16(tmem + col + lane_addr, a);
        tmem_ld_32x16(tmem + 64 + col + lane_addr, d);
        tmem_ld_wait();
        tc_fence_before();
        float U[DC_COLS];
#pragma unroll
        for (int i = 0; i < DC_COLS / 4; ++i) {
          U[4 * i] = uv[i].x - (__uint_as_float(a[4 * i]) + __uint_as_float(d[4 * i]));
          U[4 * i + 1] = uv[i].y - (__uint_as_float(a[4 * i + 1]) + __uint_as_float(d[4 * i + 1]));
          U[4 * i + 2] = uv[i].z - (__uint_as_float(a[4 * i + 2]) + __uint_as_float(d[4 * i + 2]));
          U[4 * i + 3] = uv[i].w - (__uint_as_float(a[4 * i + 3]) + __uint_as_float(d[4 * i + 3]));
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
          row[i] = make_uint4(pack_bf16x2(U[8 * i], U[8 * i + 1]), pack_bf16x2(U[8 * i + 2], U[8 * i + 3]), pack_bf16x2(U[8 * i + 4], U[8 * i + 5]),
                              pack_bf16x2(U[8 * i + 6], U[8 * i + 7]));
#pragma unroll
        for (int i = 0; i < DC_COLS; ++i) U[i] *= weight;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          split8(U, i * 8, hi[i], lo[i]);
          const uint32_t o = chunk_addr(t, col / 8 + i);
          *reinterpret_cast<uint4*>(u_p + o) = hi[i];
          *reinterpret_cast<uint4*>(u_p + CH_CHUNK + o) = lo[i];
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      if (warp == 0 && ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(smem_u32(&k_full), phase, &abort_flag, c.status, ST_TIMEOUT_SMEM_FULL));
      ok = __syncthreads_and(ok);
      if (!ok) break;
      tc_fence_after();
      if (warp == 0 && elect_one_sync()) {
        constexpr uint32_t idesc = make_idesc_bf16(DK, 128, 1, 1);
#pragma unroll
        for (int kk = 0; kk < CH / 16; ++kk) {
          const uint64_t a = make_smem_desc_sw128(k_s + kk * 2048, CH_CHUNK, 1024);
          const uint64_t d = make_smem_desc_sw128(u_s + kk * 2048, CH_CHUNK, 1024);
          umma_bf16(tmem + 128, a, d, idesc, kk ? 1u : 0u);
        }
        umma_commit(smem_u32(&s_done));
      }
      __syncwarp();
      {
        uint4* dst = reinterpret_cast<uint4*>(p.values) + (tile * 8 + col / 8) * CH + t;
        dst[0] = row[0];
        dst[CH] = row[1];
      }
      if (k + 1 < c1) fetch(k + 1);
      ok = mbar_wait_bounded(smem_u32(&s_done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      if (ok) {
        if (tid == 0 && k + 1 < c1) load_k(k + 1);                 // K has been read
        uint32_t a[DC_COLS], d[DC_COLS];
        tmem_ld_32x16(tmem + 128 + col + lane_addr, a);
        tmem_ld_32x16(tmem + 192 + col + lane_addr, d);
        tmem_ld_wait();
        tc_fence_before();
#pragma unroll
        for (int i = 0; i < DC_COLS; ++i) S[i] = fmaf(keep, S[i], __uint_as_float(a[i]) + __uint_as_float(d[i]));
      }
    }
    if (!ok && tid == 0) {                                         // no copy may land after the CTA has gone
      const uint64_t since = globaltimer_ns();
      for (int i = 0; i < 2; ++i) {
        const int loads = i ? k_loads : w_loads;
        while (loads > 0 && !mbar_try_wait(smem_u32(i ? &k_full : &w_full), (uint32_t)((loads - 1) & 1)))
          if (globaltimer_ns() - since > 50000000ull) break;
      }
    }
    if (ok && live)
#pragma unroll
      for (int i = 0; i < DC_COLS / 4; ++i) st[i] = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
    if (tid == MOVER) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  } else if (tid == 0) {
    set_status(c.status, ST_BAD_INDEX);
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kCols);
  }
}

template <int DK>
static int launch_delta_chunks(const DeltaParams& p, int n_chunks, int n_seq, cudaStream_t stream) {
  static int sms[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (sms[dev] == 0) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) return -10;
    if (cudaFuncSetAttribute(delta_solve_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, DeltaSolveCfg<DK>::kSmem) != cudaSuccess ||
        cudaFuncSetAttribute(delta_chain_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, DeltaChainCfg<DK>::kSmem) != cudaSuccess ||
        cudaFuncSetAttribute(recurrent_chunk_out_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkOutCfg<DK>::kSmem) != cudaSuccess)
      return -10;
    sms[dev] = n;
  }
  const ChunkParams& c = p.c;
  const int units = n_chunks * c.H * (c.VP / 64);
  const int most = sms[dev] * (ChunkOutCfg<DK>::kSmem + 5 * 1024 <= 113 * 1024 ? 2 : 1);
  if (launch_kernel(delta_solve_kernel<DK>, dim3(n_chunks * c.H), dim3(CHT), DeltaSolveCfg<DK>::kSmem, stream, p) != cudaSuccess) return -11;
  if (launch_kernel(delta_chain_kernel<DK>, dim3(c.VP / 64, c.H, n_seq), dim3(DC_THREADS), DeltaChainCfg<DK>::kSmem, stream, p) != cudaSuccess) return -12;
  return launch_kernel(recurrent_chunk_out_kernel<DK>, dim3(units < most ? units : most), dim3(CHT), ChunkOutCfg<DK>::kSmem, stream, c, units) == cudaSuccess ? 0 : -13;
}

}  // namespace rb
