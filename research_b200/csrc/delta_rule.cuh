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
      y[j] = s * sigmoid_f(s);
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
// The inverse: its eight 16 x 16 blocks on the diagonal by substitution in fp32, the others by mma.sync with operands in two parts.
// Warp j makes column j of blocks, transposed, X_ij^T = -(sum_(j <= k < i) X_kj^T L_ik^T) X_ii^T, so that every result is the next
// product's first operand as it lies in the registers.
// ------------------------------------------------------------------------------------------
struct DeltaParams {
  ChunkParams c;
  const float* units;      // [T, 2 G]
  const float* steps;      // [T, 2 H]
  __nv_bfloat16* w_hi;     // [chunks, H, KP / 64, CH, 64]
  __nv_bfloat16* w_lo;
  float* uv;               // [chunks, H, VP / 64, CH, 64]
  __nv_bfloat16* values;   // [T, ld_values] U
  long long ld_values;
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

// A 16 x 16 block as first operand of mma.sync (and, four accumulators of an n = 8 product after the other, as its result).
struct Block16 {
  uint32_t hi[4], lo[4];
  __device__ __forceinline__ void set(const float (&lower)[4], const float (&upper)[4], float sign) {      // columns 0 .. 7, 8 .. 15
    split_bf16x2(sign * lower[0], sign * lower[1], hi[0], lo[0]);
    split_bf16x2(sign * lower[2], sign * lower[3], hi[1], lo[1]);
    split_bf16x2(sign * upper[0], sign * upper[1], hi[2], lo[2]);
    split_bf16x2(sign * upper[2], sign * upper[3], hi[3], lo[3]);
  }
};

// acc[2] += a m^T for a block m of fp32 rows: column n of the product goes with row n of m. `m(row, column)` is the address of two elements.
template <typename Block>
__device__ __forceinline__ void block_product(float (&acc)[2][4], const Block16& a, Block m, int lane) {
  const int g = lane >> 2, c = 2 * (lane & 3);
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const float2 x = *reinterpret_cast<const float2*>(m(8 * q + g, c)), y = *reinterpret_cast<const float2*>(m(8 * q + g, c + 8));
    uint32_t h0, l0, h1, l1;
    split_bf16x2(x.x, x.y, h0, l0);
    split_bf16x2(y.x, y.y, h1, l1);
    mma_16816_bf16(acc[q], a.hi[0], a.hi[1], a.hi[2], a.hi[3], h0, h1);
    mma_16816_bf16(acc[q], a.lo[0], a.lo[1], a.lo[2], a.lo[3], h0, h1);
    mma_16816_bf16(acc[q], a.hi[0], a.hi[1], a.hi[2], a.hi[3], l0, l1);
  }
}

template <int DK>
__global__ void __launch_bounds__(CHT, 2) delta_solve_kernel(const DeltaParams p) {
  using Cfg = DeltaSolveCfg<DK>;
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ float Fs[CH], betas[CH], rks[CH];
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
  if (warp == 0) {                                       // F, step sizes, factors: four tokens per lane
    float lf[4], run = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = lane * 4 + i;
      const long long r = row0 + min(t, n - 1);
      const bool in = t < n;
      run += in ? fmaxf(p.steps[r * 2 * c.H + h] * LOG2E, -MIX_MOST) : 0.f;
      lf[i] = run;
      betas[t] = in ? p.steps[r * 2 * c.H + c.H + h] : 0.f;
      rks[t] = in ? p.units[r * 2 * G + G + hk] : 0.f;
    }
    float before = run;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += y;
    }
    const float total = __shfl_sync(0xffffffffu, before, 31);
    before -= run;
    float* gates = c.gates + ch * 3 * CH;                // log2 of a key's factor, the row's reference, the query's factor
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = lane * 4 + i;
      const float F = lf[i] + before;
      Fs[t] = F;
      gates[t] = t < n ? log2f(rks[t]) - F : -INFINITY;
      gates[CH + t] = -F;
      gates[2 * CH + t] = t < n ? p.units[(long long)(row0 + t) * 2 * G + hk] : 0.f;
    }
    if (lane == 0) c.um[ch] = make_float2(total, 0.f);
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
    {                                                    // the warp's diagonal block, a column per lane
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < i; ++j) s = fmaf(L[inverse_at(warp * 16 + i, warp * 16 + j)], x[j], s);
        x[i] = (i == (lane & 15) ? 1.f : 0.f) - s;
      }
      if (lane < 16)
#pragma unroll
        for (int i = 0; i < 16; ++i) diag[warp][i][lane] = x[i];
    }
    __syncthreads();
    Block16 Y[8];                                        // X_ij^T of this warp's j
    const int g = lane >> 2, cq = 2 * (lane & 3);
    {
      float lower[4], upper[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int m = g + (e >> 1) * 8, k = cq + (e & 1);
        lower[e] = diag[warp][k][m];
        upper[e] = diag[warp][k + 8][m];
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i == warp) Y[i].set(lower, upper, 1.f);
    }
#pragma unroll
    for (int i = 1; i < 8; ++i) {
      if (i <= warp) continue;
      float acc[2][4] = {};
#pragma unroll
      for (int k = 0; k < i; ++k)
        if (k >= warp) block_product(acc, Y[k], [&](int row, int col) { return L + inverse_at(i * 16 + row, k * 16 + col); }, lane);
      Block16 sum;
      sum.set(acc[0], acc[1], -1.f);
      float x[2][4] = {};
      block_product(x, sum, [&](int row, int col) { return &diag[i][row][col]; }, lane);
      Y[i].set(x[0], x[1], 1.f);
    }
    __syncthreads();                                     // L has been read
    // T^T with its rows (columns of T) scaled, in two parts, [CH, CH] as two tiles of 64 columns each
    auto store_inverse = [&](float s0, float s1) {       // factors of rows 16 warp + g and + 8
#pragma unroll
      for (int i = 0; i < 8; ++i) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int row = warp * 16 + g + (e & 1) * 8, col = i * 16 + (e >> 1) * 8 + cq;
          uint32_t hi = 0u, lo = 0u;
          if (i >= warp) {
            const float2 a = unpack_bf16x2(Y[i].hi[e]), b = unpack_bf16x2(Y[i].lo[e]);
            const float s = e & 1 ? s1 : s0;
            split_bf16x2((a.x + b.x) * s, (a.y + b.y) * s, hi, lo);
          }
          uint8_t* at = t_p + (col >> 6) * CH_CHUNK + chunk_addr(row, (col & 63) >> 3) + (col & 7) * 2;
          *reinterpret_cast<uint32_t*>(at) = hi;
          *reinterpret_cast<uint32_t*>(at + 2 * CH_CHUNK) = lo;
        }
      }
    };
    const int ra = warp * 16 + g, rb8 = ra + 8;
    store_inverse(betas[ra] * rks[ra] * chunk_exp2(Fs[ra]), betas[rb8] * rks[rb8] * chunk_exp2(Fs[rb8]));
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
    ok = __syncthreads_and(ok);                          // K and the inverse have been read
    if (ok) {
      const __nv_bfloat16* v = rows + c.v_col + h * c.VP;
      const int tiles = c.VP / 64;
      auto load_values = [&](int z0) {
        for (int z = z0; z < min(z0 + DK / 64, tiles); ++z) chunk_load<64>(k_s + (z - z0) * CH_CHUNK, v + z * 64, c.ld, n);
      };
      load_values(0);
      store_inverse(betas[ra], betas[rb8]);
      tc_fence_after();
#pragma unroll
      for (int z = 0; z < DK / 64; ++z) {                // W
        uint32_t w[32];
        tmem_ld_32x32(tmem + z * 64 + half * 32 + lane_addr, w);
        tmem_ld_wait();
        const long long at = ((ch * (DK / 64) + z) * CH + t) * 64 + half * 32;
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) split_bf16x2(__uint_as_float(w[i + 2 * e]), __uint_as_float(w[i + 2 * e + 1]), hi[e], lo[e]);
          *reinterpret_cast<uint4*>(p.w_hi + at + i) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(p.w_lo + at + i) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
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
          float4* dst = reinterpret_cast<float4*>(p.uv + ((ch * tiles + z0 + z) * CH + t) * 64 + half * 32);
#pragma unroll
          for (int i = 0; i < 8; ++i)
            dst[i] = make_float4(__uint_as_float(u[4 * i]), __uint_as_float(u[4 * i + 1]), __uint_as_float(u[4 * i + 2]), __uint_as_float(u[4 * i + 3]));
        }
      }
      tc_fence_before();
    }
  }
  cp_async_wait_all();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kCols);
  }
}

// The chunks of a sequence one after the other, 64 value channels of a head per CTA; the state in registers.
template <int DK>
struct DeltaChainCfg {
  static constexpr int kWBytes = CH * DK * 2;                      // one part of W; K
  static constexpr int kSBytes = DK * CH_ROWB;                     // one part of the state
  static constexpr int kSmem = 1024 + 3 * kWBytes + 2 * kSBytes + 2 * CH_CHUNK;
  static constexpr int kCols = 128;                                // W S 64 | K^T U 64
};

template <int DK>
__global__ void __launch_bounds__(CHT) delta_chain_kernel(const DeltaParams p) {
  using Cfg = DeltaChainCfg<DK>;
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t u_done, s_done;
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
  const int qd = warp & 3, half = warp >> 2, t = qd * 32 + lane;
  const uint32_t lane_addr = (uint32_t)(qd * 32) << 16;
  const int slot = c.slots[b];
  if (slot >= 0 && slot < c.num_slots) {
    const bool fresh = c.seq_lens[b] == c.cu_q[b + 1] - c.cu_q[b];
    const int c0 = c.seq_chunks[b], c1 = c.seq_chunks[b + 1];
    // key row of this thread's 32 value channels (a 64-row product: row 16 q + lane in 16 lanes)
    const int r = DK == 128 ? t : qd * 16 + lane;
    const bool holds = DK == 128 || lane < 16, live = holds && r < c.dk;
    float4* st = reinterpret_cast<float4*>(c.s + ((((long long)slot * c.H + h) * (c.VP / SC_COLS) + z * 2 + half) * c.KP + (holds ? r : 0)) * SC_COLS);
    float S[32];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !fresh) v = st[i];
      S[4 * i] = v.x; S[4 * i + 1] = v.y; S[4 * i + 2] = v.z; S[4 * i + 3] = v.w;
    }
    auto load_w = [&](int k) {
      const long long at = ((long long)k * c.H + h) * DK * CH;
#pragma unroll 4
      for (int i = tid; i < 2 * CH * (DK / 8); i += CHT) {         // parts, tiles of 64 columns, rows, pieces
        const int part = i / (CH * (DK / 8)), e = i % (CH * (DK / 8)), row = (e >> 3) % CH;
        cp_async16(w_s + part * Cfg::kWBytes + (e >> 3) / CH * CH_CHUNK + chunk_addr(row, e & 7), (part ? p.w_lo : p.w_hi) + at + e * 8, true);
      }
    };
    auto load_k = [&](int k) {
      const int4 ck = c.chunks[k];
      chunk_load<DK>(k_s, c.proj + (long long)ck.x * c.ld + c.k_col + hk * c.KP, c.ld, ck.y);
    };
    // what a thread needs of a chunk besides: its row of T diag(beta) V, the factor of its key, the chunk's decay
    float4 uv[8];
    float factor = 0.f, decay = 0.f;
    auto fetch = [&](int k) {
      const long long ch = (long long)k * c.H + h;
      const float4* src = reinterpret_cast<const float4*>(p.uv + ((ch * (c.VP / 64) + z) * CH + t) * 64 + half * 32);
#pragma unroll
      for (int i = 0; i < 8; ++i) uv[i] = src[i];
      decay = c.um[ch].x;
      factor = c.gates[ch * 3 * CH + t];
    };
    if (c0 < c1) { load_w(c0); load_k(c0); fetch(c0); }
    bool ok = true;
    for (int k = c0; k < c1; ++k) {
      const uint32_t phase = (uint32_t)((k - c0) & 1);
      const long long ch = (long long)k * c.H + h;
      const int4 ck = c.chunks[k];
      if (holds) {
        const long long at = ((ch * (c.VP / 64) + z) * c.KP + r) * 64 + half * 32;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) split_bf16x2(S[i * 8 + 2 * e], S[i * 8 + 2 * e + 1], hi[e], lo[e]);
          const uint4 a = make_uint4(hi[0], hi[1], hi[2], hi[3]), d = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          const uint32_t o = chunk_addr(r, half * 4 + i);
          *reinterpret_cast<uint4*>(s_p + o) = a;
          *reinterpret_cast<uint4*>(s_p + Cfg::kSBytes + o) = d;
          *reinterpret_cast<uint4*>(c.s_hi + at + i * 8) = a;
          *reinterpret_cast<uint4*>(c.s_lo + at + i * 8) = d;
        }
      }
      cp_async_wait_all();
      fence_proxy_async_smem();
      tc_fence_before();
      ok = __syncthreads_and(ok);
      if (!ok) break;
      tc_fence_after();
      if (warp == 0 && elect_one_sync()) {
        constexpr uint32_t idesc = make_idesc_bf16(CH, 64, 0, 1);
#pragma unroll
        for (int part = 0; part < 3; ++part)                       // W S without the product of the two small parts
#pragma unroll
          for (int kk = 0; kk < DK / 16; ++kk) {
            const uint64_t a = make_smem_desc_sw128(w_s + (part == 1 ? Cfg::kWBytes : 0) + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
            const uint64_t d = make_smem_desc_sw128(s_s + (part == 2 ? Cfg::kSBytes : 0) + kk * 2048, CH_CHUNK, 1024);
            umma_bf16(tmem, a, d, idesc, (part | kk) ? 1u : 0u);
          }
        umma_commit(smem_u32(&u_done));
      }
      __syncwarp();
      const float weight = chunk_exp2(decay + factor), keep = chunk_exp2(decay);
      ok = mbar_wait_bounded(smem_u32(&u_done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      if (ok) {
        if (k + 1 < c1) load_w(k + 1);                             // W has been read
        uint32_t v[32];
        tmem_ld_32x32(tmem + half * 32 + lane_addr, v);
        tmem_ld_wait();
        tc_fence_before();
        __nv_bfloat16* dst = p.values + (long long)(ck.x + t) * p.ld_values + h * c.VP + z * 64 + half * 32;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 x = uv[2 * i], y = uv[2 * i + 1];
          const float U[8] = {x.x - __uint_as_float(v[8 * i]),     x.y - __uint_as_float(v[8 * i + 1]), x.z - __uint_as_float(v[8 * i + 2]),
                              x.w - __uint_as_float(v[8 * i + 3]), y.x - __uint_as_float(v[8 * i + 4]), y.y - __uint_as_float(v[8 * i + 5]),
                              y.z - __uint_as_float(v[8 * i + 6]), y.w - __uint_as_float(v[8 * i + 7])};
          if (t < ck.y)
            *reinterpret_cast<uint4*>(dst + i * 8) =
                make_uint4(pack_bf16x2(U[0], U[1]), pack_bf16x2(U[2], U[3]), pack_bf16x2(U[4], U[5]), pack_bf16x2(U[6], U[7]));
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) split_bf16x2(weight * U[2 * e], weight * U[2 * e + 1], hi[e], lo[e]);
          const uint32_t o = chunk_addr(t, half * 4 + i);
          *reinterpret_cast<uint4*>(u_p + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(u_p + CH_CHUNK + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
        if (k + 1 < c1) fetch(k + 1);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      ok = __syncthreads_and(ok);
      if (!ok) break;
      tc_fence_after();
      if (warp == 0 && elect_one_sync()) {
        constexpr uint32_t idesc = make_idesc_bf16(DK, 64, 1, 1);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < CH / 16; ++kk) {
            const uint64_t a = make_smem_desc_sw128(k_s + kk * 2048, CH_CHUNK, 1024);
            const uint64_t d = make_smem_desc_sw128(u_s + part * CH_CHUNK + kk * 2048, CH_CHUNK, 1024);
            umma_bf16(tmem + 64, a, d, idesc, (part | kk) ? 1u : 0u);
          }
        umma_commit(smem_u32(&s_done));
      }
      __syncwarp();
      ok = mbar_wait_bounded(smem_u32(&s_done), phase, &abort_flag, c.status, ST_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      if (ok) {
        if (k + 1 < c1) load_k(k + 1);                             // K has been read
        uint32_t v[32];
        tmem_ld_32x32(tmem + 64 + half * 32 + lane_addr, v);
        tmem_ld_wait();
        tc_fence_before();
#pragma unroll
        for (int i = 0; i < 32; ++i) S[i] = fmaf(keep, S[i], __uint_as_float(v[i]));
      }
    }
    if (ok && live)
#pragma unroll
      for (int i = 0; i < 8; ++i) st[i] = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
  } else if (tid == 0) {
    set_status(c.status, ST_BAD_INDEX);
  }
  cp_async_wait_all();
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
  if (launch_kernel(delta_chain_kernel<DK>, dim3(c.VP / 64, c.H, n_seq), dim3(CHT), DeltaChainCfg<DK>::kSmem, stream, p) != cudaSuccess) return -12;
  ChunkParams out = c;
  out.v = p.values;
  out.ld_v = p.ld_values;
  return launch_kernel(recurrent_chunk_out_kernel<DK>, dim3(units < most ? units : most), dim3(CHT), ChunkOutCfg<DK>::kSmem, stream, out, units) == cudaSuccess ? 0 : -13;
}

}  // namespace rb
