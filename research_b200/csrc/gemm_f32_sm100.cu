// fp32 matrix products on the ordinary FMA pipes: C = A B^T with every operand, product and sum in 32-bit. The exact
// mode of models with a 32-bit residual stream runs on it; serving uses the tcgen05 kernels.
//
// A is [M, K] row-major; B is [N, K] row-major or, with b_kn, [K, N]. A batch walks blockIdx.z with one stride per
// operand (per-head products). With a tile table (mixture of experts) the tiles of one launch belong to different row groups
// and weight matrices. 64 x 64 tile, 16-deep k-blocks, 4 x 4 outputs per thread.
#include "common.cuh"

namespace rb {

constexpr int F32_BM = 64, F32_BK = 16, F32_THREADS = 256;

struct F32Group {
  const int4* tiles;                   // {first A row, valid rows (up to 128), first B row, first output column}; null: plain
  const int* num_tiles;
  int group_n;                         // output columns per group
  const unsigned long long* row_dst;   // output row r goes to this address instead of C
};

__global__ void __launch_bounds__(F32_THREADS)
gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ B, float* __restrict__ C, const float* __restrict__ bias, int M, int N, int K,
                long long lda, long long ldb, long long ldc, long long sa, long long sb, long long sc, int b_kn, int silu_cols,
                F32Group grp) {
  __shared__ float as[F32_BK][F32_BM + 4];
  __shared__ float bs[F32_BK][F32_BM + 4];
  pdl_launch_dependents();
  pdl_wait();
  A += blockIdx.z * sa;
  B += blockIdx.z * sb;
  C += blockIdx.z * sc;
  int m0 = blockIdx.y * F32_BM, n0 = blockIdx.x * F32_BM, col0 = 0;
  if (grp.tiles != nullptr) {          // blockIdx.x: tile, blockIdx.y: upper or lower 64 of its rows
    if ((int)blockIdx.x >= *grp.num_tiles) return;
    const int4 e = grp.tiles[blockIdx.x];
    m0 = e.x + m0;
    M = e.x + e.y;
    if (m0 >= M) return;
    n0 = e.z;
    N = e.z + min(F32_BM, grp.group_n - e.w);
    col0 = e.w - e.z;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += F32_BK) {
    for (int i = threadIdx.x; i < F32_BM * F32_BK; i += F32_THREADS) {
      const int r = i / F32_BK, k = i % F32_BK;
      as[k][r] = (m0 + r < M && k0 + k < K) ? A[(long long)(m0 + r) * lda + k0 + k] : 0.f;
    }
    if (!b_kn) {
      for (int i = threadIdx.x; i < F32_BM * F32_BK; i += F32_THREADS) {
        const int r = i / F32_BK, k = i % F32_BK;
        bs[k][r] = (n0 + r < N && k0 + k < K) ? B[(long long)(n0 + r) * ldb + k0 + k] : 0.f;
      }
    } else {
      for (int i = threadIdx.x; i < F32_BM * F32_BK; i += F32_THREADS) {
        const int k = i / F32_BM, r = i % F32_BM;
        bs[k][r] = (n0 + r < N && k0 + k < K) ? B[(long long)(k0 + k) * ldb + n0 + r] : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < F32_BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = as[k][ty * 4 + i]; b[i] = bs[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) {
        float* dst = grp.row_dst != nullptr ? reinterpret_cast<float*>(grp.row_dst[m]) : C + (long long)m * ldc;
        const float v = acc[i][j] + (bias != nullptr ? bias[n + col0] : 0.f);
        dst[n + col0] = n < silu_cols ? v / (1.f + expf(-v)) : v;
      }
    }
}

}  // namespace rb

using namespace rb;

extern "C" void rb_gemm_f32_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

extern "C" int rb_gemm_f32(const float* A, const float* B, float* C, const float* bias, int M, int N, int K, long long lda, long long ldb,
                           long long ldc, int batch, long long sa, long long sb, long long sc, int b_kn, int silu_cols,
                           cudaStream_t stream) {
  if (M <= 0 || N <= 0 || K <= 0 || batch <= 0 || batch > 65535) return -1;
  const dim3 grid((N + F32_BM - 1) / F32_BM, (M + F32_BM - 1) / F32_BM, batch);
  if (grid.y > 65535) return -1;
  return launch_kernel(gemm_f32_kernel, grid, dim3(F32_THREADS), 0, stream, A, B, C, bias, M, N, K, lda, ldb, ldc, sa, sb, sc, b_kn, silu_cols,
                       F32Group{nullptr, nullptr, 0, nullptr}) == cudaSuccess ? 0 : -11;
}

// Grouped product of a tile table whose tiles are 64 columns wide; B is [groups * group_n, K].
extern "C" int rb_gemm_f32_grouped(const float* A, const float* B, float* C, int K, long long lda, long long ldb, long long ldc, const void* tiles,
                                   const int* num_tiles, int max_tiles, int group_n, const unsigned long long* row_dst, cudaStream_t stream) {
  if (K <= 0 || max_tiles <= 0 || group_n <= 0 || tiles == nullptr || num_tiles == nullptr) return -1;
  return launch_kernel(gemm_f32_kernel, dim3(max_tiles, 2, 1), dim3(F32_THREADS), 0, stream, A, B, C, nullptr, 0, 0, K, lda, ldb, ldc, 0, 0, 0, 0, 0,
                       F32Group{(const int4*)tiles, num_tiles, group_n, row_dst}) == cudaSuccess ? 0 : -11;
}
