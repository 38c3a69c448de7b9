// Recurrent mixers with a matrix state per head, for sm_100a.
//
//   S_t = a_t S_(t-1) + b_t k_t v_t^T,   o_t = S_t^T q_t        (see ops/recurrent.py)
//
//   scan        token by token: decoded tokens, short portions and the exact mode. One CTA per (sequence, head, 32 value
//               channels); the state tile stays in registers over the tokens of the portion. A decoded token reads and writes
//               the state once, which is what bounds it.
//   gated_norm  RMS norm per head or over all heads, times sigmoid(gate), to the activation type
//
// State: s [slots, H, tiles, KP, 32], n [slots, H, tiles, KP], m [slots, H, tiles], all fp32. A tile of 32 value channels keeps its
// own copy of n and m, so that the CTAs of a head never share anything they write. Only the first `dk` of the KP rows are
// touched. A slot holds whatever its last user left: a portion that starts at position 0 starts from zero.
#include "common.cuh"

namespace rb {

constexpr int SC_THREADS = 256;
constexpr int SC_COLS = 32;                       // value channels of a tile
constexpr int SC_ROWS = SC_THREADS / (SC_COLS / 4);   // key rows covered by one pass of the CTA

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// log(sigmoid(z)) without cancellation at either end
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

struct ScanParams {
  const void* proj;        // [T, ld]: q | k | v (activation type)
  long long ld;
  int q_col, k_col, v_col;
  const float* small;      // [T, i | f] gate logits (gated)
  long long ld_small;
  const float* decay;      // [H] (not gated)
  const float* bias_i;     // [H]
  const float* bias_f;     // [H]
  float cap, q_scale;
  float* s;
  float* n;
  float* m;
  const int* slots;        // [B]
  const int* cu_q;         // [B+1] or null: one row per sequence
  const int* seq_lens;     // [B]
  float* out;              // [T, ldo]
  long long ldo;
  int H, dk, KP, VP, num_slots, silu, gated, rows;
  int* status;
};

// NR: key rows held by a thread (dk <= NR * SC_ROWS)
template <typename T, int NR>
__global__ void __launch_bounds__(SC_THREADS) recurrent_scan_kernel(const ScanParams p) {
  __shared__ float qs[NR * SC_ROWS], ks[NR * SC_ROWS], vs[SC_COLS];
  __shared__ float red[SC_THREADS / 32][SC_COLS];
  __shared__ float red_n[SC_THREADS / 32];
  pdl_launch_dependents();
  const int tile = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, c4 = tid & 7, r0 = tid >> 3, warp = tid >> 5, lane = tid & 31;
  pdl_wait();
  int t0 = b, t1 = b + 1;
  if (p.cu_q != nullptr) { t0 = p.cu_q[b]; t1 = p.cu_q[b + 1]; }
  int slot = p.slots[b];
  if (t1 > p.rows || slot >= p.num_slots) {
    if (tid == 0) set_status(p.status, ST_BAD_INDEX);
    return;
  }
  if (slot < 0) {                                  // padding row: defined output, no state
    for (int t = t0; t < t1; ++t)
      if (tid < SC_COLS) p.out[t * p.ldo + h * p.VP + tile * SC_COLS + tid] = 0.f;
    return;
  }
  const bool fresh = p.seq_lens[b] == t1 - t0;
  const long long unit = ((long long)slot * p.H + h) * (p.VP / SC_COLS) + tile;
  float4* st = reinterpret_cast<float4*>(p.s + unit * p.KP * SC_COLS);
  float* nt = p.n + unit * p.KP;
  float4 S[NR];
  float n[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = r0 + i * SC_ROWS;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    n[i] = 0.f;
    if (!fresh && r < p.dk) {
      S[i] = st[r * (SC_COLS / 4) + c4];
      if (p.gated) n[i] = nt[r];
    }
  }
  float m = fresh || !p.gated ? 0.f : p.m[unit];
  const T* proj = reinterpret_cast<const T*>(p.proj);
  const float decay = p.gated ? 0.f : p.decay[h];
  for (int t = t0; t < t1; ++t) {
    const T* row = proj + t * p.ld;
    for (int i = tid; i < p.dk; i += SC_THREADS) {
      float q = to_f<T>(row[p.q_col + h * p.KP + i]), k = to_f<T>(row[p.k_col + h * p.KP + i]);
      if (p.silu) { q = silu_f(q); k = silu_f(k); }
      qs[i] = q * p.q_scale;
      ks[i] = k;
    }
    if (tid < SC_COLS) {
      const float v = to_f<T>(row[p.v_col + h * p.VP + tile * SC_COLS + tid]);
      vs[tid] = p.silu ? silu_f(v) : v;
    }
    float a = decay, w = 1.f;
    if (p.gated) {
      const float* g = p.small + t * p.ld_small;
      const float gi = p.cap * tanhf((g[h] + p.bias_i[h]) / p.cap);
      const float gf = log_sigmoid_f(p.cap * tanhf((g[p.H + h] + p.bias_f[h]) / p.cap));
      const float m_new = fmaxf(gf + m, gi);
      a = expf(gf + m - m_new);
      w = expf(gi - m_new);
      m = m_new;
    }
    __syncthreads();
    const float4 v = *reinterpret_cast<const float4*>(&vs[c4 * 4]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    float nq = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = r0 + i * SC_ROWS;
      if (r < p.dk) {
        const float kw = w * ks[r], q = qs[r];
        S[i].x = fmaf(a, S[i].x, kw * v.x);
        S[i].y = fmaf(a, S[i].y, kw * v.y);
        S[i].z = fmaf(a, S[i].z, kw * v.z);
        S[i].w = fmaf(a, S[i].w, kw * v.w);
        acc.x = fmaf(q, S[i].x, acc.x);
        acc.y = fmaf(q, S[i].y, acc.y);
        acc.z = fmaf(q, S[i].z, acc.z);
        acc.w = fmaf(q, S[i].w, acc.w);
        n[i] = fmaf(a, n[i], kw);
        nq = fmaf(q, n[i], nq);
      }
    }
    // lanes of a warp: 4 key rows x 8 column groups; n . q is the same in the 8 lanes of a row
#pragma unroll
    for (int o = 8; o < 32; o <<= 1) {
      acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o);
      acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
      acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o);
      acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
      nq += __shfl_xor_sync(0xffffffffu, nq, o);
    }
    if (lane < 8) *reinterpret_cast<float4*>(&red[warp][lane * 4]) = acc;
    if (lane == 0) red_n[warp] = nq;
    __syncthreads();
    if (tid < SC_COLS) {
      float o = 0.f, d = 0.f;
#pragma unroll
      for (int i = 0; i < SC_THREADS / 32; ++i) { o += red[i][tid]; d += red_n[i]; }
      if (p.gated) o /= fmaxf(fabsf(d), expf(-m)) + 1e-6f;
      p.out[t * p.ldo + h * p.VP + tile * SC_COLS + tid] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = r0 + i * SC_ROWS;
    if (r < p.dk) {
      st[r * (SC_COLS / 4) + c4] = S[i];
      if (p.gated && c4 == 0) nt[r] = n[i];
    }
  }
  if (p.gated && tid == 0) p.m[unit] = m;
}

template <typename T>
static int launch_scan(const ScanParams& p, int B, cudaStream_t stream) {
  const dim3 grid(p.VP / SC_COLS, p.H, B);
  const int need = (p.dk + SC_ROWS - 1) / SC_ROWS;
  cudaError_t e;
  if (need <= 1) e = launch_kernel(recurrent_scan_kernel<T, 1>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 2) e = launch_kernel(recurrent_scan_kernel<T, 2>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 4) e = launch_kernel(recurrent_scan_kernel<T, 4>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 8) e = launch_kernel(recurrent_scan_kernel<T, 8>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 16) e = launch_kernel(recurrent_scan_kernel<T, 16>, grid, dim3(SC_THREADS), 0, stream, p);
  else return -1;
  return e == cudaSuccess ? 0 : -11;
}

// ------------------------------------------------------------------------------------------
// out = o / rms * weight * sigmoid(gate). One CTA per token; a warp takes whole heads. Padding channels of o are zero.
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, long long ldo, const float* __restrict__ weight,
                                                         const T* __restrict__ gate, long long ldg, T* __restrict__ out, long long ldy,
                                                         int H, int dv, int VP, int per_head, float eps) {
  __shared__ float part[8];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  const long long t = blockIdx.x;
  const float* x = o + t * ldo;
  float rs = 0.f;
  if (!per_head) {
    float s = 0.f;
    for (int i = threadIdx.x * 4; i < H * VP; i += 1024) {
      const float4 v = *reinterpret_cast<const float4*>(x + i);
      s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    s = warp_sum(s);
    if (lane == 0) part[warp] = s;
    __syncthreads();
    s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s += part[i];
    rs = 1.f / sqrtf(s / ((float)H * dv) + eps);
  }
  for (int h = warp; h < H; h += 8) {
    if (per_head) {
      float s = 0.f;
      for (int i = lane * 4; i < VP; i += 128) {
        const float4 v = *reinterpret_cast<const float4*>(x + h * VP + i);
        s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
      rs = 1.f / sqrtf(warp_sum(s) / dv + eps);
    }
    for (int i = lane * 4; i < VP; i += 128) {
      const int c = h * VP + i;
      const float4 v = *reinterpret_cast<const float4*>(x + c);
      const float4 w = *reinterpret_cast<const float4*>(weight + c);
      const T* g = gate + t * ldg + c;
      const float y0 = v.x * rs * w.x * sigmoid_f(to_f<T>(g[0])), y1 = v.y * rs * w.y * sigmoid_f(to_f<T>(g[1]));
      const float y2 = v.z * rs * w.z * sigmoid_f(to_f<T>(g[2])), y3 = v.w * rs * w.w * sigmoid_f(to_f<T>(g[3]));
      if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(out + t * ldy + c) = make_float4(y0, y1, y2, y3);
      else *reinterpret_cast<uint2*>(out + t * ldy + c) = make_uint2(pack_bf16x2(y0, y1), pack_bf16x2(y2, y3));
    }
  }
}

}  // namespace rb

using namespace rb;

extern "C" {

void rb_recurrent_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

int rb_recurrent_scan(const void* proj, long long ld, int q_col, int k_col, int v_col, const float* small, long long ld_small, const float* decay,
                      const float* bias_i, const float* bias_f, float cap, float q_scale, float* s, float* n, float* m, const int* slots,
                      const int* cu_q, const int* seq_lens, float* out, long long ldo, int H, int dk, int KP, int VP, int B, int num_slots,
                      int silu, int gated, int rows, int dtype, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || H > 65535 || B > 65535 || dk <= 0 || dk > KP || VP % SC_COLS != 0 || (gated ? small == nullptr : decay == nullptr)) return -1;
  const ScanParams p{proj, ld, q_col, k_col, v_col, small, ld_small, decay, bias_i, bias_f, cap, q_scale, s, n, m, slots, cu_q, seq_lens,
                     out, ldo, H, dk, KP, VP, num_slots, silu, gated, rows, status};
  return dtype == 0 ? launch_scan<__nv_bfloat16>(p, B, stream) : launch_scan<float>(p, B, stream);
}

int rb_gated_norm(const float* o, long long ldo, const float* weight, const void* gate, long long ldg, void* out, long long ldy, int H, int dv,
                  int VP, int per_head, int T, int dtype, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (VP % 4 != 0 || ldo % 4 != 0 || ldy % 4 != 0) return -1;
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(gated_norm_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, o, ldo, weight, (const __nv_bfloat16*)gate, ldg,
                      (__nv_bfloat16*)out, ldy, H, dv, VP, per_head, eps);
  else
    e = launch_kernel(gated_norm_kernel<float>, dim3(T), dim3(256), 0, stream, o, ldo, weight, (const float*)gate, ldg, (float*)out, ldy, H, dv, VP,
                      per_head, eps);
  return e == cudaSuccess ? 0 : -11;
}

}  // extern "C"
