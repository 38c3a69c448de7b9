// Recurrent mixers with a matrix state per head, for sm_100a.
//
//   S_t = a_t S_(t-1) + b_t k_t v_t^T,   o_t = S_t^T q_t        (see ops/recurrent.py)
//   o_t = S_(t-1)^T q_t + (sum_c u_c q_tc k_tc) v_t,  then row c of S decays by its own w_tc and takes k_tc v_t        (time mixing)
//   row c of S keeps f_tc of itself and takes (1 - f_tc) v_t,  o_t = S_t^T q_t                                         (forget mixing)
//   S decays by g_t and takes beta_t k_t (v_t - S^T k_t)^T,  o_t = S_t^T q_t                                           (delta rule)
//
//   scan        token by token: short portions and long ones of the exact mode. One CTA per (sequence, head, 32 value channels);
//               the state tile stays in registers over the tokens of the portion.
//   decode      one token per sequence: persistent CTAs stream state tiles through a ring of bulk copies
//   chunked     long portions, 128 tokens at a time on the tensor cores (tcgen05), in four launches: the gates, what every chunk
//               adds to the state (all chunks at once), the state in front of every chunk (one pass over the chunks), the
//               outputs (all chunks at once)
//   time mixing, one token per sequence: as decode, a whole head at a time, with the head's norm and the output gate
//   time mixing, forget mixing of long portions: chunked in the same way, in three launches
//   delta rule  short convolutions, SiLU and the heads' norms in a launch of their own; long portions: a triangular inverse per chunk,
//               one pass over the chunks, outputs
//   gated_norm  RMS norm per head or over all heads, times sigmoid(gate), to the activation type
//
// State: s [slots, H, tiles, KP, 32], n [slots, H, tiles, KP], m [slots, H, tiles], all fp32. A tile of 32 value channels keeps its
// own copy of n and m, so that the CTAs of a head never share anything they write. Only the first `dk` of the KP rows are
// touched. A slot holds whatever its last user left: a portion that starts at position 0 starts from zero.
#include "common.cuh"
#include "history.cuh"

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
// log(sigmoid(z)) without cancellation at either end
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

enum { FORM_PLAIN = 0, FORM_MIX = 1, FORM_FORGET = 2, FORM_DELTA = 3 };

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
  int H, dk, KP, VP, num_slots, gated, rows;
  const float* z;          // [T, ldz] time mixing: w = exp(-exp(z + w0)), column h * KP + key channel; forget mixing: logits of f
  long long ldz;
  const float* w0;         // [H * KP]
  const float* bonus;      // [H * KP]; forget mixing: the lower bound of f
  int* status;
  int ratio;               // heads that share queries and keys
  const float* units;      // [T, 2 * H / ratio] delta rule: factors of the queries, then of the keys
  const float* steps;      // [T, 2 * H] delta rule: logarithm of the decay, then the step size
};

__device__ __forceinline__ float channel_decay(float z) { return expf(-expf(z)); }

// Forget gate f = low + (1 - low) sigmoid(z) and what may be written, 1 - f.
__device__ __forceinline__ float2 forget_gate(float z, float low) {
  const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e * big;
  return make_float2(fmaf(1.f - low, z >= 0.f ? big : small, low), (1.f - low) * (z >= 0.f ? small : big));
}

// NR: key rows held by a thread (dk <= NR * SC_ROWS)
template <typename T, int NR, int FORM>
__global__ void __launch_bounds__(SC_THREADS) recurrent_scan_kernel(const ScanParams p) {
  constexpr bool MIX = FORM == FORM_MIX, FORGET = FORM == FORM_FORGET, DELTA = FORM == FORM_DELTA;
  __shared__ float qs[NR * SC_ROWS], ks[NR * SC_ROWS];
  __shared__ __align__(16) float vs[SC_COLS];
  __shared__ float ws[MIX || FORGET ? NR * SC_ROWS : 1];
  __shared__ __align__(16) float red[SC_THREADS / 32][SC_COLS];
  __shared__ __align__(16) float red_k[DELTA ? SC_THREADS / 32 : 1][SC_COLS];
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
  const float decay = p.gated || FORM != FORM_PLAIN ? 0.f : p.decay[h];
  const int hk = h / p.ratio;                      // whose queries and keys
  float bonus[MIX ? NR : 1];
  if (MIX)
#pragma unroll
    for (int i = 0; i < NR; ++i) bonus[i] = r0 + i * SC_ROWS < p.dk ? p.bonus[h * p.KP + r0 + i * SC_ROWS] : 0.f;
  for (int t = t0; t < t1; ++t) {
    const T* row = proj + t * p.ld;
    const float* unit_of = DELTA ? p.units + (long long)t * 2 * (p.H / p.ratio) + hk : nullptr;
    const float q_scale = DELTA ? p.q_scale * unit_of[0] : p.q_scale, k_scale = DELTA ? unit_of[p.H / p.ratio] : 1.f;
    for (int i = tid; i < p.dk; i += SC_THREADS) {
      qs[i] = to_f<T>(row[p.q_col + hk * p.KP + i]) * q_scale;
      if (FORGET) {
        const float2 f = forget_gate(p.z[t * p.ldz + h * p.KP + i] + p.w0[h * p.KP + i], p.bonus[h * p.KP + i]);
        ws[i] = f.x;
        ks[i] = f.y;
      } else {
        ks[i] = to_f<T>(row[p.k_col + hk * p.KP + i]) * k_scale;
      }
      if (MIX) ws[i] = channel_decay(p.z[t * p.ldz + h * p.KP + i] + p.w0[h * p.KP + i]);
    }
    if (tid < SC_COLS) {
      vs[tid] = to_f<T>(row[p.v_col + h * p.VP + tile * SC_COLS + tid]);
    }
    float a = decay, w = 1.f;
    if (DELTA) {
      const float* g = p.steps + (long long)t * 2 * p.H + h;
      a = expf(g[0]);
      w = g[p.H];
    }
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
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f), acc_k = acc;
    float nq = 0.f, kr[DELTA ? NR : 1];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = r0 + i * SC_ROWS;
      if (DELTA) {                                   // S^T k and S^T q of the state in front of the token, and q . k
        const float k = r < p.dk ? ks[r] : 0.f, q = r < p.dk ? qs[r] : 0.f;
        kr[DELTA ? i : 0] = k;
        acc_k.x = fmaf(k, S[i].x, acc_k.x);
        acc_k.y = fmaf(k, S[i].y, acc_k.y);
        acc_k.z = fmaf(k, S[i].z, acc_k.z);
        acc_k.w = fmaf(k, S[i].w, acc_k.w);
        acc.x = fmaf(q, S[i].x, acc.x);
        acc.y = fmaf(q, S[i].y, acc.y);
        acc.z = fmaf(q, S[i].z, acc.z);
        acc.w = fmaf(q, S[i].w, acc.w);
        nq = fmaf(q, k, nq);
      }
      if (FORGET && r < p.dk) {
        const float k = ks[r], q = qs[r], d = ws[r];
        S[i].x = fmaf(d, S[i].x, k * v.x);
        S[i].y = fmaf(d, S[i].y, k * v.y);
        S[i].z = fmaf(d, S[i].z, k * v.z);
        S[i].w = fmaf(d, S[i].w, k * v.w);
        acc.x = fmaf(q, S[i].x, acc.x);
        acc.y = fmaf(q, S[i].y, acc.y);
        acc.z = fmaf(q, S[i].z, acc.z);
        acc.w = fmaf(q, S[i].w, acc.w);
      }
      if (MIX && r < p.dk) {
        const float k = ks[r], q = qs[r], d = ws[r], u = bonus[MIX ? i : 0];
        const float4 kv = make_float4(k * v.x, k * v.y, k * v.z, k * v.w);
        acc.x = fmaf(q, fmaf(u, kv.x, S[i].x), acc.x);
        acc.y = fmaf(q, fmaf(u, kv.y, S[i].y), acc.y);
        acc.z = fmaf(q, fmaf(u, kv.z, S[i].z), acc.z);
        acc.w = fmaf(q, fmaf(u, kv.w, S[i].w), acc.w);
        S[i].x = fmaf(d, S[i].x, kv.x);
        S[i].y = fmaf(d, S[i].y, kv.y);
        S[i].z = fmaf(d, S[i].z, kv.z);
        S[i].w = fmaf(d, S[i].w, kv.w);
      }
      if (FORM == FORM_PLAIN && r < p.dk) {
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
      if (DELTA) {
        acc_k.x += __shfl_xor_sync(0xffffffffu, acc_k.x, o);
        acc_k.y += __shfl_xor_sync(0xffffffffu, acc_k.y, o);
        acc_k.z += __shfl_xor_sync(0xffffffffu, acc_k.z, o);
        acc_k.w += __shfl_xor_sync(0xffffffffu, acc_k.w, o);
      }
    }
    if (lane < 8) {
      *reinterpret_cast<float4*>(&red[warp][lane * 4]) = acc;
      if (DELTA) *reinterpret_cast<float4*>(&red_k[DELTA ? warp : 0][lane * 4]) = acc_k;
    }
    if (lane == 0) red_n[warp] = nq;
    const float my_v = DELTA && tid < SC_COLS ? vs[tid] : 0.f;
    __syncthreads();
    if (DELTA) {                                     // (what follows reads the sums alone: the next token's vectors may come)
      float4 sk = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < SC_THREADS / 32; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(&red_k[DELTA ? i : 0][c4 * 4]);
        sk.x += x.x; sk.y += x.y; sk.z += x.z; sk.w += x.w;
      }
      const float4 u = make_float4(w * (v.x - a * sk.x), w * (v.y - a * sk.y), w * (v.z - a * sk.z), w * (v.w - a * sk.w));
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const float k = kr[DELTA ? i : 0];
        S[i].x = fmaf(a, S[i].x, k * u.x);
        S[i].y = fmaf(a, S[i].y, k * u.y);
        S[i].z = fmaf(a, S[i].z, k * u.z);
        S[i].w = fmaf(a, S[i].w, k * u.w);
      }
    }
    if (tid < SC_COLS) {
      float o = 0.f, d = 0.f, sk = 0.f;
#pragma unroll
      for (int i = 0; i < SC_THREADS / 32; ++i) {
        o += red[i][tid];
        d += red_n[i];
        if (DELTA) sk += red_k[DELTA ? i : 0][tid];
      }
      if (p.gated) o /= fmaxf(fabsf(d), expf(-m)) + 1e-6f;
      if (DELTA) o = fmaf(a, o, d * (w * (my_v - a * sk)));
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

template <typename T, int FORM>
static int launch_scan(const ScanParams& p, int B, cudaStream_t stream) {
  const dim3 grid(p.VP / SC_COLS, p.H, B);
  const int need = (p.dk + SC_ROWS - 1) / SC_ROWS;
  cudaError_t e;
  if (need <= 1) e = launch_kernel(recurrent_scan_kernel<T, 1, FORM>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 2) e = launch_kernel(recurrent_scan_kernel<T, 2, FORM>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 4) e = launch_kernel(recurrent_scan_kernel<T, 4, FORM>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 8) e = launch_kernel(recurrent_scan_kernel<T, 8, FORM>, grid, dim3(SC_THREADS), 0, stream, p);
  else if (need <= 16) e = launch_kernel(recurrent_scan_kernel<T, 16, FORM>, grid, dim3(SC_THREADS), 0, stream, p);
  else return -1;
  return e == cudaSuccess ? 0 : -11;
}

// ------------------------------------------------------------------------------------------
// One token per sequence (row b of the batch is sequence b). The state is read and written once, which is all the time it
// takes: persistent CTAs walk over the (sequence, head, tile) units with RD_STAGES tiles in flight, bulk copies in both
// directions, the update in shared memory. The unit's vectors are fetched one unit ahead.
// ------------------------------------------------------------------------------------------
constexpr int RD_THREADS = 128, RD_STAGES = 3, RD_VEC = 3;
constexpr int RD_MAX_B = 4096;
constexpr int RD_MAX_DK = 384;                    // key rows: a ring of larger tiles does not fit

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void bulk_store(void* dst, uint32_t src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(src), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

template <typename T, int FORM>
__global__ void __launch_bounds__(RD_THREADS) recurrent_decode_kernel(const ScanParams p, int B, int units) {
  constexpr bool MIX = FORM == FORM_MIX, FORGET = FORM == FORM_FORGET, DELTA = FORM == FORM_DELTA;
  extern __shared__ __align__(128) uint8_t smem_raw[];       // RD_STAGES x [dk, 32] fp32, then the sequences' slots
  __shared__ float qs[RD_MAX_DK], ks[RD_MAX_DK];
  __shared__ float ws[MIX || FORGET ? RD_MAX_DK : 1], us[MIX ? RD_MAX_DK : 1];
  __shared__ __align__(16) float vs[SC_COLS];
  __shared__ __align__(16) float red[RD_THREADS / 32][SC_COLS];
  __shared__ __align__(16) float red_k[DELTA ? RD_THREADS / 32 : 1][SC_COLS];
  __shared__ float red_n[RD_THREADS / 32];
  __shared__ __align__(8) uint64_t full[RD_STAGES];
  __shared__ int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c4 = tid & 7, r0 = tid >> 3;
  const int tiles = p.VP / SC_COLS;
  const uint32_t ring = smem_u32(smem_raw), tile_bytes = (uint32_t)p.dk * SC_COLS * 4;
  if (tid == 0) {
    abort_flag = 0;
    for (int i = 0; i < RD_STAGES; ++i) mbar_init(smem_u32(&full[i]), 1);
    fence_mbar_init();
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  int* slots = reinterpret_cast<int*>(smem_raw + RD_STAGES * tile_bytes);      // -1: padding; bit 30: starts from zero
  for (int b = tid; b < B; b += RD_THREADS) {
    int s = p.slots[b];
    if (s >= p.num_slots) { set_status(p.status, ST_BAD_INDEX); s = -1; }
    slots[b] = s < 0 ? -1 : s | (p.seq_lens[b] == 1 ? 1 << 30 : 0);
  }
  __syncthreads();
  struct Unit { int b, h, tile, slot; bool fresh; };
  auto unit_of = [&](int u) {
    Unit x;
    x.tile = u % tiles;
    x.h = (u / tiles) % p.H;
    x.b = u / tiles / p.H;
    const int s = slots[x.b];
    x.fresh = s >= 0 && (s >> 30) != 0;
    x.slot = s < 0 ? -1 : s & ((1 << 30) - 1);
    return x;
  };
  auto state_index = [&](const Unit& x) { return ((long long)max(x.slot, 0) * p.H + x.h) * tiles + x.tile; };   // padding rows read slot 0
  int issued = 0;                                            // thread 0
  auto load = [&](int i) {                                   // thread 0: tile of this CTA's i-th unit
    const int u = blockIdx.x + i * gridDim.x;
    if (u >= units) return;
    const Unit x = unit_of(u);
    const uint32_t bar = smem_u32(&full[i % RD_STAGES]);
    mbar_expect_tx(bar, tile_bytes);
    bulk_load(ring + (i % RD_STAGES) * tile_bytes, p.s + state_index(x) * p.KP * SC_COLS, tile_bytes, bar);
    issued = i + 1;
  };
  if (tid == 0)
    for (int i = 0; i < RD_STAGES - 1; ++i) load(i);
  float q[RD_VEC], k[RD_VEC], n[RD_VEC], v = 0.f, gi = 0.f, gf = 0.f, m0 = 0.f;
  float z[MIX || FORGET ? RD_VEC : 1], bonus[MIX || FORGET ? RD_VEC : 1];
  Unit x{};
  auto fetch = [&](int u) {
    x = unit_of(u);
    const T* row = reinterpret_cast<const T*>(p.proj) + x.b * p.ld;
    const float* nt = p.n + state_index(x) * p.KP;
    const int hk = x.h / p.ratio;
    const float* unit = DELTA ? p.units + (long long)x.b * 2 * (p.H / p.ratio) + hk : nullptr;
    const float q_scale = DELTA ? p.q_scale * unit[0] : p.q_scale, k_scale = DELTA ? unit[p.H / p.ratio] : 1.f;
#pragma unroll
    for (int i = 0; i < RD_VEC; ++i) {
      const int r = tid + i * RD_THREADS;
      q[i] = k[i] = n[i] = 0.f;
      if (r < p.dk) {
        q[i] = to_f<T>(row[p.q_col + hk * p.KP + r]) * q_scale;
        if (!FORGET) k[i] = to_f<T>(row[p.k_col + hk * p.KP + r]) * k_scale;
        if (p.gated) n[i] = nt[r];
        if (MIX || FORGET) {
          z[i] = p.z[x.b * p.ldz + x.h * p.KP + r] + p.w0[x.h * p.KP + r];
          bonus[i] = p.bonus[x.h * p.KP + r];
        }
      }
    }
    if (tid < SC_COLS) v = to_f<T>(row[p.v_col + x.h * p.VP + x.tile * SC_COLS + tid]);
    if (p.gated) {
      gi = p.small[x.b * p.ld_small + x.h];
      gf = p.small[x.b * p.ld_small + p.H + x.h];
      m0 = p.m[state_index(x)];
    }
    if (DELTA) {
      gf = p.steps[(long long)x.b * 2 * p.H + x.h];
      gi = p.steps[(long long)x.b * 2 * p.H + p.H + x.h];
    }
  };
  if ((int)blockIdx.x < units) fetch(blockIdx.x);
  bool ok = true;
  int it = 0;
  for (int u = blockIdx.x; u < units; u += gridDim.x, ++it) {
    const Unit cur = x;
    const bool zero = cur.fresh;
    if (zero) m0 = n[0] = n[1] = n[2] = 0.f;
    float a = 0.f, w = 1.f, m = 0.f;
    if (p.gated) {
      gi = p.cap * tanhf((gi + p.bias_i[cur.h]) / p.cap);
      gf = log_sigmoid_f(p.cap * tanhf((gf + p.bias_f[cur.h]) / p.cap));
      m = fmaxf(gf + m0, gi);
      a = expf(gf + m0 - m);
      w = expf(gi - m);
    } else if (FORM == FORM_PLAIN) {
      a = p.decay[cur.h];
    }
    if (DELTA) {
      a = expf(gf);
      w = gi;
    }
    const long long si = state_index(cur);
    float nq = 0.f;
#pragma unroll
    for (int i = 0; i < RD_VEC; ++i) {
      const int r = tid + i * RD_THREADS;
      if (r < p.dk) {
        const float kw = DELTA ? k[i] : w * k[i];
        qs[r] = q[i];
        ks[r] = kw;
        if (DELTA) nq = fmaf(q[i], kw, nq);
        if (MIX) { ws[r] = channel_decay(z[MIX ? i : 0]); us[r] = bonus[MIX ? i : 0]; }
        if (FORGET) {
          const float2 f = forget_gate(z[FORGET ? i : 0], bonus[FORGET ? i : 0]);
          ws[r] = f.x;
          ks[r] = f.y;
        }
        if (p.gated) {
          const float nn = fmaf(a, n[i], kw);
          nq = fmaf(q[i], nn, nq);
          if (cur.slot >= 0) p.n[si * p.KP + r] = nn;
        }
      }
    }
    if (tid < SC_COLS) vs[tid] = v;
    if (p.gated && tid == 0 && cur.slot >= 0) p.m[si] = m;
    const int stage = it % RD_STAGES;
    ok = mbar_wait_bounded(smem_u32(&full[stage]), (uint32_t)((it / RD_STAGES) & 1), &abort_flag, p.status, ST_TIMEOUT_SMEM_FULL);
    ok = __syncthreads_and(ok);
    if (!ok) break;
    if (u + (int)gridDim.x < units) fetch(u + gridDim.x);
    float4* S = reinterpret_cast<float4*>(smem_raw + stage * tile_bytes);
    float4 vv = *reinterpret_cast<const float4*>(&vs[c4 * 4]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f), out_k = acc;
    const float my_v = DELTA && tid < SC_COLS ? vs[tid] : 0.f;
    if (DELTA) {                                             // S^T k and S^T q of the state in front of the token
      if (!zero)
#pragma unroll 4
        for (int r = r0; r < p.dk; r += RD_THREADS / 8) {
          const float4 s = S[r * (SC_COLS / 4) + c4];
          const float kw = ks[r], qr = qs[r];
          out_k.x = fmaf(kw, s.x, out_k.x);
          out_k.y = fmaf(kw, s.y, out_k.y);
          out_k.z = fmaf(kw, s.z, out_k.z);
          out_k.w = fmaf(kw, s.w, out_k.w);
          acc.x = fmaf(qr, s.x, acc.x);
          acc.y = fmaf(qr, s.y, acc.y);
          acc.z = fmaf(qr, s.z, acc.z);
          acc.w = fmaf(qr, s.w, acc.w);
        }
#pragma unroll
      for (int o = 8; o < 32; o <<= 1) {
        out_k.x += __shfl_xor_sync(0xffffffffu, out_k.x, o);
        out_k.y += __shfl_xor_sync(0xffffffffu, out_k.y, o);
        out_k.z += __shfl_xor_sync(0xffffffffu, out_k.z, o);
        out_k.w += __shfl_xor_sync(0xffffffffu, out_k.w, o);
      }
      if (lane < 8) *reinterpret_cast<float4*>(&red_k[DELTA ? warp : 0][lane * 4]) = out_k;
      __syncthreads();
      float4 sk = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < RD_THREADS / 32; ++i) {
        const float4 y = *reinterpret_cast<const float4*>(&red_k[DELTA ? i : 0][c4 * 4]);
        sk.x += y.x; sk.y += y.y; sk.z += y.z; sk.w += y.w;
      }
      vv = make_float4(w * (vv.x - a * sk.x), w * (vv.y - a * sk.y), w * (vv.z - a * sk.z), w * (vv.w - a * sk.w));
    }
#pragma unroll 4
    for (int r = r0; r < p.dk; r += RD_THREADS / 8) {
      float4 s = zero ? make_float4(0.f, 0.f, 0.f, 0.f) : S[r * (SC_COLS / 4) + c4];
      const float kw = ks[r], qr = DELTA ? 0.f : qs[r];
      if (FORGET) a = ws[r];
      if (MIX) {                                             // the state in front of the token, and the token with its bonus
        const float bo = us[r];
        acc.x = fmaf(qr, fmaf(bo, kw * vv.x, s.x), acc.x);
        acc.y = fmaf(qr, fmaf(bo, kw * vv.y, s.y), acc.y);
        acc.z = fmaf(qr, fmaf(bo, kw * vv.z, s.z), acc.z);
        acc.w = fmaf(qr, fmaf(bo, kw * vv.w, s.w), acc.w);
        a = ws[r];
      }
      s.x = fmaf(a, s.x, kw * vv.x);
      s.y = fmaf(a, s.y, kw * vv.y);
      s.z = fmaf(a, s.z, kw * vv.z);
      s.w = fmaf(a, s.w, kw * vv.w);
      if (!MIX && !DELTA) {
        acc.x = fmaf(qr, s.x, acc.x);
        acc.y = fmaf(qr, s.y, acc.y);
        acc.z = fmaf(qr, s.z, acc.z);
        acc.w = fmaf(qr, s.w, acc.w);
      }
      S[r * (SC_COLS / 4) + c4] = s;
    }
    fence_proxy_async_smem();
#pragma unroll
    for (int o = 8; o < 32; o <<= 1) {
      acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o);
      acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
      acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o);
      acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
    }
    if (p.gated || DELTA) nq = warp_sum(nq);
    if (lane < 8) *reinterpret_cast<float4*>(&red[warp][lane * 4]) = acc;
    if (lane == 0) red_n[warp] = nq;
    __syncthreads();
    if (tid == 0) {
      if (cur.slot >= 0) bulk_store(p.s + si * p.KP * SC_COLS, ring + stage * tile_bytes, tile_bytes);
      else asm volatile("cp.async.bulk.commit_group;" ::: "memory");
      asm volatile("cp.async.bulk.wait_group.read 1;" ::: "memory");     // the tile stored one unit ago has left its stage
      load(it + RD_STAGES - 1);
    }
    if (tid < SC_COLS) {
      float o = 0.f, d = 0.f, sk = 0.f;
#pragma unroll
      for (int i = 0; i < RD_THREADS / 32; ++i) {
        o += red[i][tid];
        d += red_n[i];
        if (DELTA) sk += red_k[DELTA ? i : 0][tid];
      }
      if (p.gated) o /= fmaxf(fabsf(d), expf(-m)) + 1e-6f;
      if (DELTA) o = fmaf(a, o, d * (w * (my_v - a * sk)));
      p.out[cur.b * p.ldo + cur.h * p.VP + cur.tile * SC_COLS + tid] = cur.slot < 0 ? 0.f : o;
    }
  }
  if (tid == 0) {
    if (!ok)                                                 // no copy may land after the CTA has gone
      for (int i = it; i < issued; ++i) {
        const uint64_t t0 = globaltimer_ns();
        while (!mbar_try_wait(smem_u32(&full[i % RD_STAGES]), (uint32_t)((i / RD_STAGES) & 1)))
          if (globaltimer_ns() - t0 > 50000000ull) break;
      }
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  }
}

template <typename T, int FORM>
static int launch_decode(const ScanParams& p, int B, cudaStream_t stream) {
  static int sms[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  const int smem = RD_STAGES * p.dk * SC_COLS * 4 + B * 4;
  if (sms[dev] == 0) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess ||
        cudaFuncSetAttribute(recurrent_decode_kernel<T, FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, RD_STAGES * RD_MAX_DK * SC_COLS * 4 + RD_MAX_B * 4) != cudaSuccess)
      return -10;
    sms[dev] = n;
  }
  const int per_sm = 200 * 1024 / (smem + 7 * 1024) > 6 ? 6 : 200 * 1024 / (smem + 7 * 1024);
  const int units = B * p.H * (p.VP / SC_COLS), grid = units < sms[dev] * per_sm ? units : sms[dev] * per_sm;
  return launch_kernel(recurrent_decode_kernel<T, FORM>, dim3(grid), dim3(RD_THREADS), smem, stream, p, B, units) == cudaSuccess ? 0 : -11;
}

// ------------------------------------------------------------------------------------------
// Chunked form. In a chunk of up to CH tokens of one sequence let F_t be the sum of the logarithms of the decays up to and
// including token t, g_j = log b_j - F_j, and (m, S, n) the state in front of the chunk. Then with B_t = max(m, max_{j<=t} g_j)
//
//   numerator_t   = sum_{j<=t} exp(g_j - B_t) (q_t . k_j) v_j  +  exp(m - B_t) S^T q_t
//   normaliser_t  = the same with v_j = 1 and n for S,           m_t = F_t + B_t
//
// and with G = max_j g_j the chunk itself contributes U = sum_j exp(g_j - G) k_j v_j^T (relative to exp(F_C + G)) to the state
// behind it. A constant decay has no normaliser and no maximum: there B_t = -F_t, G = -F_C and m = 0 throughout.
//
// Products on the tensor cores take bf16 operands; the incoming state and the weighted keys are split into two bf16 parts
// each, so that what is carried from chunk to chunk keeps 16 bits of mantissa per product and fp32 sums.
// ------------------------------------------------------------------------------------------
constexpr int CH = 128;                   // tokens of a chunk
constexpr int CHT = 256;                  // threads
constexpr int CH_ROWB = 128;              // bytes of a swizzled row: 64 bf16
constexpr int CH_CHUNK = CH * CH_ROWB;    // 64 columns of a [CH, .] tile
constexpr float LOG2E = 1.4426950408889634f;

struct ChunkParams {
  const __nv_bfloat16* proj;
  long long ld;
  int q_col, k_col, v_col;
  const float* small;
  long long ld_small;
  const float* decay;
  const float* bias_i;
  const float* bias_f;
  float cap, q_scale;
  const int4* chunks;      // {first packed row, tokens, sequence, 1 when it starts the sequence's portion}
  const int* seq_chunks;   // [n_seq + 1] first chunk of every sequence
  const int* slots;        // [n_seq]
  const int* seq_lens;     // [n_seq]
  const int* cu_q;         // [n_seq + 1]
  float* s;
  float* n;
  float* m;
  float* u;                // [chunks, H, tiles, KP, 32]
  float* un;               // [chunks, H, KP]
  float2* um;              // [chunks, H] {F_C, F_C + G}
  float* gates;            // [chunks, H, 3, CH] see recurrent_chunk_gates_kernel
  __nv_bfloat16* s_hi;     // [chunks, H, VP/64, KP, 64] state in front of the chunk
  __nv_bfloat16* s_lo;
  float* s_n;              // [chunks, H, KP]
  float* s_m;              // [chunks, H]
  float* out;
  long long ldo;
  int H, dk, KP, VP, num_slots, gated;
  int* status;
  const __nv_bfloat16* v;  // [T, ld_v] values
  long long ld_v;
  int ratio;               // heads that share queries and keys
  // delta rule: values [chunks, H, VP / 64, 8, CH, 8], the state's parts as they lie in shared memory, and the third of a token's gates is a
  // factor of its query
  const __nv_bfloat16* written;
};

__device__ __forceinline__ float chunk_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// g_j and F_j of the chunk's tokens (in units of log2), by one warp: four tokens per lane. Invalid tokens get g = -inf.
// gs[t] = g_t, bs[t] = running maximum of g (gated) or -F_t, fs[t] = F_t. Returns {F_C, max g} in every lane of the warp.
__device__ __forceinline__ float2 chunk_gates(const ChunkParams& p, int h, int row0, int n, float* gs, float* bs, float* fs) {
  const int lane = threadIdx.x & 31;
  float lf[4], li[4], F[4], run = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = lane * 4 + i;
    const float* g = p.small + (long long)(row0 + min(t, n - 1)) * p.ld_small;
    li[i] = p.gated ? g[h] : 0.f;
    lf[i] = p.gated ? g[p.H + h] : 0.f;
  }
  const float bias_i = p.gated ? p.bias_i[h] : 0.f, bias_f = p.gated ? p.bias_f[h] : 0.f;
  const float fixed = p.gated ? 0.f : logf(fmaxf(p.decay[h], 1e-30f)) * LOG2E;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (p.gated) {
      li[i] = p.cap * tanhf((li[i] + bias_i) / p.cap) * LOG2E;
      lf[i] = log_sigmoid_f(p.cap * tanhf((lf[i] + bias_f) / p.cap)) * LOG2E;
    } else {
      lf[i] = fixed;
    }
    if (lane * 4 + i >= n) lf[i] = 0.f;
    run += lf[i];
    F[i] = run;
  }
  float before = run;                                      // exclusive scan of the lanes' sums
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float y = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += y;
  }
  const float total = __shfl_sync(0xffffffffu, before, 31);
  before -= run;
  float mx = -INFINITY, g[4], top[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    F[i] += before;
    g[i] = lane * 4 + i < n ? li[i] - F[i] : -INFINITY;
    mx = fmaxf(mx, g[i]);
    top[i] = mx;
  }
  float up = mx;                                           // running maximum over the lanes before this one
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float y = __shfl_up_sync(0xffffffffu, up, o);
    if (lane >= o) up = fmaxf(up, y);
  }
  const float all = __shfl_sync(0xffffffffu, up, 31);
  float prev = __shfl_up_sync(0xffffffffu, up, 1);
  if (lane == 0) prev = -INFINITY;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    gs[lane * 4 + i] = g[i];
    bs[lane * 4 + i] = p.gated ? fmaxf(prev, top[i]) : -F[i];
    fs[lane * 4 + i] = F[i];
  }
  return make_float2(total, all);
}

// 16-byte unit u (8 columns) of row r in a [rows, 64] swizzled chunk
__device__ __forceinline__ uint32_t chunk_addr(int r, int u) { return (uint32_t)(r * CH_ROWB + ((u ^ (r & 7)) << 4)); }

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {     // zeros when not valid
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// [CH, DK] columns of a projection into swizzled chunks, asynchronously; rows past n are zero
template <int DK>
__device__ __forceinline__ void chunk_load(uint32_t dst, const __nv_bfloat16* src, long long ld, int n) {
#pragma unroll 4
  for (int i = threadIdx.x; i < CH * (DK / 8); i += CHT) {
    const int r = i / (DK / 8), u = i % (DK / 8);
    cp_async16(dst + (u >> 3) * CH_CHUNK + chunk_addr(r, u & 7), src + (r < n ? r : 0) * ld + u * 8, r < n);
  }
}

// Gates of every chunk and head, a warp each: g, B' (running maximum of g, or -F) and F per token in units of log2.
__global__ void __launch_bounds__(256) recurrent_chunk_gates_kernel(const ChunkParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const int4 ck = p.chunks[c];
  const long long ch = (long long)c * p.H + h;
  float* g = p.gates + ch * 3 * CH;
  const float2 t = chunk_gates(p, h, ck.x, ck.y, g, g + CH, g + 2 * CH);
  const float G = p.gated ? t.y : -t.x;
  if ((threadIdx.x & 31) == 0) p.um[ch] = make_float2(t.x, t.x + G);
}

// A work unit of the two kernels below: 64 value channels of one head of one chunk. Persistent CTAs walk over the units, the
// value channels of a head next to each other (they share its keys and queries in L2), and fetch a unit ahead.
struct ChunkUnit {
  int c, h, z, row0, n;
  long long ch;
};
__device__ __forceinline__ ChunkUnit chunk_unit(const ChunkParams& p, int u) {
  ChunkUnit x;
  const int zs = p.VP / 64;
  x.z = u % zs;
  x.h = (u / zs) % p.H;
  x.c = u / zs / p.H;
  const int4 ck = p.chunks[x.c];
  x.row0 = ck.x;
  x.n = ck.y;
  x.ch = (long long)x.c * p.H + x.h;
  return x;
}

// What a chunk adds to the state: U [KP, 64 value channels].
template <int DK>
struct ChunkStateCfg {
  static constexpr int kKBytes = CH * DK * 2;
  static constexpr int kSmem = 1024 + 2 * kKBytes + 2 * CH_CHUNK;      // weighted keys in two parts, two V tiles
  static constexpr int kCols = DK > 128 ? 128 : 64;
};

template <int DK>
__global__ void __launch_bounds__(CHT, DK <= 128 ? 2 : 1) recurrent_chunk_state_kernel(const ChunkParams p, int units) {
  using Cfg = ChunkStateCfg<DK>;
  constexpr int UNITS = CH * (DK / 8) / CHT;          // 16-byte pieces of K per thread
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ float gs[CH], nred[4][DK];
  __shared__ __align__(8) uint64_t done;
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* hi = smem_raw + (base - smem_u32(smem_raw));
  uint8_t* lo = hi + Cfg::kKBytes;
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
  uint4 raw[UNITS];
  float weight = 0.f;
  auto fetch = [&](const ChunkUnit& x, int buf) {
    chunk_load<64>(base + 2 * Cfg::kKBytes + buf * CH_CHUNK, p.v + x.row0 * p.ld_v + x.h * p.VP + x.z * 64, p.ld_v, x.n);
    const __nv_bfloat16* k = p.proj + x.row0 * p.ld + p.k_col + x.h * p.KP;
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
      const int e = tid + i * CHT, r = e / (DK / 8), u = e % (DK / 8);
      raw[i] = make_uint4(0u, 0u, 0u, 0u);
      if (r < x.n) raw[i] = *reinterpret_cast<const uint4*>(k + r * p.ld + u * 8);
    }
    if (tid < CH) {
      const float2 t = p.um[x.ch];
      weight = p.gates[x.ch * 3 * CH + tid] - (t.y - t.x);             // relative to exp(F_C + G)
    }
  };
  ChunkUnit x{};
  if ((int)blockIdx.x < units) { x = chunk_unit(p, blockIdx.x); fetch(x, 0); }
  bool ok = true;
  int it = 0;
  for (int u = blockIdx.x; u < units; u += gridDim.x, ++it) {
    const ChunkUnit cur = x;
    if (tid < CH) gs[tid] = chunk_exp2(weight);
    ok = __syncthreads_and(ok);                        // also: everyone is done with the unit before
    if (!ok) break;
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
      const int e = tid + i * CHT, r = e / (DK / 8), uu = e % (DK / 8);
      const float w = gs[r];
      uint4 a, b;
      auto one = [&](uint32_t v, uint32_t& l) {
        float2 f = unpack_bf16x2(v);
        f.x *= w; f.y *= w;
        const uint32_t o = pack_bf16x2(f.x, f.y);
        const float2 back = unpack_bf16x2(o);
        l = pack_bf16x2(f.x - back.x, f.y - back.y);
        return o;
      };
      a.x = one(raw[i].x, b.x); a.y = one(raw[i].y, b.y); a.z = one(raw[i].z, b.z); a.w = one(raw[i].w, b.w);
      const uint32_t at = (uu >> 3) * CH_CHUNK + chunk_addr(r, uu & 7);
      *reinterpret_cast<uint4*>(hi + at) = a;
      *reinterpret_cast<uint4*>(lo + at) = b;
    }
    cp_async_wait_all();
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 0 && elect_one_sync()) {
      const uint32_t v_s = base + 2 * Cfg::kKBytes + (it & 1) * CH_CHUNK;
#pragma unroll
      for (int m0 = 0; m0 < DK; m0 += 128) {
        const uint32_t idesc = make_idesc_bf16(DK - m0 >= 128 ? 128 : 64, 64, 1, 1);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < CH / 16; ++kk) {
            const uint64_t a = make_smem_desc_sw128(base + part * Cfg::kKBytes + (m0 / 64) * CH_CHUNK + kk * 2048, CH_CHUNK, 1024);
            const uint64_t b = make_smem_desc_sw128(v_s + kk * 2048, CH_CHUNK, 1024);
            umma_bf16(tmem + (m0 / 128) * 64, a, b, idesc, (part | kk) ? 1u : 0u);
          }
      }
      umma_commit(smem_u32(&done));
    }
    __syncwarp();
    if (u + (int)gridDim.x < units) { x = chunk_unit(p, u + gridDim.x); fetch(x, (it + 1) & 1); }
    if (p.gated && cur.z == 0) {       // the normaliser's part, while the tensor cores work: column sums of the weighted keys
      constexpr int PAIRS = DK / 2, GROUPS = 4;
      for (int i = tid; i < PAIRS * GROUPS; i += CHT) {
        const int pr = i % PAIRS, g = i / PAIRS;
        float sx = 0.f, sy = 0.f;
#pragma unroll 8
        for (int r = g * (CH / GROUPS); r < (g + 1) * (CH / GROUPS); ++r) {
          const uint32_t at = (pr >> 5) * CH_CHUNK + chunk_addr(r, (pr & 31) >> 2) + (pr & 3) * 4;
          const float2 a = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(hi + at)), b = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(lo + at));
          sx += a.x + b.x;
          sy += a.y + b.y;
        }
        nred[g][2 * pr] = sx;
        nred[g][2 * pr + 1] = sy;
      }
      __syncthreads();
      for (int i = tid; i < DK; i += CHT) p.un[cur.ch * p.KP + i] = (nred[0][i] + nred[1][i]) + (nred[2][i] + nred[3][i]);
    }
    ok = mbar_wait_bounded(smem_u32(&done), it & 1, &abort_flag, p.status, ST_TIMEOUT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    if (ok) {
      const int qd = warp & 3, half = warp >> 2;       // lanes of a TMEM quarter; the two warps of a quarter split the columns
      float* dstu = p.u + (cur.ch * (p.VP / 32) + cur.z * 2 + half) * p.KP * 32;
#pragma unroll
      for (int m0 = 0; m0 < DK; m0 += 128) {
        uint32_t v[32];
        tmem_ld_32x32(tmem + (m0 / 128) * 64 + half * 32 + ((uint32_t)(qd * 32) << 16), v);
        tmem_ld_wait();
        // a 128-row product has row 32 q + lane in quarter q, a 64-row one row 16 q + lane in its first 16 lanes
        const bool full = DK - m0 >= 128;
        const int r = m0 + (full ? qd * 32 + lane : qd * 16 + lane);
        if (full || lane < 16) {
          float4* dst = reinterpret_cast<float4*>(dstu + (long long)r * 32);
#pragma unroll
          for (int i = 0; i < 8; ++i)
            dst[i] = make_float4(__uint_as_float(v[4 * i]), __uint_as_float(v[4 * i + 1]), __uint_as_float(v[4 * i + 2]), __uint_as_float(v[4 * i + 3]));
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

// The state in front of every chunk, as two bf16 parts, and the state behind the portion. Every thread carries four value
// channels of one key row over the chunks. blockIdx: 32 key rows, tile of 32 value channels + head, sequence.
constexpr int CHAIN_AHEAD = 8;

__global__ void __launch_bounds__(256) recurrent_chunk_chain_kernel(const ChunkParams p) {
  pdl_launch_dependents();
  const int tiles = p.VP / SC_COLS;
  const int tile = blockIdx.y % tiles, h = blockIdx.y / tiles, b = blockIdx.z;
  const int c4 = threadIdx.x & 7, r = blockIdx.x * 32 + (threadIdx.x >> 3);
  pdl_wait();
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) { if (threadIdx.x == 0) set_status(p.status, ST_BAD_INDEX); return; }
  const bool fresh = p.seq_lens[b] == p.cu_q[b + 1] - p.cu_q[b];
  const int c0 = p.seq_chunks[b], c1 = p.seq_chunks[b + 1];
  const long long unit = ((long long)slot * p.H + h) * tiles + tile;
  float4* st = reinterpret_cast<float4*>(p.s + (unit * p.KP + r) * SC_COLS) + c4;
  float* nt = p.n + unit * p.KP + r;
  const bool live = r < p.dk;
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  float n = 0.f, m = 0.f;
  if (!fresh) {
    if (live) S = *st;
    if (p.gated) {
      if (live) n = *nt;
      m = p.m[unit] * LOG2E;
    }
  }
  const bool owns_n = p.gated && tile == 0 && c4 == 0;
  for (int cb = c0; cb < c1; cb += CHAIN_AHEAD) {
    float4 U[CHAIN_AHEAD];
    float un[CHAIN_AHEAD];
    float2 um[CHAIN_AHEAD];
#pragma unroll
    for (int i = 0; i < CHAIN_AHEAD; ++i) {
      const int c = cb + i;
      if (c < c1) {
        U[i] = *(reinterpret_cast<const float4*>(p.u + ((((long long)c * p.H + h) * tiles + tile) * p.KP + r) * SC_COLS) + c4);
        un[i] = p.gated ? p.un[((long long)c * p.H + h) * p.KP + r] : 0.f;
        um[i] = p.um[(long long)c * p.H + h];
      }
    }
#pragma unroll
    for (int i = 0; i < CHAIN_AHEAD; ++i) {
      const int c = cb + i;
      if (c < c1) {
        const long long ch = (long long)c * p.H + h;
        const uint32_t h0 = pack_bf16x2(S.x, S.y), h1 = pack_bf16x2(S.z, S.w);
        const float2 b0 = unpack_bf16x2(h0), b1 = unpack_bf16x2(h1);
        const long long at = ((ch * (p.VP / 64) + (tile >> 1)) * p.KP + r) * 64 + (tile & 1) * 32 + c4 * 4;
        *reinterpret_cast<uint2*>(p.s_hi + at) = make_uint2(h0, h1);
        *reinterpret_cast<uint2*>(p.s_lo + at) = make_uint2(pack_bf16x2(S.x - b0.x, S.y - b0.y), pack_bf16x2(S.z - b1.x, S.w - b1.y));
        if (owns_n) {
          p.s_n[ch * p.KP + r] = n;
          if (r == 0) p.s_m[ch] = m;
        }
        float a, w = 1.f;
        if (p.gated) {
          const float m_new = fmaxf(um[i].x + m, um[i].y);
          a = chunk_exp2(um[i].x + m - m_new);
          w = chunk_exp2(um[i].y - m_new);
          m = m_new;
        } else {
          a = chunk_exp2(um[i].x);
        }
        S.x = fmaf(a, S.x, w * U[i].x);
        S.y = fmaf(a, S.y, w * U[i].y);
        S.z = fmaf(a, S.z, w * U[i].z);
        S.w = fmaf(a, S.w, w * U[i].w);
        n = fmaf(a, n, w * un[i]);
      }
    }
  }
  if (live) {
    *st = S;
    if (p.gated && c4 == 0) *nt = n;
  }
  if (p.gated && r == 0 && c4 == 0) p.m[unit] = m / LOG2E;
}

// Outputs of a chunk.
template <int DK>
struct ChunkOutCfg {
  static constexpr int kQBytes = CH * DK * 2;
  static constexpr int kKpBytes = CH * (DK > 128 ? DK : 128) * 2;             // K, then the weights P [CH, CH]
  static constexpr int kSBytes = DK * CH_ROWB;                                // one part of the state
  static constexpr int kSvBytes = kSBytes > CH_CHUNK ? kSBytes : CH_CHUNK;    // state (first part), then V
  static constexpr int kSmem = 1024 + kQBytes + kKpBytes + kSvBytes + kSBytes;
  static constexpr int kCols = 256;                                           // scores 128 | P V 64 | Q S 64
};

template <int DK>
__global__ void __launch_bounds__(CHT, DK <= 128 ? 2 : 1) recurrent_chunk_out_kernel(const ChunkParams p, int units) {
  using Cfg = ChunkOutCfg<DK>;
  constexpr int VPT = CH * 8 / CHT;                  // 16-byte pieces of V per thread
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ __align__(16) float gs[CH], bs[CH], fs[CH], row_sum[2][CH], ns[DK];
  __shared__ float m_in;
  __shared__ __align__(8) uint64_t s_done, o_done;
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* q_p = smem_raw + (base - smem_u32(smem_raw));
  uint8_t* k_p = q_p + Cfg::kQBytes;
  uint8_t* sv_p = k_p + Cfg::kKpBytes;
  const uint32_t q_s = base, k_s = q_s + Cfg::kQBytes, sv_s = k_s + Cfg::kKpBytes, sl_s = sv_s + Cfg::kSvBytes;
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(smem_u32(&s_done), 1);
    mbar_init(smem_u32(&o_done), 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_smem), Cfg::kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_smem, t_o = tmem + 128, t_s = tmem + 192;
  pdl_launch_dependents();
  pdl_wait();
  // A unit's operands arrive in two parts, as the shared memory of the unit before becomes free; its vectors and V wait in
  // registers.
  float r_g = 0.f, r_b = 0.f, r_f = 0.f, r_n = 0.f, r_m = 0.f;
  uint4 vr[VPT];
  auto load_state = [&](uint32_t dst, const __nv_bfloat16* part, const ChunkUnit& x) {
    const __nv_bfloat16* src = part + (x.ch * (p.VP / 64) + x.z) * p.KP * 64;
#pragma unroll 4
    for (int i = tid; i < DK * 8; i += CHT) cp_async16(dst + (p.written ? i * 16 : chunk_addr(i >> 3, i & 7)), src + i * 8, true);
  };
  auto fetch_first = [&](const ChunkUnit& x) {       // Q, the state's second part, the vectors, V
    const __nv_bfloat16* rows = p.proj + x.row0 * p.ld;
    chunk_load<DK>(q_s, rows + p.q_col + x.h / p.ratio * p.KP, p.ld, x.n);
    load_state(sl_s, p.s_lo, x);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int e = tid + i * CHT, r = e >> 3;
      vr[i] = make_uint4(0u, 0u, 0u, 0u);
      if (p.written) vr[i] = reinterpret_cast<const uint4*>(p.written)[(x.ch * (p.VP / 64) + x.z) * (8 * CH) + e];
      else if (r < x.n) vr[i] = *reinterpret_cast<const uint4*>(p.v + (x.row0 + r) * p.ld_v + x.h * p.VP + x.z * 64 + (e & 7) * 8);
    }
    if (tid < CH) {
      const float* g = p.gates + x.ch * 3 * CH + tid;
      r_g = g[0];
      r_b = g[CH];
      r_f = g[2 * CH];
    }
    if (p.gated) {
      if (tid < DK) r_n = p.s_n[x.ch * p.KP + tid];
      r_m = p.s_m[x.ch];
    }
  };
  auto fetch_second = [&](const ChunkUnit& x) {      // K, the state's first part
    chunk_load<DK>(k_s, p.proj + x.row0 * p.ld + p.k_col + x.h / p.ratio * p.KP, p.ld, x.n);
    load_state(sv_s, p.s_hi, x);
  };
  ChunkUnit x{};
  if ((int)blockIdx.x < units) {
    x = chunk_unit(p, blockIdx.x);
    fetch_first(x);
    fetch_second(x);
  }
  const int qd = warp & 3, half = warp >> 2;
  const int t = qd * 32 + lane;                      // this thread's token; the two warps of a quarter split the columns
  const uint32_t lane_addr = (uint32_t)(qd * 32) << 16;
  bool ok = true;
  int it = 0;
  for (int u = blockIdx.x; u < units; u += gridDim.x, ++it) {
    const ChunkUnit cur = x;
    if (tid < CH) { gs[tid] = r_g; bs[tid] = r_b; fs[tid] = r_f; }
    if (p.gated && tid < DK) ns[tid] = r_n;
    if (tid == 0) m_in = r_m;
    cp_async_wait_all();
    fence_proxy_async_smem();
    tc_fence_before();
    ok = __syncthreads_and(ok);
    if (!ok) break;
    tc_fence_after();
    if (warp == 0 && elect_one_sync()) {
      constexpr uint32_t idesc_s = make_idesc_bf16(CH, CH, 0, 0), idesc_o = make_idesc_bf16(CH, 64, 0, 1);
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        const uint64_t a = make_smem_desc_sw128(q_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
        const uint64_t b = make_smem_desc_sw128(k_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
        umma_bf16(tmem, a, b, idesc_s, kk ? 1u : 0u);
      }
#pragma unroll
      for (int part = 0; part < 2; ++part)
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t a = make_smem_desc_sw128(q_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
          const uint64_t b = make_smem_desc_sw128((part ? sl_s : sv_s) + kk * 2048, CH_CHUNK, 1024);
          umma_bf16(t_s, a, b, idesc_o, (part | kk) ? 1u : 0u);
        }
      umma_commit(smem_u32(&s_done));
    }
    __syncwarp();
    const bool more = u + (int)gridDim.x < units;
    if (more) x = chunk_unit(p, u + gridDim.x);
    const float B = p.gated ? fmaxf(m_in, bs[t]) : bs[t], F = fs[t];
    float qn = 0.f;
    if (p.gated) {                                   // half of q . n of the incoming state
      constexpr int U = DK / 16;                     // 16-byte units per half
#pragma unroll 4
      for (int w = half * U; w < (half + 1) * U; ++w) {
        const uint4 v = *reinterpret_cast<const uint4*>(q_p + (w >> 3) * CH_CHUNK + chunk_addr(t, w & 7));
        const float4 n0 = *reinterpret_cast<const float4*>(ns + w * 8), n1 = *reinterpret_cast<const float4*>(ns + w * 8 + 4);
        float2 f;
        f = unpack_bf16x2(v.x); qn = fmaf(f.x, n0.x, fmaf(f.y, n0.y, qn));
        f = unpack_bf16x2(v.y); qn = fmaf(f.x, n0.z, fmaf(f.y, n0.w, qn));
        f = unpack_bf16x2(v.z); qn = fmaf(f.x, n1.x, fmaf(f.y, n1.y, qn));
        f = unpack_bf16x2(v.w); qn = fmaf(f.x, n1.z, fmaf(f.y, n1.w, qn));
      }
    }
    const float c_in = chunk_exp2(m_in - B);
    ok = mbar_wait_bounded(smem_u32(&s_done), it & 1, &abort_flag, p.status, ST_TIMEOUT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    float sum = 0.f;
    if (ok) {
      uint8_t* prow = k_p + half * CH_CHUNK;         // K has been read
#pragma unroll
      for (int cc = 0; cc < 2; ++cc) {
        const int j0 = half * 64 + cc * 32;
        float y[32];
        if (j0 <= qd * 32 + 31) {                    // (uniform per warp: a block on the diagonal or below it)
          uint32_t v[32];
          tmem_ld_32x32(tmem + j0 + lane_addr, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const float4 g = *reinterpret_cast<const float4*>(gs + j0 + i);
            y[i] = __uint_as_float(v[i]) * chunk_exp2(g.x - B);
            y[i + 1] = __uint_as_float(v[i + 1]) * chunk_exp2(g.y - B);
            y[i + 2] = __uint_as_float(v[i + 2]) * chunk_exp2(g.z - B);
            y[i + 3] = __uint_as_float(v[i + 3]) * chunk_exp2(g.w - B);
          }
          if (j0 + 31 > qd * 32) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (j0 + i > t) y[i] = 0.f;
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) y[i] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) sum += y[i];
#pragma unroll
        for (int w = 0; w < 4; ++w)
          *reinterpret_cast<uint4*>(prow + chunk_addr(t, cc * 4 + w)) =
              make_uint4(pack_bf16x2(y[w * 8], y[w * 8 + 1]), pack_bf16x2(y[w * 8 + 2], y[w * 8 + 3]), pack_bf16x2(y[w * 8 + 4], y[w * 8 + 5]),
                         pack_bf16x2(y[w * 8 + 6], y[w * 8 + 7]));
      }
      // V over the state's first part, which has been read too
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int e = tid + i * CHT;
        *reinterpret_cast<uint4*>(sv_p + (p.written ? chunk_addr(e % CH, e / CH) : chunk_addr(e >> 3, e & 7))) = vr[i];
      }
    }
    row_sum[half][t] = sum + c_in * qn;
    fence_proxy_async_smem();
    tc_fence_before();
    ok = __syncthreads_and(ok);
    if (!ok) break;
    tc_fence_after();
    if (warp == 0 && elect_one_sync()) {
      constexpr uint32_t idesc_o = make_idesc_bf16(CH, 64, 0, 1);
#pragma unroll
      for (int kk = 0; kk < CH / 16; ++kk) {
        const uint64_t a = make_smem_desc_sw128(k_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
        const uint64_t b = make_smem_desc_sw128(sv_s + kk * 2048, CH_CHUNK, 1024);
        umma_bf16(t_o, a, b, idesc_o, kk ? 1u : 0u);
      }
      umma_commit(smem_u32(&o_done));
    }
    __syncwarp();
    if (more) fetch_first(x);
    float f = p.q_scale;
    if (p.written) f *= F;
    if (p.gated) f /= fmaxf(fabsf((row_sum[0][t] + row_sum[1][t]) * p.q_scale), chunk_exp2(-(F + B))) + 1e-6f;
    ok = mbar_wait_bounded(smem_u32(&o_done), it & 1, &abort_flag, p.status, ST_TIMEOUT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    if (!ok) continue;                               // (the next unit's first barrier ends the loop for all)
    if (more) fetch_second(x);
    uint32_t a[32], b[32];
    tmem_ld_32x32(t_o + half * 32 + lane_addr, a);
    tmem_ld_32x32(t_s + half * 32 + lane_addr, b);
    tmem_ld_wait();
    tc_fence_before();
    if (t < cur.n) {
      float4* dst = reinterpret_cast<float4*>(p.out + (long long)(cur.row0 + t) * p.ldo + cur.h * p.VP + cur.z * 64 + half * 32);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float y[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = f * fmaf(c_in, __uint_as_float(b[4 * i + e]), __uint_as_float(a[4 * i + e]));
        dst[i] = make_float4(y[0], y[1], y[2], y[3]);
      }
    }
  }
  cp_async_wait_all();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kCols);
  }
}

template <int DK>
static int launch_chunks(const ChunkParams& p, int n_chunks, int n_seq, cudaStream_t stream) {
  static int sms[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (sms[dev] == 0) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) return -10;
    if (cudaFuncSetAttribute(recurrent_chunk_state_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkStateCfg<DK>::kSmem) != cudaSuccess ||
        cudaFuncSetAttribute(recurrent_chunk_out_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkOutCfg<DK>::kSmem) != cudaSuccess)
      return -10;
    sms[dev] = n;
  }
  const int units = n_chunks * p.H * (p.VP / 64);
  auto grid = [&](int smem) {                        // two CTAs per SM where they fit (and their TMEM does)
    const int g = sms[dev] * (smem + 5 * 1024 <= 113 * 1024 ? 2 : 1);
    return dim3(units < g ? units : g);
  };
  if (launch_kernel(recurrent_chunk_gates_kernel, dim3(n_chunks, (p.H + 7) / 8), dim3(256), 0, stream, p) != cudaSuccess) return -14;
  if (launch_kernel(recurrent_chunk_state_kernel<DK>, grid(ChunkStateCfg<DK>::kSmem), dim3(CHT), ChunkStateCfg<DK>::kSmem, stream, p, units) != cudaSuccess) return -11;
  if (launch_kernel(recurrent_chunk_chain_kernel, dim3(DK / 32, p.H * (p.VP / SC_COLS), n_seq), dim3(256), 0, stream, p) != cudaSuccess) return -12;
  return launch_kernel(recurrent_chunk_out_kernel<DK>, grid(ChunkOutCfg<DK>::kSmem), dim3(CHT), ChunkOutCfg<DK>::kSmem, stream, p, units) == cudaSuccess ? 0 : -13;
}

// ------------------------------------------------------------------------------------------
// Time mixing in chunks. With A_t the summed log2 decays of a key channel up to and including token t of the chunk (A_-1 = 0), all
// of them <= 0 and falling, and S the state in front of the chunk,
//
//   o_t = (r_t 2^A_(t-1))^T S + sum_{j<t} P_tj v_j + P_tt v_t,   P_tj = sum_c r_t k_j 2^(A_(t-1) - A_j),   P_tt = sum_c r_t u k_t
//   S'  = diag(2^A_last) S + sum_j (k_j 2^(A_last - A_j)) v_j^T
//
// Every exponent above is <= 0, but P does not factor over t and j without one that is not: 2^-A_j overflows. So P is made in
// blocks of 16 x 16 below the diagonal, whose two factors are taken relative to the token in front of the block row, both <= 1
// (mma.sync, their operands are made in registers); of a block on the diagonal the lower left quarter and the lower left quarters
// of the other two go the same way, and the four 4 x 4 triangles pair by pair in fp32. P V and the state's part run on tcgen05. Three launches: what every chunk
// adds to the state (z becomes A on the way), the chain of states, outputs with the head's norm and the output gate.
//
// Forget mixing is the same with keys 1 - f, weights that end at A_t (a token is written before it is read, P_tt = q_t . k_t) and no
// output gate. Its keys are gates, no rounded activations: they, and what is scaled by a power of A, go into every product in two parts.
// ------------------------------------------------------------------------------------------
constexpr float MIX_MOST = 64.f;      // a token that keeps less than 2^-64 keeps nothing; larger sums would cost A its last digits

struct MixParams {
  const __nv_bfloat16* proj;     // [T, ld]: r | k | v | gate
  long long ld;
  int k_col, v_col, g_col;
  float* z;                      // [T, ldz] decay logits, then A
  long long ldz;
  const float* w0;               // [H * KP]
  const float* bonus;            // [H * KP]
  const int4* chunks;
  const int* seq_chunks;
  const int* slots;
  const int* seq_lens;
  const int* cu_q;
  float* s;                      // [slots, H, tiles, KP, 32]
  float* u;                      // [chunks, H, tiles, KP, 32]
  float* last;                   // [chunks, H, KP] A of the chunk's last token
  __nv_bfloat16* s_hi;           // [chunks, H, VP/64, KP, 64]
  __nv_bfloat16* s_lo;
  const float* norm;             // [H * VP]
  float eps;
  __nv_bfloat16* out;            // [T, ldo]
  long long ldo;
  int H, dk, dv, KP, VP, num_slots;
  int* status;
  __nv_bfloat16* keys;           // [T, ld_keys] forget mixing: 1 - f [H * KP], and what bf16 lacks of it [H * KP]
  long long ld_keys;
};

// Two values as two bf16 parts each.
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 b = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - b.x, y - b.y);
}

// Forget gate for the chunked form: {log2 f (at least -MIX_MOST), 1 - f} from z log2(e), with errors of a few fp32 roundings.
// For f near 1: -log1p(-k) = 2 atanh(w) with w = k / (2 - k), and the series of atanh (w <= 1/3).
__device__ __forceinline__ float2 chunk_forget(float z2, float low) {
  const float e = chunk_exp2(-fabsf(z2)), big = __fdividef(1.f, 1.f + e), small = e * big;
  const float k = (1.f - low) * (z2 >= 0.f ? small : big);
  float kept;
  if (k < 0.5f) {
    const float w = __fdividef(k, 2.f - k), x = w * w;
    float s = fmaf(x, 1.f / 13.f, 1.f / 11.f);
    s = fmaf(x, s, 1.f / 9.f);
    s = fmaf(x, s, 1.f / 7.f);
    s = fmaf(x, s, 1.f / 5.f);
    s = fmaf(x, s, 1.f / 3.f);
    kept = -2.f * LOG2E * fmaf(w * x, s, w);
  } else {
    const float f = fmaf(1.f - low, z2 >= 0.f ? big : small, low);
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(kept) : "f"(f));
  }
  return make_float2(fmaxf(kept, -MIX_MOST), k);
}

template <int DK>
struct MixStateCfg {
  static constexpr int kKBytes = CH * DK * 2;
  static constexpr int kSmem = 1024 + 2 * kKBytes + DK / 64 * CH_CHUNK;      // weighted keys in two parts, V
  static constexpr int kCols = DK;
};

// What a chunk of one head adds to the state, and A. VP == KP == DK.
template <int DK, bool FORGET>
__global__ void __launch_bounds__(CHT, DK == 64 ? 2 : 1) time_mix_state_kernel(const MixParams p) {
  using Cfg = MixStateCfg<DK>;
  constexpr int SEGS = 2 * CHT / DK, SEG = CH / SEGS;   // a thread has two channels of SEG tokens
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ __align__(8) float sums[SEGS][DK];
  __shared__ __align__(8) uint64_t done;
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* hi = smem_raw + (base - smem_u32(smem_raw));
  uint8_t* lo = hi + Cfg::kKBytes;
  const uint32_t v_s = base + 2 * Cfg::kKBytes;
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(smem_u32(&done), 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_smem), Cfg::kCols);
    tmem_relinquish();
  }
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x / p.H, h = blockIdx.x % p.H;
  const int4 ck = p.chunks[c];
  const int row0 = ck.x, n = ck.y;
  const long long ch = (long long)c * p.H + h;
  const __nv_bfloat16* rows = p.proj + (long long)row0 * p.ld;
  chunk_load<DK>(v_s, rows + p.v_col + h * p.VP, p.ld, n);
  const int col = 2 * (tid % (DK / 2)), seg = tid / (DK / 2), t0 = seg * SEG;
  float* z = p.z + (long long)(row0 + t0) * p.ldz + h * p.KP + col;
  const __nv_bfloat16* k = rows + (long long)t0 * p.ld + p.k_col + h * p.KP + col;
  // exp(z + w0) log2(e) as one power of two; forget mixing: the bias itself
  const float2 bias = *reinterpret_cast<const float2*>(p.w0 + h * p.KP + col);
  const float w0 = FORGET ? bias.x : fmaf(bias.x, LOG2E, 0.52876637f), w1 = FORGET ? bias.y : fmaf(bias.y, LOG2E, 0.52876637f);
  const float2 low = FORGET ? *reinterpret_cast<const float2*>(p.bonus + h * p.KP + col) : make_float2(0.f, 0.f);
  float2 A[SEG];
  uint32_t keys[FORGET ? 1 : SEG];                      // (fetched before anything is stored: the stores could alias)
  float2 fresh[FORGET ? SEG : 1];                       // forget mixing: 1 - f
  const int mine = min(SEG, n - t0);
#pragma unroll
  for (int i = 0; i < SEG; ++i) A[i] = i < mine ? *reinterpret_cast<const float2*>(z + (long long)i * p.ldz) : make_float2(0.f, 0.f);
  if (!FORGET)
#pragma unroll
  for (int i = 0; i < SEG; ++i) keys[FORGET ? 0 : i] = i < mine ? *reinterpret_cast<const uint32_t*>(k + (long long)i * p.ld) : 0u;
  float2 run = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < SEG; ++i) {
    if (FORGET) {
      const float2 x = chunk_forget((A[i].x + w0) * LOG2E, low.x), y = chunk_forget((A[i].y + w1) * LOG2E, low.y);
      fresh[FORGET ? i : 0] = make_float2(i < mine && col < p.dk ? x.y : 0.f, i < mine && col + 1 < p.dk ? y.y : 0.f);
      if (i < mine) {
        run.x += x.x;
        run.y += y.x;
      }
    } else if (i < mine) {
      run.x -= fminf(chunk_exp2(fmaf(A[i].x, LOG2E, w0)), MIX_MOST);
      run.y -= fminf(chunk_exp2(fmaf(A[i].y, LOG2E, w1)), MIX_MOST);
    }
    A[i] = run;
  }
  sums[seg][col] = run.x;
  sums[seg][col + 1] = run.y;
  __syncthreads();
  float2 before = make_float2(0.f, 0.f), total = before;
#pragma unroll
  for (int i = 0; i < SEGS; ++i) {
    const float2 x = *reinterpret_cast<const float2*>(&sums[i][col]);
    if (i < seg) { before.x += x.x; before.y += x.y; }
    total.x += x.x;
    total.y += x.y;
  }
  if (seg == 0) *reinterpret_cast<float2*>(p.last + ch * p.KP + col) = total;
#pragma unroll
  for (int i = 0; i < SEG; ++i) {
    A[i].x += before.x;
    A[i].y += before.y;
    if (i < mine) *reinterpret_cast<float2*>(z + (long long)i * p.ldz) = A[i];
    float2 f;
    if (FORGET) {
      f = fresh[FORGET ? i : 0];
      if (i < mine) {
        uint32_t* key = reinterpret_cast<uint32_t*>(p.keys + (long long)(row0 + t0 + i) * p.ld_keys + h * p.KP + col);
        uint32_t hi_part, lo_part;
        split_bf16x2(f.x, f.y, hi_part, lo_part);
        key[0] = hi_part;
        key[p.H * p.KP / 2] = lo_part;
      }
    } else {
      f = unpack_bf16x2(keys[FORGET ? 0 : i]);
    }
    const float x = f.x * chunk_exp2(total.x - A[i].x), y = f.y * chunk_exp2(total.y - A[i].y);
    const uint32_t high = pack_bf16x2(x, y);
    const float2 back = unpack_bf16x2(high);
    const uint32_t at = (col >> 6) * CH_CHUNK + chunk_addr(t0 + i, (col & 63) >> 3) + (col & 7) * 2;
    *reinterpret_cast<uint32_t*>(hi + at) = high;
    *reinterpret_cast<uint32_t*>(lo + at) = pack_bf16x2(x - back.x, y - back.y);
  }
  cp_async_wait_all();
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_smem;
  if (warp == 0 && elect_one_sync()) {
    constexpr uint32_t idesc = make_idesc_bf16(DK, 64, 1, 1);
#pragma unroll
    for (int z64 = 0; z64 < DK / 64; ++z64)
#pragma unroll
      for (int part = 0; part < 2; ++part)
#pragma unroll
        for (int kk = 0; kk < CH / 16; ++kk) {
          const uint64_t a = make_smem_desc_sw128(base + part * Cfg::kKBytes + kk * 2048, CH_CHUNK, 1024);
          const uint64_t b = make_smem_desc_sw128(v_s + z64 * CH_CHUNK + kk * 2048, CH_CHUNK, 1024);
          umma_bf16(tmem + z64 * 64, a, b, idesc, (part | kk) ? 1u : 0u);
        }
    umma_commit(smem_u32(&done));
  }
  __syncwarp();
  bool ok = mbar_wait_bounded(smem_u32(&done), 0, &abort_flag, p.status, ST_TIMEOUT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  tc_fence_after();
  if (ok) {
    const int qd = warp & 3, half = warp >> 2;
    const int r = DK == 128 ? qd * 32 + lane : qd * 16 + lane;        // (a 64-row product: row 16 q + lane in 16 lanes)
#pragma unroll
    for (int z64 = 0; z64 < DK / 64; ++z64) {
      uint32_t v[32];
      tmem_ld_32x32(tmem + z64 * 64 + half * 32 + ((uint32_t)(qd * 32) << 16), v);
      tmem_ld_wait();
      if (DK == 128 || lane < 16) {
        float4* dst = reinterpret_cast<float4*>(p.u + ((ch * (p.VP / 32) + z64 * 2 + half) * p.KP + r) * 32);
#pragma unroll
        for (int i = 0; i < 8; ++i)
          dst[i] = make_float4(__uint_as_float(v[4 * i]), __uint_as_float(v[4 * i + 1]), __uint_as_float(v[4 * i + 2]), __uint_as_float(v[4 * i + 3]));
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kCols);
  }
}

// The state in front of every chunk, and behind the portion: as recurrent_chunk_chain_kernel, with a decay per key row.
__global__ void __launch_bounds__(256) time_mix_chain_kernel(const MixParams p) {
  pdl_launch_dependents();
  const int tiles = p.VP / SC_COLS;
  const int tile = blockIdx.y % tiles, h = blockIdx.y / tiles, b = blockIdx.z;
  const int c4 = threadIdx.x & 7, r = blockIdx.x * 32 + (threadIdx.x >> 3);
  pdl_wait();
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) { if (threadIdx.x == 0) set_status(p.status, ST_BAD_INDEX); return; }
  const bool fresh = p.seq_lens[b] == p.cu_q[b + 1] - p.cu_q[b];
  const int c0 = p.seq_chunks[b], c1 = p.seq_chunks[b + 1];
  float4* st = reinterpret_cast<float4*>(p.s + ((((long long)slot * p.H + h) * tiles + tile) * p.KP + r) * SC_COLS) + c4;
  const bool live = r < p.dk;
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!fresh && live) S = *st;
  for (int cb = c0; cb < c1; cb += CHAIN_AHEAD) {
    float4 U[CHAIN_AHEAD];
    float last[CHAIN_AHEAD];
#pragma unroll
    for (int i = 0; i < CHAIN_AHEAD; ++i)
      if (cb + i < c1) {
        const long long ch = (long long)(cb + i) * p.H + h;
        U[i] = *(reinterpret_cast<const float4*>(p.u + ((ch * tiles + tile) * p.KP + r) * SC_COLS) + c4);
        last[i] = p.last[ch * p.KP + r];
      }
#pragma unroll
    for (int i = 0; i < CHAIN_AHEAD; ++i)
      if (cb + i < c1) {
        const long long ch = (long long)(cb + i) * p.H + h;
        const uint32_t h0 = pack_bf16x2(S.x, S.y), h1 = pack_bf16x2(S.z, S.w);
        const float2 b0 = unpack_bf16x2(h0), b1 = unpack_bf16x2(h1);
        const long long at = ((ch * (p.VP / 64) + (tile >> 1)) * p.KP + r) * 64 + (tile & 1) * 32 + c4 * 4;
        *reinterpret_cast<uint2*>(p.s_hi + at) = make_uint2(h0, h1);
        *reinterpret_cast<uint2*>(p.s_lo + at) = make_uint2(pack_bf16x2(S.x - b0.x, S.y - b0.y), pack_bf16x2(S.z - b1.x, S.w - b1.y));
        const float a = chunk_exp2(last[i]);
        S.x = fmaf(a, S.x, U[i].x);
        S.y = fmaf(a, S.y, U[i].y);
        S.z = fmaf(a, S.z, U[i].z);
        S.w = fmaf(a, S.w, U[i].w);
      }
  }
  if (live) *st = S;
}

__device__ __forceinline__ void mma_16816_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int DK, bool FORGET>
struct MixOutCfg {
  static constexpr int kTile = CH * DK * 2;                        // r (then r 2^A), k (then V)
  static constexpr int kA = CH * DK * 4;                           // A, then both parts of the state
  static constexpr int kState = 2 * DK * DK * 2;
  static constexpr int kRest = 2 * kTile + kA + 2 * CH_CHUNK;      // forget mixing: what bf16 lacks of r 2^A, behind the state where it fits
  static constexpr int kRLow = kState + kTile <= kA ? 2 * kTile + kState : kRest;
  static constexpr int kSmem = 1024 + kRest + (FORGET && kRLow == kRest ? kTile : 0);
  static constexpr int kCols = DK;
};

// Outputs of a chunk of one head. VP == KP == DK.
template <int DK, bool FORGET>
__global__ void __launch_bounds__(CHT, DK == 64 ? 2 : 1) time_mix_out_kernel(const MixParams p) {
  using Cfg = MixOutCfg<DK, FORGET>;
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ float row_sum[2][CH];
  __shared__ __align__(8) uint64_t done;
  __shared__ uint32_t tmem_base_smem;
  __shared__ int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* r_p = smem_raw + (base - smem_u32(smem_raw));
  uint8_t* k_p = r_p + Cfg::kTile;
  uint8_t* a_p = k_p + Cfg::kTile;
  uint8_t* w_p = a_p + Cfg::kA;                                    // P [CH, CH]
  const uint32_t r_s = base, k_s = r_s + Cfg::kTile, a_s = k_s + Cfg::kTile, w_s = a_s + Cfg::kA;
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(smem_u32(&done), 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_smem), Cfg::kCols);
    tmem_relinquish();
  }
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x / p.H, h = blockIdx.x % p.H;
  const int4 ck = p.chunks[c];
  const int row0 = ck.x, n = ck.y;
  const long long ch = (long long)c * p.H + h;
  const __nv_bfloat16* rows = p.proj + (long long)row0 * p.ld;
  chunk_load<DK>(r_s, rows + h * p.KP, p.ld, n);
  if (FORGET) chunk_load<DK>(k_s, p.keys + (long long)row0 * p.ld_keys + h * p.KP, p.ld_keys, n);
  else chunk_load<DK>(k_s, rows + p.k_col + h * p.KP, p.ld, n);
  constexpr int BACK = FORGET ? 0 : 1;                             // queries read the state behind their own token, or in front of it
  {
    // A: rows of DK floats, 32-byte pieces exchanged by the row's low bits so that eight rows of a fragment meet no bank twice
    const float* A = p.z + (long long)row0 * p.ldz + h * p.KP;
#pragma unroll 4
    for (int i = tid; i < CH * (DK / 4); i += CHT) {
      const int t = i / (DK / 4), q4 = i % (DK / 4);
      cp_async16(a_s + t * DK * 4 + ((((q4 >> 1) ^ (t & 7)) << 5) | ((q4 & 1) << 4)), A + (long long)(t < n ? t : 0) * p.ldz + q4 * 4, t < n);
    }
  }
  // Addresses: row t of A is at a_p + t * 4 DK, its 32-byte piece u (channels 8u ..) at ((u ^ (t & 7)) << 5); of a tile's chunk of 64
  // channels row t is at + 128 t, its 16-byte piece u at ((u ^ (t & 7)) << 4). (Pieces beyond the eighth only have higher bits more.)
  auto a_row = [&](int t) { return a_p + t * (DK * 4); };
  auto a_piece = [&](int t, int u) { return (u ^ (t & 7)) << 5; };
  auto b_piece = [&](int t, int u) { return (u >> 3) * CH_CHUNK + (((u & 7) ^ (t & 7)) << 4); };
  auto weight_at = [&](int t, int j) { return w_p + (j >> 6) * CH_CHUNK + chunk_addr(t, (j & 63) >> 3) + (j & 7) * 2; };
  const int g = lane >> 2, cq = 2 * (lane & 3), t0 = warp * 16;    // this warp's block row of P
#pragma unroll
  for (int i = 0; i < 8; ++i) {                                    // zero its 16 rows of 256 bytes
    const int e = lane + i * 32, t = t0 + (e >> 4), u = e & 15;
    *reinterpret_cast<uint4*>(w_p + (u >> 3) * CH_CHUNK + chunk_addr(t, u & 7)) = make_uint4(0u, 0u, 0u, 0u);
  }
  cp_async_wait_all();
  __syncthreads();
  auto two_a = [&](int t, int u) {                                 // A of channels 8u + cq, 8u + cq + 1; zero in front of the chunk
    return t < 0 ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(a_row(t) + a_piece(t, u) + cq * 4);
  };
  // r_t 2^(A_(t-1) - A_ref) (forget mixing: A_t) and k_j 2^(A_ref - A_j) of those channels, as bf16 {value, what it lacks (forget mixing)}
  auto parts = [](float x, float y) {
    uint2 v = make_uint2(0u, 0u);
    if (FORGET) split_bf16x2(x, y, v.x, v.y);
    else v.x = pack_bf16x2(x, y);
    return v;
  };
  auto scaled_r = [&](int t, int u, float2 ref) {
    const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r_p + t * CH_ROWB + b_piece(t, u) + cq * 2)), a = two_a(t - BACK, u);
    return parts(x.x * chunk_exp2(a.x - ref.x), x.y * chunk_exp2(a.y - ref.y));
  };
  const __nv_bfloat16* key_rest = FORGET ? p.keys + (long long)row0 * p.ld_keys + (p.H + h) * p.KP : nullptr;      // what bf16 lacks of the keys
  auto rest_row = [&](int j) { return FORGET ? key_rest + (long long)min(j, n - 1) * p.ld_keys : nullptr; };
  auto scaled_k = [&](const uint8_t* k_row, const uint8_t* arow, const __nv_bfloat16* rest, int kb, int ab, int u, float2 ref) {
    float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_row + kb));
    const float2 a = *reinterpret_cast<const float2*>(arow + ab);
    if (FORGET) {
      const float2 y = unpack_bf16x2(__ldg(reinterpret_cast<const uint32_t*>(rest + 8 * u + cq)));
      x.x += y.x;
      x.y += y.y;
    }
    return parts(x.x * chunk_exp2(ref.x - a.x), x.y * chunk_exp2(ref.y - a.y));
  };
  // s += a b^T over 16 channels
  auto product = [&](float (&s)[4], uint2 a0, uint2 a1, uint2 a2, uint2 a3, uint2 b0, uint2 b1) {
    mma_16816_bf16(s, a0.x, a1.x, a2.x, a3.x, b0.x, b1.x);
    if (FORGET) {
      mma_16816_bf16(s, a0.y, a1.y, a2.y, a3.y, b0.x, b1.x);
      mma_16816_bf16(s, a0.x, a1.x, a2.x, a3.x, b0.y, b1.y);
    }
  };
  const uint2 none = make_uint2(0u, 0u);
  auto key_of = [](uint32_t high, uint32_t rest) {
    const float2 x = unpack_bf16x2(high), y = unpack_bf16x2(rest);
    return FORGET ? make_float2(x.x + y.x, x.y + y.y) : x;
  };
  // The blocks left of the diagonal, 8 columns at a time: rows w and 7 - w have 14 such pieces together, half of them for either warp.
  {
    int kb[DK / 8], ab[DK / 8];                                    // pieces of a row j with j % 8 == g
#pragma unroll
    for (int u = 0; u < DK / 8; ++u) { kb[u] = b_piece(g, u); ab[u] = a_piece(g, u); }
    const uint8_t* k0 = k_p + g * CH_ROWB + cq * 2;
    const uint8_t* a0 = a_row(g) + cq * 4;
    auto blocks = [&](int b0, int from, int to) {                  // block row at token b0, columns 8 from .. 8 to
      if (b0 >= n || from >= to) return;
      uint2 fa[DK / 16][4];
      float2 ref[DK / 8];
#pragma unroll
      for (int u = 0; u < DK / 8; ++u) {
        ref[u] = two_a(b0 - 1, u);
        fa[u / 2][(u & 1) * 2] = scaled_r(b0 + g, u, ref[u]);
        fa[u / 2][(u & 1) * 2 + 1] = scaled_r(b0 + g + 8, u, ref[u]);
      }
      for (int j0 = from * 8; j0 < to * 8; j0 += 8) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        const uint8_t* kr = k0 + j0 * CH_ROWB;
        const uint8_t* ar = a0 + j0 * (DK * 4);
        const __nv_bfloat16* rest = rest_row(j0 + g);
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks)
          product(s, fa[ks][0], fa[ks][1], fa[ks][2], fa[ks][3], scaled_k(kr, ar, rest, kb[2 * ks], ab[2 * ks], 2 * ks, ref[2 * ks]),
                  scaled_k(kr, ar, rest, kb[2 * ks + 1], ab[2 * ks + 1], 2 * ks + 1, ref[2 * ks + 1]));
        *reinterpret_cast<uint32_t*>(weight_at(b0 + g, j0 + cq)) = pack_bf16x2(s[0], s[1]);
        *reinterpret_cast<uint32_t*>(weight_at(b0 + g + 8, j0 + cq)) = pack_bf16x2(s[2], s[3]);
      }
    };
#pragma unroll 1
    for (int part = 0; part < 2; ++part) {
      const int low = min(warp, 7 - warp), row = part == 0 ? 7 - low : low;        // the longer row of the pair first
      if (part == 0) blocks(row * 16, warp == low ? 0 : 7 - 2 * low, warp == low ? 7 - 2 * low : 2 * row);
      else if (warp == low) blocks(row * 16, 0, 2 * row);
    }
  }
  if (t0 < n) {
    {                                                              // lower left quarter of the diagonal block
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      const uint8_t* kr = k_p + (t0 + g) * CH_ROWB + cq * 2;
      const uint8_t* ar = a_row(t0 + g) + cq * 4;
      const __nv_bfloat16* rest = rest_row(t0 + g);
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        const float2 ref0 = two_a(t0 + 7, 2 * ks), ref1 = two_a(t0 + 7, 2 * ks + 1);
        product(s, scaled_r(t0 + 8 + g, 2 * ks, ref0), none, scaled_r(t0 + 8 + g, 2 * ks + 1, ref1), none,
                scaled_k(kr, ar, rest, b_piece(g, 2 * ks), a_piece(g, 2 * ks), 2 * ks, ref0),
                scaled_k(kr, ar, rest, b_piece(g, 2 * ks + 1), a_piece(g, 2 * ks + 1), 2 * ks + 1, ref1));
      }
      *reinterpret_cast<uint32_t*>(weight_at(t0 + 8 + g, t0 + cq)) = pack_bf16x2(s[0], s[1]);
    }
    {                                                              // lower left quarters of the diagonal's two 8 x 8 blocks, in one product
      const int up = g < 4 ? 0 : 4, t = t0 + 4 + g + up, j = t0 + g + up, ref_row = t0 + 3 + 2 * up;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        const float2 ref0 = two_a(ref_row, 2 * ks), ref1 = two_a(ref_row, 2 * ks + 1);
        const uint8_t* kr = k_p + j * CH_ROWB + cq * 2;
        const uint8_t* ar = a_row(j) + cq * 4;
        const __nv_bfloat16* rest = rest_row(j);
        product(s, scaled_r(t, 2 * ks, ref0), none, scaled_r(t, 2 * ks + 1, ref1), none,
                scaled_k(kr, ar, rest, b_piece(j, 2 * ks), a_piece(j, 2 * ks), 2 * ks, ref0),
                scaled_k(kr, ar, rest, b_piece(j, 2 * ks + 1), a_piece(j, 2 * ks + 1), 2 * ks + 1, ref1));
      }
      if ((g >> 2) == (cq >> 2)) *reinterpret_cast<uint32_t*>(weight_at(t, t0 + cq + (cq < 4 ? 0 : 4))) = pack_bf16x2(s[0], s[1]);
    }
    if (lane < 24) {                                               // pairs j < t of the four 4 x 4 triangles, one per lane
      const int q = lane % 6, t = q < 1 ? 1 : q < 3 ? 2 : 3, j = q - t * (t - 1) / 2;
      const int tt = t0 + lane / 6 * 4 + t, jj = t0 + lane / 6 * 4 + j;
      const uint8_t* rr = r_p + tt * CH_ROWB;
      const uint8_t* kr = k_p + jj * CH_ROWB;
      const uint8_t* at = a_row(tt - BACK);
      const uint8_t* aj = a_row(jj);
      float s0 = 0.f, s1 = 0.f;
#pragma unroll 2
      for (int i = 0; i < DK / 8; ++i) {                           // eight channels at a time, every lane from a place of its own
        const int u = (i + lane) & (DK / 8 - 1);
        const uint4 x = *reinterpret_cast<const uint4*>(rr + b_piece(tt, u)), y = *reinterpret_cast<const uint4*>(kr + b_piece(jj, u));
        const float4* pa = reinterpret_cast<const float4*>(at + a_piece(tt - BACK, u));
        const float4* pb = reinterpret_cast<const float4*>(aj + a_piece(jj, u));
        const float4 a = pa[0], b = pb[0], c4 = pa[1], d4 = pb[1];
        const uint4 z = FORGET ? __ldg(reinterpret_cast<const uint4*>(rest_row(jj) + 8 * u)) : make_uint4(0u, 0u, 0u, 0u);
        float2 f, h2;
        f = unpack_bf16x2(x.x); h2 = key_of(y.x, z.x);
        s0 = fmaf(f.x * h2.x, chunk_exp2(a.x - b.x), s0);
        s1 = fmaf(f.y * h2.y, chunk_exp2(a.y - b.y), s1);
        f = unpack_bf16x2(x.y); h2 = key_of(y.y, z.y);
        s0 = fmaf(f.x * h2.x, chunk_exp2(a.z - b.z), s0);
        s1 = fmaf(f.y * h2.y, chunk_exp2(a.w - b.w), s1);
        f = unpack_bf16x2(x.z); h2 = key_of(y.z, z.z);
        s0 = fmaf(f.x * h2.x, chunk_exp2(c4.x - d4.x), s0);
        s1 = fmaf(f.y * h2.y, chunk_exp2(c4.y - d4.y), s1);
        f = unpack_bf16x2(x.w); h2 = key_of(y.w, z.w);
        s0 = fmaf(f.x * h2.x, chunk_exp2(c4.z - d4.z), s0);
        s1 = fmaf(f.y * h2.y, chunk_exp2(c4.w - d4.w), s1);
      }
      *reinterpret_cast<__nv_bfloat16*>(weight_at(tt, jj)) = __float2bfloat16_rn(s0 + s1);
    }
    {                                                              // the diagonal: two lanes per token
      const int t = t0 + (lane & 15);
      const float* bonus = p.bonus + h * p.KP;
      float s = 0.f;
#pragma unroll 2
      for (int i = 0; i < DK / 16; ++i) {
        const int u = (lane >> 4) * (DK / 16) + i;
        const uint4 x = *reinterpret_cast<const uint4*>(r_p + t * CH_ROWB + b_piece(t, u)), y = *reinterpret_cast<const uint4*>(k_p + t * CH_ROWB + b_piece(t, u));
        float4 b0 = make_float4(1.f, 1.f, 1.f, 1.f), b1 = b0;
        if (!FORGET) {
          b0 = *reinterpret_cast<const float4*>(bonus + u * 8);
          b1 = *reinterpret_cast<const float4*>(bonus + u * 8 + 4);
        }
        const uint4 z = FORGET ? __ldg(reinterpret_cast<const uint4*>(rest_row(t) + 8 * u)) : make_uint4(0u, 0u, 0u, 0u);
        float2 f, h2;
        f = unpack_bf16x2(x.x); h2 = key_of(y.x, z.x); s = fmaf(f.x * h2.x, b0.x, fmaf(f.y * h2.y, b0.y, s));
        f = unpack_bf16x2(x.y); h2 = key_of(y.y, z.y); s = fmaf(f.x * h2.x, b0.z, fmaf(f.y * h2.y, b0.w, s));
        f = unpack_bf16x2(x.z); h2 = key_of(y.z, z.z); s = fmaf(f.x * h2.x, b1.x, fmaf(f.y * h2.y, b1.y, s));
        f = unpack_bf16x2(x.w); h2 = key_of(y.w, z.w); s = fmaf(f.x * h2.x, b1.z, fmaf(f.y * h2.y, b1.w, s));
      }
      s += __shfl_xor_sync(0xffffffffu, s, 16);
      if (lane < 16) *reinterpret_cast<__nv_bfloat16*>(weight_at(t, t)) = __float2bfloat16_rn(s);
    }
  }
  __syncthreads();                                                 // k has been read
  chunk_load<DK>(k_s, rows + p.v_col + h * p.VP, p.ld, n);
  constexpr int PIECES = CH * (DK / 8) / CHT;
  uint4 rest_r[FORGET ? PIECES : 1];                               // forget mixing: what bf16 lacks of r 2^A
#pragma unroll
  for (int k = 0; k < PIECES; ++k) {                               // r 2^A_(t-1) (forget mixing: A_t), in place
    const int i = tid + k * CHT, t = i / (DK / 8), u = i % (DK / 8);
    if (t < BACK) continue;
    uint4* at = reinterpret_cast<uint4*>(r_p + t * CH_ROWB + b_piece(t, u));
    const float4* pa = reinterpret_cast<const float4*>(a_row(t - BACK) + a_piece(t - BACK, u));
    const float4 a = pa[0], b = pa[1];
    uint4 v = *at;
    auto one = [&](uint32_t x, float ax, float ay) {
      const float2 f = unpack_bf16x2(x);
      return parts(f.x * chunk_exp2(ax), f.y * chunk_exp2(ay));
    };
    const uint2 x = one(v.x, a.x, a.y), y = one(v.y, a.z, a.w), z = one(v.z, b.x, b.y), w = one(v.w, b.z, b.w);
    *at = make_uint4(x.x, y.x, z.x, w.x);
    if (FORGET) rest_r[FORGET ? k : 0] = make_uint4(x.y, y.y, z.y, w.y);
  }
  __syncthreads();                                                 // A has been read
  if (FORGET)
#pragma unroll
    for (int k = 0; k < PIECES; ++k) {
      const int i = tid + k * CHT, t = i / (DK / 8), u = i % (DK / 8);
      *reinterpret_cast<uint4*>(r_p + Cfg::kRLow + t * CH_ROWB + b_piece(t, u)) = rest_r[FORGET ? k : 0];
    }
  constexpr int PART = DK * DK * 2;                                // one part of the state
#pragma unroll 4
  for (int i = tid; i < 2 * (DK / 64) * DK * 8; i += CHT) {        // parts, 64 value channels, key row, 16-byte piece
    const int part = i / ((DK / 64) * DK * 8), e = i % ((DK / 64) * DK * 8), z64 = e / (DK * 8), r = (e >> 3) % DK, u = e & 7;
    const __nv_bfloat16* src = (part ? p.s_lo : p.s_hi) + ((ch * (DK / 64) + z64) * DK + r) * 64 + u * 8;
    cp_async16(a_s + part * PART + z64 * DK * CH_ROWB + chunk_addr(r, u), src, true);
  }
  cp_async_wait_all();
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_smem;
  if (warp == 0 && elect_one_sync()) {
    constexpr uint32_t idesc = make_idesc_bf16(CH, 64, 0, 1);
#pragma unroll
    for (int z64 = 0; z64 < DK / 64; ++z64) {
#pragma unroll
      for (int kk = 0; kk < CH / 16; ++kk) {
        const uint64_t a = make_smem_desc_sw128(w_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
        const uint64_t b = make_smem_desc_sw128(k_s + z64 * CH_CHUNK + kk * 2048, CH_CHUNK, 1024);
        umma_bf16(tmem + z64 * 64, a, b, idesc, kk ? 1u : 0u);
      }
#pragma unroll
      for (int part = 0; part < 2; ++part)
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t a = make_smem_desc_sw128(r_s + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
          const uint64_t b = make_smem_desc_sw128(a_s + part * PART + z64 * DK * CH_ROWB + kk * 2048, CH_CHUNK, 1024);
          umma_bf16(tmem + z64 * 64, a, b, idesc, 1u);
        }
      if (FORGET)
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t a = make_smem_desc_sw128(r_s + Cfg::kRLow + (kk >> 2) * CH_CHUNK + (kk & 3) * 32, 16, 1024);
          const uint64_t b = make_smem_desc_sw128(a_s + z64 * DK * CH_ROWB + kk * 2048, CH_CHUNK, 1024);
          umma_bf16(tmem + z64 * 64, a, b, idesc, 1u);
        }
    }
    umma_commit(smem_u32(&done));
  }
  __syncwarp();
  const int qd = warp & 3, half = warp >> 2, t = qd * 32 + lane;   // this thread's token; half the channels
  constexpr int HC = DK / 2;
  uint4 gate[HC / 8];
#pragma unroll
  for (int i = 0; i < HC / 8; ++i) {
    gate[i] = make_uint4(0u, 0u, 0u, 0u);
    if (!FORGET && t < n) gate[i] = *reinterpret_cast<const uint4*>(rows + (long long)t * p.ld + p.g_col + h * p.VP + half * HC + i * 8);
  }
  bool ok = mbar_wait_bounded(smem_u32(&done), 0, &abort_flag, p.status, ST_TIMEOUT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  tc_fence_after();
  uint32_t v[HC];
  float ss = 0.f;
  if (ok) {
#pragma unroll
    for (int i = 0; i < HC / 32; ++i) tmem_ld_32x32(tmem + half * HC + i * 32 + ((uint32_t)(qd * 32) << 16), *reinterpret_cast<uint32_t(*)[32]>(&v[i * 32]));
    tmem_ld_wait();
    tc_fence_before();
#pragma unroll
    for (int i = 0; i < HC; ++i) ss = fmaf(__uint_as_float(v[i]), __uint_as_float(v[i]), ss);
    row_sum[half][t] = ss;
  }
  __syncthreads();
  if (ok && t < n) {
    const float rs = 1.f / sqrtf((row_sum[0][t] + row_sum[1][t]) / (float)p.dv + p.eps);
    const float* w = p.norm + h * p.VP + half * HC;
    __nv_bfloat16* dst = p.out + (long long)(row0 + t) * p.ldo + h * p.VP + half * HC;
#pragma unroll
    for (int i = 0; i < HC / 8; ++i) {
      const float4 w0 = *reinterpret_cast<const float4*>(w + i * 8), w1 = *reinterpret_cast<const float4*>(w + i * 8 + 4);
      auto two = [&](int e, float wx, float wy, uint32_t gz) {
        const float2 z = unpack_bf16x2(gz);
        const float gx = FORGET ? 1.f : silu_fast(z.x), gy = FORGET ? 1.f : silu_fast(z.y);
        return pack_bf16x2(__uint_as_float(v[i * 8 + e]) * rs * wx * gx, __uint_as_float(v[i * 8 + e + 1]) * rs * wy * gy);
      };
      *reinterpret_cast<uint4*>(dst + i * 8) = make_uint4(two(0, w0.x, w0.y, gate[i].x), two(2, w0.z, w0.w, gate[i].y), two(4, w1.x, w1.y, gate[i].z),
                                                          two(6, w1.z, w1.w, gate[i].w));
    }
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kCols);
  }
}

template <int DK, bool FORGET>
static int launch_time_mix(const MixParams& p, int n_chunks, int n_seq, cudaStream_t stream) {
  static bool attr[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (!attr[dev]) {
    if (cudaFuncSetAttribute(time_mix_state_kernel<DK, FORGET>, cudaFuncAttributeMaxDynamicSharedMemorySize, MixStateCfg<DK>::kSmem) != cudaSuccess ||
        cudaFuncSetAttribute(time_mix_out_kernel<DK, FORGET>, cudaFuncAttributeMaxDynamicSharedMemorySize, MixOutCfg<DK, FORGET>::kSmem) != cudaSuccess)
      return -10;
    attr[dev] = true;
  }
  const dim3 units(n_chunks * p.H);
  if (launch_kernel(time_mix_state_kernel<DK, FORGET>, units, dim3(CHT), MixStateCfg<DK>::kSmem, stream, p) != cudaSuccess) return -11;
  if (launch_kernel(time_mix_chain_kernel, dim3(DK / 32, p.H * (p.VP / SC_COLS), n_seq), dim3(256), 0, stream, p) != cudaSuccess) return -12;
  return launch_kernel(time_mix_out_kernel<DK, FORGET>, units, dim3(CHT), MixOutCfg<DK, FORGET>::kSmem, stream, p) == cudaSuccess ? 0 : -13;
}

}  // namespace rb

#include "delta_rule.cuh"

namespace rb {

// ------------------------------------------------------------------------------------------
// Time or forget mixing, one token per sequence, heads of up to 64 channels (KP = VP = 64): a unit is a whole head of a sequence, so that its
// norm and the output gate are finished here too. As recurrent_decode_kernel: persistent CTAs, a ring of bulk copies in both
// directions, the unit's vectors fetched one unit ahead. Threads: 16 groups of 4 value channels x 8 of key rows.
// ------------------------------------------------------------------------------------------
constexpr int MD_THREADS = 128, MD_STAGES = 4, MD_DIM = 64;
constexpr int MD_BYTES = MD_DIM * MD_DIM * 4;

struct MixDecodeParams {
  const void* proj;              // [B, ld]: r | k | v | gate
  long long ld;
  int k_col, v_col, g_col;
  const float* z;                // [B, ldz]
  long long ldz;
  const float* w0;               // [H * 64]
  const float* bonus;
  const float* norm;
  float eps;
  float* s;                      // [slots, H, 2, 64, 32]
  const int* slots;
  const int* seq_lens;
  void* out;                     // [B, ldo]
  long long ldo;
  int H, dk, dv, num_slots;
  int* status;
};

template <typename T, bool FORGET>
__global__ void __launch_bounds__(MD_THREADS) time_mix_decode_kernel(const MixDecodeParams p, int units) {
  extern __shared__ __align__(128) uint8_t smem_raw[];       // MD_STAGES x [2, 64, 32] fp32
  __shared__ __align__(16) float4 rows_s[MD_DIM];            // r, k, decay, bonus of a key row
  __shared__ __align__(16) float vs[MD_DIM];
  __shared__ __align__(16) float red[MD_THREADS / 32][MD_DIM];
  __shared__ __align__(8) uint64_t full[MD_STAGES];
  __shared__ int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c4 = tid & 15, r0 = tid >> 4;
  const uint32_t ring = smem_u32(smem_raw);
  if (tid == 0) {
    abort_flag = 0;
    for (int i = 0; i < MD_STAGES; ++i) mbar_init(smem_u32(&full[i]), 1);
    fence_mbar_init();
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  struct Unit { int b, h, slot; bool fresh; };
  auto unit_of = [&](int u) {
    Unit x;
    x.b = u / p.H;
    x.h = u - x.b * p.H;
    x.slot = __ldg(p.slots + x.b);
    if (x.slot >= p.num_slots) { set_status(p.status, ST_BAD_INDEX); x.slot = -1; }
    x.fresh = __ldg(p.seq_lens + x.b) == 1;
    return x;
  };
  auto state_of = [&](const Unit& x) { return p.s + ((long long)max(x.slot, 0) * p.H + x.h) * (MD_DIM * MD_DIM); };   // padding rows read slot 0
  constexpr int MOVER = MD_THREADS - 32;                     // the thread that issues the copies (the first warp finishes the outputs)
  int issued = 0;
  auto load = [&](int i) {                                   // MOVER: state of this CTA's i-th unit
    const int u = blockIdx.x + i * gridDim.x;
    if (u >= units) return;
    const uint32_t bar = smem_u32(&full[i % MD_STAGES]);
    mbar_expect_tx(bar, MD_BYTES);
    bulk_load(ring + (i % MD_STAGES) * MD_BYTES, state_of(unit_of(u)), MD_BYTES, bar);
    issued = i + 1;
  };
  if (tid == MOVER)
    for (int i = 0; i < MD_STAGES - 1; ++i) load(i);
  float4 mine = make_float4(0.f, 0.f, 0.f, 0.f);             // threads below 64: the row's vectors; the others: v in .x
  float2 gate = make_float2(0.f, 0.f), weight = make_float2(0.f, 0.f);     // first warp: two channels of the outputs
  Unit x{};
  auto fetch = [&](int u) {
    x = unit_of(u);
    const T* row = reinterpret_cast<const T*>(p.proj) + x.b * p.ld + x.h * MD_DIM;
    const int c = x.h * MD_DIM;
    if (tid < MD_DIM) {
      mine = make_float4(to_f<T>(row[tid]), FORGET ? 0.f : to_f<T>(row[p.k_col + tid]), p.z[x.b * p.ldz + c + tid] + p.w0[c + tid], p.bonus[c + tid]);
    } else {
      mine.x = to_f<T>(row[p.v_col + tid - MD_DIM]);
    }
    if (warp == 0) {
      if (!FORGET) gate = make_float2(to_f<T>(row[p.g_col + 2 * lane]), to_f<T>(row[p.g_col + 2 * lane + 1]));
      weight = *reinterpret_cast<const float2*>(p.norm + c + 2 * lane);
    }
  };
  if ((int)blockIdx.x < units) fetch(blockIdx.x);
  bool ok = true;
  int it = 0;
  for (int u = blockIdx.x; u < units; u += gridDim.x, ++it) {
    const Unit cur = x;
    const float2 g = gate, w = weight;
    if (tid < MD_DIM) {
      if (FORGET) {
        const float2 f = forget_gate(mine.z, mine.w);
        rows_s[tid] = tid < p.dk ? make_float4(mine.x, f.y, f.x, 0.f) : make_float4(0.f, 0.f, 0.f, 0.f);
      } else {
        rows_s[tid] = make_float4(mine.x, mine.y, channel_decay(mine.z), mine.w);
      }
    } else vs[tid - MD_DIM] = mine.x;
    const int stage = it % MD_STAGES;
    ok = mbar_wait_bounded(smem_u32(&full[stage]), (uint32_t)((it / MD_STAGES) & 1), &abort_flag, p.status, ST_TIMEOUT_SMEM_FULL);
    ok = __syncthreads_and(ok);
    if (!ok) break;
    if (u + (int)gridDim.x < units) fetch(u + gridDim.x);
    float4* S = reinterpret_cast<float4*>(smem_raw + stage * MD_BYTES) + (c4 >> 3) * (MD_DIM * 8) + (c4 & 7);     // row r at S[8 r]
    const float4 v = *reinterpret_cast<const float4*>(&vs[c4 * 4]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < MD_DIM / 8; ++i) {
      const int r = r0 + i * 8;
      float4 s = cur.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : S[r * 8];
      const float4 q = rows_s[r];
      const float4 kv = make_float4(q.y * v.x, q.y * v.y, q.y * v.z, q.y * v.w);
      if (!FORGET) {
        acc.x = fmaf(q.x, fmaf(q.w, kv.x, s.x), acc.x);
        acc.y = fmaf(q.x, fmaf(q.w, kv.y, s.y), acc.y);
        acc.z = fmaf(q.x, fmaf(q.w, kv.z, s.z), acc.z);
        acc.w = fmaf(q.x, fmaf(q.w, kv.w, s.w), acc.w);
      }
      s.x = fmaf(q.z, s.x, kv.x);
      s.y = fmaf(q.z, s.y, kv.y);
      s.z = fmaf(q.z, s.z, kv.z);
      s.w = fmaf(q.z, s.w, kv.w);
      if (FORGET) {
        acc.x = fmaf(q.x, s.x, acc.x);
        acc.y = fmaf(q.x, s.y, acc.y);
        acc.z = fmaf(q.x, s.z, acc.z);
        acc.w = fmaf(q.x, s.w, acc.w);
      }
      S[r * 8] = s;
    }
    fence_proxy_async_smem();
    acc.x += __shfl_xor_sync(0xffffffffu, acc.x, 16);
    acc.y += __shfl_xor_sync(0xffffffffu, acc.y, 16);
    acc.z += __shfl_xor_sync(0xffffffffu, acc.z, 16);
    acc.w += __shfl_xor_sync(0xffffffffu, acc.w, 16);
    if (lane < 16) *reinterpret_cast<float4*>(&red[warp][c4 * 4]) = acc;
    __syncthreads();
    if (tid == MOVER) {
      if (cur.slot >= 0) bulk_store(state_of(cur), ring + stage * MD_BYTES, MD_BYTES);
      else asm volatile("cp.async.bulk.commit_group;" ::: "memory");
      asm volatile("cp.async.bulk.wait_group.read 1;" ::: "memory");     // the state stored one unit ago has left its stage
      load(it + MD_STAGES - 1);
    }
    if (warp == 0) {
      float2 o = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < MD_THREADS / 32; ++i) {
        const float2 part = *reinterpret_cast<const float2*>(&red[i][2 * lane]);
        o.x += part.x;
        o.y += part.y;
      }
      const float rs = cur.slot < 0 ? 0.f : 1.f / sqrtf(warp_sum(o.x * o.x + o.y * o.y) / (float)p.dv + p.eps);
      const float y0 = o.x * rs * w.x * (FORGET ? 1.f : g.x * sigmoid_f(g.x)), y1 = o.y * rs * w.y * (FORGET ? 1.f : g.y * sigmoid_f(g.y));
      T* dst = reinterpret_cast<T*>(p.out) + cur.b * p.ldo + cur.h * MD_DIM + 2 * lane;
      if constexpr (sizeof(T) == 4) *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
      else *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(y0, y1);
    }
  }
  if (tid == MOVER) {
    if (!ok)                                                 // no copy may land after the CTA has gone
      for (int i = it; i < issued; ++i) {
        const uint64_t t0 = globaltimer_ns();
        while (!mbar_try_wait(smem_u32(&full[i % MD_STAGES]), (uint32_t)((i / MD_STAGES) & 1)))
          if (globaltimer_ns() - t0 > 50000000ull) break;
      }
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  }
}

template <typename T, bool FORGET>
static int launch_time_mix_decode(const MixDecodeParams& p, int B, cudaStream_t stream) {
  static int sms[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -10;
  if (sms[dev] == 0) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess ||
        cudaFuncSetAttribute(time_mix_decode_kernel<T, FORGET>, cudaFuncAttributeMaxDynamicSharedMemorySize, MD_STAGES * MD_BYTES) != cudaSuccess)
      return -10;
    sms[dev] = n;
  }
  const int units = B * p.H, grid = units < sms[dev] * 3 ? units : sms[dev] * 3;
  return launch_kernel(time_mix_decode_kernel<T, FORGET>, dim3(grid), dim3(MD_THREADS), MD_STAGES * MD_BYTES, stream, p, units) == cudaSuccess ? 0 : -11;
}

// ------------------------------------------------------------------------------------------
// out = o / rms * weight * sigmoid(gate), or silu(gate), or without a gate (null). One CTA per token; a warp takes whole heads. Padding channels of o are zero.
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, long long ldo, const float* __restrict__ weight,
                                                         const T* __restrict__ gate, long long ldg, T* __restrict__ out, long long ldy,
                                                         int H, int dv, int VP, int per_head, int silu, float eps) {
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
      auto gated = [&](int e) {
        if (gate == nullptr) return 1.f;
        const float z = to_f<T>(g[e]);
        return silu ? z * sigmoid_f(z) : sigmoid_f(z);
      };
      const float y0 = v.x * rs * w.x * gated(0), y1 = v.y * rs * w.y * gated(1);
      const float y2 = v.z * rs * w.z * gated(2), y3 = v.w * rs * w.w * gated(3);
      if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(out + t * ldy + c) = make_float4(y0, y1, y2, y3);
      else *reinterpret_cast<uint2*>(out + t * ldy + c) = make_uint2(pack_bf16x2(y0, y1), pack_bf16x2(y2, y3));
    }
  }
}

// mix[s][t] = h_t + (h_(t-1) - h_t) mu[s] for the `mixes` projections of a token; 8 channels per thread. With one row per sequence
// (rows.cu_q null) the history moves on in the same pass.
template <typename T>
__global__ void __launch_bounds__(256) token_shift_kernel(const T* __restrict__ h, long long ld, const float* __restrict__ mu, int mixes, T* __restrict__ out,
                                                          long long step, long long ldo, T* __restrict__ hist, const History rows, int width, int n,
                                                          int* status) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int V = 16 / sizeof(T);
  union Vec { uint4 u[8 / V]; T e[8]; };
  const int per = width / 8;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < (long long)n * per; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / per), c = (int)(i % per) * 8;
    const RowPlace place = row_place(rows, t, status);
    const T* back = row_before(place, 1, h, ld, t, (const T*)hist, 1, width);
    Vec x, y;
#pragma unroll
    for (int j = 0; j < 8 / V; ++j) {
      x.u[j] = reinterpret_cast<const uint4*>(h + t * ld + c)[j];
      y.u[j] = back != nullptr ? reinterpret_cast<const uint4*>(back + c)[j] : make_uint4(0u, 0u, 0u, 0u);
    }
    if (rows.cu_q == nullptr && place.slot >= 0)
#pragma unroll
      for (int j = 0; j < 8 / V; ++j) reinterpret_cast<uint4*>(hist + (long long)place.slot * width + c)[j] = x.u[j];
    float a[8], d[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) { a[j] = to_f<T>(x.e[j]); d[j] = to_f<T>(y.e[j]) - a[j]; }
    for (int s = 0; s < mixes; ++s) {
      const float4* m4 = reinterpret_cast<const float4*>(mu + (long long)s * width + c);
      const float4 m0 = m4[0], m1 = m4[1];
      const float m[8] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
      Vec r;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float v = fmaf(d[j], m[j], a[j]);
        if constexpr (sizeof(T) == 4) r.e[j] = v; else r.e[j] = __float2bfloat16_rn(v);
      }
#pragma unroll
      for (int j = 0; j < 8 / V; ++j) reinterpret_cast<uint4*>(out + s * step + t * ldo + c)[j] = r.u[j];
    }
  }
}

// tanh of fp32 rows as operand of a product that is to lose nothing: fp32 as it is, bf16 as two parts side by side.
__global__ void tanh_parts_kernel(const float* __restrict__ x, int n, __nv_bfloat16* __restrict__ parts, float* __restrict__ whole, long long total) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const float v = tanhf(x[i]);
    if (whole != nullptr) {
      whole[i] = v;
    } else {
      const long long r = i / n;
      const int c = (int)(i - r * n);
      const __nv_bfloat16 hi = __float2bfloat16_rn(v);
      parts[r * 2 * n + c] = hi;
      parts[r * 2 * n + n + c] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
  }
}

}  // namespace rb

using namespace rb;

extern "C" {

// h [n, ld] -> out [mixes][n rows of ldo, `step` apart]; hist [num_slots, width]. cu_q null: one row per sequence.
int rb_token_shift(const void* h, long long ld, const float* mu, int mixes, void* out, long long step, long long ldo, void* hist, const int* cu_q,
                   const int* positions, const int* slots, int B, int num_slots, int width, int n, int dtype, int* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width % 8 != 0 || ld % 8 != 0 || ldo % 8 != 0 || step % 8 != 0 || mixes <= 0 || B <= 0) return -1;
  const History rows{cu_q, positions, slots, B, 1, num_slots};
  long long grid = ((long long)n * (width / 8) + 255) / 256;
  if (grid > 148 * 16) grid = 148 * 16;
  cudaError_t e;
  if (dtype == 0) {
    e = launch_kernel(token_shift_kernel<__nv_bfloat16>, dim3((unsigned)grid), dim3(256), 0, stream, (const __nv_bfloat16*)h, ld, mu, mixes,
                      (__nv_bfloat16*)out, step, ldo, (__nv_bfloat16*)hist, rows, width, n, status);
    if (e == cudaSuccess && cu_q != nullptr) e = launch_history_update((const __nv_bfloat16*)h, ld, rows, (__nv_bfloat16*)hist, width, stream);
  } else {
    e = launch_kernel(token_shift_kernel<float>, dim3((unsigned)grid), dim3(256), 0, stream, (const float*)h, ld, mu, mixes, (float*)out, step, ldo,
                      (float*)hist, rows, width, n, status);
    if (e == cudaSuccess && cu_q != nullptr) e = launch_history_update((const float*)h, ld, rows, (float*)hist, width, stream);
  }
  return e == cudaSuccess ? 0 : -11;
}

// x [rows, n] fp32 -> tanh as fp32 [rows, n] (whole) or as bf16 [rows, 2n] (high parts, then what they lack).
int rb_tanh_parts(const float* x, int n, void* parts, float* whole, int rows, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (n <= 0 || (parts == nullptr) == (whole == nullptr)) return -1;
  const long long total = (long long)rows * n;
  long long grid = (total + 255) / 256;
  if (grid > 148 * 8) grid = 148 * 8;
  return launch_kernel(tanh_parts_kernel, dim3((unsigned)grid), dim3(256), 0, stream, x, n, (__nv_bfloat16*)parts, whole, total) == cudaSuccess ? 0 : -11;
}

void rb_recurrent_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

int rb_recurrent_scan(const void* proj, long long ld, int q_col, int k_col, int v_col, const float* small, long long ld_small, const float* decay,
                      const float* bias_i, const float* bias_f, float cap, float q_scale, float* s, float* n, float* m, const int* slots,
                      const int* cu_q, const int* seq_lens, float* out, long long ldo, int H, int dk, int KP, int VP, int B, int num_slots,
                      int gated, int rows, const float* z, long long ldz, const float* w0, const float* bonus, int form, int ratio,
                      const float* units, const float* steps, int dtype, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || H > 65535 || B > 65535 || dk <= 0 || dk > KP || VP % SC_COLS != 0 || ratio <= 0 || H % ratio != 0) return -1;
  if (form == FORM_DELTA ? (gated || units == nullptr || steps == nullptr) : ratio != 1) return -1;
  if (form == FORM_MIX || form == FORM_FORGET) {
    if (gated || z == nullptr || w0 == nullptr || bonus == nullptr) return -1;
  } else if (form == FORM_PLAIN && (gated ? small == nullptr : decay == nullptr)) {
    return -1;
  }
  const ScanParams p{proj, ld, q_col, k_col, v_col, small, ld_small, decay, bias_i, bias_f, cap, q_scale, s, n, m, slots, cu_q, seq_lens,
                     out, ldo, H, dk, KP, VP, num_slots, gated, rows, z, ldz, w0, bonus, status, ratio, units, steps};
  const bool single = cu_q == nullptr && dk <= RD_MAX_DK && B <= RD_MAX_B;
#define RB_FORM(FORM)                                                                                                                        \
  return single ? (dtype == 0 ? launch_decode<__nv_bfloat16, FORM>(p, B, stream) : launch_decode<float, FORM>(p, B, stream))               \
                : (dtype == 0 ? launch_scan<__nv_bfloat16, FORM>(p, B, stream) : launch_scan<float, FORM>(p, B, stream))
  switch (form) {
    case FORM_PLAIN: RB_FORM(FORM_PLAIN);
    case FORM_MIX: RB_FORM(FORM_MIX);
    case FORM_FORGET: RB_FORM(FORM_FORGET);
    case FORM_DELTA: RB_FORM(FORM_DELTA);
    default: return -1;
  }
#undef RB_FORM
}

// Workspace of the chunked form in bytes.
long long rb_recurrent_chunk_workspace(int n_chunks, int H, int KP, int VP) {
  const long long ch = (long long)n_chunks * H;
  return ch * ((long long)KP * VP * 8 + KP * 8 + 3 * CH * 4 + 16) + 256;
}

// Sequences of any length, `chunks` [n_chunks] and `seq_chunks` [n_seq + 1] as ChunkParams describes; slots, seq_lens and cu_q belong to
// the same n_seq sequences. Activations in bf16.
int rb_recurrent_chunks(const void* proj, long long ld, int q_col, int k_col, int v_col, const float* small, long long ld_small, const float* decay,
                        const float* bias_i, const float* bias_f, float cap, float q_scale, float* s, float* n, float* m, const void* chunks,
                        const int* seq_chunks, const int* slots, const int* cu_q, const int* seq_lens, float* out, long long ldo, void* workspace,
                        int n_chunks, int n_seq, int H, int dk, int KP, int VP, int num_slots, int gated, int* status, cudaStream_t stream) {
  if (n_chunks <= 0 || n_seq <= 0) return 0;
  if (H <= 0 || H > 65535 || n_seq > 65535 || dk <= 0 || dk > KP || KP % 64 != 0 || VP % 64 != 0 || ld % 8 != 0 || ldo % 4 != 0 ||
      (gated ? small == nullptr : decay == nullptr) || workspace == nullptr)
    return -1;
  const long long ch = (long long)n_chunks * H;
  ChunkParams p{};
  p.proj = (const __nv_bfloat16*)proj; p.ld = ld; p.q_col = q_col; p.k_col = k_col; p.v_col = v_col;
  p.small = small; p.ld_small = ld_small; p.decay = decay; p.bias_i = bias_i; p.bias_f = bias_f; p.cap = cap; p.q_scale = q_scale;
  p.chunks = (const int4*)chunks; p.seq_chunks = seq_chunks; p.slots = slots; p.seq_lens = seq_lens; p.cu_q = cu_q;
  p.s = s; p.n = n; p.m = m; p.out = out; p.ldo = ldo;
  p.H = H; p.dk = dk; p.KP = KP; p.VP = VP; p.num_slots = num_slots; p.gated = gated; p.status = status;
  p.v = p.proj + v_col; p.ld_v = ld; p.ratio = 1;
  float* w = (float*)workspace;
  p.u = w; w += ch * KP * VP;
  p.s_hi = (__nv_bfloat16*)w; w += ch * KP * VP / 2;
  p.s_lo = (__nv_bfloat16*)w; w += ch * KP * VP / 2;
  p.un = w; w += ch * KP;
  p.s_n = w; w += ch * KP;
  p.um = (float2*)w; w += ch * 2;
  p.gates = w; w += ch * 3 * CH;
  p.s_m = w;
  switch (KP) {
    case 64: return launch_chunks<64>(p, n_chunks, n_seq, stream);
    case 128: return launch_chunks<128>(p, n_chunks, n_seq, stream);
    case 192: return launch_chunks<192>(p, n_chunks, n_seq, stream);
    case 256: return launch_chunks<256>(p, n_chunks, n_seq, stream);
    default: return -1;
  }
}

// Time mixing (forget: forget mixing, bonus holds the lower bounds) of one token per sequence down to the normed and gated output rows; heads padded to 64 channels. Activations and out
// in bf16 (dtype 0) or fp32.
int rb_time_mix_decode(const void* proj, long long ld, int k_col, int v_col, int g_col, const float* z, long long ldz, const float* w0,
                       const float* bonus, const float* norm, float eps, float* s, const int* slots, const int* seq_lens, void* out, long long ldo,
                       int B, int H, int dk, int dv, int num_slots, int forget, int dtype, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || dk <= 0 || dk > MD_DIM || dv <= 0 || dv > MD_DIM || ldo % 2 != 0) return -1;
  const MixDecodeParams p{proj, ld, k_col, v_col, g_col, z, ldz, w0, bonus, norm, eps, s, slots, seq_lens, out, ldo, H, dk, dv, num_slots, status};
  if (forget) return dtype == 0 ? launch_time_mix_decode<__nv_bfloat16, true>(p, B, stream) : launch_time_mix_decode<float, true>(p, B, stream);
  return dtype == 0 ? launch_time_mix_decode<__nv_bfloat16, false>(p, B, stream) : launch_time_mix_decode<float, false>(p, B, stream);
}

// Workspace of the chunked time mixing in bytes.
long long rb_time_mix_workspace(int n_chunks, int H, int KP) {
  const long long ch = (long long)n_chunks * H;
  return ch * ((long long)KP * KP * 8 + KP * 4) + 256;
}

// Chunked time mixing of whole portions, as rb_recurrent_chunks, down to the normed and gated output rows (bf16). z [T, ldz] is
// overwritten. KP is 64 or 128; values have as many (padded) channels as keys. keys not null: forget mixing, which leaves its keys there.
int rb_time_mix_chunks(const void* proj, long long ld, int k_col, int v_col, int g_col, float* z, long long ldz, const float* w0, const float* bonus,
                       float* s, const void* chunks, const int* seq_chunks, const int* slots, const int* cu_q, const int* seq_lens, const float* norm,
                       float eps, void* out, long long ldo, void* workspace, void* keys, long long ld_keys, int n_chunks, int n_seq, int H, int dk,
                       int dv, int KP, int num_slots, int* status, cudaStream_t stream) {
  if (n_chunks <= 0 || n_seq <= 0) return 0;
  if (H <= 0 || H * (KP / SC_COLS) > 65535 || n_seq > 65535 || dk <= 0 || dk > KP || ld % 8 != 0 || ldo % 8 != 0 || ldz % 4 != 0 || workspace == nullptr ||
      (k_col | v_col | g_col) % 8 != 0 || dv <= 0 || dv > KP || ld_keys % 8 != 0 || (keys != nullptr && ld_keys < 2 * H * KP))
    return -1;
  const long long ch = (long long)n_chunks * H;
  MixParams p{};
  p.proj = (const __nv_bfloat16*)proj; p.ld = ld; p.k_col = k_col; p.v_col = v_col; p.g_col = g_col;
  p.z = z; p.ldz = ldz; p.w0 = w0; p.bonus = bonus; p.chunks = (const int4*)chunks; p.seq_chunks = seq_chunks; p.slots = slots;
  p.seq_lens = seq_lens; p.cu_q = cu_q; p.s = s; p.norm = norm; p.eps = eps; p.out = (__nv_bfloat16*)out; p.ldo = ldo;
  p.H = H; p.dk = dk; p.dv = dv; p.KP = KP; p.VP = KP; p.num_slots = num_slots; p.status = status;
  p.keys = (__nv_bfloat16*)keys; p.ld_keys = ld_keys;
  float* w = (float*)workspace;
  p.u = w; w += ch * KP * KP;
  p.s_hi = (__nv_bfloat16*)w; w += ch * KP * KP / 2;
  p.s_lo = (__nv_bfloat16*)w; w += ch * KP * KP / 2;
  p.last = w;
  const bool forget = keys != nullptr;
  if (KP == 64) return forget ? launch_time_mix<64, true>(p, n_chunks, n_seq, stream) : launch_time_mix<64, false>(p, n_chunks, n_seq, stream);
  if (KP == 128) return forget ? launch_time_mix<128, true>(p, n_chunks, n_seq, stream) : launch_time_mix<128, false>(p, n_chunks, n_seq, stream);
  return -1;
}

// Rows of the delta rule between the joint projection and the recurrence (see DeltaRows); cu_q null: one row per sequence. With cu_q the
// histories move on in a second launch.
int rb_delta_rows(const void* proj, long long ld, const float* conv, int taps, void* hist, const int* cu_q, const int* positions, const int* slots, int B,
                  int num_slots, void* out, long long ldo, const float* small, long long ld_small, const float* rate, const float* dt_bias, float* units,
                  float* steps, int G, int H, int KP, int VP, int T, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (G <= 0 || H <= 0 || H % G != 0 || KP % 64 != 0 || VP % 64 != 0 || KP > 512 || VP > 512 || taps < 1 || taps > 16 || (taps > 1 && hist == nullptr) ||
      ld % 8 != 0 || ldo % 8 != 0 || B <= 0)
    return -1;
  DeltaRows p{proj, ld, conv, taps, hist, History{cu_q, positions, slots, B, taps - 1, num_slots}, out, ldo, small, ld_small, rate, dt_bias, units, steps,
              G, H, KP, VP, T, 1, status};
  if (cu_q != nullptr) {                                   // long enough runs that a look back is seldom fetched, enough of them to fill the machine
    const long long run = (long long)T * (2 * G + H) / (148 * 32);
    p.run = run < 1 ? 1 : run > 16 ? 16 : (int)run;
  }
  cudaError_t e = dtype == 0 ? launch_delta_rows<__nv_bfloat16>(p, stream) : launch_delta_rows<float>(p, stream);
  const int channels = 2 * G * KP + H * VP;
  if (e == cudaSuccess && cu_q != nullptr && taps > 1)
    e = dtype == 0 ? launch_history_update((const __nv_bfloat16*)proj, ld, p.rows, (__nv_bfloat16*)hist, channels, stream)
                   : launch_history_update((const float*)proj, ld, p.rows, (float*)hist, channels, stream);
  return e == cudaSuccess ? 0 : -11;
}

// Workspace of the chunked delta rule in bytes.
long long rb_delta_workspace(int n_chunks, int H, int KP, int VP) {
  const long long ch = (long long)n_chunks * H;
  return ch * ((long long)KP * VP * 4 + CH * KP * 6 + CH * VP * 6 + 3 * CH * 4 + 8) + 256;      // (room for a key head per head)
}

// The delta rule over whole portions in chunks, as rb_recurrent_chunks. rows [T, q | k | v] bf16. KP is 64 or 128.
int rb_delta_chunks(const void* rows, long long ld, int k_col, int v_col, const float* units, const float* steps, float q_scale, float* s, const void* chunks,
                    const int* seq_chunks, const int* slots, const int* cu_q, const int* seq_lens, float* out, long long ldo,
                    void* workspace, int n_chunks, int n_seq, int H, int ratio, int dk, int KP, int VP, int num_slots, int* status,
                    cudaStream_t stream) {
  if (n_chunks <= 0 || n_seq <= 0) return 0;
  if (H <= 0 || H > 65535 || n_seq > 65535 || ratio <= 0 || H % ratio != 0 || dk <= 0 || dk > KP || VP % 64 != 0 || ld % 8 != 0 ||
      ldo % 4 != 0 || k_col % 8 != 0 || v_col % 8 != 0 || workspace == nullptr)
    return -1;
  const long long ch = (long long)n_chunks * H;
  DeltaParams p{};
  ChunkParams& c = p.c;
  c.proj = (const __nv_bfloat16*)rows; c.ld = ld; c.q_col = 0; c.k_col = k_col; c.v_col = v_col; c.q_scale = q_scale;
  c.chunks = (const int4*)chunks; c.seq_chunks = seq_chunks; c.slots = slots; c.seq_lens = seq_lens; c.cu_q = cu_q;
  c.s = s; c.out = out; c.ldo = ldo;
  c.H = H; c.dk = dk; c.KP = KP; c.VP = VP; c.num_slots = num_slots; c.status = status;
  c.v = c.proj + v_col; c.ld_v = ld; c.ratio = ratio;
  p.units = units; p.steps = steps;
  float* w = (float*)workspace;
  p.uv = w; w += ch * CH * VP;
  c.s_hi = (__nv_bfloat16*)w; w += ch * KP * VP / 2;
  c.s_lo = (__nv_bfloat16*)w; w += ch * KP * VP / 2;
  p.w_hi = (__nv_bfloat16*)w; w += ch * CH * KP / 2;
  p.w_lo = (__nv_bfloat16*)w; w += ch * CH * KP / 2;
  p.keys = (__nv_bfloat16*)w; w += ch * CH * KP / 2;
  p.values = (__nv_bfloat16*)w; w += ch * CH * VP / 2;
  c.written = p.values;
  c.gates = w; w += ch * 3 * CH;
  c.um = (float2*)w;
  if (KP == 64) return launch_delta_chunks<64>(p, n_chunks, n_seq, stream);
  return KP == 128 ? launch_delta_chunks<128>(p, n_chunks, n_seq, stream) : -1;
}

int rb_gated_norm(const float* o, long long ldo, const float* weight, const void* gate, long long ldg, void* out, long long ldy, int H, int dv,
                  int VP, int per_head, int silu, int T, int dtype, float eps, cudaStream_t stream) {      // gate may be null
  if (T <= 0) return 0;
  if (VP % 4 != 0 || ldo % 4 != 0 || ldy % 4 != 0) return -1;
  cudaError_t e;
  if (dtype == 0)
    e = launch_kernel(gated_norm_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, o, ldo, weight, (const __nv_bfloat16*)gate, ldg,
                      (__nv_bfloat16*)out, ldy, H, dv, VP, per_head, silu, eps);
  else
    e = launch_kernel(gated_norm_kernel<float>, dim3(T), dim3(256), 0, stream, o, ldo, weight, (const float*)gate, ldg, (float*)out, ldy, H, dv, VP,
                      per_head, silu, eps);
  return e == cudaSuccess ? 0 : -11;
}

}  // extern "C"
