// Memory-bound transformer ops for sm_100a: RMSNorm (row and per-head), RoPE fused with the
// paged KV-cache append, SwiGLU, embedding gather, seeded sampling with log-probabilities.
// All kernels are single-pass over HBM with 16-byte accesses; rounding points follow the
// bf16 Hugging Face modules (see the functional oracles in research_b200/models/functional.py)
// so that greedy decoding matches the fp32/bf16 reference token for token.
#include "common.cuh"

namespace rb {

// ------------------------------------------------------------------------------------------
// RMSNorm: y = bf16( bf16(x * rsqrt(mean(x^2)+eps)) * w ). One warp per row.
// Reference math: rollouts/tools/functional_extractor/qwen_functional.py:46-65.
// ------------------------------------------------------------------------------------------
// The row is read from global memory once: up to 8 vectors of 8 bf16 per lane stay in
// registers (d <= 2048); longer rows fall back to a second read that hits L1/L2.
__global__ void rmsnorm_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ w,
                               __nv_bfloat16* __restrict__ y, long long rows, int d, long long ldx,
                               long long ldy, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int MAXV = 8;
  const int lane = threadIdx.x & 31;
  const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (row >= rows) return;
  const __nv_bfloat16* xr = x + row * ldx;
  __nv_bfloat16* yr = y + row * ldy;
  const int nvec = d >> 3;
  const bool in_regs = nvec <= MAXV * 32;
  uint4 keep[MAXV];
  float ss = 0.f;
  if (in_regs) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int v = lane + 32 * i;
      keep[i] = v < nvec ? *reinterpret_cast<const uint4*>(xr + v * 8) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      float2 f;
      f = unpack_bf16x2(keep[i].x); ss += f.x * f.x + f.y * f.y;
      f = unpack_bf16x2(keep[i].y); ss += f.x * f.x + f.y * f.y;
      f = unpack_bf16x2(keep[i].z); ss += f.x * f.x + f.y * f.y;
      f = unpack_bf16x2(keep[i].w); ss += f.x * f.x + f.y * f.y;
    }
  } else {
    for (int v = lane; v < nvec; v += 32) {
      uint4 u = *reinterpret_cast<const uint4*>(xr + v * 8);
      float2 f;
      f = unpack_bf16x2(u.x); ss += f.x * f.x + f.y * f.y;
      f = unpack_bf16x2(u.y); ss += f.x * f.x + f.y * f.y;
      f = unpack_bf16x2(u.z); ss += f.x * f.x + f.y * f.y;
      f = unpack_bf16x2(u.w); ss += f.x * f.x + f.y * f.y;
    }
  }
  ss = warp_sum(ss);
  const float rstd = rsqrtf(ss / (float)d + eps);
  auto emit = [&](int v, uint4 u) {
    uint4 ww = *reinterpret_cast<const uint4*>(w + v * 8);
    uint32_t xi[4] = {u.x, u.y, u.z, u.w};
    uint32_t wi[4] = {ww.x, ww.y, ww.z, ww.w};
    uint32_t oi[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 f = unpack_bf16x2(xi[j]);
      float2 g = unpack_bf16x2(wi[j]);
      // round the normalised value to bf16 before the weight multiply, like the HF module
      float a = __bfloat162float(__float2bfloat16_rn(f.x * rstd));
      float b = __bfloat162float(__float2bfloat16_rn(f.y * rstd));
      oi[j] = pack_bf16x2(a * g.x, b * g.y);
    }
    *reinterpret_cast<uint4*>(yr + v * 8) = make_uint4(oi[0], oi[1], oi[2], oi[3]);
  };
  if (in_regs) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int v = lane + 32 * i;
      if (v < nvec) emit(v, keep[i]);
    }
  } else {
    for (int v = lane; v < nvec; v += 32) emit(v, *reinterpret_cast<const uint4*>(xr + v * 8));
  }
}

// ------------------------------------------------------------------------------------------
// RoPE (rotate_half convention) + optional per-head QK RMSNorm + paged KV append.
//   qkv   : [T, (Hq + 2*Hkv) * D] bf16  (q heads, then k heads, then v heads)
//   q_out : [T, Hq * D] bf16 (rotated)
//   k_cache / v_cache : [num_blocks, Hkv, block_size, D] bf16, slot = block*block_size + off
//   cos_sin : [max_pos, D/2] float2
// One warp per (token, head). Slots < 0 are skipped (padding rows of a captured graph).
// Reference math: qwen_functional.py:68-150; cache store: inference/attention/flex_backend.py:116-142.
// ------------------------------------------------------------------------------------------
template <int D>
__global__ void rope_kv_append_kernel(const __nv_bfloat16* __restrict__ qkv, __nv_bfloat16* __restrict__ q_out,
                                      __nv_bfloat16* __restrict__ k_cache, __nv_bfloat16* __restrict__ v_cache,
                                      const int* __restrict__ positions, const int* __restrict__ slots,
                                      const float2* __restrict__ cos_sin, const __nv_bfloat16* __restrict__ q_norm_w,
                                      const __nv_bfloat16* __restrict__ k_norm_w, float norm_eps, int T, int Hq,
                                      int Hkv, int block_size, long long num_slots, int max_pos, int* status) {
  constexpr int HALF = D / 2;
  constexpr int PER_LANE = HALF / 32;  // pairs handled per lane: D=64 -> 1, D=128 -> 2
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long gw = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int heads = Hq + 2 * Hkv;
  if (gw >= (long long)T * heads) return;
  const int t = (int)(gw / heads);
  const int h = (int)(gw % heads);
  const __nv_bfloat16* src = qkv + (long long)t * heads * D + (long long)h * D;
  int pos = positions[t];
  const int slot = slots[t];
  if (pos < 0) pos = 0;
  if (pos >= max_pos) { set_status(status, ST_BAD_INDEX); pos = max_pos - 1; }

  float lo[PER_LANE], hi[PER_LANE];
#pragma unroll
  for (int j = 0; j < PER_LANE; ++j) {
    lo[j] = __bfloat162float(src[lane + 32 * j]);
    hi[j] = __bfloat162float(src[lane + 32 * j + HALF]);
  }
  __nv_bfloat16* dst;
  bool is_v = h >= Hq + Hkv;
  if (h < Hq) {
    dst = q_out + (long long)t * Hq * D + (long long)h * D;
  } else {
    if (slot < 0) return;
    if (slot >= num_slots) { set_status(status, ST_BAD_INDEX); return; }
    const int kvh = is_v ? h - Hq - Hkv : h - Hq;
    const long long blk = slot / block_size, off = slot % block_size;
    __nv_bfloat16* cache = is_v ? v_cache : k_cache;
    dst = cache + ((blk * Hkv + kvh) * block_size + off) * D;
  }
  if (is_v) {
#pragma unroll
    for (int j = 0; j < PER_LANE; ++j) {
      dst[lane + 32 * j] = __float2bfloat16_rn(lo[j]);
      dst[lane + 32 * j + HALF] = __float2bfloat16_rn(hi[j]);
    }
    return;
  }
  const __nv_bfloat16* nw = (h < Hq) ? q_norm_w : k_norm_w;
  if (nw != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER_LANE; ++j) ss += lo[j] * lo[j] + hi[j] * hi[j];
    ss = warp_sum(ss);
    const float rstd = rsqrtf(ss / (float)D + norm_eps);
#pragma unroll
    for (int j = 0; j < PER_LANE; ++j) {
      float a = __bfloat162float(__float2bfloat16_rn(lo[j] * rstd));
      float b = __bfloat162float(__float2bfloat16_rn(hi[j] * rstd));
      lo[j] = __bfloat162float(__float2bfloat16_rn(a * __bfloat162float(nw[lane + 32 * j])));
      hi[j] = __bfloat162float(__float2bfloat16_rn(b * __bfloat162float(nw[lane + 32 * j + HALF])));
    }
  }
#pragma unroll
  for (int j = 0; j < PER_LANE; ++j) {
    const float2 cs = cos_sin[(long long)pos * HALF + lane + 32 * j];
    // bf16 rounding of cos/sin and of each product mirrors q*cos + rotate_half(q)*sin in bf16
    const float c = __bfloat162float(__float2bfloat16_rn(cs.x));
    const float s = __bfloat162float(__float2bfloat16_rn(cs.y));
    const float a = __bfloat162float(__float2bfloat16_rn(lo[j] * c));
    const float b = __bfloat162float(__float2bfloat16_rn(-hi[j] * s));
    const float e = __bfloat162float(__float2bfloat16_rn(hi[j] * c));
    const float f = __bfloat162float(__float2bfloat16_rn(lo[j] * s));
    dst[lane + 32 * j] = __float2bfloat16_rn(a + b);
    dst[lane + 32 * j + HALF] = __float2bfloat16_rn(e + f);
  }
}

// ------------------------------------------------------------------------------------------
// SwiGLU: out = bf16( bf16(silu(gate)) * up ), gate|up packed as [T, 2F].
// Reference math: qwen_functional.py:251-274.
// ------------------------------------------------------------------------------------------
// `rows_dev` (optional) bounds the row count from device memory: the expert-parallel MoE layer only knows on the
// device how many routed rows it received.
__global__ void swiglu_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out,
                              long long T, int F, const int* __restrict__ rows_dev) {
  pdl_launch_dependents();
  pdl_wait();
  if (rows_dev != nullptr) {
    const long long r = *rows_dev;
    T = r < T ? (r < 0 ? 0 : r) : T;
  }
  const long long nvec = T * (F >> 3);
  const int fv = F >> 3;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < nvec;
       i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / fv;
    const int c = (int)(i % fv) * 8;
    uint4 g = *reinterpret_cast<const uint4*>(gu + t * 2 * F + c);
    uint4 u = *reinterpret_cast<const uint4*>(gu + t * 2 * F + F + c);
    uint32_t gi[4] = {g.x, g.y, g.z, g.w}, ui[4] = {u.x, u.y, u.z, u.w}, oi[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 a = unpack_bf16x2(gi[j]);
      float2 b = unpack_bf16x2(ui[j]);
      float s0 = __bfloat162float(__float2bfloat16_rn(a.x / (1.f + __expf(-a.x))));
      float s1 = __bfloat162float(__float2bfloat16_rn(a.y / (1.f + __expf(-a.y))));
      oi[j] = pack_bf16x2(s0 * b.x, s1 * b.y);
    }
    *reinterpret_cast<uint4*>(out + t * F + c) = make_uint4(oi[0], oi[1], oi[2], oi[3]);
  }
}

// SwiGLU backward: given gate|up [T,2F] and dout [T,F] writes dgate|dup [T,2F].
__global__ void swiglu_bwd_kernel(const __nv_bfloat16* __restrict__ gu, const __nv_bfloat16* __restrict__ dout,
                                  __nv_bfloat16* __restrict__ dgu, long long T, int F) {
  // 8 columns (16 bytes) per thread and step; F % 8 == 0 is checked by the launcher
  const int fv = F >> 3;
  const long long nvec = T * fv;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < nvec;
       i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / fv;
    const int c = (int)(i % fv) * 8;
    const uint4 g4 = *reinterpret_cast<const uint4*>(gu + t * 2 * F + c);
    const uint4 u4 = *reinterpret_cast<const uint4*>(gu + t * 2 * F + F + c);
    const uint4 d4 = *reinterpret_cast<const uint4*>(dout + t * F + c);
    const uint32_t gi[4] = {g4.x, g4.y, g4.z, g4.w}, ui[4] = {u4.x, u4.y, u4.z, u4.w}, di[4] = {d4.x, d4.y, d4.z, d4.w};
    uint32_t og[4], ou[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 g = unpack_bf16x2(gi[j]), u = unpack_bf16x2(ui[j]), dy = unpack_bf16x2(di[j]);
      const float s0 = 1.f / (1.f + __expf(-g.x)), s1 = 1.f / (1.f + __expf(-g.y));
      const float l0 = g.x * s0, l1 = g.y * s1;
      og[j] = pack_bf16x2(dy.x * u.x * (s0 + l0 * (1.f - s0)), dy.y * u.y * (s1 + l1 * (1.f - s1)));
      ou[j] = pack_bf16x2(dy.x * l0, dy.y * l1);
    }
    *reinterpret_cast<uint4*>(dgu + t * 2 * F + c) = make_uint4(og[0], og[1], og[2], og[3]);
    *reinterpret_cast<uint4*>(dgu + t * 2 * F + F + c) = make_uint4(ou[0], ou[1], ou[2], ou[3]);
  }
}

// ------------------------------------------------------------------------------------------
// Embedding gather: out[t, :] = table[ids[t], :]
// ------------------------------------------------------------------------------------------
__global__ void embedding_kernel(const int* __restrict__ ids, const __nv_bfloat16* __restrict__ table,
                                 __nv_bfloat16* __restrict__ out, int T, int d, int vocab, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  if (t >= T) return;
  int id = ids[t];
  if (id < 0 || id >= vocab) { if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX); id = 0; }
  const uint4* src = reinterpret_cast<const uint4*>(table + (long long)id * d);
  uint4* dst = reinterpret_cast<uint4*>(out + (long long)t * d);
  for (int v = threadIdx.x; v < (d >> 3); v += blockDim.x) dst[v] = src[v];
}

// ------------------------------------------------------------------------------------------
// Models with a 32-bit residual stream. The stream x is fp32 [T, d]; `xb` is the copy in the activation type TA
// (bf16 when serving, fp32 in exact mode) that the projections read, row stride ldb, columns d..ldb stay zero.
// ------------------------------------------------------------------------------------------
template <typename TA> __device__ __forceinline__ TA to_act(float v);
template <> __device__ __forceinline__ float to_act<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 to_act<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float from_act(float v) { return v; }
__device__ __forceinline__ float from_act(__nv_bfloat16 v) { return __bfloat162float(v); }

// Sum over the CTA (blockDim.x a multiple of 32, at most 1024); every thread receives the total.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

// Embedding row into the fp32 stream and up to two copies of it in the activation type (all strides in elements).
template <typename TA>
__global__ void stream_embed_kernel(const int* __restrict__ ids, const TA* __restrict__ table, long long ldt, float* __restrict__ x,
                                    long long ldx, TA* __restrict__ a, long long lda, TA* __restrict__ b, long long ldb, int d, int vocab,
                                    int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) { if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX); id = 0; }
  const TA* src = table + (long long)id * ldt;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const TA v = src[c];
    x[t * ldx + c] = from_act(v);
    if (a != nullptr) a[t * lda + c] = v;
    if (b != nullptr) b[t * ldb + c] = v;
  }
}

__device__ __forceinline__ float4 load_act4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load_act4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 lo = unpack_bf16x2(u.x), hi = unpack_bf16x2(u.y);
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void store_act4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store_act4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// One pass over the fp32 residual stream between two layers, a CTA per row:
//   x += mult * (y1 + y2 + sum_j w[j] e[row * k + j] + side / rms(side) * side_weight)
//                                                (absent terms are null; nothing is written back when all are; w null: ones)
//   copy = x in the activation type,  h = x / rms(x) * weight
// rows != null: h[i] comes from row rows[i] (no update). Columns are padded to a multiple of 4 with zeros.
struct StreamNormParams {
  float* x;
  long long ldx;
  const float* y1;
  const float* y2;
  long long ldy;
  const void* e;
  const float* w;
  long long lde;
  int k;
  void* copy;
  long long ldc;
  void* h;
  long long ldh;
  const float* weight;
  const float* side;
  long long ld_side;
  const float* side_weight;
  const int* rows;
  int num_src_rows, d, dp;
  float eps, mult;
  int* status;
};

template <typename TA>
__global__ void __launch_bounds__(256) stream_norm_kernel(const StreamNormParams p) {
  extern __shared__ float4 sn_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const long long r = blockIdx.x;
  long long xr = r;
  if (p.rows != nullptr) {
    xr = p.rows[r];
    if (xr < 0 || xr >= p.num_src_rows) { if (threadIdx.x == 0) set_status(p.status, ST_BAD_INDEX); xr = 0; }
  }
  float* x = p.x + xr * p.ldx;
  const bool update = p.y1 != nullptr || p.y2 != nullptr || p.e != nullptr || p.side != nullptr;
  const TA* e = reinterpret_cast<const TA*>(p.e) + r * p.k * p.lde;
  float ss = 0.f, side_scale = 0.f;
  if (p.side != nullptr) {
    float sq = 0.f;
    for (int c = threadIdx.x * 4; c < p.dp; c += blockDim.x * 4) {
      const float4 y = *reinterpret_cast<const float4*>(p.side + r * p.ld_side + c);
      sq += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
    }
    side_scale = 1.f / sqrtf(block_sum(sq, red) / (float)p.d + p.eps);
  }
  for (int c = threadIdx.x * 4; c < p.dp; c += blockDim.x * 4) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.y1 != nullptr) {
      const float4 y = *reinterpret_cast<const float4*>(p.y1 + r * p.ldy + c);
      v.x += y.x; v.y += y.y; v.z += y.z; v.w += y.w;
    }
    if (p.y2 != nullptr) {
      const float4 y = *reinterpret_cast<const float4*>(p.y2 + r * p.ldy + c);
      v.x += y.x; v.y += y.y; v.z += y.z; v.w += y.w;
    }
    if (p.e != nullptr) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = 0; j < p.k; ++j) {
        const float w = p.w != nullptr ? __ldg(p.w + r * p.k + j) : 1.f;
        const float4 y = load_act4(e + j * p.lde + c);
        a.x = fmaf(w, y.x, a.x); a.y = fmaf(w, y.y, a.y); a.z = fmaf(w, y.z, a.z); a.w = fmaf(w, y.w, a.w);
      }
      v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
    }
    if (p.side != nullptr) {
      const float4 y = *reinterpret_cast<const float4*>(p.side + r * p.ld_side + c);
      const float4 w = *reinterpret_cast<const float4*>(p.side_weight + c);
      v.x += y.x * side_scale * w.x; v.y += y.y * side_scale * w.y; v.z += y.z * side_scale * w.z; v.w += y.w * side_scale * w.w;
    }
    const float4 old = *reinterpret_cast<const float4*>(x + c);
    v.x = fmaf(p.mult, v.x, old.x); v.y = fmaf(p.mult, v.y, old.y); v.z = fmaf(p.mult, v.z, old.z); v.w = fmaf(p.mult, v.w, old.w);
    if (update) *reinterpret_cast<float4*>(x + c) = v;
    if (p.copy != nullptr) store_act4(reinterpret_cast<TA*>(p.copy) + r * p.ldc + c, v);
    sn_row[c >> 2] = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  if (p.h == nullptr) return;
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)p.d + p.eps);
  TA* h = reinterpret_cast<TA*>(p.h) + r * p.ldh;
  for (int c = threadIdx.x * 4; c < p.dp; c += blockDim.x * 4) {
    const float4 v = sn_row[c >> 2];
    const float4 w = *reinterpret_cast<const float4*>(p.weight + c);
    store_act4(h + c, make_float4(v.x * rs * w.x, v.y * rs * w.y, v.z * rs * w.z, v.w * rs * w.w));
  }
}

// One pass over the fp32 residual stream around a sublayer with a norm before and after it, a CTA per row:
//   v = y                                                    one output, or
//   v = pair_scale * (y / rms(y) * w + y2 / rms(y2) * w2)    two mixers side by side, or
//   v = sigmoid(gate) y + sum_j p[j] e[row * k + j]          a shared expert (its gate may be null) and the routed ones; choices from `experts`
//                                                            on have no row: their weight goes to `pass`, the sublayer's own input
//   x += N_post(v), copy = x, h = N_pre(x) in the activation type
// with N(z) = z / rms(z) * weight, or tanh(alpha z) * weight + bias (BOUNDED). Any of y, h and copy may be null; rows != null: h[i]
// comes from row rows[i] (no update). Columns are padded to a multiple of 4 with zeros (weights and biases there are zero too).
struct SandwichNorm { const float* weight; const float* bias; const float* alpha; };
struct SandwichParams {
  float* x; long long ldx;
  const float* y; const float* y2; long long ldy;
  const float* w; const float* w2;
  float pair_scale;
  const float* gate; long long ld_gate;
  const void* e; long long lde;
  const float* p; const int* idx; int k, experts;
  const void* pass; long long ld_pass;
  SandwichNorm post, pre;
  void* copy; long long ldc;
  void* h; long long ldh;
  const int* rows; int num_src_rows;
  int d, dp; float eps;
  int* status;
};

template <typename TA, bool BOUNDED>
__global__ void __launch_bounds__(256) stream_sandwich_kernel(const SandwichParams p) {
  extern __shared__ float4 sw_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const long long r = blockIdx.x;
  long long xr = r;
  if (p.rows != nullptr) {
    xr = p.rows[r];
    if (xr < 0 || xr >= p.num_src_rows) { if (threadIdx.x == 0) set_status(p.status, ST_BAD_INDEX); xr = 0; }
  }
  float* x = p.x + xr * p.ldx;
  const float* y = p.y + r * p.ldy;
  const float* y2 = p.y2 + r * p.ldy;
  const bool update = p.y != nullptr || p.e != nullptr;
  auto at4 = [](const float* q, int c) { return *reinterpret_cast<const float4*>(q + c); };
  auto square = [](float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
  const int step = blockDim.x * 4;
  float s1 = 1.f, s2 = 0.f;
  if (p.y2 != nullptr) {
    float a = 0.f, b = 0.f;
    for (int c = threadIdx.x * 4; c < p.dp; c += step) { a += square(at4(y, c)); b += square(at4(y2, c)); }
    s1 = p.pair_scale / sqrtf(block_sum(a, red) / (float)p.d + p.eps);
    s2 = p.pair_scale / sqrtf(block_sum(b, red) / (float)p.d + p.eps);
  }
  if (p.gate != nullptr) s1 = 1.f / (1.f + expf(-p.gate[r * p.ld_gate]));
  float through = 0.f;
  if (p.e != nullptr)
    for (int j = 0; j < p.k; ++j)
      if (p.idx[r * p.k + j] >= p.experts) through += p.p[r * p.k + j];
  const TA* e = reinterpret_cast<const TA*>(p.e) + r * p.k * p.lde;
  const TA* pass = reinterpret_cast<const TA*>(p.pass) + r * p.ld_pass;
  auto sublayer = [&](int c) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.y2 != nullptr) {
      const float4 a = at4(y, c), b = at4(y2, c), wa = at4(p.w, c), wb = at4(p.w2, c);
      return make_float4(a.x * s1 * wa.x + b.x * s2 * wb.x, a.y * s1 * wa.y + b.y * s2 * wb.y, a.z * s1 * wa.z + b.z * s2 * wb.z,
                         a.w * s1 * wa.w + b.w * s2 * wb.w);
    }
    if (p.y != nullptr) {
      const float4 a = at4(y, c);
      v = make_float4(s1 * a.x, s1 * a.y, s1 * a.z, s1 * a.w);
    }
    if (p.e != nullptr) {
      for (int j = 0; j < p.k; ++j) {
        if (__ldg(p.idx + r * p.k + j) >= p.experts) continue;
        const float w = __ldg(p.p + r * p.k + j);
        const float4 a = load_act4(e + j * p.lde + c);
        v.x = fmaf(w, a.x, v.x); v.y = fmaf(w, a.y, v.y); v.z = fmaf(w, a.z, v.z); v.w = fmaf(w, a.w, v.w);
      }
      if (through != 0.f) {
        const float4 a = load_act4(pass + c);
        v.x = fmaf(through, a.x, v.x); v.y = fmaf(through, a.y, v.y); v.z = fmaf(through, a.z, v.z); v.w = fmaf(through, a.w, v.w);
      }
    }
    return v;
  };
  auto bounded = [&](const SandwichNorm& n, float alpha, float4 v, int c) {
    const float4 w = at4(n.weight, c), b = at4(n.bias, c);
    return make_float4(fmaf(tanhf(alpha * v.x), w.x, b.x), fmaf(tanhf(alpha * v.y), w.y, b.y), fmaf(tanhf(alpha * v.z), w.z, b.z),
                       fmaf(tanhf(alpha * v.w), w.w, b.w));
  };
  TA* h = p.h != nullptr ? reinterpret_cast<TA*>(p.h) + r * p.ldh : nullptr;
  TA* copy = p.copy != nullptr ? reinterpret_cast<TA*>(p.copy) + r * p.ldc : nullptr;
  const float post_alpha = BOUNDED && update ? *p.post.alpha : 0.f, pre_alpha = BOUNDED && p.h != nullptr ? *p.pre.alpha : 0.f;
  float post_scale = 0.f;
  if (!BOUNDED && update) {
    float s = 0.f;
    for (int c = threadIdx.x * 4; c < p.dp; c += step) {
      const float4 v = sublayer(c);
      sw_row[c >> 2] = v;
      s += square(v);
    }
    post_scale = 1.f / sqrtf(block_sum(s, red) / (float)p.d + p.eps);
  }
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < p.dp; c += step) {
    float4 v = at4(x, c);
    if (update) {
      float4 n;
      if (BOUNDED) {
        n = bounded(p.post, post_alpha, sublayer(c), c);
      } else {
        const float4 a = sw_row[c >> 2], w = at4(p.post.weight, c);
        n = make_float4(a.x * post_scale * w.x, a.y * post_scale * w.y, a.z * post_scale * w.z, a.w * post_scale * w.w);
      }
      v.x += n.x; v.y += n.y; v.z += n.z; v.w += n.w;
      *reinterpret_cast<float4*>(x + c) = v;
    }
    if (copy != nullptr) store_act4(copy + c, v);
    if (h == nullptr) continue;
    if (BOUNDED) {
      store_act4(h + c, bounded(p.pre, pre_alpha, v, c));
    } else {
      sw_row[c >> 2] = v;
      ss += square(v);
    }
  }
  if (BOUNDED || h == nullptr) return;
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)p.d + p.eps);
  for (int c = threadIdx.x * 4; c < p.dp; c += step) {
    const float4 v = sw_row[c >> 2], w = at4(p.pre.weight, c);
    store_act4(h + c, make_float4(v.x * rs * w.x, v.y * rs * w.y, v.z * rs * w.z, v.w * rs * w.w));
  }
}

// out = a N(z) + b N(z^2) + c N(z^3) + e on rows of n channels (N: division by the root mean square over the row); act = {a, b, c, e}.
// Padding columns n .. np - 1 of out become zero.
template <typename TA>
__global__ void __launch_bounds__(256) poly_norm_kernel(const TA* __restrict__ z, long long ldz, const float* __restrict__ act, TA* __restrict__ out,
                                                        long long ldo, int n, int np, float eps) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const TA* row = z + (long long)blockIdx.x * ldz;
  TA* dst = out + (long long)blockIdx.x * ldo;
  float m2 = 0.f, m4 = 0.f, m6 = 0.f;
  auto powers = [&](float v) {
    const float s = v * v;
    m2 += s;
    m4 = fmaf(s, s, m4);
    m6 = fmaf(s * s, s, m6);
  };
  for (int c = threadIdx.x * 4; c < np; c += blockDim.x * 4) {      // (padding columns of z are zero)
    const float4 v = load_act4(row + c);
    powers(v.x); powers(v.y); powers(v.z); powers(v.w);
  }
  const float inv = 1.f / (float)n;
  const float a = act[0] / sqrtf(block_sum(m2, red) * inv + eps), b = act[1] / sqrtf(block_sum(m4, red) * inv + eps);
  const float k = act[2] / sqrtf(block_sum(m6, red) * inv + eps), e = act[3];
  auto one = [&](float v, int c) { return c < n ? fmaf(v, fmaf(v, fmaf(v, k, b), a), e) : 0.f; };
  for (int c = threadIdx.x * 4; c < np; c += blockDim.x * 4) {
    const float4 v = load_act4(row + c);
    store_act4(dst + c, make_float4(one(v.x, c), one(v.y, c + 1), one(v.z, c + 2), one(v.w, c + 3)));
  }
}

// Layer norm of fp32 rows with a two-pass variance; the row is kept in shared memory.
//   y == nullptr : out = LN(x[rows[i]]) * w + b                     (rows == nullptr: row i)
//   otherwise    : x += LN(y) * w + b, out = x                      (norm on the sublayer's output, residual add)
// The caller folds a layer scale into w and b.
template <typename TA>
__global__ void layernorm_kernel(const float* __restrict__ y, long long ldy, float* __restrict__ x, long long ldx,
                                 const int* __restrict__ rows,
                                 const float* __restrict__ w, const float* __restrict__ b, TA* __restrict__ out, long long ldo,
                                 int d, float eps, int num_src_rows, int* status) {
  extern __shared__ float ln_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const long long r = blockIdx.x;
  long long xr = r;
  if (rows != nullptr) {
    xr = rows[r];
    if (xr < 0 || xr >= num_src_rows) { if (threadIdx.x == 0) set_status(status, ST_BAD_INDEX); xr = 0; }
  }
  const float* src = y != nullptr ? y + r * ldy : x + xr * ldx;
  float s = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const float v = src[c];
    ln_row[c] = v;
    s += v;
  }
  const float mean = block_sum(s, red) / (float)d;
  float q = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const float v = ln_row[c] - mean;
    q += v * v;
  }
  const float rstd = 1.f / sqrtf(block_sum(q, red) / (float)d + eps);
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float v = fmaf((ln_row[c] - mean) * rstd, w[c], b[c]);
    if (y != nullptr) {
      v += x[r * ldx + c];
      x[r * ldx + c] = v;
    }
    out[r * ldo + c] = to_act<TA>(v);
  }
}

// a[t, c] = gelu_tanh(z[t, c]) * table[ids[t], col0 + c]: the gate of a per-layer token embedding.
template <typename TA>
__global__ void token_side_kernel(const float* __restrict__ z, long long ldz, const int* __restrict__ ids, const TA* __restrict__ table,
                                  long long ldt, int col0, TA* __restrict__ a, long long lda, int n, int T, int vocab, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const long long total = (long long)T * n;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / n;
    const int c = (int)(i - t * n);
    int id = ids[t];
    if (id < 0 || id >= vocab) { set_status(status, ST_BAD_INDEX); id = 0; }
    const float x = z[t * ldz + c];
    const float g = 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
    a[t * lda + c] = to_act<TA>(g * from_act(table[(long long)id * ldt + col0 + c]));
  }
}

// Gated unit on gate|up packed as [T, 2F]. limit > 0: g = min(gate, limit), u = clamp(up, +-limit), out = g sigmoid(1.702 g) (u + 1);
// otherwise out = silu(gate) * up.
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
  if (!(limit > 0.f)) return g / (1.f + expf(-g)) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}
template <typename TA>
__global__ void clamped_glu_kernel(const TA* __restrict__ gu, TA* __restrict__ out, long long T, int F, float limit) {
  pdl_launch_dependents();
  pdl_wait();
  const long long n = T * F;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / F;
    const int c = (int)(i - t * F);
    out[i] = to_act<TA>(clamped_glu(from_act(gu[t * 2 * F + c]), from_act(gu[t * 2 * F + F + c]), limit));
  }
}

// logits = cap * tanh(logits / cap), in place.
__global__ void softcap_kernel(float* __restrict__ x, long long n, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
    x[i] = cap * tanhf(x[i] / cap);
}

// ------------------------------------------------------------------------------------------
// Sampling with log-probabilities, one CTA per row of fp32 logits [B, V].
//   token  ~ softmax(logits / T)   via the Gumbel-max trick with a counter-based RNG
//            (temperature == 0 -> argmax)
//   logprob = log_softmax(logits)[token]  from the UNSCALED logits (true policy probability)
// Reference behaviour: rollouts/inference/sampling.py:10-58.
// ------------------------------------------------------------------------------------------
__device__ __forceinline__ uint64_t mix64(uint64_t z) {
  // splitmix64 finaliser: turns (seed, step) into the per-row key once per CTA
  z += 0x9E3779B97F4A7C15ull;
  z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
  z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
  return z ^ (z >> 31);
}
__device__ __forceinline__ uint32_t hash32(uint32_t idx, uint32_t k0, uint32_t k1) {
  // counter-based 32-bit mixer (murmur3 finaliser) - every (row key, column) has its own draw
  uint32_t h = (idx * 0x9E3779B1u) ^ k0;
  h ^= h >> 16; h *= 0x85EBCA6Bu;
  h ^= h >> 13; h *= 0xC2B2AE35u;
  h ^= h >> 16;
  return h + k1;
}

constexpr int SAMPLE_THREADS = 512;

__global__ void __launch_bounds__(SAMPLE_THREADS)
sample_logprob_kernel(const float* __restrict__ logits, long long ld, int V,
                      const float* __restrict__ temperature, const unsigned long long* __restrict__ seeds,
                      const unsigned long long* __restrict__ step_ptr, unsigned long long step_add,
                      int* __restrict__ out_tokens, float* __restrict__ out_logprobs,
                      float4* __restrict__ partials /*[rows][splits], splits > 1 only*/, int* __restrict__ tickets /*[rows]*/) {
  pdl_launch_dependents();
  pdl_wait();
  // grid (splits, rows): with few rows the vocabulary of a row is cut into `splits` contiguous chunks so that all
  // SMs share the transcendental work (three per element); the last CTA of a row merges the chunk records in
  // chunk order
  const int splits = gridDim.x;
  const int chunk = (((V + splits - 1) / splits) + 3) & ~3;
  const int v_lo = blockIdx.x * chunk;
  const int v_hi = min(V, v_lo + chunk);
  // The step counter lives in device memory so a captured CUDA graph draws fresh noise on
  // every replay (the host bumps the counter between replays).
  const unsigned long long step = step_add + (step_ptr != nullptr ? *step_ptr : 0ull);
  const int row = blockIdx.y;
  const float* lr = logits + (long long)row * ld;
  const float temp = temperature[row];
  const bool greedy = temp <= 0.f;
  const float inv_t = greedy ? 1.f : 1.f / temp;
  const uint64_t key = mix64(mix64(seeds[row]) ^ (step * 0x9E3779B97F4A7C15ull));
  const uint32_t k0 = (uint32_t)key, k1 = (uint32_t)(key >> 32);

  float m = -INFINITY, ssum = 0.f;     // online log-sum-exp of the unscaled logits
  float best = -INFINITY;              // best perturbed score
  int best_i = 0x7fffffff;
  const bool vec_ok = ((ld & 3) == 0) && ((reinterpret_cast<uintptr_t>(lr) & 15) == 0);
  for (int i = v_lo + threadIdx.x * 4; i < v_hi; i += SAMPLE_THREADS * 4) {
    float v[4];
    if (i + 3 < v_hi && vec_ok) {
      float4 f = __ldcs(reinterpret_cast<const float4*>(lr + i));
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = (i + j < v_hi) ? lr[i + j] : -INFINITY;
    }
    // one rescale of the running sum per 4 elements instead of a branch per element
    const float m4 = fmaxf(fmaxf(v[0], v[1]), fmaxf(v[2], v[3]));
    if (m4 > m) { ssum *= __expf(m - m4); m = m4; }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float x = v[j];          // -inf past the end: contributes exp(-inf) = 0
      ssum += __expf(x - m);
      float score = x * inv_t;
      if (!greedy) {
        const uint32_t r = hash32((uint32_t)(i + j), k0, k1);
        const float u = ((float)(r >> 8) + 0.5f) * (1.0f / 16777216.0f);  // (0,1)
        // Gumbel noise -ln(-ln u) with two fast log2 (ln x = log2 x * ln 2)
        score -= 0.6931471805599453f * __log2f(-0.6931471805599453f * __log2f(u));
      }
      if (score > best) { best = score; best_i = i + j; }
    }
  }
  // block reduction
  __shared__ float sm_m[SAMPLE_THREADS / 32], sm_s[SAMPLE_THREADS / 32], sm_b[SAMPLE_THREADS / 32];
  __shared__ int sm_i[SAMPLE_THREADS / 32];
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float m2 = __shfl_xor_sync(0xffffffffu, m, o);
    const float s2 = __shfl_xor_sync(0xffffffffu, ssum, o);
    const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
    const int i2 = __shfl_xor_sync(0xffffffffu, best_i, o);
    const float mn = fmaxf(m, m2);
    ssum = (mn == -INFINITY) ? 0.f : ssum * __expf(m - mn) + s2 * __expf(m2 - mn);
    m = mn;
    if (b2 > best || (b2 == best && i2 < best_i)) { best = b2; best_i = i2; }
  }
  if (lane == 0) { sm_m[wid] = m; sm_s[wid] = ssum; sm_b[wid] = best; sm_i[wid] = best_i; }
  __syncthreads();
  if (wid == 0) {
    constexpr int NW = SAMPLE_THREADS / 32;
    m = lane < NW ? sm_m[lane] : -INFINITY;
    ssum = lane < NW ? sm_s[lane] : 0.f;
    best = lane < NW ? sm_b[lane] : -INFINITY;
    best_i = lane < NW ? sm_i[lane] : 0x7fffffff;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float m2 = __shfl_xor_sync(0xffffffffu, m, o);
      const float s2 = __shfl_xor_sync(0xffffffffu, ssum, o);
      const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
      const int i2 = __shfl_xor_sync(0xffffffffu, best_i, o);
      const float mn = fmaxf(m, m2);
      ssum = (mn == -INFINITY) ? 0.f : ssum * __expf(m - mn) + s2 * __expf(m2 - mn);
      m = mn;
      if (b2 > best || (b2 == best && i2 < best_i)) { best = b2; best_i = i2; }
    }
    if (lane == 0) {
      if (splits > 1) {
        partials[(long long)row * splits + blockIdx.x] = make_float4(m, ssum, best, __int_as_float(best_i));
        __threadfence();
        const int tk = atomicAdd(&tickets[row], 1);
        if (tk != splits - 1) return;
        tickets[row] = 0;           // ready for the next launch
        __threadfence();
        m = -INFINITY; ssum = 0.f; best = -INFINITY; best_i = 0x7fffffff;
        for (int c = 0; c < splits; ++c) {   // chunk order: the sums do not depend on which CTA finished last
          const float4 r = __ldcg(&partials[(long long)row * splits + c]);
          const int i2 = __float_as_int(r.w);
          const float mn = fmaxf(m, r.x);
          ssum = (mn == -INFINITY) ? 0.f : ssum * __expf(m - mn) + r.y * __expf(r.x - mn);
          m = mn;
          if (r.z > best || (r.z == best && i2 < best_i)) { best = r.z; best_i = i2; }
        }
      }
      if (best_i >= V) best_i = 0;
      out_tokens[row] = best_i;
      out_logprobs[row] = lr[best_i] - (m + __logf(ssum));
    }
  }
}

// Per-token log-probability of given tokens from fp32 logits (teacher forcing / verification).
__global__ void __launch_bounds__(SAMPLE_THREADS)
token_logprob_kernel(const float* __restrict__ logits, long long ld, int V, const int* __restrict__ tokens,
                     float* __restrict__ out_logprobs) {
  const int row = blockIdx.x;
  const float* lr = logits + (long long)row * ld;
  float m = -INFINITY, ssum = 0.f;
  for (int i = threadIdx.x; i < V; i += SAMPLE_THREADS) {
    const float x = lr[i];
    if (x > m) { ssum = ssum * __expf(m - x) + 1.f; m = x; } else { ssum += __expf(x - m); }
  }
  __shared__ float sm_m[SAMPLE_THREADS / 32], sm_s[SAMPLE_THREADS / 32];
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float m2 = __shfl_xor_sync(0xffffffffu, m, o);
    const float s2 = __shfl_xor_sync(0xffffffffu, ssum, o);
    const float mn = fmaxf(m, m2);
    ssum = (mn == -INFINITY) ? 0.f : ssum * __expf(m - mn) + s2 * __expf(m2 - mn);
    m = mn;
  }
  if (lane == 0) { sm_m[wid] = m; sm_s[wid] = ssum; }
  __syncthreads();
  if (wid == 0) {
    constexpr int NW = SAMPLE_THREADS / 32;
    m = lane < NW ? sm_m[lane] : -INFINITY;
    ssum = lane < NW ? sm_s[lane] : 0.f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float m2 = __shfl_xor_sync(0xffffffffu, m, o);
      const float s2 = __shfl_xor_sync(0xffffffffu, ssum, o);
      const float mn = fmaxf(m, m2);
      ssum = (mn == -INFINITY) ? 0.f : ssum * __expf(m - mn) + s2 * __expf(m2 - mn);
      m = mn;
    }
    if (lane == 0) {
      int tok = tokens[row];
      if (tok < 0 || tok >= V) tok = 0;
      out_logprobs[row] = lr[tok] - (m + __logf(ssum));
    }
  }
}

// bf16 2-D transpose (used by the training path when an operand must change majorness).
__global__ void transpose_bf16_kernel(const __nv_bfloat16* __restrict__ in, __nv_bfloat16* __restrict__ out,
                                      int rows, int cols) {
  __shared__ __nv_bfloat16 tile[32][33];
  int x = blockIdx.x * 32 + threadIdx.x;
  int y0 = blockIdx.y * 32;
  for (int j = threadIdx.y; j < 32; j += blockDim.y) {
    int y = y0 + j;
    if (x < cols && y < rows) tile[j][threadIdx.x] = in[(long long)y * cols + x];
  }
  __syncthreads();
  int ox = blockIdx.y * 32 + threadIdx.x;
  int oy0 = blockIdx.x * 32;
  for (int j = threadIdx.y; j < 32; j += blockDim.y) {
    int oy = oy0 + j;
    if (ox < rows && oy < cols) out[(long long)oy * rows + ox] = tile[threadIdx.x][j];
  }
}

}  // namespace rb

using namespace rb;

#define RB_CHECK_LAUNCH() (cudaGetLastError() == cudaSuccess ? 0 : -11)

extern "C" void rb_ops_set_pdl(int on) { rb::pdl_enabled() = on != 0; }

extern "C" int rb_rmsnorm(const void* x, const void* w, void* y, long long rows, int d, long long ldx,
                          long long ldy, float eps, cudaStream_t stream) {
  if (d % 8 != 0 || rows <= 0) return -1;
  const int warps = rows >= 148 * 8 * 4 ? 8 : 2;   // few rows: spread them over more SMs
  const long long grid = (rows + warps - 1) / warps;
  return launch_kernel(rmsnorm_kernel, dim3((unsigned)grid), dim3(warps * 32), 0, stream, (const __nv_bfloat16*)x,
                       (const __nv_bfloat16*)w, (__nv_bfloat16*)y, rows, d, ldx, ldy, eps) == cudaSuccess ? 0 : -11;
}

extern "C" int rb_rope_kv_append(const void* qkv, void* q_out, void* k_cache, void* v_cache,
                                 const int* positions, const int* slots, const void* cos_sin,
                                 const void* q_norm_w, const void* k_norm_w, float norm_eps, int T, int Hq,
                                 int Hkv, int D, int block_size, long long num_slots, int max_pos,
                                 int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  const long long warps_total = (long long)T * (Hq + 2 * Hkv);
  const int warps = 8;
  const unsigned grid = (unsigned)((warps_total + warps - 1) / warps);
#define LAUNCH_ROPE(DD)                                                                              \
  launch_kernel(rope_kv_append_kernel<DD>, dim3(grid), dim3(warps * 32), 0, stream,                   \
      (const __nv_bfloat16*)qkv, (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, \
      positions, slots, (const float2*)cos_sin, (const __nv_bfloat16*)q_norm_w,                       \
      (const __nv_bfloat16*)k_norm_w, norm_eps, T, Hq, Hkv, block_size, num_slots, max_pos, status)
  cudaError_t e;
  if (D == 64) { e = LAUNCH_ROPE(64); }
  else if (D == 128) { e = LAUNCH_ROPE(128); }
  else return -1;
#undef LAUNCH_ROPE
  return e == cudaSuccess ? 0 : -11;
}

static int swiglu_launch(const void* gu, void* out, long long T, int F, const int* rows_dev, cudaStream_t stream) {
  if (F % 8 != 0 || T <= 0) return -1;
  const long long nvec = T * (F / 8);
  long long grid = (nvec + 255) / 256;
  if (grid > 148 * 16) grid = 148 * 16;
  return launch_kernel(swiglu_kernel, dim3((unsigned)grid), dim3(256), 0, stream, (const __nv_bfloat16*)gu,
                       (__nv_bfloat16*)out, T, F, rows_dev) == cudaSuccess ? 0 : -11;
}
extern "C" int rb_swiglu(const void* gu, void* out, long long T, int F, cudaStream_t stream) {
  return swiglu_launch(gu, out, T, F, nullptr, stream);
}
// At most T rows, and no more than *rows_dev (read on the device when the kernel runs).
extern "C" int rb_swiglu_bounded(const void* gu, void* out, long long T, int F, const int* rows_dev, cudaStream_t stream) {
  return swiglu_launch(gu, out, T, F, rows_dev, stream);
}

extern "C" int rb_swiglu_bwd(const void* gu, const void* dout, void* dgu, long long T, int F,
                             cudaStream_t stream) {
  if (F % 8 != 0 || T <= 0) return -1;
  const long long n = T * (F / 8);
  long long grid = (n + 255) / 256;
  if (grid > 148 * 32) grid = 148 * 32;
  swiglu_bwd_kernel<<<(unsigned)grid, 256, 0, stream>>>((const __nv_bfloat16*)gu, (const __nv_bfloat16*)dout,
                                                       (__nv_bfloat16*)dgu, T, F);
  return RB_CHECK_LAUNCH();
}

extern "C" int rb_embedding(const int* ids, const void* table, void* out, int T, int d, int vocab,
                            int* status, cudaStream_t stream) {
  if (d % 8 != 0 || T <= 0) return -1;
  return launch_kernel(embedding_kernel, dim3(T), dim3(128), 0, stream, ids, (const __nv_bfloat16*)table,
                       (__nv_bfloat16*)out, T, d, vocab, status) == cudaSuccess ? 0 : -11;
}

extern "C" int rb_sample_logprob(const float* logits, long long ld, int B, int V, const float* temperature,
                                 const unsigned long long* seeds, const unsigned long long* step_ptr,
                                 unsigned long long step_add, int* out_tokens, float* out_logprobs,
                                 cudaStream_t stream) {
  if (B <= 0) return 0;
  return launch_kernel(sample_logprob_kernel, dim3(1, B), dim3(SAMPLE_THREADS), 0, stream, logits, ld, V, temperature,
                       seeds, step_ptr, step_add, out_tokens, out_logprobs, (float4*)nullptr, (int*)nullptr) == cudaSuccess ? 0 : -11;
}
// Same with every row's vocabulary cut into `splits` chunks (grid splits x B). `partials` holds B * splits float4
// records, `tickets` B zero-initialised counters (they reset themselves). splits <= 0 picks about four CTAs per SM.
extern "C" int rb_sample_logprob_split(const float* logits, long long ld, int B, int V, const float* temperature,
                                       const unsigned long long* seeds, const unsigned long long* step_ptr,
                                       unsigned long long step_add, int* out_tokens, float* out_logprobs, void* partials,
                                       int* tickets, int splits, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (splits <= 0) splits = (4 * 148 + B - 1) / B;
  if (splits > 8) splits = 8;
  while (splits > 1 && V / splits < 4096) --splits;
  if (splits > 1 && (partials == nullptr || tickets == nullptr)) return -1;
  return launch_kernel(sample_logprob_kernel, dim3(splits, B), dim3(SAMPLE_THREADS), 0, stream, logits, ld, V, temperature,
                       seeds, step_ptr, step_add, out_tokens, out_logprobs, (float4*)partials, tickets) == cudaSuccess ? 0 : -11;
}

extern "C" int rb_token_logprob(const float* logits, long long ld, int B, int V, const int* tokens,
                                float* out_logprobs, cudaStream_t stream) {
  if (B <= 0) return 0;
  token_logprob_kernel<<<B, SAMPLE_THREADS, 0, stream>>>(logits, ld, V, tokens, out_logprobs);
  return RB_CHECK_LAUNCH();
}

extern "C" int rb_transpose_bf16(const void* in, void* out, int rows, int cols, cudaStream_t stream) {
  dim3 grid((cols + 31) / 32, (rows + 31) / 32);
  dim3 block(32, 8);
  transpose_bf16_kernel<<<grid, block, 0, stream>>>((const __nv_bfloat16*)in, (__nv_bfloat16*)out, rows, cols);
  return RB_CHECK_LAUNCH();
}

// dtype of the activations: 0 bf16, 1 fp32
#define RB_ACT_DISPATCH(dtype, CALL)            \
  if ((dtype) == 0) { using TA = __nv_bfloat16; CALL } \
  else if ((dtype) == 1) { using TA = float; CALL }    \
  else return -1;

extern "C" int rb_stream_embed(const int* ids, const void* table, long long ldt, float* x, long long ldx, void* a, long long lda, void* b,
                               long long ldb, int dtype, int T, int d, int vocab, int* status, cudaStream_t stream) {
  if (T <= 0 || d <= 0) return -1;
  cudaError_t e;
  RB_ACT_DISPATCH(dtype, e = launch_kernel(stream_embed_kernel<TA>, dim3(T), dim3(256), 0, stream, ids, (const TA*)table, ldt, x, ldx, (TA*)a,
                                           lda, (TA*)b, ldb, d, vocab, status);)
  return e == cudaSuccess ? 0 : -11;
}

extern "C" int rb_stream_norm(float* x, long long ldx, const float* y1, const float* y2, long long ldy, const void* e, const float* w,
                              long long lde, int k, const float* side, long long ld_side, const float* side_weight, float mult, void* copy,
                              long long ldc, void* h, long long ldh, const float* weight, const int* rows, int num_src_rows, int dtype, int n, int d,
                              int dp, float eps, int* status, cudaStream_t stream) {
  const bool update = y1 != nullptr || y2 != nullptr || e != nullptr || side != nullptr;
  if (n <= 0 || d <= 0 || dp < d || dp % 4 != 0 || dp > 12288 || (rows != nullptr && update) || (ldx | ldy | lde | ldc | ldh | ld_side) % 4 != 0) return -1;
  const StreamNormParams p{x, ldx, y1, y2, ldy, e, w, lde, k, copy, ldc, h, ldh, weight, side, ld_side, side_weight, rows, num_src_rows, d, dp, eps, mult,
                           status};
  const int threads = dp <= 512 ? 128 : 256;
  cudaError_t err;
  RB_ACT_DISPATCH(dtype, err = launch_kernel(stream_norm_kernel<TA>, dim3(n), dim3(threads), (size_t)dp * 4, stream, p);)
  return err == cudaSuccess ? 0 : -11;
}

struct SandwichArgs {            // mirrored by ops/elementwise.py
  float* x; const float* y; const float* y2; const float* w; const float* w2; const float* gate; const void* e; const float* p; const int* idx;
  const void* pass; const float* post_weight; const float* post_bias; const float* post_alpha; const float* pre_weight; const float* pre_bias;
  const float* pre_alpha; void* copy; void* h; const int* rows; int* status;
  long long ldx, ldy, ld_gate, lde, ld_pass, ldc, ldh;
  int k, experts, num_src_rows, n, d, dp, bounded, dtype;
  float pair_scale, eps;
};

extern "C" int rb_stream_sandwich(const SandwichArgs* a, cudaStream_t stream) {
  const bool update = a->y != nullptr || a->e != nullptr;
  if (a->n <= 0 || a->d <= 0 || a->dp < a->d || a->dp % 4 != 0 || a->dp > 12288 || (a->rows != nullptr && update)) return -1;
  if ((a->ldx | a->ldy | a->lde | a->ld_pass | a->ldc | a->ldh) % 4 != 0 || (a->y2 != nullptr && (a->y == nullptr || a->e != nullptr || a->gate != nullptr))) return -1;
  if ((a->e != nullptr && (a->p == nullptr || a->idx == nullptr || a->pass == nullptr)) || (update && a->post_weight == nullptr) ||
      (a->h != nullptr && a->pre_weight == nullptr))
    return -1;
  if (a->bounded && ((update && (a->post_bias == nullptr || a->post_alpha == nullptr)) || (a->h != nullptr && (a->pre_bias == nullptr || a->pre_alpha == nullptr)))) return -1;
  const SandwichParams p{a->x, a->ldx, a->y, a->y2, a->ldy, a->w, a->w2, a->pair_scale, a->gate, a->ld_gate, a->e, a->lde, a->p, a->idx, a->k, a->experts,
                         a->pass, a->ld_pass, {a->post_weight, a->post_bias, a->post_alpha}, {a->pre_weight, a->pre_bias, a->pre_alpha}, a->copy, a->ldc,
                         a->h, a->ldh, a->rows, a->num_src_rows, a->d, a->dp, a->eps, a->status};
  const int threads = a->dp <= 512 ? 128 : 256;
  const size_t smem = a->bounded ? 0 : (size_t)a->dp * 4;
  cudaError_t err;
  RB_ACT_DISPATCH(a->dtype, err = a->bounded ? launch_kernel(stream_sandwich_kernel<TA, true>, dim3(a->n), dim3(threads), smem, stream, p)
                                             : launch_kernel(stream_sandwich_kernel<TA, false>, dim3(a->n), dim3(threads), smem, stream, p);)
  return err == cudaSuccess ? 0 : -11;
}

// z [T, ldz] with np columns, n of them in use -> out [T, ldo].
extern "C" int rb_poly_norm(const void* z, long long ldz, const float* act, void* out, long long ldo, int T, int n, int np, float eps, int dtype,
                            cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n <= 0 || np < n || np % 4 != 0 || ldz % 4 != 0 || ldo % 4 != 0) return -1;
  const int threads = np <= 512 ? 128 : 256;
  cudaError_t err;
  RB_ACT_DISPATCH(dtype, err = launch_kernel(poly_norm_kernel<TA>, dim3(T), dim3(threads), 0, stream, (const TA*)z, ldz, act, (TA*)out, ldo, n, np, eps);)
  return err == cudaSuccess ? 0 : -11;
}

extern "C" int rb_token_side(const float* z, long long ldz, const int* ids, const void* table, long long ldt, int col0, void* a, long long lda, int n,
                             int T, int vocab, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || n <= 0) return -1;
  long long grid = ((long long)T * n + 255) / 256;
  if (grid > 148 * 16) grid = 148 * 16;
  cudaError_t err;
  RB_ACT_DISPATCH(dtype, err = launch_kernel(token_side_kernel<TA>, dim3((unsigned)grid), dim3(256), 0, stream, z, ldz, ids, (const TA*)table, ldt,
                                             col0, (TA*)a, lda, n, T, vocab, status);)
  return err == cudaSuccess ? 0 : -11;
}

extern "C" int rb_layernorm(const float* y, long long ldy, float* x, long long ldx, const int* rows, const float* w, const float* b, void* out,
                            long long ldo, int dtype, int n, int d, float eps, int num_src_rows, int* status, cudaStream_t stream) {
  if (n <= 0 || d <= 0 || d > 12288 || ldo < d || (y != nullptr && rows != nullptr)) return -1;
  const int threads = d <= 512 ? 128 : 256;
  cudaError_t e;
  RB_ACT_DISPATCH(dtype, e = launch_kernel(layernorm_kernel<TA>, dim3(n), dim3(threads), (size_t)d * 4, stream, y, ldy, x, ldx, rows, w, b,
                                           (TA*)out, ldo, d, eps, num_src_rows, status);)
  return e == cudaSuccess ? 0 : -11;
}

extern "C" int rb_clamped_glu(const void* gu, void* out, int dtype, long long T, int F, float limit, cudaStream_t stream) {
  if (T <= 0 || F <= 0) return -1;
  long long grid = (T * F + 255) / 256;
  if (grid > 148 * 16) grid = 148 * 16;
  cudaError_t e;
  RB_ACT_DISPATCH(dtype, e = launch_kernel(clamped_glu_kernel<TA>, dim3((unsigned)grid), dim3(256), 0, stream, (const TA*)gu, (TA*)out,
                                           T, F, limit);)
  return e == cudaSuccess ? 0 : -11;
}

extern "C" int rb_softcap(float* x, long long n, float cap, cudaStream_t stream) {
  if (n <= 0 || !(cap > 0.f)) return -1;
  long long grid = (n + 255) / 256;
  if (grid > 148 * 16) grid = 148 * 16;
  return launch_kernel(softcap_kernel, dim3((unsigned)grid), dim3(256), 0, stream, x, n, cap) == cudaSuccess ? 0 : -11;
}
