// What token-wise operations with a short look back share: the row of a token some places earlier in its sequence comes
// from the packed batch or, in front of a portion's first row, from the sequence's history
//   hist [slots, depth, channels],  hist[slot][d - 1] = the row d places before the sequence's next token.
#pragma once
#include "common.cuh"

namespace rb {

struct History {
  const int* cu_q;         // [B + 1] rows of every sequence; null: one row each
  const int* positions;    // [T]
  const int* slots;        // [B], negative: padding
  int B, depth, num_slots;
};

// Sequence of packed row t.
__device__ __forceinline__ int sequence_of(const int* cu_q, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

struct RowPlace {
  int offset;              // rows of the same portion in front of this one
  int position, slot;
};

__device__ __forceinline__ RowPlace row_place(const History& h, int t, int* status) {
  const int b = h.cu_q == nullptr ? t : sequence_of(h.cu_q, h.B, t);
  RowPlace r;
  r.offset = h.cu_q == nullptr ? 0 : t - h.cu_q[b];
  r.position = h.positions[t];
  r.slot = h.slots[b];
  if (r.slot >= h.num_slots) { set_status(status, ST_BAD_INDEX); r.slot = -1; }
  return r;
}

// The row d >= 1 places before row t, or null when there is none.
template <typename T>
__device__ __forceinline__ const T* row_before(const RowPlace& r, int d, const T* rows, long long ld, int t, const T* hist, int depth, int channels) {
  if (r.offset >= d) return rows + (long long)(t - d) * ld;
  const int back = d - r.offset;                                   // places before the portion
  if (r.slot < 0 || r.position < d || back > depth) return nullptr;
  return hist + ((long long)r.slot * depth + back - 1) * channels;
}

// Moves the histories of a packed batch on, after its rows have been used. grid (B, x), 8 channels per thread.
template <typename T>
__global__ void history_update_kernel(const T* __restrict__ rows, long long ld, const History h, T* __restrict__ hist, int channels) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, slot = h.slots[b], c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (slot < 0 || slot >= h.num_slots || c >= channels) return;
  const int t1 = h.cu_q[b + 1], n = t1 - h.cu_q[b];
  if (n <= 0) return;
  constexpr int V = 8 * sizeof(T) / 16;
  T* mine = hist + (long long)slot * h.depth * channels + c;
  for (int d = h.depth; d >= 1; --d) {                             // far ones first: they move out of the way
    const T* src = d <= n ? rows + (long long)(t1 - d) * ld + c : mine + (long long)(d - 1 - n) * channels;
#pragma unroll
    for (int i = 0; i < V; ++i)
      reinterpret_cast<uint4*>(mine + (long long)(d - 1) * channels)[i] = reinterpret_cast<const uint4*>(src)[i];
  }
}

template <typename T>
inline cudaError_t launch_history_update(const T* rows, long long ld, const History& h, T* hist, int channels, cudaStream_t stream) {
  return launch_kernel(history_update_kernel<T>, dim3(h.B, (channels / 8 + 127) / 128), dim3(128), 0, stream, rows, ld, h, hist, channels);
}

}  // namespace rb
