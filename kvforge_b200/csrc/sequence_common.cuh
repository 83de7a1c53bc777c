// What the kernels that walk a flat batch's sequences share (conventions: a step is a flat batch; sequence b owns the
// token rows qsl[b] .. qsl[b+1]-1 and the state slot state_slots[b]; a sequence without rows, a row at or beyond qsl[B]
// and a slot below zero touch nothing).
#pragma once
#include "common.cuh"

namespace kvf {

// sequence that owns token row n (qsl ascending, qsl[0] == 0), or -1 for a padding row
__device__ __forceinline__ int seq_of_row(const int* __restrict__ qsl, int B, int n) {
  if (n >= qsl[B]) return -1;
  int lo = 0, hi = B - 1;
  while (lo < hi) {  // the last b with qsl[b] <= n
    const int mid = (lo + hi + 1) >> 1;
    if (qsl[mid] <= n) lo = mid; else hi = mid - 1;
  }
  return lo;
}

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// Activations whose result is rounded to the storage type: exact library functions for float storage; for
// bfloat16 storage the fast intrinsics (an error of a few units in the last place of a float, against a rounding
// of 2^-9 right after).  With the exact forms a convolution over 2,048 x 6,144 outputs was bound by issue slots
// (some 40 instructions an output), not by its 50 MB.
template <typename T> __device__ __forceinline__ float silu_of(float x);
template <> __device__ __forceinline__ float silu_of<float>(float x) { return silu_f(x); }
template <> __device__ __forceinline__ float silu_of<bf16>(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float sigmoid_of(float x);
template <> __device__ __forceinline__ float sigmoid_of<float>(float x) { return sigmoid_f(x); }
template <> __device__ __forceinline__ float sigmoid_of<bf16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

}  // namespace kvf
