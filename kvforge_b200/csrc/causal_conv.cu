// The short causal convolution over time per channel that mixers with a running state put between their projections
// and the recurrence.
#include "sequence_common.cuh"

using namespace kvf;

namespace {

// ---------------------------------------------------------------- short causal convolution
// y[n, c] = act( b[c] + sum_j w[j, c] * u[t - (taps-1) + j, c] ), t the place of row n in its sequence; places
// before this step's first row come from the state (the last taps-1 inputs of the sequence, oldest
// first, [taps-1][C] floats), which is zero before a sequence's start.  `bias` (b) may be null.
template <typename T, int VEC> struct VecIO;
template <> struct VecIO<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct VecIO<bf16, 8> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) { bf16x8_to_float(*reinterpret_cast<const uint4*>(p), f); }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = u;
  }
};
template <typename T> struct VecIO<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = to_float<T>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = from_float<T>(f[0]); }
};

// VEC neighbouring floats (whole 16-byte loads when VEC is a multiple of four), zeros from null
template <int VEC>
__device__ __forceinline__ void load_floats(const float* p, float* f) {
  if constexpr (VEC % 4 == 0) {
#pragma unroll
    for (int e = 0; e < VEC; e += 4) {
      const float4 v = p ? *reinterpret_cast<const float4*>(p + e) : make_float4(0.f, 0.f, 0.f, 0.f);
      f[e] = v.x; f[e + 1] = v.y; f[e + 2] = v.z; f[e + 3] = v.w;
    }
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) f[e] = p ? p[e] : 0.f;
  }
}

// A thread owns VEC neighbouring channels (one 16-byte load) of `rows` consecutive token rows; TAPS > 0: the
// taps are known at compile time and a thread keeps its weights in registers.  Each output is one chain of
// fused multiply-adds over the taps, oldest first, whichever form runs.
constexpr int CONV_ROWS = 4;  // rows of a tile when a step has many

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_kernel(const T* __restrict__ x, int x_stride, const float* __restrict__ w,
                                                          const float* __restrict__ bias,
                                                          const float* __restrict__ state, long long state_stride,
                                                          const int* __restrict__ qsl, const int* __restrict__ state_slots,
                                                          int N, int B, int C, int taps_rt, int act, T* __restrict__ out,
                                                          int out_stride, int rows) {
  pdl_launch();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= C) return;
  float cb[VEC];
  load_floats<VEC>(bias ? bias + c : nullptr, cb);
  float wr[VEC][TAPS > 0 ? TAPS : 1];
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      float t[VEC];
      load_floats<VEC>(w + (size_t)j * C + c, t);
#pragma unroll
      for (int e = 0; e < VEC; ++e) wr[e][j] = t[e];
    }
  }
  if (TAPS > 0 && rows == CONV_ROWS) {
    // all of the tile's rows in one sequence: its rows + taps - 1 inputs are loaded once, together, and every row's
    // sum slides over them
    const int n0 = blockIdx.x * CONV_ROWS;
    const int b0 = n0 < N ? seq_of_row(qsl, B, n0) : -1;
    if (b0 < 0) return;
    const int first = qsl[b0], end = qsl[b0 + 1];
    if (n0 + CONV_ROWS <= end && n0 + CONV_ROWS <= N) {
      const int slot = state_slots[b0];
      const float* st = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
      const int t0 = n0 - first;
      constexpr int NIN = CONV_ROWS + (TAPS > 0 ? TAPS : 1) - 1;
      float u[NIN][VEC];
#pragma unroll
      for (int i = 0; i < NIN; ++i) {
        const int src = t0 - (TAPS - 1) + i;
        if (src >= 0) {
          VecIO<T, VEC>::load(x + (size_t)(first + src) * x_stride + c, u[i]);
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) u[i][e] = st ? st[(size_t)(TAPS - 1 + src) * C + c + e] : 0.f;
        }
      }
#pragma unroll
      for (int rr = 0; rr < CONV_ROWS; ++rr) {
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          acc[e] = cb[e];
#pragma unroll
          for (int j = 0; j < (TAPS > 0 ? TAPS : 1); ++j) acc[e] = fmaf(wr[e][j], u[rr + j][e], acc[e]);
          if (act == 1) acc[e] = silu_of<T>(acc[e]);
        }
        VecIO<T, VEC>::store(out + (size_t)(n0 + rr) * out_stride + c, acc);
      }
      return;
    }
  }
  for (int rr = 0; rr < rows; ++rr) {
    const int n = blockIdx.x * rows + rr;
    if (n >= N) return;
    const int b = seq_of_row(qsl, B, n);
    if (b < 0) return;  // this row and all after it belong to no sequence
    const int slot = state_slots[b];
    const int first = qsl[b];
    const int t = n - first;
    const float* st = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
    float acc[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = cb[e];
#pragma unroll
    for (int j = 0; j < (TAPS > 0 ? TAPS : 64); ++j) {
      if (j >= taps) break;
      const int src = t - (taps - 1) + j;
      float u[VEC];
      if (src >= 0) {
        VecIO<T, VEC>::load(x + (size_t)(first + src) * x_stride + c, u);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = st ? st[(size_t)(taps - 1 + src) * C + c + e] : 0.f;
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = fmaf(TAPS > 0 ? wr[e][TAPS > 0 ? j : 0] : w[(size_t)j * C + c + e], u[e], acc[e]);
    }
    if (act == 1) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = silu_of<T>(acc[e]);
    }
    VecIO<T, VEC>::store(out + (size_t)n * out_stride + c, acc);
  }
}

// Steps in which no sequence brings more than CONV_FEW rows (decoding): a thread owns VEC channels of ALL rows of
// one sequence, so it reads the old state, computes the rows and writes the new state itself: one launch.
constexpr int CONV_FEW = 4;

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_few_kernel(const T* __restrict__ x, int x_stride, const float* __restrict__ w,
                                                              const float* __restrict__ bias,
                                                              float* __restrict__ state, long long state_stride,
                                                              const int* __restrict__ qsl, const int* __restrict__ state_slots,
                                                              int C, int act, T* __restrict__ out, int out_stride) {
  pdl_launch();
  pdl_wait();
  const int b = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  const int first = qsl[b], q_len = qsl[b + 1] - first;
  const int slot = state_slots[b];
  if (c >= C || q_len <= 0 || q_len > CONV_FEW) return;
  float* st = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
  float wr[VEC][TAPS], cb[VEC];
  load_floats<VEC>(bias ? bias + c : nullptr, cb);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    float t[VEC];
    load_floats<VEC>(w + (size_t)j * C + c, t);
#pragma unroll
    for (int e = 0; e < VEC; ++e) wr[e][j] = t[e];
  }
  float u[TAPS - 1 + CONV_FEW][VEC];  // the state's inputs, then this step's rows
#pragma unroll
  for (int i = 0; i < TAPS - 1; ++i)
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[i][e] = st ? st[(size_t)i * C + c + e] : 0.f;
#pragma unroll
  for (int i = 0; i < CONV_FEW; ++i) {
    if (i < q_len) VecIO<T, VEC>::load(x + (size_t)(first + i) * x_stride + c, u[TAPS - 1 + i]);
    else
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[TAPS - 1 + i][e] = 0.f;
  }
#pragma unroll
  for (int i = 0; i < CONV_FEW; ++i) {
    if (i < q_len) {
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        acc[e] = cb[e];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) acc[e] = fmaf(wr[e][j], u[i + j][e], acc[e]);
        if (act == 1) acc[e] = silu_of<T>(acc[e]);
      }
      VecIO<T, VEC>::store(out + (size_t)(first + i) * out_stride + c, acc);
    }
  }
  if (st) {  // the last TAPS-1 inputs, oldest first
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
#pragma unroll
      for (int k = 0; k < TAPS - 1 + CONV_FEW; ++k)
        if (k == q_len + i) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) st[(size_t)i * C + c + e] = u[k][e];
        }
    }
  }
}

template <typename T, int VEC>
int launch_conv_few(const T* x, int x_stride, const float* w, const float* bias, float* state, long long state_stride, const int* qsl,
                    const int* state_slots, int B, int C, int taps, int act, T* out, int out_stride, cudaStream_t st) {
  const int per_cta = 128 * VEC;
  dim3 grid(B, (C + per_cta - 1) / per_cta);
  if (grid.y > 65535u) return (int)cudaErrorInvalidValue;
  if (taps == 2) return launch(causal_conv_few_kernel<T, VEC, 2>, grid, dim3(128), 0, st, x, x_stride, w, bias, state, state_stride, qsl, state_slots, C, act, out, out_stride);
  if (taps == 3) return launch(causal_conv_few_kernel<T, VEC, 3>, grid, dim3(128), 0, st, x, x_stride, w, bias, state, state_stride, qsl, state_slots, C, act, out, out_stride);
  return launch(causal_conv_few_kernel<T, VEC, 4>, grid, dim3(128), 0, st, x, x_stride, w, bias, state, state_stride, qsl, state_slots, C, act, out, out_stride);
}

template <typename T, int VEC>
int launch_conv(const T* x, int x_stride, const float* w, const float* bias, const float* state, long long state_stride, const int* qsl,
                const int* state_slots, int N, int B, int C, int taps, int act, T* out, int out_stride, cudaStream_t st) {
  const int rows = N >= 1024 ? CONV_ROWS : 1;
  const int per_cta = 128 * VEC;
  dim3 grid((N + rows - 1) / rows, (C + per_cta - 1) / per_cta);
  if (grid.y > 65535u) return (int)cudaErrorInvalidValue;
#define KVF_CONV_CASE(TP)                                                                                             \
  launch(causal_conv_kernel<T, VEC, TP>, dim3(grid), dim3(128), (size_t)(0), st, x, x_stride, w, bias, state, state_stride, qsl, state_slots, N, B, C, \
                                                        taps, act, out, out_stride, rows)
  if (taps == 2) KVF_CONV_CASE(2);
  else if (taps == 3) KVF_CONV_CASE(3);
  else if (taps == 4) KVF_CONV_CASE(4);
  else if (taps <= 64) KVF_CONV_CASE(0);
  else return (int)cudaErrorInvalidValue;
#undef KVF_CONV_CASE
  return KVF_LAUNCH_STATUS();
}

template <typename T> struct ConvVec;
template <> struct ConvVec<float> { static constexpr int N = 4; };
template <> struct ConvVec<bf16> { static constexpr int N = 8; };

// The state after the step: the last taps-1 inputs of each sequence, old ones moved up where the
// step brought fewer rows than that.  Entry i is read at i + q_len > i before entry i is written,
// and a thread owns its channel, so the move is safe in place.
template <typename T>
__global__ void __launch_bounds__(256) conv_state_kernel(const T* __restrict__ x, int x_stride, float* __restrict__ state,
                                                         long long state_stride, const int* __restrict__ qsl,
                                                         const int* __restrict__ state_slots, int C, int taps) {
  pdl_launch();
  pdl_wait();
  const int b = blockIdx.x;
  const int first = qsl[b], q_len = qsl[b + 1] - first;
  const int slot = state_slots[b];
  if (q_len <= 0 || slot < 0) return;
  float* st = state + (size_t)slot * state_stride;
  const int keep = taps - 1;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
    for (int i = 0; i < keep; ++i) {
      const int src = q_len - keep + i;
      st[(size_t)i * C + c] = src >= 0 ? to_float<T>(x[(size_t)(first + src) * x_stride + c]) : st[(size_t)(i + q_len) * C + c];
    }
  }
}

}  // namespace

#define KVF_CONV_API(SUF, T)                                                                                          \
  KVF_API int kvf_causal_conv_##SUF(const void* x, int x_stride, const float* w, const float* bias, float* state, long long state_stride, \
                                    const int* qsl, const int* state_slots, int N, int B, int C, int taps, int act,    \
                                    void* out, int out_stride, int max_q_len, cudaStream_t st) {                       \
    if (N <= 0 || B <= 0 || C <= 0) return 0;                                                                          \
    if (taps <= 0 || (unsigned)B > 65535u) return (int)cudaErrorInvalidValue;                                          \
    constexpr int V = ConvVec<T>::N;                                                                                   \
    const bool vec = C % V == 0 && x_stride % V == 0 && out_stride % V == 0 && ((uintptr_t)x % 16) == 0 &&             \
                     ((uintptr_t)out % 16) == 0 && ((uintptr_t)w % 16) == 0 && ((uintptr_t)bias % 16) == 0;            \
    if (max_q_len > 0 && max_q_len <= CONV_FEW && taps >= 2 && taps <= 4) {                                            \
      return vec ? launch_conv_few<T, V>((const T*)x, x_stride, w, bias, state, state_stride, qsl, state_slots, B, C, taps,  \
                                         act, (T*)out, out_stride, st)                                                 \
                 : launch_conv_few<T, 1>((const T*)x, x_stride, w, bias, state, state_stride, qsl, state_slots, B, C, taps,  \
                                         act, (T*)out, out_stride, st);                                                \
    }                                                                                                                  \
    int rc = vec ? launch_conv<T, V>((const T*)x, x_stride, w, bias, state, state_stride, qsl, state_slots, N, B, C, taps,   \
                                     act, (T*)out, out_stride, st)                                                     \
                 : launch_conv<T, 1>((const T*)x, x_stride, w, bias, state, state_stride, qsl, state_slots, N, B, C, taps,   \
                                     act, (T*)out, out_stride, st);                                                    \
    int gy = (C + 255) / 256;                                                                                          \
    if (gy > 65535) gy = 65535;                                                                                        \
    if (rc || taps == 1) return rc;                                                                                    \
    launch(conv_state_kernel<T>, dim3(dim3(B, gy)), dim3(256), (size_t)(0), st, (const T*)x, x_stride, state, state_stride, qsl, state_slots,    \
                                                      C, taps);                                                        \
    return KVF_LAUNCH_STATUS();                                                                                        \
  }

KVF_CONV_API(f32, float)
KVF_CONV_API(bf16, bf16)

KVF_API int kvf_conv_set_pdl(int enabled) {
  g_pdl_enabled = enabled ? 1 : 0;
  return 0;
}
