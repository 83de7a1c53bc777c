// What lies between an attention layer's input product and its attention kernel when queries and
// keys are normed per head, or when keys and values are made from one small latent per token;
// a logistic gate per head on an attention layer's output; a row added to every row of the
// residual stream.  All arithmetic is float whatever the storage type T; each result is rounded once.
#include "common.cuh"

using namespace kvf;

namespace {

// ---------------------------------------------------------------- per-head norm, rotation, cache write
// Rows of `qkv` hold nh query heads and nkv key heads of dk and nkv value heads of dv.  A warp takes
// a head at a time.  Query and key heads: x <- x / sqrt(sum(x^2) / count + eps) * w (w of dk floats shared
// by all heads; skipped without w; count: the numbers of a head that are not padding, padded places hold zeros), then the
// first `rot` dims turn by the angle pos * inv_freq[i] and are multiplied by `magnitude`, in
// interleaved pairs (2i, 2i+1) or, with split_pairs, in pairs (i, i + rot/2) (skipped when rot == 0).
// Queries are written back in place; keys and values go to their slot of the paged cache
// ([blocks][nkv][block_size][dk] and [...][dv]); a slot below zero (padding) is skipped, one beyond the
// pool raises bit 1 of the error flag.  Values may be mixed with those that an earlier layer of the same
// step left for the same token: with v_keep the values as projected are also copied to v_keep[n][nkv*dv];
// with v_first the value becomes (1 - lambda) v + lambda v_first[n] (lambda = *v_lambda, in float, rounded
// once) before it is cached.
// A CTA takes HEAD_WARPS heads of a token at a time (all of the token's when there are many tokens), and works out the token's
// cosines and sines once.  A lane keeps its pairs in registers between the sum and the rotation.
constexpr int HEAD_WARPS = 8;
constexpr int HEAD_PAIRS = 4;  // pairs a lane holds at most: heads of up to 256

template <typename T> struct Two;
template <> struct Two<float> {
  static __device__ __forceinline__ float2 load(const float* p) { return *reinterpret_cast<const float2*>(p); }
  static __device__ __forceinline__ void store(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
};
template <> struct Two<bf16> {
  static __device__ __forceinline__ float2 load(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
  static __device__ __forceinline__ void store(bf16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }
};

// PAIRS: pairs a lane holds.  SPLIT: the pairs that turn are (i, i + rot/2).  Rows and pages begin where a pair of numbers may.
template <typename T, int PAIRS, bool SPLIT>
__global__ void __launch_bounds__(HEAD_WARPS * 32) head_norm_cache_kernel(T* __restrict__ qkv, long long row_stride,
                                                               const int* __restrict__ positions,
                                                               const float* __restrict__ q_w, const float* __restrict__ k_w,
                                                               float eps, const float* __restrict__ inv_freq, int rot,
                                                               const int* __restrict__ slots, T* __restrict__ kcache,
                                                               T* __restrict__ vcache, int nh, int nkv, int dk,
                                                               int dv, int block_size, long long num_slots,
                                                               int* __restrict__ err, T* __restrict__ v_keep,
                                                               const T* __restrict__ v_first, const float* __restrict__ v_lambda,
                                                               float count, float magnitude) {
  pdl_launch();
  extern __shared__ float turn[];  // [rot / 2] cosines, [rot / 2] sines
  pdl_wait();
  const int n = blockIdx.x, heads = nh + 2 * nkv, half = rot >> 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (rot) {
    const float pos = (float)positions[n];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      float sn, cs;
      sincosf(pos * inv_freq[i], &sn, &cs);
      turn[i] = cs * magnitude;
      turn[half + i] = sn * magnitude;
    }
    __syncthreads();
  }
  T* row = qkv + (size_t)n * row_stride;
  long long slot = slots ? slots[n] : -1;
  if (slot >= num_slots) {
    if (slots && threadIdx.x == 0 && err) atomicOr(err, 2);
    slot = -2;  // beyond the pool: nothing of this token is kept
  }
  const size_t page = slot >= 0 ? (size_t)(slot / block_size) : 0, place = slot >= 0 ? (size_t)(slot % block_size) : 0;
  for (int h = blockIdx.y * HEAD_WARPS + warp; h < heads; h += gridDim.y * HEAD_WARPS) {
    const bool is_q = h < nh, is_k = !is_q && h < nh + nkv;
    if (!is_q && !is_k) {  // a value head: copied, or mixed with an earlier layer's
      const int g = h - nh - nkv;
      const T* src = row + (size_t)(nh + nkv) * dk + (size_t)g * dv;
      if (v_keep && slot >= -1)  // a row without a slot still leaves its values for the layers after
        for (int j = lane; j < dv; j += 32) v_keep[(size_t)n * nkv * dv + (size_t)g * dv + j] = src[j];
      if (slot < 0) continue;
      T* dst = vcache + ((page * nkv + g) * block_size + place) * dv;
      if (v_first) {
        const float lam = v_lambda[0];
        const T* first = v_first + (size_t)n * nkv * dv + (size_t)g * dv;
        for (int j = lane; j < dv; j += 32) dst[j] = from_float<T>(fmaf(lam, to_float<T>(first[j]), (1.f - lam) * to_float<T>(src[j])));
      } else {
        for (int j = lane; j < dv; j += 32) dst[j] = src[j];
      }
      continue;
    }
    if (is_k && slot < 0) continue;
    T* x = row + (size_t)h * dk;  // key heads follow the query heads with the same size
    const float* w = is_q ? q_w : k_w;
    if (is_q && !w && rot == 0) continue;
    T* dst = is_q ? x : kcache + ((page * nkv + (h - nh)) * block_size + place) * dk;
    float a[PAIRS], b[PAIRS], ss = 0.f;
#pragma unroll
    for (int k = 0; k < PAIRS; ++k) {
      // pair i: dims (2i, 2i+1), or (i, i + rot/2) among the dims that turn in split pairs
      const int i = lane + 32 * k;
      a[k] = b[k] = 0.f;
      if (2 * i >= dk) continue;
      if (SPLIT && i < half) {
        a[k] = to_float<T>(x[i]);
        b[k] = to_float<T>(x[i + half]);
      } else {
        const float2 v = Two<T>::load(x + 2 * i);
        a[k] = v.x;
        b[k] = v.y;
      }
      ss = fmaf(a[k], a[k], fmaf(b[k], b[k], ss));
    }
    const float r = w ? 1.f / sqrtf(warp_sum(ss) / count + eps) : 1.f;
#pragma unroll
    for (int k = 0; k < PAIRS; ++k) {
      const int i = lane + 32 * k;
      if (2 * i >= dk) continue;
      const bool turns = i < half, split = SPLIT && turns;
      const int ia = split ? i : 2 * i, ib = split ? i + half : 2 * i + 1;
      float u = a[k], v = b[k];
      if (w) {
        u = u * r * w[ia];
        v = v * r * w[ib];
      }
      if (turns) {
        float yu, yv;
        rotate_pair(u, v, turn[i], turn[half + i], yu, yv);
        u = yu;
        v = yv;
      }
      if (split) {
        dst[ia] = from_float<T>(u);
        dst[ib] = from_float<T>(v);
      } else {
        Two<T>::store(dst + ia, u, v);
      }
    }
  }
}

template <typename T>
auto head_norm_kernel(int dk, bool split) {
  if (dk <= 64) return split ? head_norm_cache_kernel<T, 1, true> : head_norm_cache_kernel<T, 1, false>;
  if (dk <= 128) return split ? head_norm_cache_kernel<T, 2, true> : head_norm_cache_kernel<T, 2, false>;
  return split ? head_norm_cache_kernel<T, HEAD_PAIRS, true> : head_norm_cache_kernel<T, HEAD_PAIRS, false>;
}

// ---------------------------------------------------------------- RMS norm of a column range
// out[n][:] = x[n][0 .. r) / sqrt(mean(x^2) + eps) * w, a warp per row; x rows may be part of wider rows.
template <typename T>
__global__ void __launch_bounds__(128) row_rmsnorm_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ w,
                                                           float eps, long long n_rows, int r, T* __restrict__ out, long long out_stride) {
  pdl_launch();
  pdl_wait();
  const long long n = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (n >= n_rows) return;
  const int lane = threadIdx.x & 31;
  const T* row = x + (size_t)n * x_stride;
  float ss = 0.f;
  for (int j = lane; j < r; j += 32) {
    const float v = to_float<T>(row[j]);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)r + eps);
  T* dst = out + (size_t)n * out_stride;
  for (int j = lane; j < r; j += 32) dst[j] = from_float<T>(to_float<T>(row[j]) * inv * w[j]);
}

// ---------------------------------------------------------------- latent keys and values
// A row of `x` holds, from column q_off, nh query heads of dk + dr numbers (the last dr of each turn
// with the position) and, from column c_off, a latent of r numbers followed by dr numbers of a key
// part that turns and is shared by all heads.  Per token, one CTA:
//   c = latent / sqrt(mean(latent^2) + eps) * c_w  -> cache row [0, r)
//   the shared key part, turned                     -> cache row [r, r + dr)
//   every head's turning query part, turned         -> qa[n][h][r .. r + dr)
// (qa rows hold nh heads of r + dr; their first r numbers are written by whoever folds the key
// up-projection into the queries).  Pairs are interleaved (2i, 2i+1), i < rot/2, rot <= dr, or with
// split_pairs (i, i + rot/2); angles pos * inv_freq[i].  The cache is [blocks][1][block_size][r + dr].
// The query heads may lie in rows of their own (`xq`, row stride q_stride; null: in `x` from q_off).
template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(const T* __restrict__ x, long long row_stride, int q_off,
                                                              int c_off, const int* __restrict__ positions,
                                                              const float* __restrict__ c_w, float eps,
                                                              const float* __restrict__ inv_freq, int rot,
                                                              const int* __restrict__ slots, T* __restrict__ cache,
                                                              T* __restrict__ qa, int nh, int dk, int dr, int r,
                                                              int block_size, long long num_slots, int* __restrict__ err,
                                                              int split_pairs, const T* __restrict__ xq, long long q_stride) {
  pdl_launch();
  pdl_wait();
  __shared__ float red[32];
  const int n = blockIdx.x;
  const T* row = x + (size_t)n * row_stride;
  const T* qsrc = xq ? xq + (size_t)n * q_stride : row + q_off;
  const float pos = (float)positions[n];
  // queries: every head's turning part
  T* qrow = qa + (size_t)n * nh * (r + dr);
  for (int idx = threadIdx.x; idx < nh * (dr / 2); idx += blockDim.x) {
    const int h = idx / (dr / 2), i = idx - h * (dr / 2);
    const T* src = qsrc + (size_t)h * (dk + dr) + dk;
    const bool split = split_pairs && 2 * i < rot;
    const int ia = split ? i : 2 * i, ib = split ? i + rot / 2 : 2 * i + 1;
    float a = to_float<T>(src[ia]), b = to_float<T>(src[ib]);
    if (2 * i < rot) {
      float sn, cs;
      sincosf(pos * inv_freq[i], &sn, &cs);
      float ya, yb;
      rotate_pair(a, b, cs, sn, ya, yb);
      a = ya;
      b = yb;
    }
    T* dst = qrow + (size_t)h * (r + dr) + r;
    dst[ia] = from_float<T>(a);
    dst[ib] = from_float<T>(b);
  }
  const long long slot = slots ? slots[n] : -1;  // uniform over the CTA
  if (slot < 0) return;
  if (slot >= num_slots) {
    if (threadIdx.x == 0 && err) atomicOr(err, 2);
    return;
  }
  const T* lat = row + c_off;
  float ss = 0.f;
  for (int j = threadIdx.x; j < r; j += blockDim.x) {
    const float v = to_float<T>(lat[j]);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)r + eps);
  T* dst = cache + (size_t)slot * (r + dr);  // one key head: a slot is a row
  for (int j = threadIdx.x; j < r; j += blockDim.x) dst[j] = from_float<T>(to_float<T>(lat[j]) * inv * c_w[j]);
  for (int i = threadIdx.x; i < dr / 2; i += blockDim.x) {
    const bool split = split_pairs && 2 * i < rot;
    const int ia = split ? i : 2 * i, ib = split ? i + rot / 2 : 2 * i + 1;
    float a = to_float<T>(lat[r + ia]), b = to_float<T>(lat[r + ib]);
    if (2 * i < rot) {
      float sn, cs;
      sincosf(pos * inv_freq[i], &sn, &cs);
      float ya, yb;
      rotate_pair(a, b, cs, sn, ya, yb);
      a = ya;
      b = yb;
    }
    dst[r + ia] = from_float<T>(a);
    dst[r + ib] = from_float<T>(b);
  }
}

// ---------------------------------------------------------------- a logistic gate per head
// y[n][h][:] *= 1 / (1 + exp(-g[n][h])), in place; g is a column range of a wider row.
template <typename T>
__global__ void head_gate_kernel(T* __restrict__ y, const T* __restrict__ g, long long g_stride, long long total, int nh,
                                 int dv) {
  pdl_launch();
  pdl_wait();
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
    const long long nhid = idx / dv;
    const long long n = nhid / nh;
    const int h = (int)(nhid - n * nh);
    const float z = to_float<T>(g[(size_t)n * g_stride + h]);
    y[idx] = from_float<T>(to_float<T>(y[idx]) * (1.f / (1.f + expf(-z))));
  }
}

// ---------------------------------------------------------------- a row added to every row
__global__ void add_row_kernel(float* __restrict__ resid, const float* __restrict__ vec, long long total, int width) {
  pdl_launch();
  pdl_wait();
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x)
    resid[idx] += vec[idx % width];
}

inline unsigned grid_for(long long total, int threads) {
  long long g = (total + threads - 1) / threads;
  return (unsigned)(g < 1 ? 1 : (g > 148 * 16 ? 148 * 16 : g));
}

}  // namespace

#define KVF_HEAD_OPS_API(SUF, T)                                                                                     \
  KVF_API int kvf_head_norm_cache_##SUF(void* qkv, long long row_stride, const int* positions, const float* q_w,     \
                                        const float* k_w, float eps, const float* inv_freq, int rot,                 \
                                        const int* slots, void* kcache, void* vcache, int n_tokens, int nh, int nkv, \
                                        int dk, int dv, int block_size, long long num_slots, int* err,               \
                                        int split_pairs, void* v_keep, const void* v_first, const float* v_lambda,   \
                                        int count, float magnitude, cudaStream_t st) {                               \
    if (n_tokens <= 0) return 0;                                                                                     \
    if (dk <= 0 || (dk & 1) || dk > 64 * HEAD_PAIRS || rot < 0 || rot > dk || (rot & 1))                             \
      return (int)cudaErrorInvalidValue;                                                                             \
    if ((v_first && !v_lambda) || count <= 0 || count > dk) return (int)cudaErrorInvalidValue;                       \
    if ((row_stride & 1) || ((((uintptr_t)qkv) | ((uintptr_t)kcache)) & (2 * sizeof(T) - 1)))                       \
      return (int)cudaErrorInvalidValue;                                                                             \
    const int groups = (nh + 2 * nkv + HEAD_WARPS - 1) / HEAD_WARPS;                                                 \
    return launch(head_norm_kernel<T>(dk, split_pairs != 0), dim3(n_tokens, n_tokens <= 256 ? groups : 1), dim3(HEAD_WARPS * 32),    \
                  (size_t)rot * sizeof(float), st, (T*)qkv, row_stride, positions, q_w, k_w, eps, inv_freq, rot,     \
                  slots, (T*)kcache, (T*)vcache, nh, nkv, dk, dv, block_size, num_slots, err,                        \
                  (T*)v_keep, (const T*)v_first, v_lambda, (float)count, magnitude);                                 \
  }                                                                                                                  \
  KVF_API int kvf_row_rmsnorm_##SUF(const void* x, long long x_stride, const float* w, float eps, long long n_rows,  \
                                    int r, void* out, long long out_stride, cudaStream_t st) {                       \
    if (n_rows <= 0) return 0;                                                                                       \
    if (r <= 0 || !w) return (int)cudaErrorInvalidValue;                                                             \
    return launch(row_rmsnorm_kernel<T>, dim3((unsigned)((n_rows + 3) / 4)), dim3(128), 0, st, (const T*)x,          \
                  x_stride, w, eps, n_rows, r, (T*)out, out_stride);                                                 \
  }                                                                                                                  \
  KVF_API int kvf_latent_prepare_##SUF(const void* x, long long row_stride, int q_off, int c_off,                    \
                                       const int* positions, const float* c_w, float eps, const float* inv_freq,     \
                                       int rot, const int* slots, void* cache, void* qa, int n_tokens, int nh,       \
                                       int dk, int dr, int r, int block_size, long long num_slots, int* err,         \
                                       int split_pairs, const void* xq, long long q_stride, cudaStream_t st) {       \
    if (n_tokens <= 0) return 0;                                                                                     \
    if (r <= 0 || dr < 0 || (dr & 1) || rot < 0 || rot > dr || (rot & 1)) return (int)cudaErrorInvalidValue;         \
    return launch(latent_prepare_kernel<T>, dim3(n_tokens), dim3(128), 0, st, (const T*)x, row_stride, q_off,        \
                  c_off, positions, c_w, eps, inv_freq, rot, slots, (T*)cache, (T*)qa, nh, dk, dr, r, block_size,    \
                  num_slots, err, split_pairs, (const T*)xq, q_stride);                                              \
  }                                                                                                                  \
  KVF_API int kvf_head_gate_##SUF(void* y, const void* g, long long g_stride, long long n_tokens, int nh, int dv,    \
                                  cudaStream_t st) {                                                                 \
    const long long total = n_tokens * nh * dv;                                                                      \
    if (total <= 0) return 0;                                                                                        \
    return launch(head_gate_kernel<T>, dim3(grid_for(total, 256)), dim3(256), 0, st, (T*)y, (const T*)g, g_stride,   \
                  total, nh, dv);                                                                                    \
  }

KVF_HEAD_OPS_API(f32, float)
KVF_HEAD_OPS_API(bf16, bf16)

KVF_API int kvf_add_row_f32(float* resid, const float* vec, long long n_rows, int width, cudaStream_t st) {
  const long long total = n_rows * width;
  if (total <= 0) return 0;
  return launch(add_row_kernel, dim3(grid_for(total, 256)), dim3(256), 0, st, resid, vec, total, width);
}

// Turn programmatic dependent launch on or off for every launch of this library (the flag is one per
// shared library).
KVF_API int kvf_routed_set_pdl(int enabled) {
  kvf::g_pdl_enabled = enabled ? 1 : 0;
  return 0;
}
