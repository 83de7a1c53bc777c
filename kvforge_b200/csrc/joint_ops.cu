// What lies around an attention layer whose query (and key) rows are normed as one vector before they are split into
// heads and whose result is gated before the output projection; and a learned vector per position that joins the
// residual stream after the embedding.
//
//   joint_norm_cache : biases, RMS norm over all query numbers and over all key numbers of a token, rotation, keys and values to
//                      the cache
//   output_gate      : out = mult * y * sigmoid(g), one gate a head or one a channel
//   add_position_rows: resid[n] += table[position of n]
//
// All arithmetic is float whatever the storage type T; each result is rounded once.
#include "common.cuh"

using namespace kvf;

namespace {

// V neighbouring numbers of the storage type (or of a float slice) at a time
template <typename T, int V> struct Pack;
template <typename T> struct Pack<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = to_float<T>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = from_float<T>(f[0]); }
};
template <> struct Pack<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct Pack<bf16, 4> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a);
    u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  }
};

// ---------------------------------------------------------------- joint norm of q and of k, cache write
// A row holds  q [nh*dk] | k [nkv*dk] | v [nkv*dv] | rest  (nkv == 0: no keys and values, the rest follows q).  The row
// comes from `y` (storage type) or, when `parts` is given, as the sum of nsplit float slices (slice order; row stride
// `width`).  q and k become (x + bias) / sqrt(sum x^2 / count + eps) * w  with one sum over all of q and one over all of
// k (`count`: the numbers of a head that are not padding; padded places hold zeros), without `qw` they are only
// biased; v is only biased.  Then the first `rot` numbers of every q and k head turn by the angle pos * inv_freq[i] and are
// multiplied by `magnitude`, in interleaved pairs (2i, 2i+1) or in split pairs (i, i + rot/2) (rot == 0: none do).  q goes back to `y` in place, k and v to the token's slot of the cache
// ([blocks][nkv][block_size][dk] and [...][dv]); with `parts` the rest goes to `y` as well.  A slot below zero (padding)
// writes no key and no value, one beyond the pool raises bit 1 of the error flag.  One CTA a token.
struct JointParams {
  void* y;
  long long ldy;
  const float* parts;
  int nsplit;
  long long split_stride;
  int width;
  const float* bias;  // [nh*dk + nkv*dk + nkv*dv] or null
  const float* qw;    // [nh*dk] or null
  const float* kw;    // [nkv*dk]
  float q_count, k_count, eps;
  const int* positions;
  const float* inv_freq;  // [rot / 2]
  int rot, interleaved;
  float magnitude;
  const int* slots;
  void* kcache;
  void* vcache;
  int nh, nkv, dk, dv, block_size;
  long long num_slots;
  int* err;
};

template <typename T, int V>
__global__ void __launch_bounds__(1024) joint_norm_cache_kernel(const JointParams p) {
  pdl_launch();
  extern __shared__ __align__(16) float row[];  // q and k of the token, then the cosines and sines of its angles
  __shared__ float red[64];
  const int n = blockIdx.x;
  const int q_dim = p.nh * p.dk, k_dim = p.nkv * p.dk, v_dim = p.nkv * p.dv, qk = q_dim + k_dim;
  T* y = (T*)p.y + (size_t)n * p.ldy;
  const float* pt = p.parts ? p.parts + (size_t)n * p.width : nullptr;
  pdl_wait();
  auto fetch = [&](int c, float* f) {
    if (pt) {
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = 0.f;
#pragma unroll 8
      for (int s = 0; s < p.nsplit; ++s) {
        float t[V];
        Pack<float, V>::load(pt + (size_t)s * p.split_stride + c, t);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] += t[e];
      }
    } else {
      Pack<T, V>::load(y + c, f);
    }
  };
  const int half = p.rot >> 1;
  float* cs = row + qk;
  float* sn = cs + half;
  const float pos = p.rot ? (float)p.positions[n] : 0.f;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * V; c < qk; c += blockDim.x * V) {
    float f[V];
    fetch(c, f);
    if (p.bias) {
      float b[V];
      Pack<float, V>::load(p.bias + c, b);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] += b[e];
    }
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s = fmaf(f[e], f[e], s);
    if (c < q_dim) sq += s; else sk += s;
    if (p.qw) {
      float w[V];
      Pack<float, V>::load(c < q_dim ? p.qw + c : p.kw + (c - q_dim), w);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= w[e];
    }
    Pack<float, V>::store(row + c, f);  // lacks the norm's one factor for all of q or of k
  }
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * p.inv_freq[i], &s, &c);
    cs[i] = c * p.magnitude;
    sn[i] = s * p.magnitude;
  }
  float rq = 1.f, rk = 1.f;
  if (p.qw) {
    // both sums through one pair of barriers, in a tree that depends on the sizes alone
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      red[warp] = sq;
      red[32 + warp] = sk;
    }
    __syncthreads();
    const int nw = blockDim.x >> 5;
    sq = warp_sum(lane < nw ? red[lane] : 0.f);
    sk = warp_sum(lane < nw ? red[32 + lane] : 0.f);
    rq = 1.f / sqrtf(sq / p.q_count + p.eps);
    if (k_dim) rk = 1.f / sqrtf(sk / p.k_count + p.eps);
  } else if (p.rot) {
    __syncthreads();  // a pair's numbers and its angle may be another thread's
  }
  long long slot = -1;
  if (p.nkv) {
    slot = p.slots[n];
    if (slot >= p.num_slots) {
      if (threadIdx.x == 0 && p.err) atomicOr(p.err, 2);
      slot = -1;
    }
  }
  const size_t page = slot >= 0 ? (size_t)(slot / p.block_size) : 0, place = slot >= 0 ? (size_t)(slot % p.block_size) : 0;
  for (int c = threadIdx.x * V; c < qk; c += blockDim.x * V) {  // nobody writes the row any more
    float f[V];
    Pack<float, V>::load(row + c, f);
    const bool is_q = c < q_dim;
    const float r = is_q ? rq : rk;
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] *= r;
    const int j0 = c % p.dk;  // V numbers of one head from its j0 on
    if (j0 < p.rot) {
      if (V == 4 && p.interleaved && j0 + 4 <= p.rot) {  // whole pairs
#pragma unroll
        for (int e = 0; e < V; e += 2) {
          float a, b;
          const int i = (j0 + e) >> 1;
          rotate_pair(f[e], f[(e + 1) % V], cs[i], sn[i], a, b);
          f[e] = a;
          f[(e + 1) % V] = b;
        }
      } else if (V == 4 && !p.interleaved && (half & 3) == 0 && (p.dk & 3) == 0) {  // four pairs' numbers of one side
        const bool first = j0 < half;
        const int d = first ? half : -half, i = first ? j0 : j0 - half;
        float other[V], c4[V], s4[V];
        Pack<float, V>::load(row + c + d, other);
        Pack<float, V>::load(cs + i, c4);
        Pack<float, V>::load(sn + i, s4);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          float a, b;
          other[e] *= r;
          rotate_pair(first ? f[e] : other[e], first ? other[e] : f[e], c4[e], s4[e], a, b);
          f[e] = first ? a : b;
        }
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const int j = j0 + e;
          if (j >= p.rot) continue;
          const bool first = p.interleaved ? !(j & 1) : j < half;
          const int d = p.interleaved ? (first ? 1 : -1) : (first ? half : -half);  // where the pair's other number is
          const int i = p.interleaved ? j >> 1 : (first ? j : j - half);
          const float other = row[c + e + d] * r, own = row[c + e] * r;
          float a, b;
          if (first)
            rotate_pair(own, other, cs[i], sn[i], a, b);
          else
            rotate_pair(other, own, cs[i], sn[i], a, b);
          f[e] = first ? a : b;
        }
      }
    }
    if (is_q) {
      Pack<T, V>::store(y + c, f);
    } else if (slot >= 0) {
      const int k = c - q_dim, g = k / p.dk;
      Pack<T, V>::store((T*)p.kcache + ((page * p.nkv + g) * p.block_size + place) * p.dk + (k - g * p.dk), f);
    }
  }
  if (slot >= 0) {
    for (int c = threadIdx.x * V; c < v_dim; c += blockDim.x * V) {
      float f[V];
      fetch(qk + c, f);
      if (p.bias) {
        float b[V];
        Pack<float, V>::load(p.bias + qk + c, b);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] += b[e];
      }
      const int g = c / p.dv;
      Pack<T, V>::store((T*)p.vcache + ((page * p.nkv + g) * p.block_size + place) * p.dv + (c - g * p.dv), f);
    }
  }
  if (pt) {
    for (int c = qk + v_dim + threadIdx.x * V; c < p.width; c += blockDim.x * V) {
      float f[V];
      fetch(c, f);
      Pack<T, V>::store(y + c, f);
    }
  }
}

template <typename T>
int joint_norm_cache(const JointParams& p, int n_tokens, cudaStream_t st) {
  auto al = [](const void* q, size_t b) { return q == nullptr || ((uintptr_t)q % b) == 0; };
  const bool vec = p.dk % 4 == 0 && p.dv % 4 == 0 && p.ldy % 4 == 0 && p.width % 4 == 0 && p.split_stride % 4 == 0 &&
                   al(p.y, 4 * sizeof(T)) && al(p.parts, 16) && al(p.bias, 16) && al(p.qw, 16) && al(p.kw, 16) &&
                   al(p.kcache, 4 * sizeof(T)) && al(p.vcache, 4 * sizeof(T));
  const size_t smem = ((size_t)(p.nh + p.nkv) * p.dk + p.rot) * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  auto kern = vec ? joint_norm_cache_kernel<T, 4> : joint_norm_cache_kernel<T, 1>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  // few tokens: a thread for every four numbers, so that all slices of a row are asked for at once
  const int units = p.width / (vec ? 4 : 1);
  const int threads = n_tokens > 148 || units <= 256 ? 256 : units <= 512 ? 512 : 1024;
  return launch(kern, dim3(n_tokens), dim3(threads), smem, st, p);
}

// ---------------------------------------------------------------- a logistic gate on an attention layer's result
// out[n][c] = mult * y[n][c] / (1 + exp(-g)),  g = gate[n][c], or gate[n][c / dv] with one gate a head.
template <typename T> __device__ __forceinline__ float logistic(float z);
template <> __device__ __forceinline__ float logistic<float>(float z) { return 1.f / (1.f + expf(-z)); }
// rounded to 8 bits of mantissa right after: the fast intrinsics' error of a few units in the last place does not show
template <> __device__ __forceinline__ float logistic<bf16>(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

template <typename T, int V>
__global__ void __launch_bounds__(256) output_gate_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ gate, long long ldg,
                                                           int per_head, float mult, T* __restrict__ out, long long ldo, int C, int dv) {
  pdl_launch();
  pdl_wait();
  const long long n = blockIdx.x;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * V; c < C; c += gridDim.y * blockDim.x * V) {
    float f[V], g[V];
    Pack<T, V>::load(y + n * ldy + c, f);
    if (per_head) {
      const float s = logistic<T>(to_float<T>(gate[n * ldg + c / dv]));
#pragma unroll
      for (int e = 0; e < V; ++e) g[e] = s;
    } else {
      Pack<T, V>::load(gate + n * ldg + c, g);
#pragma unroll
      for (int e = 0; e < V; ++e) g[e] = logistic<T>(g[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] *= g[e] * mult;
    Pack<T, V>::store(out + n * ldo + c, f);
  }
}

// ---------------------------------------------------------------- a learned vector per position
template <typename T>
__global__ void __launch_bounds__(256) add_position_rows_kernel(float* __restrict__ resid, const T* __restrict__ table,
                                                                 const int* __restrict__ positions, int W, int rows, int* __restrict__ err) {
  pdl_launch();
  pdl_wait();
  const int n = blockIdx.x;
  const int pos = positions[n];
  if (pos < 0 || pos >= rows) {
    if (threadIdx.x == 0 && err) atomicOr(err, 16);
    return;
  }
  float* h = resid + (size_t)n * W;
  const T* t = table + (size_t)pos * W;
  for (int i = threadIdx.x; i < W; i += blockDim.x) h[i] += to_float<T>(t[i]);
}

}  // namespace

KVF_API int kvf_joint_set_pdl(int enabled) {
  g_pdl_enabled = enabled ? 1 : 0;
  return 0;
}

#define KVF_JOINT_API(SUF, T)                                                                                           \
  KVF_API int kvf_joint_norm_cache_##SUF(void* y, long long ldy, const float* parts, int nsplit, long long split_stride, \
                                         int width, const float* bias, const float* qw, const float* kw, int q_count,   \
                                         int k_count, float eps, const int* positions, const float* inv_freq, int rot,  \
                                         int interleaved, float magnitude, const int* slots, void* kcache, void* vcache, \
                                         int n_tokens, int nh, int nkv, int dk, int dv, int block_size,                 \
                                         long long num_slots, int* err, cudaStream_t st) {                              \
    if (n_tokens <= 0) return 0;                                                                                        \
    if (nh <= 0 || nkv < 0 || dk <= 0 || dv <= 0 || (nkv && (!slots || !kcache || !vcache || block_size <= 0)) ||       \
        rot < 0 || rot > dk || (rot & 1) || (rot && (!positions || !inv_freq)) || (parts && nsplit <= 0) || (qw && (q_count <= 0 || (nkv && (!kw || k_count <= 0)))))                             \
      return (int)cudaErrorInvalidValue;                                                                                \
    JointParams p;                                                                                                      \
    p.y = y; p.ldy = ldy; p.parts = parts; p.nsplit = nsplit; p.split_stride = split_stride; p.width = width;           \
    p.bias = bias; p.qw = qw; p.kw = kw; p.q_count = (float)q_count; p.k_count = (float)k_count; p.eps = eps;           \
    p.positions = positions; p.inv_freq = inv_freq; p.rot = rot; p.interleaved = interleaved; p.magnitude = magnitude;  \
    p.slots = slots; p.kcache = kcache; p.vcache = vcache; p.nh = nh; p.nkv = nkv; p.dk = dk; p.dv = dv;                \
    p.block_size = block_size; p.num_slots = num_slots; p.err = err;                                                    \
    return joint_norm_cache<T>(p, n_tokens, st);                                                                        \
  }                                                                                                                     \
  KVF_API int kvf_output_gate_##SUF(const void* y, long long ldy, const void* gate, long long ldg, int per_head,        \
                                    float mult, void* out, long long ldo, int n_tokens, int nh, int dv,                 \
                                    cudaStream_t st) {                                                                  \
    if (n_tokens <= 0 || nh <= 0) return 0;                                                                             \
    if (dv <= 0 || !gate) return (int)cudaErrorInvalidValue;                                                            \
    const int C = nh * dv;                                                                                              \
    constexpr size_t B = 4 * sizeof(T);                                                                                 \
    const bool vec = dv % 4 == 0 && ldy % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)y % B) == 0 && ((uintptr_t)out % B) == 0 && \
                     (per_head || (ldg % 4 == 0 && ((uintptr_t)gate % B) == 0));                                        \
    const int per = 256 * (vec ? 4 : 1);                                                                                \
    dim3 grid(n_tokens, (C + per - 1) / per);                                                                           \
    if (grid.y > 65535u) grid.y = 65535u;                                                                               \
    return launch(vec ? output_gate_kernel<T, 4> : output_gate_kernel<T, 1>, grid, dim3(256), 0, st, (const T*)y, ldy,  \
                  (const T*)gate, ldg, per_head, mult, (T*)out, ldo, C, dv);                                            \
  }                                                                                                                     \
  KVF_API int kvf_add_position_rows_##SUF(float* resid, const void* table, const int* positions, int n_tokens, int W,   \
                                          int rows, int* err, cudaStream_t st) {                                        \
    if (n_tokens <= 0) return 0;                                                                                        \
    if (W <= 0 || rows <= 0) return (int)cudaErrorInvalidValue;                                                         \
    return launch(add_position_rows_kernel<T>, dim3(n_tokens), dim3(256), 0, st, resid, (const T*)table, positions, W,  \
                  rows, err);                                                                                           \
  }

KVF_JOINT_API(f32, float)
KVF_JOINT_API(bf16, bf16)
