// A state space per head whose step size follows the token (Mamba-2's recurrence), around the walk of decay_walk.cuh:
//
//   d_t = softplus(dt_t + dt_bias_h),  a_t = exp(-exp(A_log_h) d_t)
//   S_t = a_t S_(t-1) + B_t (d_t x_t)^T      (S: [N][dv] floats per head; B and C are shared by groups of heads)
//   y_t = S_t^T C_t + D_h x_t
//
//   prepare   : a CTA per token: step sizes and decays, d x, B and C as floats.  Nothing here depends on the state.
//   walk      : decay_walk with one decay a token and head, or for many tokens decay_chunks.
//   wide_norm : what follows a recurrence: the read-out (plus D x), gated before or after a norm over wide parts of the
//               row (one part, or several equal ones), times a weight.
//
// Everything is float whatever the storage type T of projections and results.
#include "decay_chunks.cuh"

using namespace kvf;

namespace {

__device__ __forceinline__ float softplus_exact(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

template <typename T, int V> struct Run;
template <typename T> struct Run<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = to_float<T>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = from_float<T>(f[0]); }
};
template <> struct Run<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct Run<bf16, 4> {
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

// x: rows of  x [H*dv] | B [G*N] | C [G*N]  after convolution and activation; dt: rows of [H] logits.
template <typename T, int V>
__global__ void __launch_bounds__(256) state_space_prepare_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ dt,
                                                                   long long lddt, const float* __restrict__ dt_bias,
                                                                   const float* __restrict__ a_log, int log_form, int H, int dv, int gn,
                                                                   float* __restrict__ decay, float* __restrict__ cn,
                                                                   float* __restrict__ bn, float* __restrict__ vn) {
  pdl_launch();
  extern __shared__ float step[];  // [H]
  pdl_wait();
  const long long n = blockIdx.x;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    const float d = softplus_exact(to_float<T>(dt[n * lddt + h]) + dt_bias[h]);
    step[h] = d;
    const float l = -expf(a_log[h]) * d;
    decay[n * H + h] = log_form ? l : expf(l);
  }
  __syncthreads();
  const T* row = x + n * ldx;
  const int inner = H * dv;
  for (int c = threadIdx.x * V; c < inner + 2 * gn; c += blockDim.x * V) {
    float f[V];
    Run<T, V>::load(row + c, f);
    if (c < inner) {
      const float d = step[c / dv];
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= d;
      Run<float, V>::store(vn + n * inner + c, f);
    } else if (c < inner + gn) {
      Run<float, V>::store(bn + n * gn + (c - inner), f);
    } else {
      Run<float, V>::store(cn + n * gn + (c - inner - gn), f);
    }
  }
}

// ---------------------------------------------------------------- wide norm and gate
// Part g of token n (C / parts numbers): u = o + skip[c / dvh] * xs[c]; with gate_first u *= act(z[c]);
// y = u / sqrt(mean(u^2) + eps) * w[c]; without gate_first y *= act(z[c]); out = mult * y, rounded once.
// act: 0 no gate, 1 silu, 2 the logistic function.  One CTA a (part, token).
struct WideNormParams {
  const float* o;
  long long ldo;
  const float* skip;  // [C / dvh] or null
  const void* xs;
  long long ldxs;
  int dvh;
  const void* z;
  long long ldz;
  int act, gate_first;
  const float* w;
  float eps, mult;
  int C, part;  // numbers in a row, in a part
  void* out;
  long long ldout;
};

__device__ __forceinline__ float gate_of(float z, int act, bool exact) {
  const float s = exact ? 1.f / (1.f + expf(-z)) : __fdividef(1.f, 1.f + __expf(-z));
  return act == 1 ? z * s : s;
}

template <typename T, int V>
__global__ void __launch_bounds__(256) wide_norm_gate_kernel(const WideNormParams p) {
  pdl_launch();
  extern __shared__ __align__(16) float u[];  // [part]
  __shared__ float red[32];
  constexpr bool EXACT = sizeof(T) == 4;  // float storage: the library's exponential; bfloat16: the fast one
  pdl_wait();
  const int parts = p.C / p.part;
  const long long n = blockIdx.x / parts;
  const int c0 = (int)(blockIdx.x - n * parts) * p.part;
  const float* o = p.o + n * p.ldo + c0;
  const T* xs = p.skip ? (const T*)p.xs + n * p.ldxs + c0 : nullptr;
  const T* z = p.act ? (const T*)p.z + n * p.ldz + c0 : nullptr;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < p.part; i += blockDim.x * V) {
    float f[V];
    Run<float, V>::load(o + i, f);
    if (xs) {
      float x[V];
      Run<T, V>::load(xs + i, x);
      const float d = p.skip[(c0 + i) / p.dvh];
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = fmaf(d, x[e], f[e]);
    }
    if (z && p.gate_first) {
      float g[V];
      Run<T, V>::load(z + i, g);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= gate_of(g[e], p.act, EXACT);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(f[e], f[e], ss);
    Run<float, V>::store(u + i, f);
  }
  ss = block_sum(ss, red);
  const float r = p.mult / sqrtf(ss / (float)p.part + p.eps);
  T* out = (T*)p.out + n * p.ldout + c0;
  for (int i = threadIdx.x * V; i < p.part; i += blockDim.x * V) {  // a thread reads what it wrote itself
    float f[V], w[V];
    Run<float, V>::load(u + i, f);
    Run<float, V>::load(p.w + c0 + i, w);
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] = f[e] * r * w[e];
    if (z && !p.gate_first) {
      float g[V];
      Run<T, V>::load(z + i, g);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= gate_of(g[e], p.act, EXACT);
    }
    Run<T, V>::store(out + i, f);
  }
}

template <typename T>
int wide_norm_gate(const WideNormParams& p, long long n_tokens, cudaStream_t st) {
  auto al = [](const void* q, size_t b) { return q == nullptr || ((uintptr_t)q % b) == 0; };
  constexpr size_t TB = 4 * sizeof(T);
  const bool vec = p.part % 4 == 0 && p.ldo % 4 == 0 && p.ldout % 4 == 0 && al(p.o, 16) && al(p.w, 16) && al(p.out, TB) &&
                   (!p.skip || (p.dvh % 4 == 0 && p.ldxs % 4 == 0 && al(p.xs, TB))) && (!p.act || (p.ldz % 4 == 0 && al(p.z, TB)));
  const size_t smem = (size_t)p.part * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  auto kern = vec ? wide_norm_gate_kernel<T, 4> : wide_norm_gate_kernel<T, 1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const long long ctas = n_tokens * (p.C / p.part);
  if (ctas > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  const int threads = p.part >= 2048 ? 256 : p.part >= 256 ? 128 : 64;
  return launch(kern, dim3((unsigned)ctas), dim3(threads), smem, st, p);
}

}  // namespace

// x: rows of  x [H*dv] | B [G*N] | C [G*N]; dt: rows of [H]; out: float [N_tokens][H*dv] (row stride out_stride), the
// read-out without the D term.  state: float, slot i at state + i * state_stride, [H][N][dv].  Scratch: decay [tokens][H],
// cn and bn [tokens][G*N], vn [tokens][H*dv], and for the chunked form raw [tokens][G][64] (else null).  Two launches,
// three in the chunked form.
#define KVF_STATE_SPACE_API(SUF, T)                                                                                     \
  KVF_API int kvf_state_space_##SUF(const void* x, long long ldx, const void* dt, long long lddt, const float* dt_bias, \
                                    const float* a_log, float* state, long long state_stride, float* out,               \
                                    long long out_stride, const int* qsl, const int* state_slots, int B,                \
                                    long long n_tokens, int H, int G, int ns, int dv, float* decay, float* cn,          \
                                    float* bn, float* vn, int max_q_len, float* raw, cudaStream_t st) {                             \
    if (B <= 0 || n_tokens <= 0) return 0;                                                                              \
    if (H <= 0 || G <= 0 || H % G || ns <= 0 || ns > 512 || dv <= 0 || (unsigned)B > 65535u || (unsigned)H > 65535u ||  \
        n_tokens > 0x7fffffffLL)                                                                                        \
      return (int)cudaErrorInvalidValue;                                                                                \
    const int gn = G * ns;                                                                                              \
    auto al = [](const void* q, size_t b) { return ((uintptr_t)q % b) == 0; };                                          \
    const bool vec = dv % 4 == 0 && gn % 4 == 0 && ldx % 4 == 0 && al(x, 4 * sizeof(T)) && al(vn, 16) && al(bn, 16) &&  \
                     al(cn, 16);                                                                                        \
    int rc = launch(vec ? state_space_prepare_kernel<T, 4> : state_space_prepare_kernel<T, 1>,                          \
                    dim3((unsigned)n_tokens), dim3(256), (size_t)H * sizeof(float), st, (const T*)x, ldx,               \
                    (const T*)dt, lddt, dt_bias, a_log, raw ? 1 : 0, H, dv, gn, decay, cn, bn, vn);                                  \
    if (rc) return rc;                                                                                                  \
    if (raw)                                                                                                            \
      return decay_chunks<true>(cn, bn, vn, decay, raw, state, state_stride, out, out_stride, qsl, state_slots, B,      \
                                n_tokens, H, H / G, ns, dv, st);                                                        \
    return decay_walk<true>(cn, bn, vn, decay, state, state_stride, out, out_stride, qsl, state_slots, B, H, H / G, ns, \
                            dv, max_q_len, st);                                                                         \
  }                                                                                                                     \
  KVF_API int kvf_wide_norm_gate_##SUF(const float* o, long long ldo, const float* skip, const void* xs, long long ldxs, \
                                       int dvh, const void* z, long long ldz, int act, int gate_first, const float* w,  \
                                       float eps, float mult, long long n_tokens, int C, int parts, void* out,          \
                                       long long ldout, cudaStream_t st) {                                              \
    if (n_tokens <= 0 || C <= 0) return 0;                                                                              \
    if (parts <= 0 || C % parts || act < 0 || act > 2 || (act && !z) || (skip && (!xs || dvh <= 0 || C % dvh)) || !w)   \
      return (int)cudaErrorInvalidValue;                                                                                \
    WideNormParams p;                                                                                                   \
    p.o = o; p.ldo = ldo; p.skip = skip; p.xs = xs; p.ldxs = ldxs; p.dvh = dvh; p.z = z; p.ldz = ldz; p.act = act;      \
    p.gate_first = gate_first; p.w = w; p.eps = eps; p.mult = mult; p.C = C; p.part = C / parts; p.out = out;           \
    p.ldout = ldout;                                                                                                    \
    return wide_norm_gate<T>(p, n_tokens, st);                                                                          \
  }

KVF_STATE_SPACE_API(f32, float)
KVF_STATE_SPACE_API(bf16, bf16)
