// A matrix memory with exponential gates (the mLSTM of "xLSTM: Extended Long Short-Term Memory", Beck et al.) around the walk
// of decay_walk.cuh.  Per head, with log gates  i_t = cap tanh(zi_t / cap)  and  f_t = logsigmoid(cap tanh(zf_t / cap)):
//
//   m_t = max(f_t + m_(t-1), i_t)                                          (running maximum, zero before the first token)
//   S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T        (S: [dk][dv])
//   n_t = e^(f_t + m_(t-1) - m_t) n_(t-1) + e^(i_t - m_t) k_t
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
//
// n is one more column of S: the column whose value is always one.  So the state of a head is [dk][dvx] floats, dvx = dv
// columns of S, then n, then columns of zeros up to a multiple of four, and the walk's read-out of column dv is n . q.  The running
// maxima of the heads follow the heads' matrices in the slot: [H][dk][dvx] | m [H].
//
//   gates   : per (sequence, head) the log gates and the running maximum, token by token; leaves per token and head
//             the decay (or its logarithm), the inflow e^(i - m) and the floor e^(-m)
//   prepare : q times its scale, k, and v times the inflow, widened to float
//   step    : both for steps that bring one token a sequence, one launch
//   walk    : decay_walk with one decay a token and head, or for many tokens decay_chunks (every logarithm of a decay is at
//             most zero: m_t is at least f_t + m_(t-1))
//   read    : the division, every head over its root mean square, the weight, act(gate)
//
// Everything is float whatever the storage type T of projections and results; the gates' logits come as floats.
#include "decay_chunks.cuh"

using namespace kvf;

namespace {

constexpr float READ_EPS = 1e-6f;  // joins the divisor of the read-out
constexpr int GATE_CHUNK = 512;    // tokens a CTA of the gates kernel takes at a time, at most

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

struct GateParams {
  const float* z;          // logits [N][*]: input gates from column 0, forget gates from column f_off
  long long ldz;
  int nsplit;              // the logits are the sum of so many slices (slice order), split_stride apart
  long long split_stride;
  int f_off;
  const float* ib;         // [H]
  const float* fb;         // [H]
  float cap;
  float* m;                // running maximum of head h of slot s: m[s * state_stride + h]
  long long state_stride;
  const int* qsl;
  const int* slots;
  int H, log_form;
  float* decay;            // [N][H]
  float* inflow;           // [N][H]
  float* floor_;           // [N][H]
};

// (log input gate, log forget gate) of token n and head h
__device__ __forceinline__ void log_gates(const GateParams& p, long long n, int h, float& li, float& lf) {
  float zi = 0.f, zf = 0.f;
#pragma unroll 8
  for (int s = 0; s < p.nsplit; ++s) {
    const float* row = p.z + (size_t)s * p.split_stride + n * p.ldz;
    zi += row[h];
    zf += row[p.f_off + h];
  }
  li = p.cap * tanhf((zi + p.ib[h]) / p.cap);
  const float y = p.cap * tanhf((zf + p.fb[h]) / p.cap);
  lf = fminf(y, 0.f) - log1pf(expf(-fabsf(y)));
}

__device__ __forceinline__ void leave_gates(const GateParams& p, long long n, int h, float li, float lf, float before, float m) {
  const float l = (lf + before) - m;
  p.decay[n * p.H + h] = p.log_form ? l : expf(l);
  p.inflow[n * p.H + h] = expf(li - m);
  p.floor_[n * p.H + h] = expf(-m);
}

// A CTA per (head, sequence).  The maximum is carried by one thread, token by token, so it is the same bits however the
// sequence is cut into steps; while it goes through one stretch of tokens the other warps work out the next stretch's log gates and
// write the stretch before's results.
__global__ void __launch_bounds__(GATE_CHUNK + 32) memory_gates_kernel(const GateParams p) {
  pdl_launch();
  pdl_wait();
  __shared__ __align__(16) float fs[3][GATE_CHUNK], is[3][GATE_CHUNK], ms[3][GATE_CHUNK + 4];  // ms[.][3]: the maximum before the stretch
  const int h = blockIdx.x, b = blockIdx.y, chunk = blockDim.x - 32, t = threadIdx.x;
  const int begin = p.qsl[b], len = p.qsl[b + 1] - begin, slot = p.slots[b];
  if (len <= 0 || slot < 0) return;
  float* mem = p.m + (size_t)slot * p.state_stride + h;
  const int chunks = (len + chunk - 1) / chunk;
  float m = t == chunk ? *mem : 0.f;
  for (int it = 0; it < chunks + 2; ++it) {
    if (t < chunk) {
      if (it < chunks && it * chunk + t < len) {
        float li, lf;
        log_gates(p, begin + it * chunk + t, h, li, lf);
        fs[it % 3][t] = lf;
        is[it % 3][t] = li;
      }
      const int done = it - 2;
      if (done >= 0 && done * chunk + t < len) {
        const float* mm = ms[done % 3] + 3;
        leave_gates(p, begin + done * chunk + t, h, is[done % 3][t], fs[done % 3][t], mm[t], mm[t + 1]);
      }
    } else if (t == chunk && it >= 1 && it <= chunks) {
      const int c = it - 1, n = min(chunk, len - c * chunk);
      const float *f = fs[c % 3], *i = is[c % 3];
      float* mm = ms[c % 3] + 3;
      mm[0] = m;
      int j = 0;
      // Rounding is monotone: max(a, b) + f, rounded, is the larger of a + f and b + f, rounded.  So what eight tokens make of the inputs among
      // them is worked out beside the chain, which is eight additions and one maximum for eight tokens, with the same bits.
      for (; j + 8 <= n; j += 8) {
        float fj[8], c[8], a[8];
        *reinterpret_cast<float4*>(fj) = *reinterpret_cast<const float4*>(f + j);
        *reinterpret_cast<float4*>(fj + 4) = *reinterpret_cast<const float4*>(f + j + 4);
        *reinterpret_cast<float4*>(c) = *reinterpret_cast<const float4*>(i + j);
        *reinterpret_cast<float4*>(c + 4) = *reinterpret_cast<const float4*>(i + j + 4);
#pragma unroll
        for (int e = 1; e < 8; ++e) c[e] = fmaxf(fj[e] + c[e - 1], c[e]);
#pragma unroll
        for (int e = 0; e < 8; ++e) a[e] = fj[e] + (e ? a[e - 1] : m);
#pragma unroll
        for (int e = 0; e < 8; ++e) a[e] = fmaxf(a[e], c[e]);
        m = a[7];
        *reinterpret_cast<float4*>(mm + 1 + j) = *reinterpret_cast<const float4*>(a);
        *reinterpret_cast<float4*>(mm + 5 + j) = *reinterpret_cast<const float4*>(a + 4);
      }
      for (; j < n; ++j) mm[j + 1] = m = fmaxf(f[j] + m, i[j]);
    }
    __syncthreads();
  }
  if (t == chunk) *mem = m;
}

struct PrepareParams {
  const void* x;  // projections: q heads from q_off, k heads from k_off, v heads from v_off
  long long ldx;
  int q_off, k_off, v_off;
  float q_scale;
  int dk, dv, dvx;
  float* qn;      // [N][H * dk]
  float* kn;      // [N][H * dk]
  float* vn;      // [N][H * dvx]
};

// The numbers of heads h0 .. h1 - 1 of a token widened to float; `in`: their inflow.
template <typename T, int V>
__device__ __forceinline__ void widen(const PrepareParams& p, long long n, int H, int h0, int h1, const float* in) {
  const T* row = (const T*)p.x + n * p.ldx;
  const int qk = H * p.dk, part = (h1 - h0) * p.dk, all = 2 * part + (h1 - h0) * p.dvx;
  for (int u0 = threadIdx.x * V; u0 < all; u0 += blockDim.x * V) {
    float f[V];
    // the place among all q, then all k, then all v columns
    const int c = u0 < part ? h0 * p.dk + u0 : u0 < 2 * part ? qk + h0 * p.dk + (u0 - part) : 2 * qk + h0 * p.dvx + (u0 - 2 * part);
    if (c < qk) {
      Run<T, V>::load(row + p.q_off + c, f);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= p.q_scale;
      Run<float, V>::store(p.qn + n * qk + c, f);
    } else if (c < 2 * qk) {
      Run<T, V>::load(row + p.k_off + (c - qk), f);
      Run<float, V>::store(p.kn + n * qk + (c - qk), f);
    } else {
      const int u = c - 2 * qk, h = u / p.dvx, j = u - h * p.dvx;
      const float g = in[h - h0];
      if (j < p.dv) {
        Run<T, V>::load(row + p.v_off + h * p.dv + j, f);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] *= g;
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] = j + e == p.dv ? g : 0.f;
      }
      Run<float, V>::store(p.vn + n * H * p.dvx + u, f);
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) memory_prepare_kernel(const PrepareParams p, int H, const float* __restrict__ inflow) {
  pdl_launch();
  pdl_wait();
  widen<T, V>(p, blockIdx.x, H, 0, H, inflow + (size_t)blockIdx.x * H);
}

// Gates and widening of a step in which no sequence brings more than one token: a CTA per sequence and STEP_HEADS heads.
constexpr int STEP_HEADS = 4;
template <typename T, int V>
__global__ void __launch_bounds__(256) memory_step_kernel(const PrepareParams p, const GateParams g) {
  pdl_launch();
  __shared__ float in[STEP_HEADS];
  pdl_wait();
  const int b = blockIdx.x, n = g.qsl[b], slot = g.slots[b];
  if (g.qsl[b + 1] - n != 1 || slot < 0) return;
  const int h0 = blockIdx.y * STEP_HEADS, h1 = min(g.H, h0 + STEP_HEADS);
  for (int h = h0 + threadIdx.x; h < h1; h += blockDim.x) {
    float* mem = g.m + (size_t)slot * g.state_stride + h;
    float li, lf;
    log_gates(g, n, h, li, lf);
    const float before = *mem, m = fmaxf(lf + before, li);
    leave_gates(g, n, h, li, lf, before, m);
    in[h - h0] = expf(li - m);
    *mem = m;
  }
  __syncthreads();
  widen<T, V>(p, n, g.H, h0, h1, in);
}

// A warp per (token, head).  out = y / sqrt(mean(y^2) + eps) * w * sigmoid(gate) (without a gate: * 1), y the read-out over its divisor.
// NIT: how many times 32 * V numbers a lane keeps in registers (a head has at most NIT * 32 * V).
__device__ __forceinline__ float logistic(float z, bool exact) { return exact ? 1.f / (1.f + expf(-z)) : __fdividef(1.f, 1.f + __expf(-z)); }

template <typename T, int V, int NIT>
__global__ void __launch_bounds__(128) memory_read_kernel(const float* __restrict__ o, long long ldo, const float* __restrict__ floor_,
                                                           const T* __restrict__ gate, long long ldg, const float* __restrict__ w, float eps,
                                                           long long pairs, int H, int dv, int dvx, T* __restrict__ out, long long ldout) {
  pdl_launch();
  pdl_wait();
  constexpr bool EXACT = sizeof(T) == 4;  // float storage: the library's exponential; bfloat16: the fast one, rounded right after
  const long long pair = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (pair >= pairs) return;
  const int lane = threadIdx.x & 31;
  const long long n = pair / H;
  const int h = (int)(pair - n * H);
  const float* row = o + n * ldo + (size_t)h * dvx;
  const T* g = gate ? gate + n * ldg + (size_t)h * dv : nullptr;
  float f[NIT][V], z[NIT][V], wv[NIT][V];  // everything is asked for before the first number is used
#pragma unroll
  for (int it = 0; it < NIT; ++it) {
    const int j = (it * 32 + lane) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) f[it][e] = z[it][e] = wv[it][e] = 0.f;
    if (j >= dv) continue;
    Run<float, V>::load(row + j, f[it]);
    Run<float, V>::load(w + (size_t)h * dv + j, wv[it]);
    if (g) Run<T, V>::load(g + j, z[it]);
  }
  const float one_over = 1.f / (fmaxf(fabsf(row[dv]), floor_[pair]) + READ_EPS);
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < NIT; ++it)
#pragma unroll
    for (int e = 0; e < V; ++e) {
      f[it][e] *= one_over;
      ss = fmaf(f[it][e], f[it][e], ss);
    }
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
  T* dst = out + n * ldout + (size_t)h * dv;
#pragma unroll
  for (int it = 0; it < NIT; ++it) {
    const int j = (it * 32 + lane) * V;
    if (j >= dv) continue;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      f[it][e] = f[it][e] * r * wv[it][e];
      if (g) f[it][e] *= logistic(z[it][e], EXACT);
    }
    Run<T, V>::store(dst + j, f[it]);
  }
}

constexpr int READ_MAX = 1024;  // numbers of a head's value

template <typename T>
auto memory_read(bool vec, int dv) {
  if (vec) return dv <= 128 ? memory_read_kernel<T, 4, 1> : dv <= 256 ? memory_read_kernel<T, 4, 2> : memory_read_kernel<T, 4, READ_MAX / 128>;
  return dv <= 64 ? memory_read_kernel<T, 1, 2> : memory_read_kernel<T, 1, READ_MAX / 32>;
}

inline bool aligned(const void* p, size_t n) { return p == nullptr || ((uintptr_t)p % n) == 0; }

template <typename T>
int memory_run(const GateParams& g0, const PrepareParams& p, float* state, float* out, long long ldo, int B, long long N, int max_q_len,
               float* raw, cudaStream_t st) {
  GateParams g = g0;
  g.log_form = raw ? 1 : 0;
  const int H = g.H;
  const bool vec = p.dk % 4 == 0 && p.dv % 4 == 0 && p.ldx % 4 == 0 && (p.q_off | p.k_off | p.v_off) % 4 == 0 && aligned(p.x, 4 * sizeof(T)) &&
                   aligned(p.qn, 16) && aligned(p.kn, 16) && aligned(p.vn, 16);
  int rc;
  if (max_q_len == 1) {
    rc = launch(vec ? memory_step_kernel<T, 4> : memory_step_kernel<T, 1>, dim3(B, (H + STEP_HEADS - 1) / STEP_HEADS), dim3(256), 0, st, p, g);
    if (rc) return rc;
  } else {
    rc = launch(memory_gates_kernel, dim3(H, B), dim3((max_q_len > 0 && max_q_len <= 128 ? 128 : GATE_CHUNK) + 32), 0, st, g);
    if (rc) return rc;
    rc = launch(vec ? memory_prepare_kernel<T, 4> : memory_prepare_kernel<T, 1>, dim3((unsigned)N), dim3(256), 0, st, p, H, (const float*)g.inflow);
    if (rc) return rc;
  }
  if (raw)
    return decay_chunks<true>(p.qn, p.kn, p.vn, g.decay, raw, state, g.state_stride, out, ldo, g.qsl, g.slots, B, N, H, 1, p.dk, p.dvx, st);
  return decay_walk<true>(p.qn, p.kn, p.vn, g.decay, state, g.state_stride, out, ldo, g.qsl, g.slots, B, H, 1, p.dk, p.dvx, max_q_len, st);
}

}  // namespace

// Columns of a head's state for values of dv numbers: dv of S, one of n, zeros up to a multiple of four.
KVF_API int kvf_memory_columns(int dv) { return (dv + 4) & ~3; }

// x: rows of the projections (q heads from q_off, k heads from k_off: H of dk each; v heads from v_off: H of dv).  z: float rows of the gates'
// logits, nsplit slices.  state: float, slot i at state + i * state_stride: [H][dk][dvx] | m [H], dvx = kvf_memory_columns(dv).
// out: float [N][H * dvx] (row stride ldo), undivided, n . q in column dv of a head; floor_ [N][H]: e^(-m).  Scratch: decay and inflow
// [N][H], qn and kn [N][H * dk], vn [N][H * dvx], and for the chunked form raw [N][H][64] (else null).  max_q_len: the most rows a sequence
// of the step brings (0: unknown).  Two launches when it is one, three otherwise, four in the chunked form.
#define KVF_MEMORY_API(SUF, T)                                                                                          \
  KVF_API int kvf_matrix_memory_##SUF(const void* x, long long ldx, int q_off, int k_off, int v_off, float q_scale,     \
                                      const float* z, long long ldz, int nsplit, long long split_stride, int f_off,     \
                                      const float* ib, const float* fb, float cap, float* state,                        \
                                      long long state_stride, float* out, long long ldo, const int* qsl,                \
                                      const int* state_slots, int B, long long N, int H, int dk, int dv, float* decay,  \
                                      float* inflow, float* floor_, float* qn, float* kn, float* vn, int max_q_len,     \
                                      float* raw, cudaStream_t st) {                                                    \
    if (B <= 0 || N <= 0) return 0;                                                                                     \
    if (H <= 0 || dk <= 0 || dk > 512 || dv <= 0 || nsplit <= 0 || f_off < H || !(cap > 0.f) || (unsigned)B > 65535u || \
        (unsigned)H > 8192u || N > 0x7fffffffLL)                                                                        \
      return (int)cudaErrorInvalidValue;                                                                                \
    PrepareParams p;                                                                                                    \
    p.x = x; p.ldx = ldx; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.q_scale = q_scale; p.dk = dk; p.dv = dv; \
    p.dvx = kvf_memory_columns(dv); p.qn = qn; p.kn = kn; p.vn = vn;                                                    \
    GateParams g;                                                                                                       \
    g.z = z; g.ldz = ldz; g.nsplit = nsplit; g.split_stride = split_stride; g.f_off = f_off; g.ib = ib; g.fb = fb;      \
    g.cap = cap; g.m = state + (size_t)H * dk * p.dvx; g.state_stride = state_stride; g.qsl = qsl;                      \
    g.slots = state_slots; g.H = H; g.decay = decay; g.inflow = inflow; g.floor_ = floor_;                              \
    return memory_run<T>(g, p, state, out, ldo, B, N, max_q_len, raw, st);                                              \
  }                                                                                                                     \
  KVF_API int kvf_memory_read_##SUF(const float* o, long long ldo, const float* floor_, const void* gate,               \
                                    long long ldg, const float* w, float eps, long long N, int H, int dv, void* out,    \
                                    long long ldout, cudaStream_t st) {                                                 \
    const long long pairs = N * H;                                                                                      \
    if (pairs <= 0) return 0;                                                                                           \
    if (dv <= 0 || dv > READ_MAX || !w || !floor_) return (int)cudaErrorInvalidValue;                                   \
    const bool vec = dv % 4 == 0 && ldo % 4 == 0 && ldg % 4 == 0 && ldout % 4 == 0 && aligned(o, 16) && aligned(w, 16) && \
                     aligned(gate, 4 * sizeof(T)) && aligned(out, 4 * sizeof(T));                                       \
    return launch(memory_read<T>(vec, dv), dim3((unsigned)((pairs + 3) / 4)),                                           \
                  dim3(128), 0, st, o, ldo, floor_, (const T*)gate, ldg, w, eps, pairs, H, dv, kvf_memory_columns(dv),  \
                  (T*)out, ldout);                                                                                      \
  }

KVF_MEMORY_API(f32, float)
KVF_MEMORY_API(bf16, bf16)

KVF_API int kvf_memory_set_pdl(int enabled) {
  g_pdl_enabled = enabled ? 1 : 0;
  return 0;
}
