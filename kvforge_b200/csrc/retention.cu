// Retention: linear attention with one fixed decay a head, no softmax and no denominator.
//
//   S_t = a_h S_(t-1) + k_t v_t^T        (S: [dk][dv] floats per head, in the request's state slot)
//   o_t = S_t^T q_t
//
// q, k and v may pass silu first.  q and k turn with the position on their first `rot` dims (pairs (i, i + rot/2), or (2i, 2i+1)); k is then
// multiplied by k_scale.  Everything from the rotation on is float whatever the storage type T of the projections.
//
//   prepare : a warp per (token, head of q, k or v): rotation, scaling, widening to float.  Nothing here depends
//             on the state, so it runs over all tokens at once.
//   walk    : csrc/decay_walk.cuh, or for many tokens csrc/decay_chunks.cuh.
//   gate    : every head's read-out divided by its root mean square and multiplied by act(gate).
#include "decay_chunks.cuh"

using namespace kvf;

namespace {

// what a projected number becomes before anything else: act 0 itself, 1 silu
__device__ __forceinline__ float entry(float z, int act) { return act ? z / (1.f + expf(-z)) : z; }

template <typename T>
__global__ void __launch_bounds__(128) retention_prepare_kernel(const T* __restrict__ x, long long x_stride, int q_off, int k_off,
                                                                 int v_off, const int* __restrict__ positions,
                                                                 const float* __restrict__ inv_freq, int rot, int split_pairs,
                                                                 float k_scale, int act, long long n_tokens, int H, int dk, int dv,
                                                                 float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ vn) {
  pdl_launch();
  pdl_wait();
  const long long unit = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (unit >= n_tokens * 3 * H) return;
  const long long n = unit / (3 * H);
  const int u = (int)(unit - n * 3 * H), kind = u / H, h = u - kind * H;
  const int lane = threadIdx.x & 31;
  const T* row = x + (size_t)n * x_stride;
  if (kind == 2) {
    const T* src = row + v_off + (size_t)h * dv;
    float* dst = vn + ((size_t)n * H + h) * dv;
    for (int j = lane; j < dv; j += 32) dst[j] = entry(to_float<T>(src[j]), act);
    return;
  }
  const T* src = row + (kind == 0 ? q_off : k_off) + (size_t)h * dk;
  float* dst = (kind == 0 ? qn : kn) + ((size_t)n * H + h) * dk;
  const float mul = kind == 0 ? 1.f : k_scale;
  const float pos = (float)positions[n];
  for (int i = lane; i < dk / 2; i += 32) {
    const bool turns = 2 * i < rot;
    const int ia = (turns && split_pairs) ? i : 2 * i, ib = (turns && split_pairs) ? i + rot / 2 : 2 * i + 1;
    float a = entry(to_float<T>(src[ia]), act), b = entry(to_float<T>(src[ib]), act);
    if (turns) {
      float sn, cs;
      sincosf(pos * inv_freq[i], &sn, &cs);
      float ya, yb;
      rotate_pair(a, b, cs, sn, ya, yb);
      a = ya;
      b = yb;
    }
    dst[ia] = a * mul;
    dst[ib] = b * mul;
  }
  if ((dk & 1) && lane == 0) dst[dk - 1] = entry(to_float<T>(src[dk - 1]), act) * mul;
}

// What follows the walk: every head's read-out divided by its root mean square (no weight) and multiplied by
// act(gate), a warp per (token, head).  act: 0 none, 1 silu, 2 the logistic function; float arithmetic, one rounding.
template <typename T>
__global__ void __launch_bounds__(128) retention_gate_kernel(const float* __restrict__ o, long long o_stride, const T* __restrict__ gate,
                                                              long long gate_stride, float eps, int act, long long pairs, int H, int dv,
                                                              T* __restrict__ out, long long out_stride) {
  pdl_launch();
  pdl_wait();
  const long long pair = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (pair >= pairs) return;
  const int lane = threadIdx.x & 31;
  const long long n = pair / H;
  const int h = (int)(pair - n * H);
  const float* row = o + (size_t)n * o_stride + (size_t)h * dv;
  float ss = 0.f;
  for (int j = lane; j < dv; j += 32) ss = fmaf(row[j], row[j], ss);
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)dv + eps);
  const T* g = gate ? gate + (size_t)n * gate_stride + (size_t)h * dv : nullptr;
  T* dst = out + (size_t)n * out_stride + (size_t)h * dv;
  for (int j = lane; j < dv; j += 32) {
    float y = row[j] * inv;
    if (act) {
      const float z = to_float<T>(g[j]), sg = 1.f / (1.f + expf(-z));
      y *= act == 1 ? z * sg : sg;
    }
    dst[j] = from_float<T>(y);
  }
}

}  // namespace

// x: rows of the projections (q heads from q_off, k heads from k_off, v heads from v_off; H heads each of dk, dk, dv).
// qn, kn [N][H*dk] and vn [N][H*dv]: float scratch.  state: float, slot i at state + i * state_stride, [H][dk][dv].
// out: float [N][H*dv] (row stride out_stride).  decay: float [H].  max_q_len: the most rows a sequence of the step brings
// (0: unknown); a step of single tokens stages one token, not sixteen.  With `raw` (float scratch [N][H][64]) and log_decay
// (float [H]) the chunked form runs.  Two launches, three in the chunked form.
#define KVF_RETENTION_API(SUF, T)                                                                                       \
  KVF_API int kvf_retention_##SUF(const void* x, long long x_stride, int q_off, int k_off, int v_off,                   \
                                  const int* positions, const float* inv_freq, int rot, int split_pairs,                \
                                  float k_scale, int act, const float* decay, float* state, long long state_stride, float* out,  \
                                  long long out_stride, const int* qsl, const int* state_slots, int B, long long N,     \
                                  int H, int dk, int dv, float* qn, float* kn, float* vn, int max_q_len,                \
                                  const float* log_decay, float* raw,                                                   \
                                  cudaStream_t st) {                                                                    \
    if (B <= 0 || N <= 0) return 0;                                                                                     \
    if (H <= 0 || dk <= 0 || dk > 512 || dv <= 0 || rot < 0 || rot > dk || (rot & 1) || (unsigned)B > 65535u ||         \
        (unsigned)H > 65535u)                                                                                           \
      return (int)cudaErrorInvalidValue;                                                                                \
    const long long units = N * 3 * H;                                                                                  \
    int rc = launch(retention_prepare_kernel<T>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, st, (const T*)x,      \
                    x_stride, q_off, k_off, v_off, positions, inv_freq, rot, split_pairs, k_scale, act, N, H, dk, dv, qn,    \
                    kn, vn);                                                                                            \
    if (rc) return rc;                                                                                                  \
    if (raw)                                                                                                            \
      return decay_chunks<false>(qn, kn, vn, log_decay, raw, state, state_stride, out, out_stride, qsl, state_slots, B, \
                                 N, H, 1, dk, dv, st);                                                                  \
    return decay_walk<false>(qn, kn, vn, decay, state, state_stride, out, out_stride, qsl, state_slots, B, H, 1, dk, dv, \
                             max_q_len, st);                                                                            \
  }

#define KVF_RETENTION_GATE_API(SUF, T)                                                                                  \
  KVF_API int kvf_retention_gate_##SUF(const float* o, long long o_stride, const void* gate, long long gate_stride,     \
                                       float eps, int act, long long N, int H, int dv, void* out, long long out_stride, \
                                       cudaStream_t st) {                                                               \
    const long long pairs = N * H;                                                                                      \
    if (pairs <= 0) return 0;                                                                                           \
    if ((act && !gate) || act < 0 || act > 2 || dv <= 0) return (int)cudaErrorInvalidValue;                             \
    return launch(retention_gate_kernel<T>, dim3((unsigned)((pairs + 3) / 4)), dim3(128), 0, st, o, o_stride,           \
                  (const T*)gate, gate_stride, eps, act, pairs, H, dv, (T*)out, out_stride);                            \
  }

KVF_RETENTION_GATE_API(f32, float)
KVF_RETENTION_GATE_API(bf16, bf16)
KVF_RETENTION_API(f32, float)
KVF_RETENTION_API(bf16, bf16)
