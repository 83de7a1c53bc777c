// The recurrence of decay_walk.cuh over many tokens of a sequence, chunk by chunk of 64 tokens instead of token by token.
// Inside a chunk (tokens 0 .. n-1, state S before it, g_t the sum of the decays' logarithms up to and with token t):
//
//   o_t = e^(g_t) S^T q_t + sum_(s <= t) e^(g_t - g_s) (q_t . k_s) v_s
//   S  <- e^(g_(n-1)) S + sum_s e^(g_(n-1) - g_s) k_s v_s^T
//
// so that a chunk is three small matrix products on the FP32 pipes and the chain over a sequence has one link a chunk.
// Every exponent is at most zero: nothing grows, whatever the decays are.  The sums of logarithms are double
// (a step that forgets everything makes them large, and their differences must not lose the small steps beside it); all
// other arithmetic is float.  The result differs from the
// walk's by the order of the sums (rounding), and so does the result of a sequence that is cut at other places.
//
//   scores : raw[n][key head][s] = q_n . k_(chunk start + s), a CTA per (chunk, key head): heads that share keys share it.
//   chunks : a CTA owns (sequence, head, tile of DVT value columns), holds its part of S in shared memory and goes through
//            the sequence's chunks; the next chunk's rows come in by cp.async while one is worked on.  The inner dimension of
//            [q | scores] x [S ; v] is cut into slices, one for every DVT threads, whose sums are added through shared memory
//            (in slice order); the product of keys and values is cut over even and odd tokens.
//
// What bounds such products is shared memory, not the FP32 pipes: a thread's register tile is 8 x 8 (8 x 4 or 4 x 4 in the
// second product), read as 16-byte words whose rows lie 4 words apart modulo the banks.
#pragma once
#include "decay_walk.cuh"

namespace kvf {

constexpr int CH = 64;        // tokens a chunk
constexpr int CH_LD = CH + 4;  // row length of the scores in shared memory

__device__ __forceinline__ void cp_async16(float* dst, const float* src, bool valid) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  const int sz = valid ? 16 : 0;  // 0: the 16 bytes are filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src), "r"(sz));
}

// two floats in one 64-bit register pair, and one instruction for both multiply-adds
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t both(float a) {
  pair_t r;
  asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(a));
  return r;
}
__device__ __forceinline__ void fma_pair(pair_t& acc, pair_t a, pair_t b) { asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(acc) : "l"(a), "l"(b)); }
__device__ __forceinline__ pair_t mul_pair(pair_t a, pair_t b) {
  pair_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ float2 floats_of(pair_t a) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(a));
  return f;
}
struct alignas(16) Quad {
  pair_t lo, hi;
};
__device__ __forceinline__ Quad load_quad(const float* p) { return *reinterpret_cast<const Quad*>(p); }

// Which chunk of which sequence is number `idx` of the step: sequences in order, each with ceil(rows / CH) chunks.
// False when the step has fewer.
__device__ __forceinline__ bool find_chunk(const int* __restrict__ qsl, int B, int idx, int& first, int& rows) {
  const int lane = threadIdx.x & 31;
  int before = 0;
  for (int b0 = 0; b0 < B; b0 += 32) {
    const int b = b0 + lane;
    const int lo = b < B ? qsl[b] : 0, len = b < B ? qsl[b + 1] - lo : 0;
    int n = len > 0 ? (len + CH - 1) / CH : 0;
    int incl = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += up;
    }
    const int mine = idx - before - (incl - n);  // my sequence's chunk, if it is mine
    const unsigned hit = __ballot_sync(0xffffffffu, mine >= 0 && mine < n);
    if (hit) {
      const int src = __ffs(hit) - 1;
      const int c = __shfl_sync(0xffffffffu, mine, src);
      first = __shfl_sync(0xffffffffu, lo, src) + c * CH;
      rows = min(CH, __shfl_sync(0xffffffffu, len, src) - c * CH);
      return true;
    }
    before += __shfl_sync(0xffffffffu, incl, 31);
  }
  return false;
}

static __global__ void __launch_bounds__(256) chunk_scores_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                                                            const int* __restrict__ qsl, int B, int key_heads, int dk,
                                                            float* __restrict__ raw) {
  pdl_launch();
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  int first, rows;
  if (!find_chunk(qsl, B, blockIdx.x, first, rows)) return;
  const int kh = blockIdx.y, ld = dk + 4;
  float* Q = sm;
  float* K = sm + CH * ld;
  const int per = dk >> 2;
  for (int idx = threadIdx.x; idx < CH * per; idx += blockDim.x) {
    const int t = idx / per, j = (idx - t * per) << 2;
    const size_t g = ((size_t)(first + (t < rows ? t : 0)) * key_heads + kh) * dk + j;
    cp_async16(Q + t * ld + j, qn + g, t < rows);
    cp_async16(K + t * ld + j, kn + g, t < rows);
  }
  asm volatile("cp.async.commit_group;\n" ::);
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const int sg = threadIdx.x & 15, tg = threadIdx.x >> 4;  // 16 x 16 threads; rows tg + 16 i, columns sg + 16 j
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k = 0; k < dk; k += 4) {
    float4 q4[4], k4[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      q4[i] = *reinterpret_cast<const float4*>(Q + (tg + 16 * i) * ld + k);
      k4[i] = *reinterpret_cast<const float4*>(K + (sg + 16 * i) * ld + k);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        acc[i][j] = fmaf(q4[i].w, k4[j].w, fmaf(q4[i].z, k4[j].z, fmaf(q4[i].y, k4[j].y, fmaf(q4[i].x, k4[j].x, acc[i][j]))));
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = tg + 16 * i;
    if (t >= rows) continue;
    float* dst = raw + ((size_t)(first + t) * key_heads + kh) * CH;
#pragma unroll
    for (int j = 0; j < 4; ++j) dst[sg + 16 * j] = acc[i][j];
  }
}

// floats of a stage (q, scores, k, v, logarithms of a chunk), and how many of the slices' sums fit where q and the scores lie
template <int DVT> __host__ __device__ constexpr int stage_floats(int dk) { return 2 * CH * (dk + 4) + CH * CH_LD + CH * DVT + CH; }
template <int DVT> __host__ __device__ constexpr int slices_in_stage(int dk) {
  const int fit = (CH * (dk + 4) + CH * CH_LD) / (CH * DVT), all = 256 / DVT;
  return fit < all ? fit : all;
}

// log_decay: float [H], or with TOK [N][H]: the logarithm of the decay of a (token and) head, finite and at most zero.
template <int DVT, bool TOK>
__global__ void __launch_bounds__(256) decay_chunks_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                                                                const float* __restrict__ vn, const float* __restrict__ raw,
                                                                const float* __restrict__ log_decay, float* __restrict__ state,
                                                                long long state_stride, float* __restrict__ out, long long out_stride,
                                                                const int* __restrict__ qsl, const int* __restrict__ state_slots, int H,
                                                                int heads_per_key, int dk, int dv) {
  pdl_launch();
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  constexpr int NT = 256, CG = DVT / 4, NS = NT / DVT;  // NS slices of the inner dimension, DVT threads each
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * DVT;
  const int q_begin = qsl[b], q_len = qsl[b + 1] - q_begin;
  const int slot = state_slots[b];
  if (q_len <= 0 || slot < 0) return;
  const int tid = threadIdx.x, ld = dk + 4;
  const int kh = h / heads_per_key, key_heads = H / heads_per_key;
  float* S = sm;                          // [dk][DVT]
  float* part = S + dk * DVT;             // the slices' sums that do not fit where q and the scores were
  double* gs = reinterpret_cast<double*>(part + (NS - slices_in_stage<DVT>(dk)) * CH * DVT);  // [CH] g_t
  float* es = reinterpret_cast<float*>(gs + CH);  // [CH] e^(g_t)
  float* ws = es + CH;                    // [CH] e^(g_(n-1) - g_t)
  float* stages = ws + CH;
  const int stage = stage_floats<DVT>(dk);  // q, scores, k, v, logarithms

  float* sbase = state + (size_t)slot * state_stride + (size_t)h * dk * dv + c0;
  for (int idx = tid; idx < dk * CG; idx += NT) {
    const int r = idx / CG, c = (idx - r * CG) << 2;
    *reinterpret_cast<float4*>(S + r * DVT + c) = c0 + c < dv ? *reinterpret_cast<const float4*>(sbase + (size_t)r * dv + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  auto issue = [&](int c) {
    float* Q = stages + (c & 1) * stage;
    float* P = Q + CH * ld;
    float* K = P + CH * CH_LD;
    float* V = K + CH * ld;
    float* L = V + CH * DVT;
    const int t0 = c * CH, n = min(CH, q_len - t0), n4 = (n + 3) & ~3, per = dk >> 2;
    const size_t row0 = (size_t)(q_begin + t0) * key_heads + kh;
    for (int t = tid >> 5; t < n; t += NT / 32) {  // a warp a row
      const float* qr = qn + (row0 + (size_t)t * key_heads) * dk;
      const float* kr = kn + (row0 + (size_t)t * key_heads) * dk;
      for (int j = tid & 31; j < per; j += 32) {
        cp_async16(Q + t * ld + 4 * j, qr + 4 * j, true);
        cp_async16(K + t * ld + 4 * j, kr + 4 * j, true);
      }
    }
    for (int t = tid >> 4; t < n; t += NT / 16) {  // half a warp a row; nothing after the row's own token is used
      const int j = tid & 15;
      if (4 * j <= t) cp_async16(P + t * CH_LD + 4 * j, raw + (row0 + (size_t)t * key_heads) * CH + 4 * j, true);
    }
    for (int idx = tid; idx < n4 * CG; idx += NT) {  // rows past the last token, up to a multiple of four, are zeros
      const int t = idx / CG, j = (idx - t * CG) << 2;
      const bool ok = t < n && c0 + j < dv;
      cp_async16(V + t * DVT + j, vn + (ok ? ((size_t)(q_begin + t0 + t) * H + h) * dv + c0 + j : 0), ok);
    }
    if (TOK)
      for (int t = tid; t < n; t += NT) cp_async(L + t, log_decay + (size_t)(q_begin + t0 + t) * H + h, false);
  };

  const int chunks = (q_len + CH - 1) / CH;
  // first product: slice `sl` of the inner dimension, columns 8 cg .. + 7 of tokens tg + 8 i
  const int sl = tid / DVT, u = tid % DVT, cg = u % (DVT / 8), tg = u / (DVT / 8);
  // second product: rows r .. of S and four columns, every other token
  constexpr int KR = DVT / 4;
  const int late = tid >> 7, tile = tid & 127, sr = (tile / CG) * KR, sc = (tile % CG) << 2;
  auto slice_sums = [&](float* Q, int i) {
    const int fit = slices_in_stage<DVT>(dk);
    return i < fit ? Q + i * (CH * DVT) : part + (i - fit) * (CH * DVT);
  };
  issue(0);
  asm volatile("cp.async.commit_group;\n" ::);
  for (int c = 0; c < chunks; ++c) {
    if (c + 1 < chunks) issue(c + 1);
    asm volatile("cp.async.commit_group;\n" ::);
    asm volatile("cp.async.wait_group 1;\n" ::);
    __syncthreads();
    float* Q = stages + (c & 1) * stage;
    float* P = Q + CH * ld;
    const float* K = P + CH * CH_LD;
    const float* V = K + CH * ld;
    const float* L = V + CH * DVT;
    const int t0 = c * CH, n = min(CH, q_len - t0), n4 = (n + 3) & ~3;
    // ---- the sums of logarithms and their exponentials
    if (tid < 32) {
      double a, d;  // tokens 2 lane and 2 lane + 1
      const int l2 = 2 * tid;
      if (TOK) {
        a = l2 < n ? (double)L[l2] : 0.0;
        d = l2 + 1 < n ? (double)L[l2 + 1] : 0.0;
      } else {
        a = l2 < n ? (double)log_decay[h] : 0.0;
        d = l2 + 1 < n ? (double)log_decay[h] : 0.0;
      }
      double incl = a + d;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, incl, o);
        if (tid >= o) incl += up;
      }
      const double total = __shfl_sync(0xffffffffu, incl, 31), g0 = incl - d, g1 = incl;
      gs[l2] = g0;
      gs[l2 + 1] = g1;
      es[l2] = expf((float)g0);
      es[l2 + 1] = expf((float)g1);
      ws[l2] = expf((float)(total - g0));
      ws[l2 + 1] = expf((float)(total - g1));
    }
    __syncthreads();
    // ---- scores: what a later token of the chunk keeps of an earlier one, zero for the ones to come
    for (int t = tid >> 4; t < n; t += NT / 16) {
      const int s = (tid & 15) << 2;
      float4 p4 = make_float4(0.f, 0.f, 0.f, 0.f);
      if (s <= t) {
        p4 = *reinterpret_cast<float4*>(P + t * CH_LD + s);
        const double gt = gs[t];
        p4.x *= expf((float)(gt - gs[s]));
        p4.y = s + 1 <= t ? p4.y * expf((float)(gt - gs[s + 1])) : 0.f;
        p4.z = s + 2 <= t ? p4.z * expf((float)(gt - gs[s + 2])) : 0.f;
        p4.w = s + 3 <= t ? p4.w * expf((float)(gt - gs[s + 3])) : 0.f;
      }
      *reinterpret_cast<float4*>(P + t * CH_LD + s) = p4;
    }
    __syncthreads();
    // ---- o = e^g (q S) + scores v: the inner dimension dk + n4 in NS slices
    pair_t acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0ull;
    const int inner = dk + n4, size = (((inner >> 2) + NS - 1) / NS) << 2;
    const int lo = sl * size, hi = min(inner, lo + size);
    if (tg < n) {
      auto tiles = [&](const float* A, int lda, const float* B, int k0, int k1) {  // acc += A[tokens][k] B[k][columns]
#pragma unroll 1
        for (int k = k0; k < k1; k += 4) {
          float4 a4[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) a4[i] = *reinterpret_cast<const float4*>(A + (tg + 8 * i) * lda + k);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const Quad b0 = load_quad(B + (k + j) * DVT + 8 * cg), b1 = load_quad(B + (k + j) * DVT + 8 * cg + 4);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const pair_t a = both(j == 0 ? a4[i].x : j == 1 ? a4[i].y : j == 2 ? a4[i].z : a4[i].w);
              fma_pair(acc[i][0], a, b0.lo);
              fma_pair(acc[i][1], a, b0.hi);
              fma_pair(acc[i][2], a, b1.lo);
              fma_pair(acc[i][3], a, b1.hi);
            }
          }
        }
      };
      if (lo < dk) {
        tiles(Q, ld, S, lo, min(hi, dk));
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const pair_t e = both(es[tg + 8 * i]);
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = mul_pair(acc[i][j], e);
        }
      }
      if (hi > dk) tiles(P, CH_LD, V, max(lo, dk) - dk, hi - dk);
    }
    __syncthreads();  // q, the scores and S have been read: the slices' sums may lie where q and the scores were
    if (tg < n) {
      float* sums = slice_sums(Q, sl);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        *reinterpret_cast<Quad*>(sums + (tg + 8 * i) * DVT + 8 * cg) = Quad{acc[i][0], acc[i][1]};
        *reinterpret_cast<Quad*>(sums + (tg + 8 * i) * DVT + 8 * cg + 4) = Quad{acc[i][2], acc[i][3]};
      }
    }
    // ---- S <- e^(g of the last token) S + sum_t e^(..) k_t v_t^T: even tokens by the first half of the threads, odd by the second
    const float keep = es[n - 1];
    pair_t up[KR / 2][4];  // rows 2 i and 2 i + 1 of column e
#pragma unroll
    for (int i = 0; i < KR / 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) up[i][e] = 0ull;
    if (sr < dk) {
#pragma unroll 4
      for (int t = late; t < n; t += 2) {
        const float4 v4 = *reinterpret_cast<const float4*>(V + t * DVT + sc);
        const float w = ws[t];
        const pair_t v0 = both(v4.x * w), v1 = both(v4.y * w), v2 = both(v4.z * w), v3 = both(v4.w * w);
#pragma unroll
        for (int i = 0; i < KR / 4; ++i) {
          const Quad k4 = load_quad(K + t * ld + sr + 4 * i);
          fma_pair(up[2 * i][0], k4.lo, v0);
          fma_pair(up[2 * i][1], k4.lo, v1);
          fma_pair(up[2 * i][2], k4.lo, v2);
          fma_pair(up[2 * i][3], k4.lo, v3);
          fma_pair(up[2 * i + 1][0], k4.hi, v0);
          fma_pair(up[2 * i + 1][1], k4.hi, v1);
          fma_pair(up[2 * i + 1][2], k4.hi, v2);
          fma_pair(up[2 * i + 1][3], k4.hi, v3);
        }
      }
    }
    auto join = [&](float scale) {
#pragma unroll
      for (int i = 0; i < KR; i += 2) {
        if (sr + i >= dk) break;  // dk is a multiple of four
        float4* d0 = reinterpret_cast<float4*>(S + (sr + i) * DVT + sc);
        float4* d1 = reinterpret_cast<float4*>(S + (sr + i + 1) * DVT + sc);
        const float4 a4 = *d0, b4 = *d1;
        const float2 u0 = floats_of(up[i / 2][0]), u1 = floats_of(up[i / 2][1]), u2 = floats_of(up[i / 2][2]), u3 = floats_of(up[i / 2][3]);
        *d0 = make_float4(fmaf(scale, a4.x, u0.x), fmaf(scale, a4.y, u1.x), fmaf(scale, a4.z, u2.x), fmaf(scale, a4.w, u3.x));
        *d1 = make_float4(fmaf(scale, b4.x, u0.y), fmaf(scale, b4.y, u1.y), fmaf(scale, b4.z, u2.y), fmaf(scale, b4.w, u3.y));
      }
    };
    if (!late) join(keep);
    __syncthreads();
    if (late) join(1.f);
    // ---- the slices' sums become the read-out
    for (int idx = tid; idx < n * CG; idx += NT) {
      const int t = idx / CG, col = (idx % CG) << 2;
      if (c0 + col >= dv) continue;
      float4 o4 = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const float4 p4 = *reinterpret_cast<const float4*>(slice_sums(Q, i) + t * DVT + col);
        o4.x += p4.x; o4.y += p4.y; o4.z += p4.z; o4.w += p4.w;
      }
      *reinterpret_cast<float4*>(out + (size_t)(q_begin + t0 + t) * out_stride + (size_t)h * dv + c0 + col) = o4;
    }
    __syncthreads();  // the stage and S are free for what comes next
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  for (int idx = tid; idx < dk * CG; idx += NT) {
    const int r = idx / CG, c = (idx - r * CG) << 2;
    if (c0 + c < dv) *reinterpret_cast<float4*>(sbase + (size_t)r * dv + c) = *reinterpret_cast<const float4*>(S + r * DVT + c);
  }
}

template <int DVT, bool TOK>
int launch_chunks(const float* qn, const float* kn, const float* vn, const float* raw, const float* log_decay, float* state, long long state_stride,
                  float* out, long long out_stride, const int* qsl, const int* state_slots, int B, int H, int heads_per_key, int dk, int dv,
                  cudaStream_t st) {
  const size_t smem = (size_t)(dk * DVT + (256 / DVT - slices_in_stage<DVT>(dk)) * CH * DVT + 4 * CH + 2 * stage_floats<DVT>(dk)) * sizeof(float);
  auto kern = decay_chunks_kernel<DVT, TOK>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  return launch(kern, dim3((dv + DVT - 1) / DVT, H, B), dim3(256), smem, st, qn, kn, vn, raw, log_decay, state, state_stride, out, out_stride, qsl,
                state_slots, H, heads_per_key, dk, dv);
}

// Two launches.  raw: float scratch [N][H / heads_per_key][CH].  dk at most 128; dk, dv, state_stride and out_stride multiples of
// four, every pointer on a 16-byte boundary.
template <bool TOK>
int decay_chunks(const float* qn, const float* kn, const float* vn, const float* log_decay, float* raw, float* state, long long state_stride,
                 float* out, long long out_stride, const int* qsl, const int* state_slots, int B, long long N, int H, int heads_per_key, int dk,
                 int dv, cudaStream_t st) {
  if (dk > 128 || (dk & 3) || (dv & 3) || (state_stride & 3) || (out_stride & 3)) return (int)cudaErrorInvalidValue;
  const uintptr_t all = (uintptr_t)qn | (uintptr_t)kn | (uintptr_t)vn | (uintptr_t)raw | (uintptr_t)state | (uintptr_t)out;
  if (all & 15) return (int)cudaErrorInvalidValue;
  const int key_heads = H / heads_per_key;
  const size_t smem = (size_t)2 * CH * (dk + 4) * sizeof(float);
  cudaError_t e = cudaFuncSetAttribute(chunk_scores_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  int rc = launch(chunk_scores_kernel, dim3((unsigned)(N / CH + B), key_heads), dim3(256), smem, st, qn, kn, qsl, B, key_heads, dk, raw);
  if (rc) return rc;
  // a CTA fills an SM and takes about as long with narrow tiles as with wide ones: narrow only if all run at once
  if (dv > 16 && (long long)B * H * ((dv + 15) / 16) > 148)
    return launch_chunks<32, TOK>(qn, kn, vn, raw, log_decay, state, state_stride, out, out_stride, qsl, state_slots, B, H, heads_per_key, dk, dv, st);
  return launch_chunks<16, TOK>(qn, kn, vn, raw, log_decay, state, state_stride, out, out_stride, qsl, state_slots, B, H, heads_per_key, dk, dv, st);
}

}  // namespace kvf
