// The walk of a recurrence whose state is a matrix a head that decays by one number a head and gains an outer product:
//
//   S_t = a_t S_(t-1) + k_t v_t^T        (S: [dk][dv] floats per head, in the request's state slot)
//   o_t = S_t^T q_t
//
// with a_t fixed per head (retention) or one number per token and head (a state space whose step size follows the token),
// and with keys and queries of a head's own or shared by groups of neighbouring heads.
//
// A CTA owns (sequence, head, tile of CT value columns) and walks the sequence's tokens in order.  A
// column's dk rows are spread over KS neighbouring lanes, R rows each in registers (in runs of four: rows
// 4 (j KS + s) .. + 3 for lane s, so that q and k come from shared memory four at a time).  Per token a
// lane makes  S <- a S + k v  and its part of  S^T q  in one pass; the parts are added in a tree whose
// shape follows dk alone.  Chunks of TC tokens come in through a cp.async double buffer; the state tile passes through
// shared memory so that global memory sees whole rows.
//
// The state after a token is the same bits however the sequence was cut into steps (the walk is token by token,
// and every sum has an order fixed by dk alone, however many rows a lane holds), so a token's output does not
// depend on the cut, the batch or the slot.  A sequence without rows, or with a slot below zero (padding), touches nothing.
#pragma once
#include "common.cuh"

namespace kvf {

constexpr int TC = 16;  // tokens per chunk of the walk, at most

__device__ __forceinline__ void cp_async(float* dst, const float* src, bool wide) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  if (wide)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src));
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(d), "l"(src));
}

// R rows a lane (a multiple of four); blockDim.x = KS * CT (a multiple of 32, at most 256); KS a power of two, at most 32.
// The sum over a column's rows has one order whatever R is: runs of four rows are added in order, and the runs are then
// added in a binary tree that joins the halves of the (padded) row range first and neighbouring runs last; a lane's own runs
// are the upper levels of that tree and the shuffles over the KS lanes the lower ones.  So R can follow the batch (few
// sequences: fewer rows a lane and more lanes) without changing a bit of the result.
template <int R, bool TOK>
__global__ void __launch_bounds__(256) decay_walk_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                                                          const float* __restrict__ vn, const float* __restrict__ decay,
                                                          float* __restrict__ state, long long state_stride,
                                                          float* __restrict__ out, long long out_stride,
                                                          const int* __restrict__ qsl, const int* __restrict__ state_slots,
                                                          int H, int heads_per_key, int dk, int dv, int KS, int CT, int tc) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  constexpr int NJ = R / 4;  // runs of four rows a lane
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * CT;
  const int q_begin = qsl[b], q_len = qsl[b + 1] - q_begin;
  const int slot = state_slots[b];
  if (q_len <= 0 || slot < 0) return;
  const int dkp = KS * R, tid = threadIdx.x, nthreads = blockDim.x;
  const int s = tid & (KS - 1), col = tid / KS;
  const int ncol = min(CT, dv - c0);
  const int lds = CT + 1;
  float* St = sm;                       // [dkp][CT + 1]: the state tile on its way in and out
  const int st_floats = (dkp * lds + 3) & ~3;
  // tc tokens a chunk (16, or as many as the step's longest sequence brings when that is fewer)
  const int tokens4 = TOK ? (tc + 3) & ~3 : 0;
  const int stage = tc * (2 * dkp + CT) + tokens4;  // q [tc][dkp], k [tc][dkp], v [tc][CT], and with TOK the decays [tc]
  float* buf = sm + st_floats;
  const float a_fixed = TOK ? 0.f : decay[h];
  const int kh = h / heads_per_key, key_heads = H / heads_per_key;

  float* sbase = state + (size_t)slot * state_stride + (size_t)h * dk * dv + c0;
  // whole rows go four numbers at a time (columns of the CTA beyond the tile's hold whatever lies there, and nothing reads them)
  const bool tile4 = dkp == dk && (ncol & 3) == 0 && (CT & 3) == 0 && (dv & 3) == 0 && (((uintptr_t)sbase) & 15) == 0;
  if (tile4) {
    const int c4 = ncol >> 2;
    for (int idx = tid; idx < dk * c4; idx += nthreads) {
      const int r = idx / c4, c = (idx - r * c4) << 2;
      const float4 t4 = *reinterpret_cast<const float4*>(sbase + (size_t)r * dv + c);
      float* d = St + r * lds + c;
      d[0] = t4.x; d[1] = t4.y; d[2] = t4.z; d[3] = t4.w;
    }
  } else {
    for (int idx = tid; idx < dkp * CT; idx += nthreads) {
      const int r = idx / CT, c = idx - r * CT;
      St[r * lds + c] = (r < dk && c < ncol) ? sbase[(size_t)r * dv + c] : 0.f;
    }
    // what no copy ever writes is zero for good: rows of q and k beyond dk, value columns beyond the tile's
    for (int idx = tid; idx < 2 * stage; idx += nthreads) buf[idx] = 0.f;
  }
  __syncthreads();
  // register i of lane s holds row ((i / 4) * KS + s) * 4 + i % 4: run i / 4 of the lane is run (i / 4) * KS + s of the column
  float S[R];
#pragma unroll
  for (int i = 0; i < R; ++i) S[i] = St[(((i >> 2) * KS + s) * 4 + (i & 3)) * lds + col];

  const bool wide_qk = (dk & 3) == 0, wide_v = (dv & 3) == 0 && (c0 & 3) == 0 && (ncol & 3) == 0;
  auto issue = [&](int chunk) {
    float* bq = buf + (chunk & 1) * stage;
    float* bk = bq + tc * dkp;
    float* bv = bk + tc * dkp;
    const int t0 = chunk * tc, nt = min(tc, q_len - t0);
    const int per = wide_qk ? dk / 4 : dk;
    for (int idx = tid; idx < nt * per; idx += nthreads) {
      const int t = idx / per, j = (idx - t * per) * (wide_qk ? 4 : 1);
      const size_t g = ((size_t)(q_begin + t0 + t) * key_heads + kh) * dk + j;
      cp_async(bq + t * dkp + j, qn + g, wide_qk);
      cp_async(bk + t * dkp + j, kn + g, wide_qk);
    }
    const int perv = wide_v ? ncol / 4 : ncol;
    for (int idx = tid; idx < nt * perv; idx += nthreads) {
      const int t = idx / perv, j = (idx - t * perv) * (wide_v ? 4 : 1);
      cp_async(bv + t * CT + j, vn + ((size_t)(q_begin + t0 + t) * H + h) * dv + c0 + j, wide_v);
    }
    if (TOK) {
      float* ba = bv + tc * CT;
      for (int t = tid; t < nt; t += nthreads) cp_async(ba + t, decay + (size_t)(q_begin + t0 + t) * H + h, false);
    }
  };

  const int nchunks = (q_len + tc - 1) / tc;
  issue(0);
  asm volatile("cp.async.commit_group;\n" ::);
  for (int c = 0; c < nchunks; ++c) {
    if (c + 1 < nchunks) issue(c + 1);
    asm volatile("cp.async.commit_group;\n" ::);
    asm volatile("cp.async.wait_group 1;\n" ::);
    __syncthreads();
    const float* bq = buf + (c & 1) * stage;
    const float* bk = bq + tc * dkp;
    const float* bv = bk + tc * dkp;
    const int t0 = c * tc, nt = min(tc, q_len - t0);
    float* orow = out + (size_t)(q_begin + t0) * out_stride + (size_t)h * dv + c0 + col;
    const float4* q = reinterpret_cast<const float4*>(bq) + s;
    const float4* k = reinterpret_cast<const float4*>(bk) + s;
    const float* v = bv + col;
    const float* ba = bv + tc * CT;
    const bool writes = s == 0 && col < ncol;
#pragma unroll(R >= 32 ? 2 : 4)
    for (int t = 0; t < nt; ++t) {
      const float vv = *v, a = TOK ? ba[t] : a_fixed;
      float pg[NJ];
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const float4 k4 = k[j * KS], q4 = q[j * KS];
        S[4 * j] = fmaf(a, S[4 * j], __fmul_rn(k4.x, vv));
        S[4 * j + 1] = fmaf(a, S[4 * j + 1], __fmul_rn(k4.y, vv));
        S[4 * j + 2] = fmaf(a, S[4 * j + 2], __fmul_rn(k4.z, vv));
        S[4 * j + 3] = fmaf(a, S[4 * j + 3], __fmul_rn(k4.w, vv));
        pg[j] = fmaf(S[4 * j + 3], q4.w, fmaf(S[4 * j + 2], q4.z, fmaf(S[4 * j + 1], q4.y, __fmul_rn(S[4 * j], q4.x))));
      }
#pragma unroll
      for (int half = NJ / 2; half > 0; half >>= 1) {
#pragma unroll
        for (int j = 0; j < half; ++j) pg[j] = __fadd_rn(pg[j], pg[j + half]);
      }
      float p = pg[0];
      // the lanes' parts, the halves of the row range first; levels a column has no lanes for are skipped (KS is one for the CTA)
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
        if (o < KS) p = __fadd_rn(p, __shfl_xor_sync(0xffffffffu, p, o));
      if (writes) *orow = p;
      q += dkp / 4;
      k += dkp / 4;
      v += CT;
      orow += out_stride;
    }
    __syncthreads();  // the chunk is used up: the copy after next may overwrite it
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
#pragma unroll
  for (int i = 0; i < R; ++i) St[(((i >> 2) * KS + s) * 4 + (i & 3)) * lds + col] = S[i];
  __syncthreads();
  if (tile4) {
    const int c4 = ncol >> 2;
    for (int idx = tid; idx < dk * c4; idx += nthreads) {
      const int r = idx / c4, c = (idx - r * c4) << 2;
      const float* d = St + r * lds + c;
      *reinterpret_cast<float4*>(sbase + (size_t)r * dv + c) = make_float4(d[0], d[1], d[2], d[3]);
    }
    return;
  }
  for (int idx = tid; idx < dk * ncol; idx += nthreads) {
    const int r = idx / ncol, c = idx - r * ncol;
    sbase[(size_t)r * dv + c] = St[r * lds + c];
  }
}

inline int pow2_at_least(int v) {
  int p = 1;
  while (p < v) p <<= 1;
  return p;
}

template <int R, bool TOK>
int launch_walk(const float* qn, const float* kn, const float* vn, const float* decay, float* state, long long state_stride, float* out,
                long long out_stride, const int* qsl, const int* state_slots, int B, int H, int heads_per_key, int dk, int dv, int tc, cudaStream_t st) {
  const int KS = pow2_at_least((dk + R - 1) / R);
  if (KS > 32) return (int)cudaErrorInvalidValue;
  int CT = (R >= 32 ? 128 : 256) / KS;  // 32 rows a lane take 128 registers: smaller CTAs fit an SM better
  const int cols = pow2_at_least(dv);
  if (CT > cols) CT = cols;
  if (CT * KS < 32) CT = 32 / KS;
  // few (sequence, head) pairs: narrower tiles, so that there are CTAs for every SM
  while (CT * KS > 64 && CT > 4 && (long long)B * H * ((dv + CT - 1) / CT) < 148) CT >>= 1;
  const int dkp = KS * R;
  const size_t smem = (size_t)(((dkp * (CT + 1) + 3) & ~3) + 2 * (tc * (2 * dkp + CT) + (TOK ? (tc + 3) & ~3 : 0))) * sizeof(float);
  auto kern = decay_walk_kernel<R, TOK>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch(kern, dim3((dv + CT - 1) / CT, H, B), dim3(KS * CT), smem, st, qn, kn, vn, decay, state, state_stride, out, out_stride,
                qsl, state_slots, H, heads_per_key, dk, dv, KS, CT, tc);
}

// Rows a lane: as many (up to 32) as still leave a warp for every warp scheduler of the device; a state of few heads in a
// step of few sequences is spread thin instead, since the walk over a sequence is a chain that only other lanes can hide
// (one sequence of 2,048 tokens, 16 heads of 128 x 128: 536 us with 32 rows a lane, 460 us with 16 or 8, 480 us with 4;
// eight sequences of 256 tokens: 219, 244, 247 and 336 us).
inline int rows_per_lane(int B, int H, int dk, int dv) {
  int best = 32;
  for (int r = 32; r >= 4; r >>= 1) {
    if ((dk + r - 1) / r > 32) break;  // more lanes a column than a warp has
    best = r;
    if ((long long)B * H * dv * pow2_at_least((dk + r - 1) / r) / 32 >= 4 * 148) break;
  }
  return best;
}

// decay: float [H], or with TOK [N][H].  qn, kn: [N][H / heads_per_key * dk], vn: [N][H * dv].  max_q_len: the most rows a
// sequence of the step brings (0: unknown); a step of single tokens stages one token, not sixteen.
template <bool TOK>
int decay_walk(const float* qn, const float* kn, const float* vn, const float* decay, float* state, long long state_stride, float* out,
               long long out_stride, const int* qsl, const int* state_slots, int B, int H, int heads_per_key, int dk, int dv, int max_q_len,
               cudaStream_t st) {
  const int r = rows_per_lane(B, H, dk, dv);
  const int tc = max_q_len > 0 && max_q_len < TC ? max_q_len : TC;
#define KVF_WALK(R) launch_walk<R, TOK>(qn, kn, vn, decay, state, state_stride, out, out_stride, qsl, state_slots, B, H, heads_per_key, dk, dv, tc, st)
  if (r == 4) return KVF_WALK(4);
  if (r == 8) return KVF_WALK(8);
  if (r == 16) return KVF_WALK(16);
  return KVF_WALK(32);
#undef KVF_WALK
}

}  // namespace kvf
