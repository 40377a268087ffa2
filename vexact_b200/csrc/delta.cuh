// Gated delta rule between its projections: per head, an N x P fp32 state S carried per sequence,
//     S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// with k and q the unit vectors of their convolved projections (q also times scale), g = exp(-exp(A_log) dt) and
// beta = sigmoid(b).  Convolutions and dt = softplus(. + dt_bias) are ssm_conv's.
//
// Activation row of a token: [q: G N | k: G N | v: H P]; head h uses q / k head h / (H / G).  q and k come as they left
// the convolution: their lengths are divided out in fp32 here.  Sequences and state slots as in ssm.cuh.
//
//   delta_scan_kernel    token by token: decode, short portions, fp32 models
//   delta_prep_kernel    long portions, what a chunk of 64 tokens does without the state, all chunks at once
//   delta_chunk_kernel   long portions, the state's walk over the chunks (delta_chunk.cuh)
#pragma once
#include "ssm.cuh"

namespace b200 {

struct DeltaParams {
  SsmSeqs seqs;
  const void* act;             // [T, act_stride]
  long long act_stride;
  const float* dt;             // [T, heads]
  const void* b;               // [T, b_stride], `heads` columns
  long long b_stride;
  const float* A_log;          // [heads]
  float* state;                // [slots, heads, N, P]
  void* o;                     // [T, heads * P]
  int heads, groups, N, P;
  float scale;
  int min_len, max_len;        // sequences of other lengths are another kernel's
};

constexpr float DELTA_UNIT_EPS = 1e-6f;   // x / sqrt(sum x^2 + eps)

// ------------------------------------------------------------------ token by token
// One CTA per (64-wide slice of P, head, sequence); thread = 4 columns of P x every 16th of the N state rows, held in
// fp32 registers across the sequence's tokens.  With r_k = S^T k and r_q = S^T q of the state BEFORE the token,
//     u = beta (v - g r_k),   o = g r_q + (k . q) u,   S <- g S + k u^T,
// so one pass over the state gives both sums and a token costs one barrier.
// Algorithmic bytes at one token per sequence: the state once in, once out (8 N P per head).
constexpr int DELTA_TB = 4;

template <typename T, int NR>
__global__ void __launch_bounds__(SSM_SCAN_THREADS) delta_scan_kernel(const DeltaParams p) {
  __shared__ float sq[DELTA_TB][NR * 16], sk[DELTA_TB][NR * 16];
  __shared__ float sv[DELTA_TB][SSM_SCAN_P];
  __shared__ float s_g[DELTA_TB], s_beta[DELTA_TB], s_kq[DELTA_TB], s_rk[DELTA_TB], s_rq[DELTA_TB];
  __shared__ __align__(16) float part[2][2][8][SSM_SCAN_P];   // [parity][k, q][warp][column]
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.z, t0, len, fresh, slot) || len < p.min_len || len > p.max_len) return;
  const int h = blockIdx.y, p0 = blockIdx.x * SSM_SCAN_P;
  const int N = p.N, P = p.P, tid = threadIdx.x, lane = tid & 31;
  const int pl = tid & 15, ng = tid >> 4, warp = tid >> 5;
  const int pc = p0 + pl * 4;                       // P is a multiple of 8: four columns are in or out together
  const bool pin = pc < P;
  const int grp = h / (p.heads / p.groups);
  const long long inner = (long long)p.heads * P, qk = (long long)p.groups * N;
  const T* act = reinterpret_cast<const T*>(p.act);
  const float a_head = -expf(p.A_log[h]);
  float S[NR][4];
  float* st = slot < 0 ? nullptr : p.state + ((long long)slot * p.heads + h) * N * P;
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int n = r * 16 + ng;
    S[r][0] = S[r][1] = S[r][2] = S[r][3] = 0.f;
    if (st && !fresh && pin && n < N) load4(st + (long long)n * P + pc, S[r]);
  }
  int par = 0;
  for (int b = 0; b < len; b += DELTA_TB) {
    const int nt = min(DELTA_TB, len - b);
    for (int e = tid; e < nt * NR * 16; e += SSM_SCAN_THREADS) {
      const int i = e / (NR * 16), n = e % (NR * 16);
      const T* row = act + (long long)(t0 + b + i) * p.act_stride + (long long)grp * N;
      sq[i][n] = n < N ? to_f32(row[n]) : 0.f;
      sk[i][n] = n < N ? to_f32(row[qk + n]) : 0.f;
    }
    for (int e = tid; e < nt * SSM_SCAN_P; e += SSM_SCAN_THREADS) {
      const int i = e / SSM_SCAN_P, c = e % SSM_SCAN_P;
      sv[i][c] = p0 + c < P ? to_f32(act[(long long)(t0 + b + i) * p.act_stride + 2 * qk + (long long)h * P + p0 + c]) : 0.f;
    }
    __syncthreads();
    if (warp < nt) {
      float qq = 0.f, kk = 0.f, kq = 0.f;
      for (int n = lane; n < NR * 16; n += 32) {
        const float q = sq[warp][n], k = sk[warp][n];
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
        kq = fmaf(k, q, kq);
      }
      qq = warp_sum(qq);
      kk = warp_sum(kk);
      kq = warp_sum(kq);
      if (lane == 0) {
        const float rq = p.scale / sqrtf(qq + DELTA_UNIT_EPS), rk = 1.f / sqrtf(kk + DELTA_UNIT_EPS);
        const long long t = t0 + b + warp;
        s_rq[warp] = rq;
        s_rk[warp] = rk;
        s_kq[warp] = kq * rq * rk;
        s_g[warp] = expf(a_head * p.dt[t * p.heads + h]);
        s_beta[warp] = 1.f / (1.f + expf(-to_f32(reinterpret_cast<const T*>(p.b)[t * p.b_stride + h])));
      }
    }
    __syncthreads();
    for (int i = 0; i < nt; ++i, par ^= 1) {
      const float g = s_g[i], beta = s_beta[i], rk = s_rk[i], rq = s_rq[i];
      float ak[4] = {0.f, 0.f, 0.f, 0.f}, aq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const float k = sk[i][r * 16 + ng] * rk, q = sq[i][r * 16 + ng] * rq;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          ak[c] = fmaf(k, S[r][c], ak[c]);
          aq[c] = fmaf(q, S[r][c], aq[c]);
        }
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        ak[c] += __shfl_xor_sync(0xffffffffu, ak[c], 16);
        aq[c] += __shfl_xor_sync(0xffffffffu, aq[c], 16);
      }
      if ((tid & 16) == 0) {
        *reinterpret_cast<float4*>(&part[par][0][warp][pl * 4]) = make_float4(ak[0], ak[1], ak[2], ak[3]);
        *reinterpret_cast<float4*>(&part[par][1][warp][pl * 4]) = make_float4(aq[0], aq[1], aq[2], aq[3]);
      }
      __syncthreads();      // (the other parity's sums may still be read: the next token writes those)
      float xk[4] = {0.f, 0.f, 0.f, 0.f}, xq[4] = {0.f, 0.f, 0.f, 0.f}, u[4];
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float4 a = *reinterpret_cast<const float4*>(&part[par][0][w][pl * 4]);
        const float4 c = *reinterpret_cast<const float4*>(&part[par][1][w][pl * 4]);
        xk[0] += a.x; xk[1] += a.y; xk[2] += a.z; xk[3] += a.w;
        xq[0] += c.x; xq[1] += c.y; xq[2] += c.z; xq[3] += c.w;
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) u[c] = beta * (sv[i][pl * 4 + c] - g * xk[c]);
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const float k = sk[i][r * 16 + ng] * rk;
#pragma unroll
        for (int c = 0; c < 4; ++c) S[r][c] = fmaf(g, S[r][c], k * u[c]);
      }
      if (ng == 0 && pin) {
        float o[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) o[c] = fmaf(g, xq[c], s_kq[i] * u[c]);
        store4(reinterpret_cast<T*>(p.o) + (long long)(t0 + b + i) * inner + (long long)h * P + pc, o);
      }
    }
    __syncthreads();
  }
  if (st && pin) {
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int n = r * 16 + ng;
      if (n < N) store4(st + (long long)n * P + pc, S[r]);
    }
  }
}

template <typename T>
inline int delta_scan_launch(const DeltaParams& p, cudaStream_t st) {
  const dim3 grid((unsigned)((p.P + SSM_SCAN_P - 1) / SSM_SCAN_P), (unsigned)p.heads, (unsigned)p.seqs.num_seqs);
  const dim3 block(SSM_SCAN_THREADS);
  if (p.N <= 32) launch_k(delta_scan_kernel<T, 2>, grid, block, 0, st, p);
  else if (p.N <= 64) launch_k(delta_scan_kernel<T, 4>, grid, block, 0, st, p);
  else if (p.N <= 128) launch_k(delta_scan_kernel<T, 8>, grid, block, 0, st, p);
  else if (p.N <= 256) launch_k(delta_scan_kernel<T, 16>, grid, block, 0, st, p);
  else if (p.N <= 512) launch_k(delta_scan_kernel<T, 32>, grid, block, 0, st, p);
  else return B200_ERR_SHAPE;
  return launch_status();
}

inline int delta_check(const DeltaParams& p) {
  if (!ssm_seqs_ok(p.seqs) || !p.act || !p.dt || !p.b || !p.A_log || !p.state || !p.o || p.heads <= 0 || p.groups <= 0 ||
      p.N <= 0 || p.P <= 0)
    return B200_ERR_ARG;
  if (p.heads % p.groups != 0 || p.P % 8 != 0 || p.N % 8 != 0 || p.act_stride % 8 != 0 || p.heads > 65535 ||
      p.seqs.num_seqs > 65535 || ((reinterpret_cast<uintptr_t>(p.act) | reinterpret_cast<uintptr_t>(p.o)) & 15))
    return B200_ERR_SHAPE;
  return B200_OK;
}

}  // namespace b200

// Token-by-token recurrence of the sequences that bring min_len .. max_len tokens.  act rows [q | k | v] after the
// convolution, dt [T, heads] after softplus, b [T, ..] before the sigmoid; o [T, heads * P]; state [slots, heads, N, P].
extern "C" int b200_delta_scan(const void* act, long long act_row_stride, const void* dt_f32, const void* b,
                               long long b_row_stride, const void* A_log_f32, void* state_f32, void* o,
                               const void* query_start_loc, const void* context_lens, const void* state_slots, int num_seqs,
                               int num_slots, int heads, int groups, int N, int P, float scale, int min_len, int max_len,
                               int dtype, void* stream) {
  using namespace b200;
  DeltaParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
                act, act_row_stride, (const float*)dt_f32, b, b_row_stride, (const float*)A_log_f32, (float*)state_f32, o,
                heads, groups, N, P, scale, min_len, max_len};
  if (int rc = delta_check(p)) return rc;
  if (dtype != 0 && dtype != 1) return B200_ERR_ARG;
  return dtype == 0 ? delta_scan_launch<__nv_bfloat16>(p, (cudaStream_t)stream)
                    : delta_scan_launch<float>(p, (cudaStream_t)stream);
}
