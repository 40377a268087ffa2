// Chunked tensor-core form of the gated delta rule (bf16 activations), for portions longer than a few tokens.
//
// Inside a chunk of 64 tokens let c_i = sum_(m <= i) log g_m, S the state before the chunk, k_i and q_i the unit vectors.
// Unrolling the recurrence gives for the written values u_i
//     (I + A) U = diag(beta) (V - diag(e^c) K S),      A_ij = beta_i (k_i . k_j) e^(c_i - c_j)  for j < i,
// and with Tb = (I + A)^-1 diag(beta) (unit lower triangular inverse: forward substitution, fp32)
//     U  = Tb (V - diag(e^c) K S)
//     O  = diag(e^c) Q S + M U,                        M_ij = (q_i . k_j) e^(c_i - c_j)  for j <= i
//     S' = e^(c_last) S + sum_j e^(c_last - c_j) k_j u_j^T.
// This is the compact (WY) form of a product of Householder-like factors (Yang, Wang, Zhang, Shen, Kim: "Parallelizing
// Linear Transformers with the Delta Rule over Sequence Length").
//
// Tb and M do not depend on the state: delta_prep_kernel makes them for every (chunk, head) at once.  delta_chunk_kernel
// then walks a sequence's chunks, one CTA per (slice of PS state columns, head, sequence), with S in fp32 registers (MMA
// accumulators); the state never travels through memory between chunks.
//
// q, k and v as they left the convolution are exact bf16 operands (the lengths of q and k are fp32 factors kept apart);
// whatever is fp32 (Tb, M, S, U and its decayed copy) enters a product as a bf16 pair hi + lo, which keeps 16 bits of it:
// two products against an exact operand, three (hi hi, lo hi, hi lo) between two pairs.
//
// Tb and M are stored in the order of the A fragments the second kernel reads (a lane's four registers of a 16 x 16 tile
// are 16 contiguous bytes), so they go from memory straight into registers.
#pragma once
#include "delta.cuh"
#include "ssm_chunk.cuh"   // cp.async, split_bf2, fragment loads

namespace b200 {

constexpr int DLC_L = 64;                  // tokens of a chunk
constexpr int DLC_THREADS = 128;
constexpr int DLC_FRAG = 4 * 4 * 32;       // uint4 of one 64 x 64 matrix in fragment order: [row tile][k step][lane]
constexpr int DLC_MATS = 4;                // Tb hi, Tb lo, M hi, M lo
constexpr int DLC_VECS = 3;                // c, 1 / |k|, scale / |q|

// Chunk slots of a step: sequence s starts at slot t0 / 64 + s, so neighbours never share one and T / 64 + S are enough.
__device__ __forceinline__ long long dlc_slot(int t0, int s, int chunk) { return t0 / DLC_L + s + chunk; }

struct DeltaChunkParams {
  DeltaParams d;
  uint4* mats;                 // [slots, heads, DLC_MATS, DLC_FRAG]
  float* vecs;                 // [slots, heads, DLC_VECS, 64]
};

template <int NMAX>
struct DlpLayout {
  static constexpr int LDN = NMAX + 8;
  static constexpr int TILE = DLC_L * LDN * 2;
  static constexpr int LDA = DLC_L + 4;
  static constexpr int BYTES = 2 * TILE + DLC_L * LDA * 4 + 4 * DLC_L * 4;
};

template <int NMAX>
__global__ void __launch_bounds__(DLC_THREADS) delta_prep_kernel(const DeltaChunkParams cp) {
  using L = DlpLayout<NMAX>;
  const DeltaParams& p = cp.d;
  extern __shared__ __align__(16) uint8_t dlc_smem[];
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  const int seq = blockIdx.z, chunk = blockIdx.x, h = blockIdx.y;
  if (!ssm_seq(p.seqs, seq, t0, len, fresh, slot) || len < p.min_len || chunk * DLC_L >= len) return;
  const int base = chunk * DLC_L, n = min(DLC_L, len - base), N = p.N;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int grp = h / (p.heads / p.groups), n16 = (N + 15) / 16;
  const uint32_t smem = ptx::smem_u32(dlc_smem), s_q = smem, s_k = smem + L::TILE;
  float* s_a = reinterpret_cast<float*>(dlc_smem + 2 * L::TILE);
  float* s_c = s_a + DLC_L * L::LDA;
  float *s_beta = s_c + DLC_L, *s_rk = s_beta + DLC_L, *s_rq = s_rk + DLC_L;
  const __nv_bfloat16* act = reinterpret_cast<const __nv_bfloat16*>(p.act);
  for (int e = tid; e < DLC_L * (NMAX / 8); e += DLC_THREADS) {
    const int r = e / (NMAX / 8), v = e % (NMAX / 8);
    const bool in = r < n && v * 8 < N;
    const __nv_bfloat16* src = act + (long long)(t0 + base + (in ? r : 0)) * p.act_stride + (long long)grp * N + (in ? v * 8 : 0);
    cp_async16(s_q + (uint32_t)(r * L::LDN + v * 8) * 2, src, in);
    cp_async16(s_k + (uint32_t)(r * L::LDN + v * 8) * 2, src + (long long)p.groups * N, in);
  }
  cp_async_commit();
  if (warp == 0) {             // inclusive sums of log g: two tokens per lane, then across the warp
    const float a = -expf(p.A_log[h]);
    auto log_g = [&](int i) { return i < n ? a * p.dt[(long long)(t0 + base + i) * p.heads + h] : 0.f; };
    const float v0 = log_g(2 * lane), v1 = v0 + log_g(2 * lane + 1);
    float before = v1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float q = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += q;
    }
    before -= v1;
    s_c[2 * lane] = before + v0;
    s_c[2 * lane + 1] = before + v1;
  } else if (warp >= 2) {
    const int i = tid - 64;
    s_beta[i] = i < n ? 1.f / (1.f + expf(-bf2f(reinterpret_cast<const __nv_bfloat16*>(p.b)[(long long)(t0 + base + i) * p.b_stride + h])))
                      : 0.f;
  }
  cp_async_wait<0>();
  __syncthreads();
  {                            // lengths: thread = (row, q or k)
    const int r = tid & 63, which = tid >> 6;
    const uint4* row = reinterpret_cast<const uint4*>(dlc_smem + (which ? L::TILE : 0) + r * L::LDN * 2);
    float ss = 0.f;
    for (int v = 0; v < n16 * 2; ++v) {
      const uint4 x = row[v];
      const uint32_t w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        float a, b;
        unpack_bf2(w[k], a, b);
        ss = fmaf(a, a, ss);
        ss = fmaf(b, b, ss);
      }
    }
    if (which) s_rk[r] = 1.f / sqrtf(ss + DELTA_UNIT_EPS);
    else s_rq[r] = p.scale / sqrtf(ss + DELTA_UNIT_EPS);
  }
  __syncthreads();
  const long long at = dlc_slot(t0, seq, chunk) * p.heads + h;
  uint4* mats = cp.mats + at * (DLC_MATS * DLC_FRAG);
  float* vecs = cp.vecs + at * (DLC_VECS * DLC_L);
  if (tid < DLC_L) {
    vecs[tid] = s_c[tid];
    vecs[DLC_L + tid] = s_rk[tid];
    vecs[2 * DLC_L + tid] = s_rq[tid];
  }
  // warp w: rows 16 w .. of K K^T and Q K^T, keys up to the diagonal tile
  const int r0 = 16 * warp, i0 = r0 + g4, i1 = i0 + 8;
  for (int kt = 0; kt <= warp; ++kt) {
    float kk[2][4] = {}, qk[2][4] = {};
#pragma unroll 4
    for (int s = 0; s < n16; ++s) {
      uint32_t ak[4], aq[4], b[4];
      abm_frag_a(s_k, L::LDN, r0, s * 16, lane, ak);
      abm_frag_a(s_q, L::LDN, r0, s * 16, lane, aq);
      abm_frag_b_rows(s_k, L::LDN, kt * 16, s * 16, lane, b);
      mma_bf16_16816(kk[0], ak[0], ak[1], ak[2], ak[3], b[0], b[1]);
      mma_bf16_16816(kk[1], ak[0], ak[1], ak[2], ak[3], b[2], b[3]);
      mma_bf16_16816(qk[0], aq[0], aq[1], aq[2], aq[3], b[0], b[1]);
      mma_bf16_16816(qk[1], aq[0], aq[1], aq[2], aq[3], b[2], b[3]);
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      float m[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e < 2 ? i0 : i1, j = kt * 16 + q * 8 + 2 * t4 + (e & 1);
        const float d = j <= i ? expf(s_c[i] - s_c[j]) * s_rk[j] : 0.f;
        m[e] = qk[q][e] * s_rq[i] * d;
        s_a[i * L::LDA + j] = j < i ? s_beta[i] * s_rk[i] * d * kk[q][e] : 0.f;
      }
      split_bf2(m[0], m[1], hi[2 * q], lo[2 * q]);
      split_bf2(m[2], m[3], hi[2 * q + 1], lo[2 * q + 1]);
    }
    // accumulator quads (row, row + 8) x (columns, columns + 8) are the A fragment's registers in this order
    uint4* m = mats + 2 * DLC_FRAG + (warp * 4 + kt) * 32 + lane;
    m[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    m[DLC_FRAG] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  __syncthreads();
  // column `tid` of (I + A)^-1 by forward substitution, times beta of the column
  if (tid < DLC_L) {
    float x[DLC_L];
#pragma unroll
    for (int i = 0; i < DLC_L; ++i) {
      float s0 = i == tid ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
      const float4* row = reinterpret_cast<const float4*>(s_a + i * L::LDA);
#pragma unroll
      for (int k = 0; k < (i + 3) / 4; ++k) {
        const float4 a = row[k];     // entries on and past the diagonal inside a row's tile are zero
        s0 = fmaf(-a.x, x[4 * k], s0);
        if (4 * k + 1 < i) s1 = fmaf(-a.y, x[4 * k + 1], s1);
        if (4 * k + 2 < i) s2 = fmaf(-a.z, x[4 * k + 2], s2);
        if (4 * k + 3 < i) s3 = fmaf(-a.w, x[4 * k + 3], s3);
      }
      x[i] = (s0 + s1) + (s2 + s3);
    }
    const float beta = s_beta[tid];
    // element (i, j = tid) of the fragment order: tile (i / 16, j / 16), lane (i % 8) * 4 + (j % 8) / 2, register
    // (i / 8 % 2) + 2 (j / 8 % 2), half j % 2
    __nv_bfloat16* th = reinterpret_cast<__nv_bfloat16*>(mats);
    const int j = tid;
#pragma unroll
    for (int i = 0; i < DLC_L; ++i) {
      if ((i >> 4) < (j >> 4)) continue;       // tiles above the diagonal are never read
      const int q = (((i >> 4) * 4 + (j >> 4)) * 32 + (i & 7) * 4 + ((j & 7) >> 1)) * 8 + (((i >> 3) & 1) + 2 * ((j >> 3) & 1)) * 2 + (j & 1);
      const float v = x[i] * beta;
      const __nv_bfloat16 top = f2bf(v);
      th[q] = top;
      th[q + DLC_FRAG * 8] = f2bf(v - bf2f(top));
    }
  }
}

template <int NMAX, int PS>
struct DlcLayout {
  // one stage where two would leave room for a single CTA on an SM: the other CTA's products cover the copies
  static constexpr int STAGES = NMAX <= 64 || (NMAX <= 128 && PS <= 16) ? 2 : 1;
  static constexpr int LDN = NMAX + 8, LDP = PS + 8;          // padded pitches: ldmatrix rows in distinct banks
  static constexpr int QK = DLC_L * LDN * 2, X = DLC_L * LDP * 2, ST = NMAX * LDP * 2;
  static constexpr int STAGE = 2 * QK + X + DLC_VECS * DLC_L * 4;    // q, k, v, vectors
  static constexpr int BYTES = STAGES * STAGE + 4 * X + 2 * ST;      // + (R, then U) hi lo, decayed U hi lo, state hi lo
};

template <int NMAX, int PS>
__global__ void __launch_bounds__(DLC_THREADS) delta_chunk_kernel(const DeltaChunkParams cp) {
  using L = DlcLayout<NMAX, PS>;
  const DeltaParams& p = cp.d;
  constexpr int NT = NMAX / 64, PT = PS / 8;
  extern __shared__ __align__(16) uint8_t dlc_smem[];
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  const int seq = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * PS;
  if (!ssm_seq(p.seqs, seq, t0, len, fresh, slot) || len < p.min_len) return;
  const int N = p.N, P = p.P, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int n16 = (N + 15) / 16, grp = h / (p.heads / p.groups);
  const long long inner = (long long)p.heads * P, qk = (long long)p.groups * N;
  const uint32_t smem = ptx::smem_u32(dlc_smem);
  const uint32_t s_r = smem + L::STAGES * L::STAGE, s_ud = s_r + 2 * L::X, s_st = s_ud + 2 * L::X;
  const __nv_bfloat16* act = reinterpret_cast<const __nv_bfloat16*>(p.act);
  const long long slot0 = dlc_slot(t0, seq, 0);

  auto load = [&](int c) {     // chunk c into its stage; rows past the sequence and columns past N / P are zero
    const uint32_t b = smem + (c % L::STAGES) * L::STAGE;
    const int base = c * DLC_L;
    for (int e = tid; e < DLC_L * (NMAX / 8); e += DLC_THREADS) {
      const int r = e / (NMAX / 8), v = e % (NMAX / 8);
      const bool in = base + r < len && v * 8 < N;
      const __nv_bfloat16* src = act + (long long)(t0 + (in ? base + r : 0)) * p.act_stride + (long long)grp * N + (in ? v * 8 : 0);
      cp_async16(b + (uint32_t)(r * L::LDN + v * 8) * 2, src, in);
      cp_async16(b + L::QK + (uint32_t)(r * L::LDN + v * 8) * 2, src + qk, in);
    }
    for (int e = tid; e < DLC_L * (PS / 8); e += DLC_THREADS) {
      const int r = e / (PS / 8), v = e % (PS / 8);
      const bool in = base + r < len && p0 + v * 8 < P;
      const __nv_bfloat16* src =
          act + (long long)(t0 + (in ? base + r : 0)) * p.act_stride + 2 * qk + (long long)h * P + (in ? p0 + v * 8 : 0);
      cp_async16(b + 2 * L::QK + (uint32_t)(r * L::LDP + v * 8) * 2, src, in);
    }
    const float* vec = cp.vecs + ((slot0 + c) * p.heads + h) * (DLC_VECS * DLC_L);
    if (tid < DLC_VECS * DLC_L / 4) cp_async16(b + 2 * L::QK + L::X + tid * 16, vec + tid * 4, true);
    cp_async_commit();
  };
  load(0);

  float S[NT][PT][4];   // rows 16 (warp + 4 i) + g4 (+ 8), columns 8 j + 2 t4 (+ 1)
  float* st = slot < 0 ? nullptr : p.state + ((long long)slot * p.heads + h) * N * P;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < PT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = 16 * (warp + 4 * i) + g4 + (e >> 1) * 8, c = p0 + 8 * j + 2 * t4 + (e & 1);
        S[i][j][e] = st && !fresh && n < N && c < P ? st[(long long)n * P + c] : 0.f;
      }
  // fp32 accumulator tile (rows row0 + g4 and + 8) as hi and lo tiles of bytes `step` apart
  auto publish = [&](uint32_t at, int step, int row0, const float (&x)[PT][4], float f0, float f1) {
#pragma unroll
    for (int j = 0; j < PT; ++j)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const float f = half ? f1 : f0;
        uint32_t hi, lo;
        split_bf2(x[j][2 * half] * f, x[j][2 * half + 1] * f, hi, lo);
        uint8_t* d = dlc_smem + (at - smem) + ((row0 + g4 + 8 * half) * L::LDP + 8 * j + 2 * t4) * 2;
        *reinterpret_cast<uint32_t*>(d) = hi;
        *reinterpret_cast<uint32_t*>(d + step) = lo;
      }
  };
#pragma unroll
  for (int i = 0; i < NT; ++i) publish(s_st, L::ST, 16 * (warp + 4 * i), S[i], 1.f, 1.f);

  const int chunks = (len + DLC_L - 1) / DLC_L, r0 = 16 * warp;
  for (int c = 0; c < chunks; ++c) {
    const uint32_t sQ = smem + (c % L::STAGES) * L::STAGE, sK = sQ + L::QK, sV = sK + L::QK;
    const float* s_c = reinterpret_cast<const float*>(dlc_smem + (sV - smem) + L::X);
    const float *s_rk = s_c + DLC_L, *s_rq = s_rk + DLC_L;
    const int base = c * DLC_L;
    const uint4* mats = cp.mats + ((slot0 + c) * p.heads + h) * (DLC_MATS * DLC_FRAG) + warp * 128 + lane;
    uint4 th[4], tl[4];              // this warp's rows of Tb
#pragma unroll
    for (int kt = 0; kt < 4; ++kt)
      if (kt <= warp) {
        th[kt] = mats[kt * 32];
        tl[kt] = mats[DLC_FRAG + kt * 32];
      }
    cp_async_wait<0>();
    __syncthreads();                 // the tiles and the state are in place, everyone has left chunk c - 1
    if (L::STAGES == 2 && c + 1 < chunks) load(c + 1);
    const float c0 = s_c[r0 + g4], c1 = s_c[r0 + g4 + 8], last = s_c[DLC_L - 1];
    const float e0 = expf(c0), e1 = expf(c1);
    // K S and Q S of this warp's rows
    float ks[PT][4] = {}, qs[PT][4] = {};
#pragma unroll 4
    for (int kk = 0; kk < n16; ++kk) {
      uint32_t ak[4], aq[4];
      abm_frag_a(sK, L::LDN, r0, kk * 16, lane, ak);
      abm_frag_a(sQ, L::LDN, r0, kk * 16, lane, aq);
#pragma unroll
      for (int j = 0; j < PT; j += 2)
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          uint32_t b[4];
          abm_frag_b_cols(s_st + part * L::ST, L::LDP, kk * 16, j * 8, lane, b);
          mma_bf16_16816(ks[j], ak[0], ak[1], ak[2], ak[3], b[0], b[1]);
          mma_bf16_16816(ks[j + 1], ak[0], ak[1], ak[2], ak[3], b[2], b[3]);
          mma_bf16_16816(qs[j], aq[0], aq[1], aq[2], aq[3], b[0], b[1]);
          mma_bf16_16816(qs[j + 1], aq[0], aq[1], aq[2], aq[3], b[2], b[3]);
        }
    }
    {                                // R = V - e^c K S
      const float f0 = e0 * s_rk[r0 + g4], f1 = e1 * s_rk[r0 + g4 + 8];
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float a, b;
          unpack_bf2(*reinterpret_cast<const uint32_t*>(dlc_smem + (sV - smem) + ((r0 + g4 + 8 * half) * L::LDP + 8 * j + 2 * t4) * 2),
                     a, b);
          const float f = half ? f1 : f0;
          ks[j][2 * half] = a - f * ks[j][2 * half];
          ks[j][2 * half + 1] = b - f * ks[j][2 * half + 1];
        }
      publish(s_r, L::X, r0, ks, 1.f, 1.f);
    }
    __syncthreads();
    // product of a pair of fragment rows (this warp's) with a pair of 64 x PS tiles
    auto pair_product = [&](float (&acc)[PT][4], const uint4 (&ah)[4], const uint4 (&al)[4], uint32_t tile) {
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > warp) break;
#pragma unroll
        for (int j = 0; j < PT; j += 2) {
          uint32_t b[4], bl[4];
          abm_frag_b_cols(tile, L::LDP, kt * 16, j * 8, lane, b);
          abm_frag_b_cols(tile + L::X, L::LDP, kt * 16, j * 8, lane, bl);
          mma_bf16_16816(acc[j], ah[kt].x, ah[kt].y, ah[kt].z, ah[kt].w, b[0], b[1]);
          mma_bf16_16816(acc[j + 1], ah[kt].x, ah[kt].y, ah[kt].z, ah[kt].w, b[2], b[3]);
          mma_bf16_16816(acc[j], al[kt].x, al[kt].y, al[kt].z, al[kt].w, b[0], b[1]);
          mma_bf16_16816(acc[j + 1], al[kt].x, al[kt].y, al[kt].z, al[kt].w, b[2], b[3]);
          mma_bf16_16816(acc[j], ah[kt].x, ah[kt].y, ah[kt].z, ah[kt].w, bl[0], bl[1]);
          mma_bf16_16816(acc[j + 1], ah[kt].x, ah[kt].y, ah[kt].z, ah[kt].w, bl[2], bl[3]);
        }
      }
    };
    float u[PT][4] = {};
    pair_product(u, th, tl, s_r);
#pragma unroll
    for (int kt = 0; kt < 4; ++kt)   // this warp's rows of M
      if (kt <= warp) {
        th[kt] = mats[2 * DLC_FRAG + kt * 32];
        tl[kt] = mats[3 * DLC_FRAG + kt * 32];
      }
    __syncthreads();                 // R has been read: U takes its place
    publish(s_r, L::X, r0, u, 1.f, 1.f);
    publish(s_ud, L::X, r0, u, expf(last - c0) * s_rk[r0 + g4], expf(last - c1) * s_rk[r0 + g4 + 8]);
    __syncthreads();
    if (base + r0 < len) {
      const float f0 = e0 * s_rq[r0 + g4], f1 = e1 * s_rq[r0 + g4 + 8];
#pragma unroll
      for (int j = 0; j < PT; ++j) {
        qs[j][0] *= f0;
        qs[j][1] *= f0;
        qs[j][2] *= f1;
        qs[j][3] *= f1;
      }
      pair_product(qs, th, tl, s_r);
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = base + r0 + g4 + 8 * half, col = p0 + 8 * j + 2 * t4;
          if (r < len && col < P)
            *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.o) + (long long)(t0 + r) * inner + (long long)h * P + col) =
                pack_bf2(qs[j][2 * half], qs[j][2 * half + 1]);
        }
    }
    // the state after the chunk
    const float keep = expf(last);
    const int ktiles = (min(DLC_L, len - base) + 15) / 16;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int n0 = 16 * (warp + 4 * i);
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= keep;
      if (n0 < N) {
#pragma unroll
        for (int kt = 0; kt < DLC_L / 16; ++kt) {
          if (kt >= ktiles) break;
          uint32_t a[4];
          frag_a_trans(sK, L::LDN, n0, kt * 16, lane, a);
#pragma unroll
          for (int j = 0; j < PT; j += 2)
#pragma unroll
            for (int part = 0; part < 2; ++part) {
              uint32_t b[4];
              abm_frag_b_cols(s_ud + part * L::X, L::LDP, kt * 16, j * 8, lane, b);
              mma_bf16_16816(S[i][j], a[0], a[1], a[2], a[3], b[0], b[1]);
              mma_bf16_16816(S[i][j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
      }
      publish(s_st, L::ST, n0, S[i], 1.f, 1.f);   // (every warp read the old state two barriers ago)
    }
    if (L::STAGES == 1 && c + 1 < chunks) {
      __syncthreads();
      load(c + 1);
    }
  }
  if (st) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int n = 16 * (warp + 4 * i) + g4 + 8 * half, c = p0 + 8 * j + 2 * t4;
          if (n < N && c < P)
            *reinterpret_cast<float2*>(st + (long long)n * P + c) = make_float2(S[i][j][2 * half], S[i][j][2 * half + 1]);
        }
  }
}

template <int NMAX>
inline int delta_prep_launch(const DeltaChunkParams& p, int max_len, cudaStream_t st) {
  constexpr int smem = DlpLayout<NMAX>::BYTES;
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, delta_prep_kernel<NMAX>, smem)) return rc;
  launch_k(delta_prep_kernel<NMAX>,
           dim3((unsigned)((max_len + DLC_L - 1) / DLC_L), (unsigned)p.d.heads, (unsigned)p.d.seqs.num_seqs),
           dim3(DLC_THREADS), (size_t)smem, st, p);
  return launch_status();
}

template <int NMAX, int PS>
inline int delta_chunk_launch(const DeltaChunkParams& p, cudaStream_t st) {
  constexpr int smem = DlcLayout<NMAX, PS>::BYTES;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, delta_chunk_kernel<NMAX, PS>, smem)) return rc;
  launch_k(delta_chunk_kernel<NMAX, PS>,
           dim3((unsigned)((p.d.P + PS - 1) / PS), (unsigned)p.d.heads, (unsigned)p.d.seqs.num_seqs), dim3(DLC_THREADS),
           (size_t)smem, st, p);
  return launch_status();
}

}  // namespace b200

// The recurrence of b200_delta_scan on tensor cores (bf16), for the sequences that bring at least min_len tokens (at most
// max_new of them).  Scratch for T / 64 + num_seqs chunks: mats 32 KB and vecs 768 bytes per chunk and head.  N <= 256.
// slice: state columns per CTA (16 or 32; a choice of speed only).
extern "C" int b200_delta_chunk_scan(const void* act, long long act_row_stride, const void* dt_f32, const void* b,
                                     long long b_row_stride, const void* A_log_f32, void* state_f32, void* o, void* mats,
                                     void* vecs_f32, const void* query_start_loc, const void* context_lens,
                                     const void* state_slots, int num_seqs, int num_slots, int heads, int groups, int N,
                                     int P, float scale, int min_len, int max_new, int slice, void* stream) {
  using namespace b200;
  DeltaChunkParams p{{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
                      act, act_row_stride, (const float*)dt_f32, b, b_row_stride, (const float*)A_log_f32, (float*)state_f32,
                      o, heads, groups, N, P, scale, min_len < 1 ? 1 : min_len, 0x7fffffff},
                     (uint4*)mats, (float*)vecs_f32};
  if (int rc = delta_check(p.d)) return rc;
  if (!mats || !vecs_f32 || max_new <= 0 || (slice != 16 && slice != 32)) return B200_ERR_ARG;
  if (N > 256 || ((reinterpret_cast<uintptr_t>(mats) | reinterpret_cast<uintptr_t>(vecs_f32)) & 15)) return B200_ERR_SHAPE;
  const cudaStream_t st = (cudaStream_t)stream;
  int rc = N <= 64 ? delta_prep_launch<64>(p, max_new, st)
                   : (N <= 128 ? delta_prep_launch<128>(p, max_new, st) : delta_prep_launch<256>(p, max_new, st));
  if (rc) return rc;
  if (slice == 16) {
    if (N <= 64) return delta_chunk_launch<64, 16>(p, st);
    if (N <= 128) return delta_chunk_launch<128, 16>(p, st);
    return delta_chunk_launch<256, 16>(p, st);
  }
  if (N <= 64) return delta_chunk_launch<64, 32>(p, st);
  if (N <= 128) return delta_chunk_launch<128, 32>(p, st);
  return delta_chunk_launch<256, 32>(p, st);
}
