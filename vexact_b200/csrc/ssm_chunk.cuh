// Chunked tensor-core form of the state-space recurrence (bf16 activations), for portions longer than a few tokens.
//
// With cum_i = sum_(k <= i) -exp(A_log) dt_k inside a chunk of SSC_L tokens and S the state before the chunk,
//     y_i  = sum_(j <= i) (C_i . B_j) exp(cum_i - cum_j) dt_j x_j  +  exp(cum_i) S^T C_i  +  D x_i
//     S'   = exp(cum_last) S + sum_j exp(cum_last - cum_j) dt_j B_j x_j^T
// so a chunk is four small products.  One CTA owns a (sequence, head, slice of PS state columns) and walks the
// sequence's chunks with S in fp32 registers (MMA accumulators): the state never travels through memory between
// chunks.  B, C and x are exact bf16 operands; whatever is fp32 (the decay-weighted scores, the state, the
// decay-weighted x) enters its product as a bf16 pair hi + lo with both products accumulated in fp32, which keeps
// 16 bits of it.  Tiles of the next chunk arrive by cp.async while this one is computed.
//
// Warp w of 4 owns token rows 16 w .. 16 w + 15 of the chunk for y and state rows 16 w .. (then every 64) for S.  Two or
// more CTAs share an SM, so that one's matrix products run under another's copies, exponentials and barriers.
#pragma once
#include "attn_bwd_mma.cuh"   // abm_frag_a, abm_frag_b_rows, abm_frag_b_cols (ldmatrix fragment loads)
#include "ssm.cuh"

namespace b200 {

constexpr int SSC_L = 64;
constexpr int SSC_THREADS = 128;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;   // 0 source bytes: the 16 destination bytes are zeroed
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// v = hi + lo as a bf16 pair (16 bits of mantissa together).
__device__ __forceinline__ void split_bf2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf2(a, b);
  float ha, hb;
  unpack_bf2(hi, ha, hb);
  lo = pack_bf2(a - ha, b - hb);
}

// A fragment (16 x 16) of the transpose of a row-major [k][m] tile.
__device__ __forceinline__ void frag_a_trans(uint32_t base, int ld, int m0, int k0, int lane, uint32_t (&a)[4]) {
  const int r = lane & 7, mi = lane >> 3;
  ldmatrix_x4_trans(base + (uint32_t)((k0 + r + (mi >> 1) * 8) * ld + m0 + (mi & 1) * 8) * 2, a[0], a[1], a[2], a[3]);
}

struct SsmChunkParams {
  SsmSeqs seqs;
  const __nv_bfloat16* act;   // [T, act_stride]: x | B | C
  long long act_stride;
  const float* dt;            // [T, heads]
  const float* A_log;
  const float* D;
  float* state;               // [slots, heads, N, P]
  __nv_bfloat16* y;           // [T, heads * P]
  int heads, groups, N, P;
  int min_len;
};

template <int NMAX, int PS>
struct SscLayout {
  static constexpr int STAGES = NMAX <= 128 ? 2 : 1;
  static constexpr int LDN = NMAX + 8, LDP = PS + 8;          // padded pitches: ldmatrix rows in distinct banks
  static constexpr int BC = SSC_L * LDN * 2;                   // bytes of one B or C tile
  static constexpr int X = SSC_L * LDP * 2;
  static constexpr int ST = NMAX * LDP * 2;
  static constexpr int STAGE = 2 * BC + X + SSC_L * 4;         // B, C, x, dt
  static constexpr int BYTES = STAGES * STAGE + 2 * X + 2 * ST + SSC_L * 4;
};

template <int NMAX, int PS>
__global__ void __launch_bounds__(SSC_THREADS) ssm_chunk_kernel(const SsmChunkParams p) {
  using L = SscLayout<NMAX, PS>;
  constexpr int NT = NMAX / 64;                      // state row tiles per warp
  constexpr bool KEEP_C = NMAX <= 128;               // the warp's rows of C stay in registers
  constexpr int PT = PS / 8;
  extern __shared__ __align__(16) uint8_t ssc_smem[];
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.z, t0, len, fresh, slot) || len < p.min_len) return;
  const int h = blockIdx.y, p0 = blockIdx.x * PS;
  const int N = p.N, P = p.P, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n16 = (N + 15) / 16, g4 = lane >> 2, t4 = lane & 3;
  const int grp = h / (p.heads / p.groups);
  const long long inner = (long long)p.heads * P;
  const float a_head = -expf(p.A_log[h]), d_head = p.D[h];
  const uint32_t smem = ptx::smem_u32(ssc_smem);
  const uint32_t s_xp = smem + L::STAGES * L::STAGE;        // decay-weighted x: hi, lo
  const uint32_t s_st = s_xp + 2 * L::X;                    // state before the chunk: hi, lo
  float* s_cum = reinterpret_cast<float*>(ssc_smem + L::STAGES * L::STAGE + 2 * L::X + 2 * L::ST);

  auto load = [&](int c) {   // chunk c into its stage; rows past the sequence and columns past N / P are zero
    const uint32_t b = smem + (c % L::STAGES) * L::STAGE;
    const int base = c * SSC_L;
    for (int e = tid; e < SSC_L * (NMAX / 8); e += SSC_THREADS) {
      const int r = e / (NMAX / 8), v = e % (NMAX / 8);
      const bool in = base + r < len && v * 8 < N;
      const __nv_bfloat16* src =
          p.act + (long long)(t0 + (in ? base + r : 0)) * p.act_stride + inner + (long long)grp * N + (in ? v * 8 : 0);
      cp_async16(b + (uint32_t)(r * L::LDN + v * 8) * 2, src, in);
      cp_async16(b + L::BC + (uint32_t)(r * L::LDN + v * 8) * 2, src + (long long)p.groups * N, in);
    }
    for (int e = tid; e < SSC_L * (PS / 8); e += SSC_THREADS) {
      const int r = e / (PS / 8), v = e % (PS / 8);
      const bool in = base + r < len && p0 + v * 8 < P;
      const __nv_bfloat16* src =
          p.act + (long long)(t0 + (in ? base + r : 0)) * p.act_stride + (long long)h * P + p0 + (in ? v * 8 : 0);
      cp_async16(b + 2 * L::BC + (uint32_t)(r * L::LDP + v * 8) * 2, src, in);
    }
    if (tid < SSC_L) {
      const bool in = base + tid < len;
      cp_async4(b + 2 * L::BC + L::X + tid * 4, p.dt + (long long)(t0 + (in ? base + tid : 0)) * p.heads + h, in);
    }
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
  auto publish_state = [&]() {
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int n0 = 16 * (warp + 4 * i);
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split_bf2(S[i][j][2 * half], S[i][j][2 * half + 1], hi, lo);
          uint8_t* d = ssc_smem + (s_st - smem) + ((n0 + g4 + 8 * half) * L::LDP + 8 * j + 2 * t4) * 2;
          *reinterpret_cast<uint32_t*>(d) = hi;
          *reinterpret_cast<uint32_t*>(d + L::ST) = lo;
        }
    }
  };
  publish_state();

  const int chunks = (len + SSC_L - 1) / SSC_L;
  for (int c = 0; c < chunks; ++c) {
    const uint32_t sB = smem + (c % L::STAGES) * L::STAGE, sC = sB + L::BC, sX = sC + L::BC;
    const float* s_dt = reinterpret_cast<const float*>(ssc_smem + (sX - smem) + L::X);
    const int base = c * SSC_L;
    cp_async_wait<0>();
    __syncthreads();          // the tiles and the state are in place, everyone has left chunk c - 1
    if (L::STAGES == 2 && c + 1 < chunks) load(c + 1);
    if (warp == 0) {          // inclusive sums of -exp(A_log) dt: two tokens per lane, then across the warp
      const float v0 = a_head * s_dt[2 * lane], v1 = v0 + a_head * s_dt[2 * lane + 1];
      float before = v1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float q = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += q;
      }
      before -= v1;
      s_cum[2 * lane] = before + v0;
      s_cum[2 * lane + 1] = before + v1;
    }
    __syncthreads();
    const float last = s_cum[SSC_L - 1];
    for (int e = tid; e < SSC_L * (PS / 2); e += SSC_THREADS) {
      const int r = e / (PS / 2), v = e % (PS / 2);
      const float f = expf(last - s_cum[r]) * s_dt[r];
      float a, b;
      unpack_bf2(*reinterpret_cast<const uint32_t*>(ssc_smem + (sX - smem) + (r * L::LDP + 2 * v) * 2), a, b);
      uint32_t hi, lo;
      split_bf2(f * a, f * b, hi, lo);
      uint8_t* d = ssc_smem + (s_xp - smem) + (r * L::LDP + 2 * v) * 2;
      *reinterpret_cast<uint32_t*>(d) = hi;
      *reinterpret_cast<uint32_t*>(d + L::X) = lo;
    }
    __syncthreads();

    const int r0 = 16 * warp;
    if (base + r0 < len) {
      float y[PT][4];
#pragma unroll
      for (int j = 0; j < PT; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
      uint32_t cf[KEEP_C ? NMAX / 16 : 1][4];
      if constexpr (KEEP_C) {
#pragma unroll
        for (int kk = 0; kk < NMAX / 16; ++kk)
          if (kk < n16) abm_frag_a(sC, L::LDN, r0, kk * 16, lane, cf[kk]);
      }
      // exp(cum_i) C_i . S
#pragma unroll
      for (int kk = 0; kk < NMAX / 16; ++kk) {
        if (kk >= n16) break;
        uint32_t a[4];
        if constexpr (KEEP_C) {
#pragma unroll
          for (int e = 0; e < 4; ++e) a[e] = cf[kk][e];
        } else {
          abm_frag_a(sC, L::LDN, r0, kk * 16, lane, a);
        }
#pragma unroll
        for (int j = 0; j < PT; j += 2) {
          uint32_t b[4];
#pragma unroll
          for (int part = 0; part < 2; ++part) {
            abm_frag_b_cols(s_st + part * L::ST, L::LDP, kk * 16, j * 8, lane, b);
            mma_bf16_16816(y[j], a[0], a[1], a[2], a[3], b[0], b[1]);
            mma_bf16_16816(y[j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
          }
        }
      }
      const float cum0 = s_cum[r0 + g4], cum1 = s_cum[r0 + g4 + 8];
      const float e0 = expf(cum0), e1 = expf(cum1);
#pragma unroll
      for (int j = 0; j < PT; ++j) {
        y[j][0] *= e0;
        y[j][1] *= e0;
        y[j][2] *= e1;
        y[j][3] *= e1;
      }
      // keys 32 at a time up to the diagonal tile
      for (int kt = 0; kt <= warp; kt += 2) {
        float gacc[4][4] = {};
#pragma unroll
        for (int kk = 0; kk < NMAX / 16; ++kk) {
          if (kk >= n16) break;
          uint32_t a[4], b[4], b2[4];
          if constexpr (KEEP_C) {
#pragma unroll
            for (int e = 0; e < 4; ++e) a[e] = cf[kk][e];
          } else {
            abm_frag_a(sC, L::LDN, r0, kk * 16, lane, a);
          }
          abm_frag_b_rows(sB, L::LDN, kt * 16, kk * 16, lane, b);
          abm_frag_b_rows(sB, L::LDN, kt * 16 + 16, kk * 16, lane, b2);
          mma_bf16_16816(gacc[0], a[0], a[1], a[2], a[3], b[0], b[1]);
          mma_bf16_16816(gacc[1], a[0], a[1], a[2], a[3], b[2], b[3]);
          mma_bf16_16816(gacc[2], a[0], a[1], a[2], a[3], b2[0], b2[1]);
          mma_bf16_16816(gacc[3], a[0], a[1], a[2], a[3], b2[2], b2[3]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          if (kt + half > warp) break;
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const float(&gv)[4] = gacc[2 * half + q];
            const int j0 = (kt + half) * 16 + q * 8 + 2 * t4;
            const float c0 = s_cum[j0], c1 = s_cum[j0 + 1], d0 = s_dt[j0], d1 = s_dt[j0 + 1];
            const int i0 = r0 + g4, i1 = i0 + 8;
            const float w00 = j0 <= i0 ? gv[0] * (__expf(cum0 - c0) * d0) : 0.f;
            const float w01 = j0 + 1 <= i0 ? gv[1] * (__expf(cum0 - c1) * d1) : 0.f;
            const float w10 = j0 <= i1 ? gv[2] * (__expf(cum1 - c0) * d0) : 0.f;
            const float w11 = j0 + 1 <= i1 ? gv[3] * (__expf(cum1 - c1) * d1) : 0.f;
            split_bf2(w00, w01, hi[2 * q], lo[2 * q]);
            split_bf2(w10, w11, hi[2 * q + 1], lo[2 * q + 1]);
          }
#pragma unroll
          for (int j = 0; j < PT; j += 2) {
            uint32_t b[4];
            abm_frag_b_cols(sX, L::LDP, (kt + half) * 16, j * 8, lane, b);
            mma_bf16_16816(y[j], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
            mma_bf16_16816(y[j + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
            mma_bf16_16816(y[j], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
            mma_bf16_16816(y[j + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = r0 + g4 + 8 * half, col = p0 + 8 * j + 2 * t4;
          if (base + r < len && col < P) {
            float a, b;
            unpack_bf2(*reinterpret_cast<const uint32_t*>(ssc_smem + (sX - smem) + (r * L::LDP + 8 * j + 2 * t4) * 2), a, b);
            *reinterpret_cast<uint32_t*>(p.y + (long long)(t0 + base + r) * inner + (long long)h * P + col) =
                pack_bf2(y[j][2 * half] + d_head * a, y[j][2 * half + 1] + d_head * b);
          }
        }
    }
    // the state after the chunk
    const float keep = expf(last);
    const int ktiles = (min(SSC_L, len - base) + 15) / 16;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int n0 = 16 * (warp + 4 * i);
#pragma unroll
      for (int j = 0; j < PT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= keep;
      if (n0 < N) {
#pragma unroll
        for (int kt = 0; kt < SSC_L / 16; ++kt) {
          if (kt >= ktiles) break;
          uint32_t a[4], b[4];
          frag_a_trans(sB, L::LDN, n0, kt * 16, lane, a);
#pragma unroll
          for (int j = 0; j < PT; j += 2)
#pragma unroll
            for (int part = 0; part < 2; ++part) {
              abm_frag_b_cols(s_xp + part * L::X, L::LDP, kt * 16, j * 8, lane, b);
              mma_bf16_16816(S[i][j], a[0], a[1], a[2], a[3], b[0], b[1]);
              mma_bf16_16816(S[i][j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
      }
    }
    __syncthreads();          // every warp has read the old state
    publish_state();
    if (L::STAGES == 1 && c + 1 < chunks) load(c + 1);
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

template <int NMAX, int PS>
inline int ssm_chunk_launch(const SsmChunkParams& p, cudaStream_t st) {
  constexpr int smem = SscLayout<NMAX, PS>::BYTES;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, ssm_chunk_kernel<NMAX, PS>, smem)) return rc;
  launch_k(ssm_chunk_kernel<NMAX, PS>, dim3((unsigned)((p.P + PS - 1) / PS), (unsigned)p.heads, (unsigned)p.seqs.num_seqs),
           dim3(SSC_THREADS), (size_t)smem, st, p);
  return launch_status();
}

}  // namespace b200

// The recurrence of b200_ssm_scan on tensor cores, bf16, for the sequences that bring at least min_len tokens.
// P and N multiples of 8, N <= 256.  slice: state columns per CTA (16 or 32; a choice of speed only).
extern "C" int b200_ssm_chunk_scan(const void* act, long long act_row_stride, const void* dt_f32, const void* A_log_f32,
                                   const void* D_f32, void* state_f32, void* y, const void* query_start_loc,
                                   const void* context_lens, const void* state_slots, int num_seqs, int num_slots,
                                   int heads, int groups, int N, int P, int min_len, int slice, void* stream) {
  using namespace b200;
  SsmChunkParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
                   (const __nv_bfloat16*)act, act_row_stride, (const float*)dt_f32, (const float*)A_log_f32,
                   (const float*)D_f32, (float*)state_f32, (__nv_bfloat16*)y, heads, groups, N, P, min_len};
  if (!ssm_seqs_ok(p.seqs) || !act || !dt_f32 || !A_log_f32 || !D_f32 || !state_f32 || !y || heads <= 0 || groups <= 0 ||
      N <= 0 || P <= 0 || (slice != 16 && slice != 32))
    return B200_ERR_ARG;
  if (heads % groups != 0 || P % 8 != 0 || N % 8 != 0 || N > 256 || act_row_stride % 8 != 0 || heads > 65535 ||
      num_seqs > 65535 || (reinterpret_cast<uintptr_t>(act) & 15))
    return B200_ERR_SHAPE;
  const cudaStream_t st = (cudaStream_t)stream;
  if (slice == 16) {
    if (N <= 64) return ssm_chunk_launch<64, 16>(p, st);
    if (N <= 128) return ssm_chunk_launch<128, 16>(p, st);
    return ssm_chunk_launch<256, 16>(p, st);
  }
  if (N <= 64) return ssm_chunk_launch<64, 32>(p, st);
  if (N <= 128) return ssm_chunk_launch<128, 32>(p, st);
  return ssm_chunk_launch<256, 32>(p, st);
}
