// minGRU: a gated recurrence whose gates read the current token only, element by element over `width` channels,
//     z = sigmoid(zp + z_bias),  u = xp + x_bias,  c = u + 1/2 where u >= 0 and sigmoid(u) where u < 0,
//     S_t = (1 - z) S_(t-1) + z c,      out = S_t * silu(gp) * out_scale,
// with zp, xp and gp columns of a projection row.  The state is fp32, [slots, width]; sequences and state slots as in ssm.cuh.
//
//   gru_scan_kernel    token by token: decode, short portions, fp32 models
//   gru_chunk_kernel   long portions: tiles of tokens as a scan of the maps S -> a S + b
//
// Algorithmic bytes per token: the three columns once, out once (and the state once in, once out per sequence): HBM bandwidth.
#pragma once
#include "ssm.cuh"

namespace b200 {

struct GruParams {
  SsmSeqs seqs;
  const void* proj;            // [T, proj_stride]
  long long proj_stride;
  int z_off, x_off, g_off;     // first columns
  const float* z_bias;         // [width]
  const float* x_bias;         // [width]
  float* state;                // [slots, width]
  void* out;                   // [T, out_stride]
  long long out_stride;
  int width;
  float out_scale;
  int min_len, max_len;        // sequences of other lengths are another kernel's
};

// a = 1 - z and b = z c of one channel and token, and o = silu(g).  In bf16 models three exponentials share a reciprocal:
// they are kept below 2^40, so that their product stays in range (a gate below 2^-40 comes out as 2^-40).
template <typename T>
__device__ __forceinline__ void gru_gates(float zp, float u, float g, float& a, float& b, float& o) {
  if constexpr (sizeof(T) == 2) {
    constexpr float kMost = 27.725887f;      // ln 2^40
    const float ez = __expf(fminf(-zp, kMost)), eu = __expf(fminf(-u, kMost)), eg = __expf(fminf(-g, kMost));
    const float dz = 1.f + ez, du = 1.f + eu, dg = 1.f + eg, inv = __fdividef(1.f, dz * du * dg);
    const float z = du * dg * inv;
    a = ez * z;
    b = z * (u >= 0.f ? u + 0.5f : dz * dg * inv);
    o = g * (dz * du * inv);
  } else {
    const float z = 1.f / (1.f + expf(-zp));
    a = 1.f / (1.f + expf(zp));
    b = z * (u >= 0.f ? u + 0.5f : 1.f / (1.f + expf(-u)));
    o = silu_f32(g);
  }
}

// ------------------------------------------------------------------ token by token
// A thread owns four channels of a sequence and walks its tokens, GRU_AHEAD of them requested together.
constexpr int GRU_THREADS = 128, GRU_AHEAD = 4;

template <typename T>
__global__ void __launch_bounds__(GRU_THREADS) gru_scan_kernel(const GruParams p) {
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.y, t0, len, fresh, slot) || len < p.min_len || len > p.max_len) return;
  const int c = (blockIdx.x * GRU_THREADS + threadIdx.x) * 4;
  if (c >= p.width) return;
  float* st = slot < 0 ? nullptr : p.state + (long long)slot * p.width + c;
  float S[4] = {0.f, 0.f, 0.f, 0.f}, zb[4], xb[4];
  if (st && !fresh) load4(st, S);
  load4(p.z_bias + c, zb);
  load4(p.x_bias + c, xb);
  const T* row = reinterpret_cast<const T*>(p.proj) + (long long)t0 * p.proj_stride + c;
  T* out = reinterpret_cast<T*>(p.out) + (long long)t0 * p.out_stride + c;
  for (int j = 0; j < len; j += GRU_AHEAD) {
    float z[GRU_AHEAD][4], x[GRU_AHEAD][4], g[GRU_AHEAD][4];
#pragma unroll
    for (int q = 0; q < GRU_AHEAD; ++q) {
      const T* r = row + (long long)min(j + q, len - 1) * p.proj_stride;
      load4(r + p.z_off, z[q]);
      load4(r + p.x_off, x[q]);
      load4(r + p.g_off, g[q]);
    }
#pragma unroll
    for (int q = 0; q < GRU_AHEAD; ++q) {
      if (j + q >= len) break;
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        float a, b, o;
        gru_gates<T>(z[q][k] + zb[k], x[q][k] + xb[k], g[q][k], a, b, o);
        S[k] = fmaf(a, S[k], b);
        y[k] = S[k] * o * p.out_scale;
      }
      store4(out + (long long)(j + q) * p.out_stride, y);
    }
  }
  if (st) store4(st, S);
}

// ------------------------------------------------------------------ tiles of tokens
// A CTA owns 4 CL channels of a sequence: a thread four channels of GRU_RUN neighbouring tokens, CL lanes beside each other in
// the channels.  A tile is GROUPS runs of GRU_RUN tokens.  Every thread composes the maps of its run, the runs' maps are
// scanned per channel (a warp each, the runs on its lanes), and every thread walks its run from the state its scan gives it.
// The next tile's rows are requested ahead of the work on this one.
constexpr int GRU_RUN = 4, GRU_WARPS = 8;

template <int CL>
__global__ void __launch_bounds__(GRU_WARPS * 32) gru_chunk_kernel(const GruParams p) {
  using T = __nv_bfloat16;
  constexpr int GROUPS = GRU_WARPS * 32 / CL, TILE = GROUPS * GRU_RUN, CH = 4 * CL;
  constexpr int PER_LANE = GROUPS / 32, PER_WARP = CH / GRU_WARPS;
  __shared__ float s_a[CH][GROUPS + 1], s_b[CH][GROUPS + 1];     // a run's map, then s_b: the state ahead of the run
  __shared__ float s_carry[CH];
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.y, t0, len, fresh, slot) || len < p.min_len || len > p.max_len) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, cl = tid % CL, grp = tid / CL;
  const int c0 = blockIdx.x * CH, c = c0 + cl * 4;
  const bool in = c < p.width;                     // width is a multiple of 8
  const int cc = in ? c : 0;
  float* st = slot < 0 ? nullptr : p.state + (long long)slot * p.width;
  if (tid < CH) s_carry[tid] = st && !fresh && c0 + tid < p.width ? st[c0 + tid] : 0.f;
  float zb[4], xb[4];
  load4(p.z_bias + cc, zb);
  load4(p.x_bias + cc, xb);
  const T* proj = reinterpret_cast<const T*>(p.proj) + (long long)t0 * p.proj_stride + cc;
  T* out = reinterpret_cast<T*>(p.out) + (long long)t0 * p.out_stride + cc;
  uint2 raw[GRU_RUN][3];
  auto request = [&](int base) {
#pragma unroll
    for (int q = 0; q < GRU_RUN; ++q) {
      const T* r = proj + (long long)min(base + grp * GRU_RUN + q, len - 1) * p.proj_stride;
      raw[q][0] = *reinterpret_cast<const uint2*>(r + p.z_off);
      raw[q][1] = *reinterpret_cast<const uint2*>(r + p.x_off);
      raw[q][2] = *reinterpret_cast<const uint2*>(r + p.g_off);
    }
  };
  request(0);
  for (int base = 0; base < len; base += TILE) {
    const int first = base + grp * GRU_RUN;
    float a[GRU_RUN][4], b[GRU_RUN][4], o[GRU_RUN][4], A[4] = {1.f, 1.f, 1.f, 1.f}, B[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int q = 0; q < GRU_RUN; ++q) {
      float z[4], x[4], g[4];
      unpack_bf2(raw[q][0].x, z[0], z[1]);
      unpack_bf2(raw[q][0].y, z[2], z[3]);
      unpack_bf2(raw[q][1].x, x[0], x[1]);
      unpack_bf2(raw[q][1].y, x[2], x[3]);
      unpack_bf2(raw[q][2].x, g[0], g[1]);
      unpack_bf2(raw[q][2].y, g[2], g[3]);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        gru_gates<T>(z[k] + zb[k], x[k] + xb[k], g[k], a[q][k], b[q][k], o[q][k]);
        if (first + q >= len) {                     // past the end: the state stays
          a[q][k] = 1.f;
          b[q][k] = 0.f;
        }
        A[k] *= a[q][k];
        B[k] = fmaf(a[q][k], B[k], b[q][k]);
      }
    }
    if (base + TILE < len) request(base + TILE);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      s_a[cl * 4 + k][grp] = A[k];
      s_b[cl * 4 + k][grp] = B[k];
    }
    __syncthreads();
#pragma unroll
    for (int w = 0; w < PER_WARP; ++w) {
      const int ch = warp * PER_WARP + w;
      float ra[PER_LANE], rb[PER_LANE], la = 1.f, lb = 0.f;
#pragma unroll
      for (int i = 0; i < PER_LANE; ++i) {
        ra[i] = s_a[ch][lane * PER_LANE + i];
        rb[i] = s_b[ch][lane * PER_LANE + i];
        la *= ra[i];
        lb = fmaf(ra[i], lb, rb[i]);
      }
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {            // (la, lb): the maps of this lane's runs and all before, composed
        const float pa = __shfl_up_sync(0xffffffffu, la, d), pb = __shfl_up_sync(0xffffffffu, lb, d);
        if (lane >= d) {
          lb = fmaf(la, pb, lb);
          la *= pa;
        }
      }
      float ea = __shfl_up_sync(0xffffffffu, la, 1), eb = __shfl_up_sync(0xffffffffu, lb, 1);
      if (lane == 0) {
        ea = 1.f;
        eb = 0.f;
      }
      const float carry = s_carry[ch];
      float S = fmaf(ea, carry, eb);
#pragma unroll
      for (int i = 0; i < PER_LANE; ++i) {
        s_b[ch][lane * PER_LANE + i] = S;
        S = fmaf(ra[i], S, rb[i]);
      }
      __syncwarp();
      if (lane == 31) s_carry[ch] = S;
    }
    __syncthreads();
    float S[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) S[k] = s_b[cl * 4 + k][grp];
#pragma unroll
    for (int q = 0; q < GRU_RUN; ++q) {
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        S[k] = fmaf(a[q][k], S[k], b[q][k]);
        y[k] = S[k] * o[q][k] * p.out_scale;
      }
      if (in && first + q < len) store4(out + (long long)(first + q) * p.out_stride, y);
    }
    __syncthreads();                                // the runs' states have been read
  }
  if (tid < CH && st && c0 + tid < p.width) st[c0 + tid] = s_carry[tid];
}

template <typename T>
inline int gru_scan_launch(const GruParams& p, cudaStream_t st) {
  const dim3 grid((unsigned)((p.width / 4 + GRU_THREADS - 1) / GRU_THREADS), (unsigned)p.seqs.num_seqs);
  launch_k(gru_scan_kernel<T>, grid, dim3(GRU_THREADS), 0, st, p);
  return launch_status();
}

inline int gru_check(const GruParams& p) {
  if (!ssm_seqs_ok(p.seqs) || !p.proj || !p.z_bias || !p.x_bias || !p.state || !p.out || p.width <= 0 || p.z_off < 0 ||
      p.x_off < 0 || p.g_off < 0)
    return B200_ERR_ARG;
  if (p.width % 8 || p.proj_stride % 8 || p.z_off % 8 || p.x_off % 8 || p.g_off % 8 || p.out_stride % 8 ||
      p.seqs.num_seqs > 65535 || ((reinterpret_cast<uintptr_t>(p.proj) | reinterpret_cast<uintptr_t>(p.out)) & 15))
    return B200_ERR_SHAPE;
  return B200_OK;
}

}  // namespace b200

// The sequences that bring min_len .. max_len tokens, token by token; dtype 0 = bf16, 1 = fp32 (proj and out).
extern "C" int b200_gru_scan(const void* proj, long long proj_row_stride, int z_off, int x_off, int g_off,
                             const void* z_bias_f32, const void* x_bias_f32, void* state_f32, void* out,
                             long long out_row_stride, const void* query_start_loc, const void* context_lens,
                             const void* state_slots, int num_seqs, int num_slots, int width, float out_scale, int min_len,
                             int max_len, int dtype, void* stream) {
  using namespace b200;
  GruParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
              proj, proj_row_stride, z_off, x_off, g_off, (const float*)z_bias_f32, (const float*)x_bias_f32,
              (float*)state_f32, out, out_row_stride, width, out_scale, min_len, max_len};
  if (int rc = gru_check(p)) return rc;
  if (dtype != 0 && dtype != 1) return B200_ERR_ARG;
  return dtype == 0 ? gru_scan_launch<__nv_bfloat16>(p, (cudaStream_t)stream) : gru_scan_launch<float>(p, (cudaStream_t)stream);
}

// The same recurrence in tiles of tokens (bf16), for the sequences that bring at least min_len tokens.  channels: of a CTA, 16
// or 32 (speed only).
extern "C" int b200_gru_chunk_scan(const void* proj, long long proj_row_stride, int z_off, int x_off, int g_off,
                                   const void* z_bias_f32, const void* x_bias_f32, void* state_f32, void* out,
                                   long long out_row_stride, const void* query_start_loc, const void* context_lens,
                                   const void* state_slots, int num_seqs, int num_slots, int width, float out_scale,
                                   int min_len, int channels, void* stream) {
  using namespace b200;
  GruParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
              proj, proj_row_stride, z_off, x_off, g_off, (const float*)z_bias_f32, (const float*)x_bias_f32,
              (float*)state_f32, out, out_row_stride, width, out_scale, min_len, 0x7fffffff};
  if (int rc = gru_check(p)) return rc;
  if (channels != 16 && channels != 32) return B200_ERR_ARG;
  const dim3 grid((unsigned)((width + channels - 1) / channels), (unsigned)num_seqs), block(GRU_WARPS * 32);
  if (channels == 16) launch_k(gru_chunk_kernel<4>, grid, block, 0, (cudaStream_t)stream, p);
  else launch_k(gru_chunk_kernel<8>, grid, block, 0, (cudaStream_t)stream, p);
  return launch_status();
}
