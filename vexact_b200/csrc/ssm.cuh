// State-space (Mamba-2) mixer between its two projections.
//
// Input row of a token: [z: H*P | x: H*P | B: G*N | C: G*N | dt: H] (the output of the in-projection).
//   1. x, B, C: causal convolution per channel (`taps` inputs, the last one the current token) + bias, silu;
//      dt: softplus(dt + dt_bias) in fp32.                                              ssm_conv_*_kernel
//   2. per head, S an N x P fp32 state carried per sequence:
//         S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t
//                                                                                        ssm_scan_kernel (token by
//      token; decode, short portions, fp32 models) or the chunked tensor-core form of ssm_chunk.cuh
//   3. y * silu(z), RMS norm in equal parts, times the norm weight.                      ssm_gate_norm_kernel
//
// Sequences are described by query_start_loc [S + 1] and context_lens [S] (tokens after this step); `state_slots`
// [S] names the slot that holds a sequence's convolution inputs and state, -1 = none (a padded sequence: nothing is
// read or written).  A sequence whose step starts at position 0 starts from zeros whatever its slot holds.
#pragma once
#include "hyper.cuh"   // load4 / store4 / to_f32 / from_f32

namespace b200 {

struct SsmSeqs {
  const int* query_start_loc;  // [S + 1]
  const int* context_lens;     // [S]
  const int* state_slots;      // [S]
  int num_seqs;
  int num_slots;
};

// One sequence's place in the step: false when there is nothing to do for it.
__device__ __forceinline__ bool ssm_seq(const SsmSeqs& q, int s, int& t0, int& len, bool& fresh, int& slot) {
  t0 = q.query_start_loc[s];
  len = q.query_start_loc[s + 1] - t0;
  fresh = q.context_lens[s] <= len;
  slot = q.state_slots[s];
  if (slot >= q.num_slots) {
    if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, slot);
    slot = -1;
  }
  return len > 0;
}

__device__ __forceinline__ float silu_f32(float v) { return v / (1.f + expf(-v)); }
// silu of an activation that is stored in T.
template <typename T>
__device__ __forceinline__ float silu_as(float v) { return silu_f32(v); }
template <>
__device__ __forceinline__ float silu_as<__nv_bfloat16>(float v) { return __fdividef(v, 1.f + __expf(-v)); }
__device__ __forceinline__ float softplus_f32(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

struct SsmConvParams {
  SsmSeqs seqs;
  const void* proj;            // [T, proj_stride], see the row layout above
  long long proj_stride;
  int conv_off, dt_off;        // columns of the first convolved channel and of dt
  int channels, heads, taps;
  const float* w;              // [channels, taps]
  const float* bias;           // [channels]
  const float* dt_bias;        // [heads]
  void* conv_state;            // [slots, taps - 1, channels], the projection's own values
  void* act;                   // [T, channels]
  float* dt;                   // [T, heads]
  long long num_tokens;
};

// Output of channel c for token j of a sequence that starts at packed token t0.
template <typename T>
__device__ __forceinline__ float ssm_conv_at(const SsmConvParams& p, const T* proj, const T* st, int c, long long t0,
                                             int j) {
  float a = p.bias[c];
  for (int k = 0; k < p.taps; ++k) {
    const int i = j - (p.taps - 1) + k;          // token of the sequence's step this tap reads
    float v = 0.f;
    if (i >= 0) v = to_f32(proj[(t0 + i) * p.proj_stride + p.conv_off + c]);
    else if (st) v = to_f32(st[(long long)(i + p.taps - 1) * p.channels + c]);
    a = fmaf(p.w[c * p.taps + k], v, a);
  }
  return silu_as<T>(a);
}

// The last taps - 1 inputs of (old state, this step's inputs) become the state.  Ascending k reads only entries at or
// above the one it writes.
template <typename T>
__device__ __forceinline__ void ssm_conv_shift(const SsmConvParams& p, const T* proj, T* st, bool fresh, int c,
                                               long long t0, int len) {
  for (int k = 0; k + 1 < p.taps; ++k) {
    const int i = len - (p.taps - 1) + k;
    T v = from_f32<T>(0.f);
    if (i >= 0) v = proj[(t0 + i) * p.proj_stride + p.conv_off + c];
    else if (!fresh) v = st[(long long)(i + p.taps - 1) * p.channels + c];
    st[(long long)k * p.channels + c] = v;
  }
}

// Decode and short portions: one thread per (sequence, channel) walks the sequence's tokens and moves the state on.
template <typename T>
__global__ void __launch_bounds__(128) ssm_conv_seq_kernel(const SsmConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * 128 + threadIdx.x;
  int len, slot, t0;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.y, t0, len, fresh, slot)) return;
  const T* proj = reinterpret_cast<const T*>(p.proj);
  if (c < p.channels) {
    T* st = slot < 0 ? nullptr
                     : reinterpret_cast<T*>(p.conv_state) + (long long)slot * (p.taps - 1) * p.channels;
    T* act = reinterpret_cast<T*>(p.act);
    if (len == 1 && p.taps == 4 && st) {   // a decoded token: every load at once, then the shift from registers
      const float4 w = *reinterpret_cast<const float4*>(p.w + (long long)c * 4);
      const T zero = from_f32<T>(0.f), x = proj[(long long)t0 * p.proj_stride + p.conv_off + c];
      const T s0 = fresh ? zero : st[c], s1 = fresh ? zero : st[p.channels + c], s2 = fresh ? zero : st[2 * p.channels + c];
      float a = p.bias[c];
      a = fmaf(w.x, to_f32(s0), a);
      a = fmaf(w.y, to_f32(s1), a);
      a = fmaf(w.z, to_f32(s2), a);
      a = fmaf(w.w, to_f32(x), a);
      act[(long long)t0 * p.channels + c] = from_f32<T>(silu_as<T>(a));
      st[c] = s1;
      st[p.channels + c] = s2;
      st[2 * p.channels + c] = x;
      return;
    }
    for (int j = 0; j < len; ++j)
      act[(long long)(t0 + j) * p.channels + c] =
          from_f32<T>(ssm_conv_at<T>(p, proj, fresh ? nullptr : st, c, t0, j));
    if (st) ssm_conv_shift<T>(p, proj, st, fresh, c, t0, len);
  } else if (c < p.channels + p.heads) {
    const int h = c - p.channels;
    for (int j = 0; j < len; ++j)
      p.dt[(long long)(t0 + j) * p.heads + h] =
          softplus_f32(to_f32(proj[(long long)(t0 + j) * p.proj_stride + p.dt_off + h]) + p.dt_bias[h]);
  }
}

constexpr int SSM_CONV_TILE = 16;   // tokens per CTA of the tiled form

// Long portions: a thread owns one channel of SSM_CONV_TILE packed tokens; the state is only read (the shift is a
// launch of its own, because other CTAs may still need the old inputs).
template <typename T>
__global__ void __launch_bounds__(128) ssm_conv_tile_kernel(const SsmConvParams p) {
  __shared__ int s_seq;
  pdl_trigger();
  pdl_wait();
  const long long tile0 = (long long)blockIdx.y * SSM_CONV_TILE;
  if (threadIdx.x == 0) {   // sequence of the tile's first token: the last one that starts at or before it
    int lo = 0, hi = p.seqs.num_seqs - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.seqs.query_start_loc[mid] <= tile0) lo = mid;
      else hi = mid - 1;
    }
    s_seq = lo;
  }
  __syncthreads();
  const int c = blockIdx.x * 128 + threadIdx.x;
  const T* proj = reinterpret_cast<const T*>(p.proj);
  int s = s_seq, len, slot, t0;
  bool fresh;
  ssm_seq(p.seqs, s, t0, len, fresh, slot);
  if (sizeof(T) == 2 && p.taps <= 4 && p.channels % 256 == 0 && (int)blockIdx.x * 128 < p.channels && tile0 >= t0 &&
      tile0 + SSM_CONV_TILE <= t0 + len) {
    if ((int)blockIdx.x * 256 >= p.channels) return;
    // a tile inside one sequence: two channels per thread, every input loaded up front
    const int c2 = (blockIdx.x * 128 + threadIdx.x) * 2;
    float2 w[4], in[SSM_CONV_TILE + 3];
    const int j0 = (int)(tile0 - t0);
#pragma unroll
    for (int i = 0; i < SSM_CONV_TILE + 3; ++i) {
      const int q = j0 - 3 + i;
      in[i] = make_float2(0.f, 0.f);
      if (q >= 0) {
        unpack_bf2(*reinterpret_cast<const uint32_t*>(proj + (t0 + (long long)q) * p.proj_stride + p.conv_off + c2), in[i].x,
                   in[i].y);
      } else if (!fresh && slot >= 0 && q + p.taps - 1 >= 0) {
        unpack_bf2(*reinterpret_cast<const uint32_t*>(reinterpret_cast<const T*>(p.conv_state) +
                                                      ((long long)slot * (p.taps - 1) + q + p.taps - 1) * p.channels + c2),
                   in[i].x, in[i].y);
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int kk = k - (4 - p.taps);
      w[k] = kk >= 0 ? make_float2(p.w[c2 * p.taps + kk], p.w[(c2 + 1) * p.taps + kk]) : make_float2(0.f, 0.f);
    }
    const float2 bias = *reinterpret_cast<const float2*>(p.bias + c2);
    T* out = reinterpret_cast<T*>(p.act) + tile0 * p.channels + c2;
#pragma unroll
    for (int i = 0; i < SSM_CONV_TILE; ++i) {
      float a = bias.x, b = bias.y;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        a = fmaf(w[k].x, in[i + k].x, a);
        b = fmaf(w[k].y, in[i + k].y, b);
      }
      *reinterpret_cast<uint32_t*>(out + (long long)i * p.channels) = pack_bf2(silu_as<T>(a), silu_as<T>(b));
    }
    return;
  }
  const bool is_dt = c >= p.channels;
  if (c >= p.channels + p.heads) return;
  if (!is_dt && p.taps <= 4) {
    // sliding window in registers
    float w[4], win[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      w[k] = k >= 4 - p.taps ? p.w[c * p.taps + k - (4 - p.taps)] : 0.f;
      win[k] = 0.f;
    }
    const float bias = p.bias[c];
    bool refill = true;
    for (int i = 0; i < SSM_CONV_TILE; ++i) {
      const long long t = tile0 + i;
      if (t >= p.num_tokens) return;
      while (t >= t0 + len && s + 1 < p.seqs.num_seqs) {
        ++s;
        ssm_seq(p.seqs, s, t0, len, fresh, slot);
        refill = true;
      }
      const int j = (int)(t - t0);
      if (j >= len) return;   // padding tokens past the last sequence
      if (refill) {           // the three inputs before token j
        refill = false;
#pragma unroll
        for (int k = 1; k < 4; ++k) {
          const int q = j - 4 + k;
          float v = 0.f;
          if (q >= 0) v = to_f32(proj[(t0 + q) * p.proj_stride + p.conv_off + c]);
          else if (!fresh && slot >= 0 && q + p.taps - 1 >= 0)
            v = to_f32((reinterpret_cast<const T*>(p.conv_state) +
                        ((long long)slot * (p.taps - 1) + q + p.taps - 1) * p.channels)[c]);
          win[k] = v;
        }
      }
#pragma unroll
      for (int k = 0; k < 3; ++k) win[k] = win[k + 1];
      win[3] = to_f32(proj[t * p.proj_stride + p.conv_off + c]);
      float a = bias;
#pragma unroll
      for (int k = 0; k < 4; ++k) a = fmaf(w[k], win[k], a);
      reinterpret_cast<T*>(p.act)[t * p.channels + c] = from_f32<T>(silu_as<T>(a));
    }
    return;
  }
  for (int i = 0; i < SSM_CONV_TILE; ++i) {
    const long long t = tile0 + i;
    if (t >= p.num_tokens) return;
    while (t >= t0 + len && s + 1 < p.seqs.num_seqs) {
      ++s;
      ssm_seq(p.seqs, s, t0, len, fresh, slot);
    }
    if (t - t0 >= len) return;
    if (is_dt) {
      const int h = c - p.channels;
      p.dt[t * p.heads + h] = softplus_f32(to_f32(proj[t * p.proj_stride + p.dt_off + h]) + p.dt_bias[h]);
    } else {
      const T* st = fresh || slot < 0 ? nullptr
                                      : reinterpret_cast<const T*>(p.conv_state) + (long long)slot * (p.taps - 1) * p.channels;
      reinterpret_cast<T*>(p.act)[t * p.channels + c] = from_f32<T>(ssm_conv_at<T>(p, proj, st, c, t0, (int)(t - t0)));
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) ssm_conv_shift_kernel(const SsmConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * 128 + threadIdx.x;
  int len, slot, t0;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.y, t0, len, fresh, slot) || slot < 0 || c >= p.channels) return;
  ssm_conv_shift<T>(p, reinterpret_cast<const T*>(p.proj),
                    reinterpret_cast<T*>(p.conv_state) + (long long)slot * (p.taps - 1) * p.channels, fresh, c, t0, len);
}

// ------------------------------------------------------------------ token-by-token scan
// One CTA per (64-wide slice of P, head, sequence).  Thread = 4 values of P x every 16th of the N state rows, held in
// fp32 registers across the sequence's tokens.  Tokens go through shared memory SSM_SCAN_TB at a time; the partial
// sums over N meet in a fixed order.
// Algorithmic bytes at one token per sequence: the state once in, once out (8 N P per head).
constexpr int SSM_SCAN_TB = 4;
constexpr int SSM_SCAN_P = 64;
constexpr int SSM_SCAN_THREADS = 256;

struct SsmScanParams {
  SsmSeqs seqs;
  const void* act;             // [T, act_stride]: x | B | C
  long long act_stride;
  const float* dt;             // [T, heads]
  const float* A_log;          // [heads]
  const float* D;              // [heads]
  float* state;                // [slots, heads, N, P]
  void* y;                     // [T, heads * P]
  int heads, groups, N, P;
  int min_len, max_len;        // sequences of other lengths are another kernel's
};

template <typename T, int NR>
__global__ void __launch_bounds__(SSM_SCAN_THREADS) ssm_scan_kernel(const SsmScanParams p) {
  __shared__ float sB[SSM_SCAN_TB][NR * 16], sC[SSM_SCAN_TB][NR * 16];
  __shared__ float sx[SSM_SCAN_TB][SSM_SCAN_P];
  __shared__ float sdt[SSM_SCAN_TB];
  __shared__ float part[SSM_SCAN_TB][8][SSM_SCAN_P];
  pdl_trigger();
  pdl_wait();
  int t0, len, slot;
  bool fresh;
  if (!ssm_seq(p.seqs, blockIdx.z, t0, len, fresh, slot) || len < p.min_len || len > p.max_len) return;
  const int h = blockIdx.y, p0 = blockIdx.x * SSM_SCAN_P;
  const int N = p.N, P = p.P, tid = threadIdx.x;
  const int pl = tid & 15, ng = tid >> 4, warp = tid >> 5;
  const int pc = p0 + pl * 4;                       // P is a multiple of 8: four columns are in or out together
  const bool pin = pc < P;
  const int g = h / (p.heads / p.groups);
  const long long inner = (long long)p.heads * P;
  const T* act = reinterpret_cast<const T*>(p.act);
  const float a_head = -expf(p.A_log[h]), d_head = p.D[h];
  float S[NR][4];
  float* st = slot < 0 ? nullptr : p.state + ((long long)slot * p.heads + h) * N * P;
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int n = r * 16 + ng;
    S[r][0] = S[r][1] = S[r][2] = S[r][3] = 0.f;
    if (st && !fresh && pin && n < N) load4(st + (long long)n * P + pc, S[r]);
  }
  for (int b = 0; b < len; b += SSM_SCAN_TB) {
    const int nt = min(SSM_SCAN_TB, len - b);
    for (int e = tid; e < nt * NR * 16; e += SSM_SCAN_THREADS) {
      const int i = e / (NR * 16), n = e % (NR * 16);
      const T* row = act + (long long)(t0 + b + i) * p.act_stride + inner + g * N;
      sB[i][n] = n < N ? to_f32(row[n]) : 0.f;
      sC[i][n] = n < N ? to_f32(row[(long long)p.groups * N + n]) : 0.f;
    }
    for (int e = tid; e < nt * SSM_SCAN_P; e += SSM_SCAN_THREADS) {
      const int i = e / SSM_SCAN_P, c = e % SSM_SCAN_P;
      sx[i][c] = p0 + c < P ? to_f32(act[(long long)(t0 + b + i) * p.act_stride + (long long)h * P + p0 + c]) : 0.f;
    }
    if (tid < nt) sdt[tid] = p.dt[(long long)(t0 + b + tid) * p.heads + h];
    __syncthreads();
    for (int i = 0; i < nt; ++i) {
      const float dt = sdt[i], decay = expf(a_head * dt);
      float x[4], y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < 4; ++k) x[k] = dt * sx[i][pl * 4 + k];
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const float bn = sB[i][r * 16 + ng], cn = sC[i][r * 16 + ng];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          S[r][k] = fmaf(decay, S[r][k], bn * x[k]);
          y[k] = fmaf(cn, S[r][k], y[k]);
        }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) y[k] += __shfl_xor_sync(0xffffffffu, y[k], 16);
      if ((tid & 16) == 0)
        *reinterpret_cast<float4*>(&part[i][warp][pl * 4]) = make_float4(y[0], y[1], y[2], y[3]);
    }
    __syncthreads();
    for (int e = tid; e < nt * SSM_SCAN_P; e += SSM_SCAN_THREADS) {
      const int i = e / SSM_SCAN_P, c = e % SSM_SCAN_P;
      if (p0 + c < P) {
        float v = d_head * sx[i][c];
#pragma unroll
        for (int w = 0; w < 8; ++w) v += part[i][w][c];
        reinterpret_cast<T*>(p.y)[(long long)(t0 + b + i) * inner + (long long)h * P + p0 + c] = from_f32<T>(v);
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
inline int ssm_scan_launch(const SsmScanParams& p, cudaStream_t st) {
  const dim3 grid((unsigned)((p.P + SSM_SCAN_P - 1) / SSM_SCAN_P), (unsigned)p.heads, (unsigned)p.seqs.num_seqs);
  const dim3 block(SSM_SCAN_THREADS);
  if (p.N <= 16) launch_k(ssm_scan_kernel<T, 1>, grid, block, 0, st, p);
  else if (p.N <= 32) launch_k(ssm_scan_kernel<T, 2>, grid, block, 0, st, p);
  else if (p.N <= 64) launch_k(ssm_scan_kernel<T, 4>, grid, block, 0, st, p);
  else if (p.N <= 128) launch_k(ssm_scan_kernel<T, 8>, grid, block, 0, st, p);
  else if (p.N <= 256) launch_k(ssm_scan_kernel<T, 16>, grid, block, 0, st, p);
  else if (p.N <= 512) launch_k(ssm_scan_kernel<T, 32>, grid, block, 0, st, p);
  else return B200_ERR_SHAPE;
  return launch_status();
}

// ------------------------------------------------------------------ gate + grouped RMS norm
// out = rms_norm_by_part(y * silu(z)) * w.  One CTA per (token, part).  The heads of y, z and out are P columns wide;
// the true width of a head is `p_true` <= P (columns p_true .. P are padding: never read, written as zero), the parts
// divide the heads * p_true true columns.
struct SsmGateNormParams {
  const void* y;
  const void* z;
  long long y_stride, z_stride, out_stride;
  const float* w;   // [heads * P] in the padded layout
  void* out;
  int heads, P, p_true, parts;
  float eps;
  int norm_first;   // 1: the norm is of y alone and the gate multiplies its result; 0: the norm is of y * silu(z)
};

// The common case (heads unpadded, parts of a multiple of 8 up to 2048 columns, bf16): one warp per (token, part), its
// gated values in registers.
template <bool NORM_FIRST>
__global__ void __launch_bounds__(256) ssm_gate_norm_warp_kernel(const SsmGateNormParams p, long long pairs) {
  pdl_trigger();
  pdl_wait();
  const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= pairs) return;
  const int lane = threadIdx.x & 31, n = p.heads * p.P / p.parts;
  const long long t = id / p.parts;
  const int j0 = (int)(id - t * p.parts) * n;
  const __nv_bfloat16* y = reinterpret_cast<const __nv_bfloat16*>(p.y) + t * p.y_stride + j0;
  const __nv_bfloat16* z = reinterpret_cast<const __nv_bfloat16*>(p.z) + t * p.z_stride + j0;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + t * p.out_stride + j0;
  uint4 a[8], b[8];
#pragma unroll
  for (int c = 0; c < 8; ++c) {
    const int i = (c * 32 + lane) * 8;
    if (i < n) {
      a[c] = *reinterpret_cast<const uint4*>(y + i);
      b[c] = *reinterpret_cast<const uint4*>(z + i);
    }
  }
  float g[8][8], ss = 0.f;
#pragma unroll
  for (int c = 0; c < 8; ++c) {
    const int i = (c * 32 + lane) * 8;
    if (i < n) {
      const uint32_t av[4] = {a[c].x, a[c].y, a[c].z, a[c].w}, bv[4] = {b[c].x, b[c].y, b[c].z, b[c].w};
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        float y0, y1, z0, z1;
        unpack_bf2(av[k], y0, y1);
        unpack_bf2(bv[k], z0, z1);
        g[c][2 * k] = NORM_FIRST ? y0 : y0 * silu_as<__nv_bfloat16>(z0);
        g[c][2 * k + 1] = NORM_FIRST ? y1 : y1 * silu_as<__nv_bfloat16>(z1);
        ss = fmaf(g[c][2 * k], g[c][2 * k], ss);
        ss = fmaf(g[c][2 * k + 1], g[c][2 * k + 1], ss);
      }
    }
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)n + p.eps);
#pragma unroll
  for (int c = 0; c < 8; ++c) {
    const int i = (c * 32 + lane) * 8;
    if (i < n) {
      float w[8];
      load4(p.w + j0 + i, *reinterpret_cast<float(*)[4]>(w));
      load4(p.w + j0 + i + 4, *reinterpret_cast<float(*)[4]>(w + 4));
      uint32_t o[4];
      const uint32_t bv[4] = {b[c].x, b[c].y, b[c].z, b[c].w};
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        float z0 = 1.f, z1 = 1.f;
        if constexpr (NORM_FIRST) {
          unpack_bf2(bv[k], z0, z1);
          z0 = silu_as<__nv_bfloat16>(z0);
          z1 = silu_as<__nv_bfloat16>(z1);
        }
        o[k] = pack_bf2(g[c][2 * k] * inv * w[2 * k] * z0, g[c][2 * k + 1] * inv * w[2 * k + 1] * z1);
      }
      *reinterpret_cast<uint4*>(out + i) = make_uint4(o[0], o[1], o[2], o[3]);
    }
  }
}

// Narrow parts (a multiple of 8 up to 8 LANES columns, heads unpadded, bf16): LANES lanes per (token, part), eight columns each.
template <int LANES, bool NORM_FIRST>
__global__ void __launch_bounds__(256) ssm_gate_norm_narrow_kernel(const SsmGateNormParams p, long long pairs) {
  pdl_trigger();
  pdl_wait();
  const long long id = (long long)blockIdx.x * (256 / LANES) + threadIdx.x / LANES;
  const int n = p.heads * p.P / p.parts, i = (threadIdx.x % LANES) * 8;
  const bool in = id < pairs && i < n;
  const long long t = in ? id / p.parts : 0;
  const int j = in ? (int)(id - t * p.parts) * n + i : 0;
  uint4 a = make_uint4(0, 0, 0, 0), b = a;
  float w[8] = {};
  if (in) {
    a = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.y) + t * p.y_stride + j);
    b = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.z) + t * p.z_stride + j);
    load4(p.w + j, *reinterpret_cast<float(*)[4]>(w));
    load4(p.w + j + 4, *reinterpret_cast<float(*)[4]>(w + 4));
  }
  const uint32_t av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
  float g[8], z[8], ss = 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    unpack_bf2(av[k], g[2 * k], g[2 * k + 1]);
    unpack_bf2(bv[k], z[2 * k], z[2 * k + 1]);
  }
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    z[k] = silu_as<__nv_bfloat16>(z[k]);
    if (!NORM_FIRST) g[k] *= z[k];
    ss = fmaf(g[k], g[k], ss);
  }
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = 1.f / sqrtf(ss / (float)n + p.eps);
  if (!in) return;
  uint32_t o[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float f0 = NORM_FIRST ? z[2 * k] : 1.f, f1 = NORM_FIRST ? z[2 * k + 1] : 1.f;
    o[k] = pack_bf2(g[2 * k] * inv * w[2 * k] * f0, g[2 * k + 1] * inv * w[2 * k + 1] * f1);
  }
  *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(p.out) + t * p.out_stride + j) = make_uint4(o[0], o[1], o[2], o[3]);
}

template <int LANES>
inline int ssm_gate_norm_narrow(const SsmGateNormParams& p, long long pairs, cudaStream_t st) {
  launch_k(p.norm_first ? ssm_gate_norm_narrow_kernel<LANES, true> : ssm_gate_norm_narrow_kernel<LANES, false>,
           dim3((unsigned)((pairs * LANES + 255) / 256)), dim3(256), 0, st, p, pairs);
  return launch_status();
}

template <typename T>
__global__ void __launch_bounds__(256) ssm_gate_norm_kernel(const SsmGateNormParams p) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int n = p.heads * p.p_true / p.parts, j0 = blockIdx.y * n;
  const T* y = reinterpret_cast<const T*>(p.y) + t * p.y_stride;
  const T* z = reinterpret_cast<const T*>(p.z) + t * p.z_stride;
  T* out = reinterpret_cast<T*>(p.out) + t * p.out_stride;
  const bool plain = p.p_true == p.P;
  // factor of y inside the norm, and of the normed value after it
  auto inner_gate = [&](float v) { return p.norm_first ? 1.f : silu_f32(v); };
  auto outer_gate = [&](float v) { return p.norm_first ? silu_f32(v) : 1.f; };
  auto column = [&](int j) { return plain ? j : (j / p.p_true) * p.P + j % p.p_true; };
  constexpr int KEEP = 8;
  float keep[KEEP][4];
  float ss = 0.f;
  if (plain && n % 4 == 0) {
    const int chunks = n >> 2;
#pragma unroll
    for (int c = 0; c < KEEP; ++c) {
      const int i = c * blockDim.x + threadIdx.x;
      keep[c][0] = keep[c][1] = keep[c][2] = keep[c][3] = 0.f;
      if (i < chunks) {
        float a[4], b[4];
        load4(y + j0 + i * 4, a);
        load4(z + j0 + i * 4, b);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          keep[c][k] = a[k] * inner_gate(b[k]);
          ss = fmaf(keep[c][k], keep[c][k], ss);
        }
      }
    }
    for (int i = KEEP * blockDim.x + threadIdx.x; i < chunks; i += blockDim.x) {
      float a[4], b[4];
      load4(y + j0 + i * 4, a);
      load4(z + j0 + i * 4, b);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float v = a[k] * inner_gate(b[k]);
        ss = fmaf(v, v, ss);
      }
    }
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)n + p.eps);
#pragma unroll
    for (int c = 0; c < KEEP; ++c) {
      const int i = c * blockDim.x + threadIdx.x;
      if (i < chunks) {
        float w[4], o[4];
        load4(p.w + j0 + i * 4, w);
        float b[4];
        if (p.norm_first) load4(z + j0 + i * 4, b);
#pragma unroll
        for (int k = 0; k < 4; ++k) o[k] = keep[c][k] * inv * w[k] * (p.norm_first ? silu_f32(b[k]) : 1.f);
        store4(out + j0 + i * 4, o);
      }
    }
    for (int i = KEEP * blockDim.x + threadIdx.x; i < chunks; i += blockDim.x) {
      float a[4], b[4], w[4], o[4];
      load4(y + j0 + i * 4, a);
      load4(z + j0 + i * 4, b);
      load4(p.w + j0 + i * 4, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) o[k] = a[k] * inner_gate(b[k]) * inv * w[k] * outer_gate(b[k]);
      store4(out + j0 + i * 4, o);
    }
    return;
  }
  for (int j = threadIdx.x; j < n; j += blockDim.x) {
    const int c = column(j0 + j);
    const float v = to_f32(y[c]) * inner_gate(to_f32(z[c]));
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)n + p.eps);
  for (int j = threadIdx.x; j < n; j += blockDim.x) {
    const int c = column(j0 + j);
    out[c] = from_f32<T>(to_f32(y[c]) * inner_gate(to_f32(z[c])) * inv * p.w[c] * outer_gate(to_f32(z[c])));
  }
  if (!plain && blockIdx.y == 0)
    for (int h = threadIdx.x; h < p.heads; h += blockDim.x)
      for (int k = p.p_true; k < p.P; ++k) out[h * p.P + k] = from_f32<T>(0.f);
}

inline bool ssm_seqs_ok(const SsmSeqs& q) {
  return q.query_start_loc && q.context_lens && q.state_slots && q.num_seqs > 0 && q.num_slots > 0;
}

}  // namespace b200

// tiled: 0 = one thread walks a sequence's tokens and moves the state on (decode, short portions); 1 = long portions
// (tokens in tiles, then the state in a second launch).  dtype: 0 = bf16, 1 = fp32.
extern "C" int b200_ssm_conv(const void* proj, long long proj_row_stride, int conv_off, int dt_off, int channels,
                             int heads, int taps, const void* w_f32, const void* bias_f32, const void* dt_bias_f32,
                             void* conv_state, void* act, void* dt_f32, const void* query_start_loc,
                             const void* context_lens, const void* state_slots, int num_seqs, int num_slots,
                             long long num_tokens, int tiled, int dtype, void* stream) {
  using namespace b200;
  SsmConvParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
                  proj, proj_row_stride, conv_off, dt_off, channels, heads, taps, (const float*)w_f32,
                  (const float*)bias_f32, (const float*)dt_bias_f32, conv_state, act, (float*)dt_f32, num_tokens};
  if (!ssm_seqs_ok(p.seqs) || !proj || !w_f32 || !bias_f32 || !dt_bias_f32 || (!conv_state && taps > 1) || !act ||
      !dt_f32 || channels <= 0 || heads <= 0 || taps < 1 || num_tokens < 0 || (dtype != 0 && dtype != 1))
    return B200_ERR_ARG;
  if (num_seqs > 65535) return B200_ERR_SHAPE;
  if (num_tokens == 0) return B200_OK;
  const cudaStream_t st = (cudaStream_t)stream;
  const unsigned cb = (unsigned)((channels + heads + 127) / 128);
  if (!tiled) {
    if (dtype == 0) launch_k(ssm_conv_seq_kernel<__nv_bfloat16>, dim3(cb, num_seqs), dim3(128), 0, st, p);
    else launch_k(ssm_conv_seq_kernel<float>, dim3(cb, num_seqs), dim3(128), 0, st, p);
    return launch_status();
  }
  const long long tiles = (num_tokens + SSM_CONV_TILE - 1) / SSM_CONV_TILE;
  if (tiles > 65535) return B200_ERR_SHAPE;
  if (dtype == 0) {
    launch_k(ssm_conv_tile_kernel<__nv_bfloat16>, dim3(cb, (unsigned)tiles), dim3(128), 0, st, p);
    if (taps > 1) launch_k(ssm_conv_shift_kernel<__nv_bfloat16>, dim3(cb, num_seqs), dim3(128), 0, st, p);
  } else {
    launch_k(ssm_conv_tile_kernel<float>, dim3(cb, (unsigned)tiles), dim3(128), 0, st, p);
    if (taps > 1) launch_k(ssm_conv_shift_kernel<float>, dim3(cb, num_seqs), dim3(128), 0, st, p);
  }
  return launch_status();
}

extern "C" int b200_ssm_scan(const void* act, long long act_row_stride, const void* dt_f32, const void* A_log_f32,
                             const void* D_f32, void* state_f32, void* y, const void* query_start_loc,
                             const void* context_lens, const void* state_slots, int num_seqs, int num_slots, int heads,
                             int groups, int N, int P, int min_len, int max_len, int dtype, void* stream) {
  using namespace b200;
  SsmScanParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
                  act, act_row_stride, (const float*)dt_f32, (const float*)A_log_f32, (const float*)D_f32,
                  (float*)state_f32, y, heads, groups, N, P, min_len, max_len};
  if (!ssm_seqs_ok(p.seqs) || !act || !dt_f32 || !A_log_f32 || !D_f32 || !state_f32 || !y || heads <= 0 || groups <= 0 ||
      N <= 0 || P <= 0 || (dtype != 0 && dtype != 1))
    return B200_ERR_ARG;
  if (heads % groups != 0 || P % 8 != 0 || heads > 65535 || num_seqs > 65535) return B200_ERR_SHAPE;
  return dtype == 0 ? ssm_scan_launch<__nv_bfloat16>(p, (cudaStream_t)stream)
                    : ssm_scan_launch<float>(p, (cudaStream_t)stream);
}

extern "C" int b200_ssm_gate_norm(const void* y, long long y_row_stride, const void* z, long long z_row_stride,
                                  const void* w_f32, void* out, long long out_row_stride, long long T, int heads, int P,
                                  int p_true, int parts, float eps, int norm_first, int dtype, void* stream) {
  using namespace b200;
  if (!y || !z || !w_f32 || !out || T < 0 || heads <= 0 || P <= 0 || p_true <= 0 || p_true > P || parts <= 0 ||
      (dtype != 0 && dtype != 1))
    return B200_ERR_ARG;
  if ((heads * p_true) % parts != 0 || P % 8 != 0 || y_row_stride % 8 != 0 || z_row_stride % 8 != 0 ||
      out_row_stride % 8 != 0 || parts > 65535 || T > 0x7fffffffLL)
    return B200_ERR_SHAPE;
  if (T == 0) return B200_OK;
  SsmGateNormParams p{y, z, y_row_stride, z_row_stride, out_row_stride, (const float*)w_f32, out, heads, P, p_true,
                      parts, eps, norm_first};
  const int n = heads * p_true / parts;
  auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (dtype == 0 && p_true == P && n % 8 == 0 && n <= 2048 && aligned(y) && aligned(z) && aligned(out) && aligned(w_f32)) {
    const long long pairs = T * parts;
    if (n <= 64) return ssm_gate_norm_narrow<8>(p, pairs, (cudaStream_t)stream);
    if (n <= 128) return ssm_gate_norm_narrow<16>(p, pairs, (cudaStream_t)stream);
    if (n <= 256) return ssm_gate_norm_narrow<32>(p, pairs, (cudaStream_t)stream);
    launch_k(norm_first ? ssm_gate_norm_warp_kernel<true> : ssm_gate_norm_warp_kernel<false>,
             dim3((unsigned)((pairs + 7) / 8)), dim3(256), 0, (cudaStream_t)stream, p, pairs);
    return launch_status();
  }
  const int threads = n <= 512 ? 64 : (n <= 2048 ? 128 : 256);
  if (dtype == 0)
    launch_k(ssm_gate_norm_kernel<__nv_bfloat16>, dim3((unsigned)T, (unsigned)parts), dim3(threads), 0,
             (cudaStream_t)stream, p);
  else
    launch_k(ssm_gate_norm_kernel<float>, dim3((unsigned)T, (unsigned)parts), dim3(threads), 0, (cudaStream_t)stream, p);
  return launch_status();
}
