// Between the projections and attention over per-head pages: short convolution, query / key norm, rotation, paged store.
//
// Projection row of a token: [q: H * DK | k: G * DK | ...], the values anywhere in it or none.  Every part is optional:
//   convolution   y_t = sum_j w[j] u_(t - taps + 1 + j) per channel of q and k, no bias, no activation, zeros before the
//                 sequence's first token; the last taps - 1 inputs of a sequence are its state (slots as in ssm.cuh)
//   values        columns of the row, or (keys as values) the convolved keys before norm and rotation; columns of the row may be
//                 mixed with another row of the same token, (1 - mix) v + mix first
//   norm          x / sqrt(mean(x^2) + eps) * w per head (w [DK], or none), or over all heads of q, and of k, at once
//                 (w [H * DK], [G * DK]).  The rotation that follows keeps lengths as long as rot_mag is 1, so a norm without
//                 a weight may as well be meant behind it
//   rotation      the first rot_dims columns of a head turn in pairs (2i, 2i + 1) or (i, i + rot_dims / 2) by
//                 position * inv_freq[i]; cosine and sine are multiplied by rot_mag
// q goes to rows of its own, k and v to their pages.  fp32 from the projection's values to the stored ones.
//
// LPH lanes own a head, eight neighbouring columns each (of every 8 * LPH); a CTA walks up to PREP_TOKENS tokens, PREP_BATCH
// rows requested together, with the convolution's weights and window in registers.  The convolution's state is moved on here
// in steps that bring one token per sequence, and by ssm_conv_shift_kernel afterwards in others (other CTAs may still need the
// old inputs).
// Algorithmic bytes per token: the row once, q, k and v once: HBM bandwidth.
#pragma once
#include "latent.cuh"   // latent_seq_of
#include "ssm.cuh"      // sequences and state slots, ssm_conv_shift_kernel

namespace b200 {

constexpr int PREP_MAX_WARPS = 10, PREP_TOKENS = 8, PREP_BATCH = 4, PREP_MAX_PAIRS = 128;
constexpr int PREP_NORM_NONE = 0, PREP_NORM_HEAD = 1, PREP_NORM_ALL = 2;

struct AttnPrepParams {
  SsmSeqs seqs;                // looked at with a convolution only
  const void* proj;
  long long proj_stride;
  int v_off;                   // first value column, -1: keys as values
  const long long* positions;
  const int* slot_mapping;     // -1 = do not store
  const float* conv_w;         // [taps, (H + G) * DK] or null
  void* conv_state;            // [slots, taps - 1, (H + G) * DK]
  int taps;
  int one_each;                // no sequence brings more than one token
  int shift;                   // ..: its state is moved on here
  int norm;
  const float* q_norm;
  const float* k_norm;
  int dim;                     // columns of a head that exist (the rest is padding and zero)
  float eps;
  const float* inv_freq;       // [rot_dims / 2]
  int rot_dims, rot_half;
  float rot_mag;
  void* q_out;                 // [T, H * DK]
  void* k_cache;               // [num_slots, G * DK]
  void* v_cache;               // [num_slots, G * DV]
  int heads, kv_heads, DK, DV;
  long long num_tokens, num_slots;
  int per_cta;                 // tokens of a CTA
  const void* v_first;         // [T, v_first_stride]: values mixed in, or null
  long long v_first_stride;
  float v_mix;
};

// Eight neighbouring values.
template <typename T>
struct Eight;
template <>
struct Eight<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void zero() { v = make_uint4(0, 0, 0, 0); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    unpack_bf2(v.x, f[0], f[1]);
    unpack_bf2(v.y, f[2], f[3]);
    unpack_bf2(v.z, f[4], f[5]);
    unpack_bf2(v.w, f[6], f[7]);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[8]) {
    *reinterpret_cast<uint4*>(p) =
        make_uint4(pack_bf2(f[0], f[1]), pack_bf2(f[2], f[3]), pack_bf2(f[4], f[5]), pack_bf2(f[6], f[7]));
  }
};
template <>
struct Eight<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = reinterpret_cast<const float4*>(p)[0];
    b = reinterpret_cast<const float4*>(p)[1];
  }
  __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&f)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
  }
};
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  Eight<float> e;
  e.load(p);
  e.get(f);
}

// 1 / sqrt(v) in a model that stores T.
template <typename T>
__device__ __forceinline__ float inv_sqrt_as(float v) { return sizeof(T) == 2 ? rsqrtf(v) : 1.f / sqrtf(v); }

// 8 * LPH * NC >= DK.  TAPS: 0 no convolution, 4 up to four taps (weights and window in registers), -1 any number.
template <typename T, int LPH, int NC, int TAPS>
__global__ void __launch_bounds__(PREP_MAX_WARPS * 32, 2) attn_prep_kernel(const AttnPrepParams p) {
  constexpr int B = PREP_BATCH, HPW = 32 / LPH;
  __shared__ __align__(16) float s_cos[PREP_TOKENS][PREP_MAX_PAIRS], s_sin[PREP_TOKENS][PREP_MAX_PAIRS];
  __shared__ float s_turn[PREP_MAX_WARPS][256 * NC];      // heads' columns, for pairs that are not eight columns apart
  __shared__ float s_red[PREP_TOKENS][2][PREP_MAX_WARPS], s_inv[PREP_TOKENS][2];
  __shared__ int s_j[PREP_TOKENS], s_slot[PREP_TOKENS];   // token's place in its sequence's step, state slot (-1: zeros)
  __shared__ int s_store[PREP_TOKENS];                    // cache slot, -1: none
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5, sub = lane / LPH, hl = lane % LPH;
  const long long t0 = (long long)blockIdx.x * p.per_cta;
  const int tokens = (int)min((long long)p.per_cta, p.num_tokens - t0);
  const int half = p.rot_dims >> 1, qk_heads = p.heads + p.kv_heads, channels = qk_heads * p.DK;
  const int h0 = warp * HPW + sub, stride = warps * HPW, rounds = (qk_heads + stride - 1) / stride;
  const T* proj = reinterpret_cast<const T*>(p.proj) + t0 * p.proj_stride;
  const T* state = reinterpret_cast<const T*>(p.conv_state);
  // Lanes without a head or without columns of it work on the head's first columns and store nothing.
  int col[NC];
  bool mine[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    mine[c] = (c * LPH + hl) * 8 < p.DK;
    col[c] = mine[c] ? (c * LPH + hl) * 8 : 0;
  }
  Eight<T> raw[B][NC];
  auto rows = [&](int q0, int h) {      // projection rows of a batch, all requested together
#pragma unroll
    for (int b = 0; b < B; ++b)
      if (q0 + b < tokens)
#pragma unroll
        for (int c = 0; c < NC; ++c) raw[b][c].load(proj + (q0 + b) * p.proj_stride + h * p.DK + col[c]);
  };
  rows(0, min(h0, qk_heads - 1));       // on their way while the tables are made
  for (int e = threadIdx.x; e < tokens * half; e += blockDim.x) {
    const int q = e / half, i = e - q * half;
    float s, c;
    sincosf((float)p.positions[t0 + q] * p.inv_freq[i], &s, &c);
    s_sin[q][i] = s * p.rot_mag;
    s_cos[q][i] = c * p.rot_mag;
  }
  if (threadIdx.x < tokens) {
    const long long t = t0 + threadIdx.x, store = p.slot_mapping[t];
    if (store >= p.num_slots) report_status(B200_STATUS_BAD_INDEX, (int)store);
    s_store[threadIdx.x] = store < p.num_slots ? (int)store : -1;
    if (TAPS != 0) {
      const int* qsl = p.seqs.query_start_loc;
      // one token each and no empty sequence before this one: the token's number is the sequence's
      const bool same = p.one_each && t < p.seqs.num_seqs && qsl[t] == (int)t && qsl[t + 1] == (int)t + 1;
      const int s = same ? (int)t : latent_seq_of(qsl, p.seqs.num_seqs, t);
      int first, len, slot;
      bool fresh;
      const bool live = ssm_seq(p.seqs, s, first, len, fresh, slot) && t < first + len;
      s_j[threadIdx.x] = live ? (int)(t - first) : 0;
      // a padding token convolves zeros; below -1: a fresh sequence, whose state is written but not read
      s_slot[threadIdx.x] = !live || slot < 0 ? -1 : fresh ? -2 - slot : slot;
    }
  }
  __syncthreads();

  constexpr int WT = TAPS == 4 ? 4 : 1, PAST = TAPS == 4 ? 3 : 1;
  float w[WT][NC][8], past[PAST][NC][8];        // the convolution's weights of a head, the inputs before the current one
  auto weights = [&](int h) {
    if constexpr (TAPS == 4) {
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          const int kk = k - (4 - p.taps);
#pragma unroll
          for (int e = 0; e < 8; ++e) w[k][c][e] = 0.f;
          if (kk >= 0) load8(p.conv_w + (long long)kk * channels + h * p.DK + col[c], w[k][c]);
        }
    }
  };
  // input i of the step of token q's sequence (negative: before the step, from its state)
  auto input = [&](int q, int h, int i, int c, float (&u)[8]) {
    const int ch = h * p.DK + col[c], slot = s_slot[q];
    Eight<T> r;
    r.zero();
    if (i >= 0) r.load(proj + (q - s_j[q] + i) * p.proj_stride + ch);
    else if (slot >= 0 && i + p.taps - 1 >= 0) r.load(state + ((long long)slot * (p.taps - 1) + i + p.taps - 1) * channels + ch);
    r.get(u);
  };
  auto window = [&](int q, int h) {             // the inputs before token q
    if constexpr (TAPS == 4) {
#pragma unroll
      for (int k = 0; k < 3; ++k)
#pragma unroll
        for (int c = 0; c < NC; ++c) input(q, h, s_j[q] - 3 + k, c, past[k][c]);
    }
  };
  // the (convolved) values of token q = q0 + b; zeros in columns the head does not have
  auto values = [&](int q, int b, int h, float (&x)[NC][8]) {
    if (TAPS == 4 && b > 0 && (s_j[q] == 0 || s_slot[q] == -1)) window(q, h);     // not the sequence of the token before
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      raw[b][c].get(x[c]);
      if constexpr (TAPS == 4) {
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float u = x[c][e];
          const float a = fmaf(w[1][c][e], past[1][c][e], w[0][c][e] * past[0][c][e]);
          x[c][e] = fmaf(w[3][c][e], u, fmaf(w[2][c][e], past[2][c][e], a));
          past[0][c][e] = past[1][c][e];
          past[1][c][e] = past[2][c][e];
          past[2][c][e] = u;
        }
      } else if constexpr (TAPS == -1) {
#pragma unroll
        for (int e = 0; e < 8; ++e) x[c][e] = 0.f;
        for (int k = 0; k < p.taps; ++k) {
          float u[8], wk[8];
          input(q, h, s_j[q] - (p.taps - 1) + k, c, u);
          load8(p.conv_w + (long long)k * channels + h * p.DK + col[c], wk);
#pragma unroll
          for (int e = 0; e < 8; ++e) x[c][e] = fmaf(wk[e], u[e], x[c][e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if (TAPS != 0 && sizeof(T) == 2) x[c][e] = round_bf(x[c][e]);   // a value of the model dtype, like a projected one
        if (!mine[c]) x[c][e] = 0.f;
      }
    }
  };
  auto squares = [&](const float (&x)[NC][8]) {
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int k = 0; k < 8; ++k) ss = fmaf(x[c][k], x[c][k], ss);
    return ss;
  };

  if (p.norm == PREP_NORM_ALL) {
    for (int q0 = 0; q0 < tokens; q0 += B) {
      float ss[B][2] = {};
      for (int r = 0; r < rounds; ++r) {
        const int hr = h0 + r * stride, h = min(hr, qk_heads - 1);
        if (r != 0 || q0 != 0) rows(q0, h);
        weights(h);
        window(q0, h);
#pragma unroll
        for (int b = 0; b < B; ++b) {
          if (q0 + b >= tokens) break;
          float x[NC][8];
          values(q0 + b, b, h, x);
          const float s = squares(x);
          if (hr < qk_heads) ss[b][h < p.heads ? 0 : 1] += s;
        }
      }
#pragma unroll
      for (int b = 0; b < B; ++b)
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const float s = warp_sum(ss[b][k]);
          if (lane == 0 && q0 + b < tokens) s_red[q0 + b][k][warp] = s;
        }
    }
    __syncthreads();
    if (threadIdx.x < 2 * tokens) {
      const int q = threadIdx.x >> 1, k = threadIdx.x & 1;
      float ss = 0.f;
      for (int i = 0; i < warps; ++i) ss += s_red[q][k][i];
      s_inv[q][k] = inv_sqrt_as<T>(ss / (float)((k ? p.kv_heads : p.heads) * p.dim) + p.eps);
    }
    __syncthreads();
  }
  const float per_dim = 1.f / (float)p.dim;
  for (int r = 0; r < rounds; ++r) {
    const int hr = h0 + r * stride, h = min(hr, qk_heads - 1), kvh = h - p.heads;
    const bool is_q = h < p.heads, live = hr < qk_heads;
    float nw[NC][8];
    weights(h);
    if (p.norm != PREP_NORM_NONE) {
      const float* src = is_q ? p.q_norm : p.k_norm;
      if (p.norm == PREP_NORM_ALL) src += (is_q ? h : kvh) * p.DK;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
#pragma unroll
        for (int e = 0; e < 8; ++e) nw[c][e] = 1.f;
        if (src) load8(src + col[c], nw[c]);
      }
    }
    T* qk_out = is_q ? reinterpret_cast<T*>(p.q_out) + (t0 * p.heads + h) * p.DK : reinterpret_cast<T*>(p.k_cache) + kvh * p.DK;
    T* v_out = reinterpret_cast<T*>(p.v_cache) + kvh * p.DV;
    for (int q0 = 0; q0 < tokens; q0 += B) {
      if (r != 0 || q0 != 0 || p.norm == PREP_NORM_ALL) rows(q0, h);
      if (q0 == 0 || s_j[q0] == 0 || s_slot[q0] == -1) window(q0, h);
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const int q = q0 + b;
        if (q >= tokens) break;
        float x[NC][8];
        values(q, b, h, x);
        if constexpr (TAPS == 4) {
          if (p.shift && p.taps > 1 && live && s_slot[q] != -1) {     // past: the last three inputs, this token's included
            const int slot = s_slot[q] < -1 ? -2 - s_slot[q] : s_slot[q];
            T* st = reinterpret_cast<T*>(p.conv_state) + (long long)slot * (p.taps - 1) * channels + h * p.DK;
#pragma unroll
            for (int k = 0; k < 3; ++k)
              if (k + 1 > 4 - p.taps)
#pragma unroll
                for (int c = 0; c < NC; ++c)
                  if (mine[c]) Eight<T>::store(st + (long long)(k - (4 - p.taps)) * channels + col[c], past[k][c]);
          }
        }
        const int slot = s_store[q];
        const bool write = live && (is_q || slot >= 0);
        if (write && !is_q && p.v_off < 0) {
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (mine[c]) Eight<T>::store(v_out + (long long)slot * p.kv_heads * p.DV + col[c], x[c]);
        }
        if (p.norm != PREP_NORM_NONE) {
          float inv;
          if (p.norm == PREP_NORM_ALL) {
            inv = s_inv[q][is_q ? 0 : 1];
          } else {
            float ss = squares(x);
#pragma unroll
            for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            inv = inv_sqrt_as<T>(fmaf(ss, per_dim, p.eps));
          }
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int k = 0; k < 8; ++k) x[c][k] = x[c][k] * inv * nw[c][k];
        }
        if (half > 0 && !p.rot_half) {
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (col[c] < p.rot_dims) {
              const float4 co = *reinterpret_cast<const float4*>(&s_cos[q][col[c] >> 1]);
              const float4 si = *reinterpret_cast<const float4*>(&s_sin[q][col[c] >> 1]);
              const float cs[4] = {co.x, co.y, co.z, co.w}, sn[4] = {si.x, si.y, si.z, si.w};
#pragma unroll
              for (int k = 0; k < 4; ++k)
                if (col[c] + 2 * k < p.rot_dims) {
                  const float u = x[c][2 * k], z = x[c][2 * k + 1];
                  x[c][2 * k] = u * cs[k] - z * sn[k];
                  x[c][2 * k + 1] = z * cs[k] + u * sn[k];
                }
            }
        } else if (NC == 1 && half > 0 && half % 8 == 0) {    // a lane's columns turn with those of another lane
          const bool low = col[0] < half;
          const int other = lane + (low ? half >> 3 : -(half >> 3)), pair = low ? col[0] : col[0] - half;
          float u[8];
#pragma unroll
          for (int k = 0; k < 8; ++k) u[k] = __shfl_sync(0xffffffffu, x[0][k], other);
          if (col[0] < p.rot_dims) {
            float co[8], si[8];
            load8(&s_cos[q][pair], co);
            load8(&s_sin[q][pair], si);
#pragma unroll
            for (int k = 0; k < 8; ++k) x[0][k] = fmaf(x[0][k], co[k], low ? -u[k] * si[k] : u[k] * si[k]);
          }
        } else if (half > 0) {
          float* turn = s_turn[warp] + sub * (LPH * 8 * NC);
          __syncwarp();
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (mine[c])
#pragma unroll
              for (int k = 0; k < 8; ++k) turn[col[c] + k] = x[c][k];
          __syncwarp();
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int k = 0; k < 8; ++k) {
              const int e = col[c] + k;
              if (e < half) x[c][k] = x[c][k] * s_cos[q][e] - turn[e + half] * s_sin[q][e];
              else if (e < p.rot_dims) x[c][k] = x[c][k] * s_cos[q][e - half] + turn[e - half] * s_sin[q][e - half];
            }
        }
        if (write) {
          T* dst = qk_out + (is_q ? (long long)q * p.heads : (long long)slot * p.kv_heads) * p.DK;
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (mine[c]) Eight<T>::store(dst + col[c], x[c]);
        }
      }
    }
  }
  if (p.v_off < 0) return;
  const int width = p.kv_heads * p.DV;       // a multiple of 8
  for (int q = 0; q < tokens; ++q) {
    if (s_store[q] < 0) continue;
    for (int e = threadIdx.x * 8; e < width; e += blockDim.x * 8) {
      Eight<T> v;
      float f[8];
      v.load(proj + q * p.proj_stride + p.v_off + e);
      v.get(f);
      if (p.v_first) {
        float first[8];
        v.load(reinterpret_cast<const T*>(p.v_first) + (t0 + q) * p.v_first_stride + e);
        v.get(first);
#pragma unroll
        for (int k = 0; k < 8; ++k) f[k] = fmaf(p.v_mix, first[k], (1.f - p.v_mix) * f[k]);
      }
      Eight<T>::store(reinterpret_cast<T*>(p.v_cache) + (long long)s_store[q] * width + e, f);
    }
  }
}

template <typename T, int LPH, int NC>
inline int attn_prep_launch(AttnPrepParams& p, cudaStream_t st) {
  p.per_cta = p.num_tokens >= 148 * PREP_TOKENS ? PREP_TOKENS : 1;
  const int need = ((p.heads + p.kv_heads) * LPH + 31) / 32;
  const dim3 grid((unsigned)((p.num_tokens + p.per_cta - 1) / p.per_cta));
  const dim3 block(32 * (need < PREP_MAX_WARPS ? need : PREP_MAX_WARPS));
  if (!p.conv_w) {
    launch_k(attn_prep_kernel<T, LPH, NC, 0>, grid, block, 0, st, p);
    return launch_status();
  }
  if constexpr (NC == 1) {
    if (p.taps <= 4) {
      launch_k(attn_prep_kernel<T, LPH, NC, 4>, grid, block, 0, st, p);
      return launch_status();
    }
  }
  launch_k(attn_prep_kernel<T, LPH, NC, -1>, grid, block, 0, st, p);
  return launch_status();
}

template <typename T>
inline int attn_prep_dispatch(AttnPrepParams& p, cudaStream_t st) {
  p.shift = p.conv_w && p.one_each && p.taps <= 4 && p.DK <= 256;
  int rc = p.DK <= 64    ? attn_prep_launch<T, 8, 1>(p, st)
           : p.DK <= 128 ? attn_prep_launch<T, 16, 1>(p, st)
           : p.DK <= 256 ? attn_prep_launch<T, 32, 1>(p, st)
                         : attn_prep_launch<T, 32, 2>(p, st);
  if (rc || !p.conv_w || p.shift || p.taps == 1) return rc;
  SsmConvParams c{};
  c.seqs = p.seqs;
  c.proj = p.proj;
  c.proj_stride = p.proj_stride;
  c.channels = (p.heads + p.kv_heads) * p.DK;
  c.taps = p.taps;
  c.conv_state = p.conv_state;
  launch_k(ssm_conv_shift_kernel<T>, dim3((unsigned)((c.channels + 127) / 128), (unsigned)p.seqs.num_seqs), dim3(128), 0, st, c);
  return launch_status();
}

}  // namespace b200

// See the head of this file.  proj rows [q: heads * DK | k: kv_heads * DK | ..]; v_off -1: keys as values (DV = DK).
// conv_w_f32 [taps, (heads + kv_heads) * DK] or NULL; conv_state [num_state_slots, taps - 1, the same] (unused with one
// tap); one_token_each: no sequence brings more than one token.  norm: 0 none, 1 per head (weights NULL: ones), 2 over all
// heads.  v_first NULL: values as they are projected.
extern "C" int b200_attn_prep(const void* proj, long long proj_row_stride, int v_off, const void* positions_i64,
                              const void* slot_mapping_i32, const void* conv_w_f32, void* conv_state, int taps,
                              const void* query_start_loc, const void* context_lens, const void* state_slots, int num_seqs,
                              int num_state_slots, int one_token_each, int norm, const void* q_norm_f32,
                              const void* k_norm_f32, int dim, float eps, const void* inv_freq_f32, int rot_dims,
                              int rot_half, float rot_mag, const void* v_first, long long v_first_row_stride, float v_mix,
                              void* q_out, void* k_cache, void* v_cache, long long T, int heads, int kv_heads, int DK, int DV,
                              long long num_slots, int dtype, void* stream) {
  using namespace b200;
  if (!proj || !positions_i64 || !slot_mapping_i32 || !q_out || !k_cache || !v_cache || T < 0 || heads <= 0 || kv_heads <= 0 ||
      DK <= 0 || DV <= 0 || dim <= 0 || dim > DK || (dtype != 0 && dtype != 1) || norm < PREP_NORM_NONE ||
      norm > PREP_NORM_ALL || (norm == PREP_NORM_ALL && (!q_norm_f32 || !k_norm_f32)) || (!q_norm_f32 != !k_norm_f32) || (v_first && v_off < 0) || rot_dims < 0 || rot_dims > dim ||
      (rot_dims && !inv_freq_f32))
    return B200_ERR_ARG;
  if (conv_w_f32 && (taps < 1 || (taps > 1 && !conv_state) || !query_start_loc || !context_lens || !state_slots ||
                     num_seqs <= 0 || num_seqs > 65535))
    return B200_ERR_ARG;
  if (DK % 8 || DV % 8 || proj_row_stride % 8 || rot_dims % 2 || rot_dims > 2 * PREP_MAX_PAIRS || DK > 512 || v_off < -1 ||
      v_off % 8 > 0 || v_first_row_stride % 8 || (reinterpret_cast<uintptr_t>(v_first) & 15) || (v_off < 0 && DV != DK) || T > 0x7fffffffLL ||
      ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_out)) & 15))
    return B200_ERR_SHAPE;
  if (T == 0) return B200_OK;
  AttnPrepParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_state_slots},
                   proj, proj_row_stride, v_off, (const long long*)positions_i64, (const int*)slot_mapping_i32,
                   (const float*)conv_w_f32, conv_state, taps, one_token_each, 0, norm, (const float*)q_norm_f32,
                   (const float*)k_norm_f32, dim, eps, (const float*)inv_freq_f32, rot_dims, rot_half, rot_mag, q_out, k_cache, v_cache, heads,
                   kv_heads, DK, DV, T, num_slots, 1, v_first, v_first_row_stride, v_mix};
  const cudaStream_t st = (cudaStream_t)stream;
  return dtype == 0 ? attn_prep_dispatch<__nv_bfloat16>(p, st) : attn_prep_dispatch<float>(p, st);
}
