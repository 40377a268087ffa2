// Between the projections and attention over per-head pages: short convolution, query / key norm, rotation, paged store.
//
// Projection row of a token: [q: H * DK | k: G * DK | ...], the values anywhere in it or none.  Every part is optional:
//   convolution   y_t = sum_j w[j] u_(t - taps + 1 + j) per channel of q and k, no bias, no activation, zeros before the
//                 sequence's first token; the last taps - 1 inputs of a sequence are its state (slots as in ssm.cuh)
//   values        columns of the row, or (keys as values) the convolved keys before norm and rotation
//   norm          x / sqrt(mean(x^2) + eps) * w per head (w [DK]), or over all heads of q, and of k, at once (w [H * DK],
//                 [G * DK])
//   rotation      the first rot_dims columns of a head turn in pairs (2i, 2i + 1) or (i, i + rot_dims / 2) by
//                 position * inv_freq[i]; cosine and sine are multiplied by rot_mag
// q goes to rows of its own, k and v to their pages.  fp32 from the projection's values to the stored ones.
//
// A warp owns heads, a lane VEC neighbouring columns of every 32 * VEC; a CTA walks up to PREP_TOKENS tokens, PREP_BATCH
// rows requested together, with the convolution's weights and window in registers.  The convolution's state is moved on here in steps that bring one token per sequence,
// and by ssm_conv_shift_kernel afterwards in others (other CTAs may still need the old inputs).
// Algorithmic bytes per token: the row once, q, k and v once: HBM bandwidth.
#pragma once
#include "latent.cuh"   // latent_seq_of
#include "ssm.cuh"      // sequences and state slots, ssm_conv_shift_kernel

namespace b200 {

constexpr int PREP_WARPS = 8, PREP_TOKENS = 8, PREP_BATCH = 4, PREP_MAX_PAIRS = 128;
constexpr int PREP_REGISTER_NC = 2;      // heads of up to 256 columns keep four taps in registers
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
  int taps, shift;             // shift: every sequence brings one token, its state is moved on here
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
};

template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    load4(p, v);
  } else if constexpr (sizeof(T) == 2) {
    unpack_bf2(*reinterpret_cast<const uint32_t*>(p), v[0], v[1]);
  } else {
    const float2 t = *reinterpret_cast<const float2*>(p);
    v[0] = t.x;
    v[1] = t.y;
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) store4(p, v);
  else if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf2(v[0], v[1]);
  else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}

// VEC * 32 * NC >= DK.  TAPS: 0 no convolution, 4 up to four taps (weights and window in registers), -1 any number.
template <typename T, int VEC, int NC, int TAPS>
__global__ void __launch_bounds__(PREP_WARPS * 32) attn_prep_kernel(const AttnPrepParams p) {
  constexpr int B = PREP_BATCH;
  __shared__ float s_cos[PREP_TOKENS][PREP_MAX_PAIRS], s_sin[PREP_TOKENS][PREP_MAX_PAIRS];
  __shared__ float s_turn[PREP_WARPS][VEC * 32 * NC];     // a head's columns, for pairs that lie in different lanes
  __shared__ float s_red[PREP_TOKENS][2][PREP_WARPS];
  __shared__ int s_j[PREP_TOKENS], s_slot[PREP_TOKENS];   // token's place in its sequence's step, state slot (-1: zeros)
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long t0 = (long long)blockIdx.x * p.per_cta;
  const int tokens = (int)min((long long)p.per_cta, p.num_tokens - t0);
  const int half = p.rot_dims >> 1, channels = (p.heads + p.kv_heads) * p.DK;
  const int qk_heads = p.heads + p.kv_heads, stride = PREP_WARPS * gridDim.y, h0 = blockIdx.y * PREP_WARPS + warp;
  const T* proj = reinterpret_cast<const T*>(p.proj);
  const T* state = reinterpret_cast<const T*>(p.conv_state);
  int cols[NC];                // this lane's columns of a head, clamped
  bool mine[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    mine[c] = (c * 32 + lane) * VEC < p.DK;
    cols[c] = mine[c] ? (c * 32 + lane) * VEC : 0;
  }
  // projection rows of the batch q0 .. q0 + B - 1, all requested together
  auto rows = [&](int q0, int h, float (&x)[B][NC][VEC]) {
#pragma unroll
    for (int b = 0; b < B; ++b)
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        load_vec<T, VEC>(proj + (t0 + min(q0 + b, tokens - 1)) * p.proj_stride + h * p.DK + cols[c], x[b][c]);
        if (!mine[c])
#pragma unroll
          for (int k = 0; k < VEC; ++k) x[b][c][k] = 0.f;
      }
  };
  float x[B][NC][VEC];
  if (h0 < qk_heads) rows(0, h0, x);         // on their way while the tables are made
  for (int e = threadIdx.x; e < tokens * half; e += PREP_WARPS * 32) {
    const int q = e / half, i = e - q * half;
    float s, c;
    sincosf((float)p.positions[t0 + q] * p.inv_freq[i], &s, &c);
    s_sin[q][i] = s * p.rot_mag;
    s_cos[q][i] = c * p.rot_mag;
  }
  if (TAPS != 0 && threadIdx.x < tokens) {
    const long long t = t0 + threadIdx.x;
    const int s = latent_seq_of(p.seqs.query_start_loc, p.seqs.num_seqs, t);
    int first, len, slot;
    bool fresh;
    const bool live = ssm_seq(p.seqs, s, first, len, fresh, slot) && t < first + len;
    s_j[threadIdx.x] = live ? (int)(t - first) : 0;
    // a padding token convolves zeros; below -1: a fresh sequence, whose state is written but not read
    s_slot[threadIdx.x] = !live || slot < 0 ? -1 : fresh ? -2 - slot : slot;
  }
  __syncthreads();

  constexpr int WT = TAPS == 4 ? 4 : 1, PAST = TAPS == 4 ? 3 : 1;
  float w[WT][NC][VEC], past[PAST][NC][VEC];     // the convolution's weights of a head, the inputs before the current one
  auto weights = [&](int h) {
    if constexpr (TAPS == 4) {
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          const int kk = k - (4 - p.taps);
#pragma unroll
          for (int e = 0; e < VEC; ++e) w[k][c][e] = 0.f;
          if (kk >= 0 && mine[c]) load_vec<float, VEC>(p.conv_w + (long long)kk * channels + h * p.DK + cols[c], w[k][c]);
        }
    }
  };
  // input i of the step of token q's sequence (negative: before the step, from its state), columns of group c
  auto input = [&](int q, int h, int i, int c, float (&u)[VEC]) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) u[k] = 0.f;
    if (!mine[c]) return;
    const int ch = h * p.DK + cols[c], slot = s_slot[q];
    if (i >= 0) load_vec<T, VEC>(proj + (t0 + q - s_j[q] + i) * p.proj_stride + ch, u);
    else if (slot >= 0 && i + p.taps - 1 >= 0) load_vec<T, VEC>(state + ((long long)slot * (p.taps - 1) + i + p.taps - 1) * channels + ch, u);
  };
  // x: the inputs of token q -> the convolution's values
  auto convolve = [&](int q, int h, float (&x)[NC][VEC]) {
    if constexpr (TAPS == 4) {
      if (q == 0 || s_j[q] == 0 || s_slot[q] == -1) {      // the window does not go on from the token before
#pragma unroll
        for (int k = 0; k < 3; ++k)
#pragma unroll
          for (int c = 0; c < NC; ++c) input(q, h, s_j[q] - 3 + k, c, past[k][c]);
      }
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const float u = x[c][e];
          x[c][e] = fmaf(w[3][c][e], u, fmaf(w[2][c][e], past[2][c][e], fmaf(w[1][c][e], past[1][c][e], w[0][c][e] * past[0][c][e])));
          past[0][c][e] = past[1][c][e];
          past[1][c][e] = past[2][c][e];
          past[2][c][e] = u;
        }
    } else if constexpr (TAPS == -1) {
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float a[VEC] = {};
        for (int k = 0; k < p.taps; ++k) {
          float u[VEC], wk[VEC];
          input(q, h, s_j[q] - (p.taps - 1) + k, c, u);
          load_vec<float, VEC>(p.conv_w + (long long)k * channels + h * p.DK + cols[c], wk);
#pragma unroll
          for (int e = 0; e < VEC; ++e) a[e] = fmaf(wk[e], u[e], a[e]);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[c][e] = a[e];
      }
    }
    if constexpr (TAPS != 0 && sizeof(T) == 2) {     // a convolved value is a value of the model dtype, like a projected one
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[c][e] = round_bf(x[c][e]);
    }
  };
  auto squares = [&](const float (&x)[NC][VEC]) {
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(x[c][k], x[c][k], ss);
    return ss;
  };

  if (p.norm == PREP_NORM_ALL) {       // one CTA holds every head of its tokens (gridDim.y is 1)
    for (int q0 = 0; q0 < tokens; q0 += B) {
      float ss[B][2] = {};
      for (int h = h0; h < qk_heads; h += stride) {
        if (h != h0 || q0 != 0) rows(q0, h, x);
        weights(h);
#pragma unroll
        for (int b = 0; b < B; ++b) {
          if (q0 + b >= tokens) break;
          if (TAPS == 4 && b == 0 && q0 != 0)        // the window of another batch's head has gone
#pragma unroll
            for (int k = 0; k < PAST; ++k)
#pragma unroll
              for (int c = 0; c < NC; ++c) input(q0, h, s_j[q0] - 3 + k, c, past[k][c]);
          convolve(q0 + b, h, x[b]);
          ss[b][h < p.heads ? 0 : 1] += squares(x[b]);
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
  }
  for (int h = h0; h < qk_heads; h += stride) {
    const bool is_q = h < p.heads;
    const int kvh = h - p.heads;
    float nw[NC][VEC];
    weights(h);
    if (p.norm != PREP_NORM_NONE) {
      const float* src = is_q ? p.q_norm : p.k_norm;
      if (p.norm == PREP_NORM_ALL) src += (is_q ? h : kvh) * p.DK;
#pragma unroll
      for (int c = 0; c < NC; ++c) load_vec<float, VEC>(src + cols[c], nw[c]);
    }
    for (int q0 = 0; q0 < tokens; q0 += B) {
      if (h != h0 || q0 != 0 || p.norm == PREP_NORM_ALL) rows(q0, h, x);
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const int q = q0 + b;
        if (q >= tokens) break;
        float (&v)[NC][VEC] = x[b];
        convolve(q, h, v);
        if constexpr (TAPS == 4) {
          if (p.shift && p.taps > 1 && s_slot[q] != -1) {      // past: the last three inputs, this token's included
            const int slot = s_slot[q] < -1 ? -2 - s_slot[q] : s_slot[q];
            T* st = reinterpret_cast<T*>(p.conv_state) + (long long)slot * (p.taps - 1) * channels + h * p.DK;
#pragma unroll
            for (int k = 0; k < 3; ++k)
              if (k + 1 > 4 - p.taps)
#pragma unroll
                for (int c = 0; c < NC; ++c)
                  if (mine[c]) store_vec<T, VEC>(st + (long long)(k - (4 - p.taps)) * channels + cols[c], past[k][c]);
          }
        }
        const long long t = t0 + q;
        long long slot = p.slot_mapping[t];
        if (slot >= p.num_slots) {
          if (lane == 0 && h == h0) report_status(B200_STATUS_BAD_INDEX, (int)slot);
          slot = -1;
        }
        if (!is_q && slot < 0) continue;
        if (!is_q && p.v_off < 0) {
          T* dst = reinterpret_cast<T*>(p.v_cache) + (slot * p.kv_heads + kvh) * p.DV;
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (mine[c]) store_vec<T, VEC>(dst + cols[c], v[c]);
        }
        if (p.norm != PREP_NORM_NONE) {
          float ss = 0.f, n = (float)p.dim;
          if (p.norm == PREP_NORM_HEAD) {
            ss = warp_sum(squares(v));
          } else {
#pragma unroll
            for (int k = 0; k < PREP_WARPS; ++k) ss += s_red[q][is_q ? 0 : 1][k];
            n *= (float)(is_q ? p.heads : p.kv_heads);
          }
          const float inv = 1.f / sqrtf(ss / n + p.eps);
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[c][k] = v[c][k] * inv * nw[c][k];
        }
        if (half > 0 && p.rot_half) {
          __syncwarp();
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (mine[c] && cols[c] < p.rot_dims) {
#pragma unroll
              for (int k = 0; k < VEC; ++k) s_turn[warp][cols[c] + k] = v[c][k];
            }
          __syncwarp();
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
              const int col = cols[c] + k;
              if (col < half) v[c][k] = v[c][k] * s_cos[q][col] - s_turn[warp][col + half] * s_sin[q][col];
              else if (col < p.rot_dims) v[c][k] = v[c][k] * s_cos[q][col - half] + s_turn[warp][col - half] * s_sin[q][col - half];
            }
        } else if (half > 0) {
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int k = 0; k < VEC; k += 2) {
              const int col = cols[c] + k;
              if (col < p.rot_dims) {
                const float u = v[c][k], z = v[c][k + 1], co = s_cos[q][col >> 1], si = s_sin[q][col >> 1];
                v[c][k] = u * co - z * si;
                v[c][k + 1] = z * co + u * si;
              }
            }
        }
        T* dst = is_q ? reinterpret_cast<T*>(p.q_out) + (t * p.heads + h) * p.DK
                      : reinterpret_cast<T*>(p.k_cache) + (slot * p.kv_heads + kvh) * p.DK;
#pragma unroll
        for (int c = 0; c < NC; ++c)
          if (mine[c]) store_vec<T, VEC>(dst + cols[c], v[c]);
      }
    }
  }
  if (p.v_off < 0) return;
  const int width = p.kv_heads * p.DV;       // a multiple of 8
  for (int e = (int)(blockIdx.y * PREP_WARPS * 32 + threadIdx.x) * 4; e < width * tokens; e += (int)gridDim.y * PREP_WARPS * 32 * 4) {
    const int q = e / width, col = e - q * width;
    const long long slot = p.slot_mapping[t0 + q];
    if (slot < 0 || slot >= p.num_slots) continue;
    float v[4];
    load4(proj + (t0 + q) * p.proj_stride + p.v_off + col, v);
    store4(reinterpret_cast<T*>(p.v_cache) + slot * width + col, v);
  }
}

template <typename T, int VEC, int NC>
inline int attn_prep_launch(AttnPrepParams& p, cudaStream_t st) {
  p.per_cta = p.num_tokens >= 148 * PREP_TOKENS ? PREP_TOKENS : 1;
  const long long gx = (p.num_tokens + p.per_cta - 1) / p.per_cta;
  const int need = (p.heads + p.kv_heads + PREP_WARPS - 1) / PREP_WARPS;
  const dim3 grid((unsigned)gx, (unsigned)(p.norm == PREP_NORM_ALL ? 1 : need < 65535 ? need : 65535));
  const dim3 block(PREP_WARPS * 32);
  if (!p.conv_w) {
    launch_k(attn_prep_kernel<T, VEC, NC, 0>, grid, block, 0, st, p);
    return launch_status();
  }
  if constexpr (NC <= PREP_REGISTER_NC) {
    if (p.taps <= 4) {
      launch_k(attn_prep_kernel<T, VEC, NC, 4>, grid, block, 0, st, p);
      return launch_status();
    }
  }
  launch_k(attn_prep_kernel<T, VEC, NC, -1>, grid, block, 0, st, p);
  return launch_status();
}

template <typename T>
inline int attn_prep_dispatch(AttnPrepParams& p, int one_token_each, cudaStream_t st) {
  p.shift = p.conv_w && one_token_each && p.taps <= 4 && p.DK <= 128 * PREP_REGISTER_NC;
  int rc = p.DK <= 64    ? attn_prep_launch<T, 2, 1>(p, st)
           : p.DK <= 128 ? attn_prep_launch<T, 4, 1>(p, st)
           : p.DK <= 256 ? attn_prep_launch<T, 4, 2>(p, st)
                         : attn_prep_launch<T, 4, 8>(p, st);
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
// tap); one_token_each: no sequence brings more than one token.  norm: 0 none, 1 per head, 2 over all heads.
extern "C" int b200_attn_prep(const void* proj, long long proj_row_stride, int v_off, const void* positions_i64,
                              const void* slot_mapping_i32, const void* conv_w_f32, void* conv_state, int taps,
                              const void* query_start_loc, const void* context_lens, const void* state_slots, int num_seqs,
                              int num_state_slots, int one_token_each, int norm, const void* q_norm_f32,
                              const void* k_norm_f32, int dim, float eps, const void* inv_freq_f32, int rot_dims,
                              int rot_half, float rot_mag, void* q_out, void* k_cache, void* v_cache, long long T, int heads,
                              int kv_heads, int DK, int DV, long long num_slots, int dtype, void* stream) {
  using namespace b200;
  if (!proj || !positions_i64 || !slot_mapping_i32 || !q_out || !k_cache || !v_cache || T < 0 || heads <= 0 || kv_heads <= 0 ||
      DK <= 0 || DV <= 0 || dim <= 0 || dim > DK || (dtype != 0 && dtype != 1) || norm < PREP_NORM_NONE ||
      norm > PREP_NORM_ALL || (norm && (!q_norm_f32 || !k_norm_f32)) || rot_dims < 0 || rot_dims > dim ||
      (rot_dims && !inv_freq_f32))
    return B200_ERR_ARG;
  if (conv_w_f32 && (taps < 1 || (taps > 1 && !conv_state) || !query_start_loc || !context_lens || !state_slots ||
                     num_seqs <= 0 || num_seqs > 65535))
    return B200_ERR_ARG;
  if (DK % 8 || DV % 8 || proj_row_stride % 8 || rot_dims % 2 || rot_dims > 2 * PREP_MAX_PAIRS || DK > 1024 || v_off < -1 ||
      v_off % 4 > 0 || (v_off < 0 && DV != DK) || T > 0x7fffffffLL)
    return B200_ERR_SHAPE;
  if (T == 0) return B200_OK;
  AttnPrepParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_state_slots},
                   proj, proj_row_stride, v_off, (const long long*)positions_i64, (const int*)slot_mapping_i32,
                   (const float*)conv_w_f32, conv_state, taps, 0, norm, (const float*)q_norm_f32, (const float*)k_norm_f32,
                   dim, eps, (const float*)inv_freq_f32, rot_dims, rot_half, rot_mag, q_out, k_cache, v_cache, heads,
                   kv_heads, DK, DV, T, num_slots, 1};
  const cudaStream_t st = (cudaStream_t)stream;
  return dtype == 0 ? attn_prep_dispatch<__nv_bfloat16>(p, one_token_each, st) : attn_prep_dispatch<float>(p, one_token_each, st);
}
