// One residual stream (fp32) with a norm on both sides of every sublayer, fused across the boundary of two sublayers.
//
// For every token, with y the output of the sublayer just done:
//     x  <- x + y / sqrt(mean(y^2) + eps) * post            (start of the model: x = 0 and y the embedding row)
//     x  <- x + add                                         (optional vector, the same for every token)
//     xn  = x / sqrt(mean(x^2) + eps) * norm                (the next sublayer's input)
// y comes as rows, or as what a mixture of experts leaves: expert-sorted rows of which a token sums `topk` (found through
// scatter_index), plus a row of the shared expert; that sum is then never a tensor of its own.
//
// One CTA per token, everything in registers between the two reductions.  `rows` picks tokens at the end of a model;
// nothing is written back then.
//
// Without `post` (PRE) the sublayer's result is not normed, and may be multiplied column by column by a gate of the token:
//     x  <- x + y * sigmoid(gate + gate_bias) (+ add)       (start of the model: x = the embedding row)
//
// The norms may be dynamic tanh instead, tanh(alpha x) * w + b with one number alpha, which reduces nothing:
//     x <- x + tanh(post_alpha y) * post + post_bias (+ add),    xn = tanh(norm_alpha x) * norm + norm_bias
// A thread then owns four columns, keeps the norms' vectors in registers and walks tokens, ROWS at a time.  At the start of a model y is
// the embedding row times embed_scale, under either norm.
// Algorithmic bytes per token: 8 W (x) + b W (topk + shared rows of y) + b W (xn), b = 2 or 4: HBM bandwidth.
#pragma once
#include "attn_extras.cuh"   // tanh_as
#include "hyper.cuh"   // load4 / store4 / to_f32 / from_f32

namespace b200 {

struct ResidualParams {
  float* x;                   // [T, W]
  const void* y;              // [T or y_rows, y_stride], or null (then `extra` or ids)
  long long y_stride, y_rows;
  const int* scatter_index;   // [T, topk] rows of y to sum, or null (row t)
  int topk;
  const void* extra;          // [T, extra_stride] added to y, or null
  long long extra_stride;
  const void* embed;          // [vocab, W] or null
  const long long* ids;       // [T]
  long long vocab;
  const int* rows;            // [R] source token of each output row, or null (row r is token r)
  long long num_tokens;
  const float* post;          // [W]
  const float* add;           // [W] or null
  const float* norm_w;        // [W] or null (no xn)
  float eps;
  void* xn;                   // [R, xn_stride]; columns W .. xn_cols are zeroed
  long long xn_stride;
  int xn_cols;
  int W;
  int write_back;
  long long num_rows;
  float embed_scale;
  // dynamic tanh (residual_tanh_kernel)
  const float* post_bias;     // [W]
  const float* norm_bias;     // [W]
  float post_alpha, norm_alpha;
  // gate of the sublayer's result (PRE)
  const void* gate;           // [T, gate_stride] or null
  long long gate_stride;
  const float* gate_bias;     // [W] or null
};

template <typename T>
__device__ __forceinline__ void load4_tail(const T* p, int left, float (&v)[4]) {
#pragma unroll
  for (int k = 0; k < 4; ++k) v[k] = k < left ? to_f32(p[k]) : 0.f;
}

// CH: register chunks of four columns per thread (W <= threads * CH * 4); MAXT: threads at most; PICK: y is expert-sorted;
// PRE: no norm of y.
template <typename T, int CH, int MAXT, bool PICK, bool PRE>
__global__ void __launch_bounds__(MAXT) residual_step_kernel(const ResidualParams p) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const long long r = blockIdx.x;
  long long t = p.rows ? p.rows[r] : r;
  if (t < 0 || t >= p.num_tokens) {
    if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, (int)t);
    t = 0;
  }
  const int W = p.W;
  const bool vec = W % 4 == 0;
  auto get = [&](const auto* row, int i, float (&v)[4]) {
    if (vec) load4(row + i, v);
    else load4_tail(row + i, W - i, v);
  };
  const T* src = nullptr;      // the one row of y, or of the embedding
  if (p.ids) {
    long long id = p.ids[t];
    if (id < 0 || id >= p.vocab) {
      if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, (int)id);
      id = 0;
    }
    src = reinterpret_cast<const T*>(p.embed) + id * W;
  } else if (!PICK && p.y) {
    src = reinterpret_cast<const T*>(p.y) + t * p.y_stride;
  }
  const T* extra = p.extra ? reinterpret_cast<const T*>(p.extra) + t * p.extra_stride : nullptr;
  const int* pick = PICK ? p.scatter_index + t * p.topk : nullptr;
  float* xrow = p.x + t * (long long)W;
  int pos[8];                  // the token's rows of a mixture, looked up once
  if constexpr (PICK)
#pragma unroll
    for (int k = 0; k < 8; ++k) pos[k] = k < p.topk ? pick[k] : -1;
  float v[CH][4], x[CH][4], w[CH][4], nw[CH][4];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {   // every load that depends on nothing, ahead of the first use
    const int i = (c * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int k = 0; k < 4; ++k) v[c][k] = x[c][k] = w[c][k] = nw[c][k] = 0.f;
    if (i >= W) continue;
    if (src) get(src, i, v[c]);
    if (p.ids) {
#pragma unroll
      for (int k = 0; k < 4; ++k) v[c][k] *= p.embed_scale;
    } else {
      get(xrow, i, x[c]);
    }
    if constexpr (!PRE) {
      get(p.post, i, w[c]);
    } else if (p.gate) {          // w: the gate ahead of its sigmoid
      get(reinterpret_cast<const T*>(p.gate) + t * p.gate_stride, i, w[c]);
      float b[4] = {0.f, 0.f, 0.f, 0.f};
      if (p.gate_bias) get(p.gate_bias, i, b);
#pragma unroll
      for (int k = 0; k < 4; ++k) w[c][k] += b[k];
    }
    if (p.norm_w) get(p.norm_w, i, nw[c]);
  }
  auto add_row = [&](const T* row, int i, float (&a)[4]) {
    float e[4];
    get(row, i, e);
#pragma unroll
    for (int q = 0; q < 4; ++q) a[q] += e[q];
  };
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i >= W) continue;
    if constexpr (PICK) {
      auto one = [&](int row) {
        if (row >= 0 && row < p.y_rows) add_row(reinterpret_cast<const T*>(p.y) + row * p.y_stride, i, v[c]);
        else if (threadIdx.x == 0 && c == 0) report_status(B200_STATUS_BAD_INDEX, row);
      };
#pragma unroll
      for (int k0 = 0; k0 < 8; k0 += 4) {
        if (vec && k0 + 4 <= p.topk) {      // four rows requested together, added in order
          float e[4][4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int row = pos[k0 + k];
            const bool ok = row >= 0 && row < p.y_rows;
            if (!ok && threadIdx.x == 0 && c == 0) report_status(B200_STATUS_BAD_INDEX, row);
            load4(reinterpret_cast<const T*>(p.y) + (ok ? row : 0) * p.y_stride + i, e[k]);
            if (!ok) e[k][0] = e[k][1] = e[k][2] = e[k][3] = 0.f;
          }
#pragma unroll
          for (int k = 0; k < 4; ++k)
#pragma unroll
            for (int q = 0; q < 4; ++q) v[c][q] += e[k][q];
        } else {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (k0 + k < p.topk) one(pos[k0 + k]);
        }
      }
      for (int k = 8; k < p.topk; ++k) one(pick[k]);
    }
    if (extra) add_row(extra, i, v[c]);
    if constexpr (!PRE) {
#pragma unroll
      for (int k = 0; k < 4; ++k) ss = fmaf(v[c][k], v[c][k], ss);
    }
  }
  float inv_y = 1.f;
  if constexpr (!PRE) {
    ss = block_sum(ss, red);
    inv_y = 1.f / sqrtf(ss / (float)W + p.eps);
    ss = 0.f;
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i >= W) continue;
    float a[4] = {0.f, 0.f, 0.f, 0.f};
    if (p.add) get(p.add, i, a);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if constexpr (PRE) {
        const float s = !p.gate ? 1.f : sizeof(T) == 2 ? sigmoid_fast(w[c][k]) : 1.f / (1.f + expf(-w[c][k]));
        x[c][k] = x[c][k] + v[c][k] * s + a[k];
      } else {
        x[c][k] = x[c][k] + v[c][k] * inv_y * w[c][k] + a[k];
      }
      ss = fmaf(x[c][k], x[c][k], ss);      // columns past W are zero in every term
    }
    if (p.write_back) {
      if (vec) store4(xrow + i, x[c]);
      else
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (i + k < W) xrow[i + k] = x[c][k];
    }
  }
  if (!p.norm_w) return;
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)W + p.eps);
  T* orow = reinterpret_cast<T*>(p.xn) + r * p.xn_stride;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i >= W) continue;
    float o[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) o[k] = x[c][k] * inv * nw[c][k];
    if (vec) store4(orow + i, o);
    else
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (i + k < W) orow[i + k] = from_f32<T>(o[k]);
  }
  for (int i = W + threadIdx.x; i < p.xn_cols; i += blockDim.x) orow[i] = from_f32<T>(0.f);
}

// The boundary under dynamic tanh.  A thread owns four neighbouring columns; a CTA takes batches of ROWS tokens and, where y
// comes as rows, has the next batch on its way while it works on one.
template <typename T, int ROWS, bool PICK>
__global__ void __launch_bounds__(128) residual_tanh_kernel(const ResidualParams p) {
  constexpr bool AHEAD = ROWS > 1 && !PICK;
  pdl_trigger();
  pdl_wait();
  const int W = p.W, i = (blockIdx.y * 128 + threadIdx.x) * 4;
  const bool vec = W % 4 == 0;
  auto get = [&](const auto* row, float (&v)[4]) {
    if (vec) load4(row + i, v);
    else load4_tail(row + i, W - i, v);
  };
  const long long first = (long long)blockIdx.x * ROWS, stride = (long long)gridDim.x * ROWS;
  if (i >= W) {                // columns past the width: zeros
    if (p.norm_w)
      for (long long r0 = first; r0 < p.num_rows; r0 += stride)
        for (int q = 0; q < ROWS && r0 + q < p.num_rows; ++q)
          for (int k = i; k < min(i + 4, p.xn_cols); ++k) reinterpret_cast<T*>(p.xn)[(r0 + q) * p.xn_stride + k] = from_f32<T>(0.f);
    return;
  }
  auto token = [&](long long r) {
    r = min(r, p.num_rows - 1);
    if (!p.rows) return r;
    const long long t = p.rows[r];
    if (t >= 0 && t < p.num_tokens) return t;
    if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, (int)t);
    return 0ll;
  };
  // what the sublayer left (v) and the residual (x) of the batch that starts at r0
  auto fetch = [&](long long r0, float (&v)[ROWS][4], float (&x)[ROWS][4]) {
    long long tok[ROWS];
#pragma unroll
    for (int q = 0; q < ROWS; ++q) {
      const long long t = tok[q] = token(r0 + q);
#pragma unroll
      for (int k = 0; k < 4; ++k) v[q][k] = x[q][k] = 0.f;
      if (p.ids) {
        long long id = p.ids[t];
        if (id < 0 || id >= p.vocab) {
          if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, (int)id);
          id = 0;
        }
        get(reinterpret_cast<const T*>(p.embed) + id * W, v[q]);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[q][k] *= p.embed_scale;
      } else {
        get(p.x + t * (long long)W, x[q]);
        if (!PICK && p.y) get(reinterpret_cast<const T*>(p.y) + t * p.y_stride, v[q]);
      }
    }
    if constexpr (PICK) {        // expert-sorted rows: four of every token requested together, added in order
      for (int k0 = 0; k0 < p.topk; k0 += 4) {
        int pos[ROWS][4];
#pragma unroll
        for (int q = 0; q < ROWS; ++q)
#pragma unroll
          for (int k = 0; k < 4; ++k) pos[q][k] = k0 + k < p.topk ? p.scatter_index[tok[q] * p.topk + k0 + k] : -1;
#pragma unroll
        for (int q = 0; q < ROWS; ++q) {
          float e[4][4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int row = pos[q][k];
            const bool ok = row >= 0 && row < p.y_rows;
            if (!ok && k0 + k < p.topk && threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, row);
            e[k][0] = e[k][1] = e[k][2] = e[k][3] = 0.f;
            if (ok) get(reinterpret_cast<const T*>(p.y) + row * p.y_stride, e[k]);
          }
#pragma unroll
          for (int k = 0; k < 4; ++k)
#pragma unroll
            for (int j = 0; j < 4; ++j) v[q][j] += e[k][j];
        }
      }
    }
    if (p.extra) {
      float e[ROWS][4];
#pragma unroll
      for (int q = 0; q < ROWS; ++q) get(reinterpret_cast<const T*>(p.extra) + tok[q] * p.extra_stride, e[q]);
#pragma unroll
      for (int q = 0; q < ROWS; ++q)
#pragma unroll
        for (int k = 0; k < 4; ++k) v[q][k] += e[q][k];
    }
  };
  float v[ROWS][4], x[ROWS][4];
  if (first < p.num_rows) fetch(first, v, x);
  float w[4], wb[4], nw[4] = {}, nb[4] = {}, add[4] = {};
  get(p.post, w);
  get(p.post_bias, wb);
  if (p.norm_w) {
    get(p.norm_w, nw);
    get(p.norm_bias, nb);
  }
  if (p.add) get(p.add, add);
#pragma unroll
  for (int k = 0; k < 4; ++k) wb[k] += add[k];
  for (long long r0 = first; r0 < p.num_rows; r0 += stride) {
    float v2[ROWS][4], x2[ROWS][4];
    const bool more = r0 + stride < p.num_rows;
    if (AHEAD && more) fetch(r0 + stride, v2, x2);
#pragma unroll
    for (int q = 0; q < ROWS; ++q) {
      if (r0 + q >= p.num_rows) break;
      float o[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        x[q][k] += fmaf(tanh_as<T>(p.post_alpha * v[q][k]), w[k], wb[k]);
        o[k] = fmaf(tanh_as<T>(p.norm_alpha * x[q][k]), nw[k], nb[k]);
      }
      float* xrow = p.x + token(r0 + q) * (long long)W + i;
      T* orow = reinterpret_cast<T*>(p.xn) + (r0 + q) * p.xn_stride + i;
      if (vec) {
        if (p.write_back) store4(xrow, x[q]);
        if (p.norm_w) store4(orow, o);
      } else {
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          if (p.write_back && i + k < W) xrow[k] = x[q][k];
          if (p.norm_w && i + k < p.xn_cols) orow[k] = from_f32<T>(i + k < W ? o[k] : 0.f);
        }
      }
    }
    if (!more) break;
    if constexpr (AHEAD) {
#pragma unroll
      for (int q = 0; q < ROWS; ++q)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          v[q][k] = v2[q][k];
          x[q][k] = x2[q][k];
        }
    } else {
      fetch(r0 + stride, v, x);
    }
  }
}

template <typename T, bool PICK>
inline int residual_tanh_launch(const ResidualParams& p, cudaStream_t st) {
  constexpr int MANY = PICK ? 4 : 2, BATCHES = 8;
  const unsigned gy = (unsigned)(((p.norm_w ? p.xn_cols : p.W) + 511) / 512);
  const long long many = (p.num_rows + MANY * BATCHES - 1) / (MANY * BATCHES);
  if (many * gy >= 148 * 2)
    launch_k(residual_tanh_kernel<T, MANY, PICK>, dim3((unsigned)many, gy), dim3(128), 0, st, p);
  else
    launch_k(residual_tanh_kernel<T, 1, PICK>, dim3((unsigned)p.num_rows, gy), dim3(128), 0, st, p);
  return launch_status();
}

template <typename T, bool PICK, bool PRE = false>
inline int residual_launch(const ResidualParams& p, long long rows, cudaStream_t st) {
  if constexpr (!PRE) {
    if (!p.post) return residual_launch<T, PICK, true>(p, rows, st);
    if (p.post_bias) return residual_tanh_launch<T, PICK>(p, st);
  }
  const int chunks = (p.W + 3) / 4;
  const dim3 g((unsigned)rows);
  int threads = 64;
  while (threads < 256 && chunks > threads) threads <<= 1;
  if (chunks <= threads) launch_k(residual_step_kernel<T, 1, 256, PICK, PRE>, g, dim3(threads), 0, st, p);
  else if (chunks <= 512) launch_k(residual_step_kernel<T, 2, 256, PICK, PRE>, g, dim3(256), 0, st, p);
  else if (chunks <= 1024) launch_k(residual_step_kernel<T, 2, 512, PICK, PRE>, g, dim3(512), 0, st, p);
  else if (chunks <= 4096) launch_k(residual_step_kernel<T, 4, 1024, PICK, PRE>, g, dim3(1024), 0, st, p);
  else return B200_ERR_SHAPE;
  return launch_status();
}

}  // namespace b200

// dtype: 0 = bf16, 1 = fp32 (embed, y, extra and xn; the residual and the norm weights are always fp32).
extern "C" int b200_residual_step(void* x_f32, const void* y, long long y_row_stride, long long y_rows,
                                  const void* scatter_index_i32, int topk, const void* extra, long long extra_row_stride,
                                  const void* embed, const void* ids_i64, long long vocab, const void* rows_i32,
                                  long long num_tokens, long long num_rows, int W, const void* post_f32,
                                  const void* add_f32, const void* norm_w_f32, float eps, float embed_scale,
                                  const void* post_bias_f32, float post_alpha, const void* norm_bias_f32,
                                  float norm_alpha, const void* gate, long long gate_row_stride,
                                  const void* gate_bias_f32, void* xn, long long xn_row_stride, int xn_cols,
                                  int write_back, int dtype, void* stream) {
  using namespace b200;
  if (!x_f32 || num_tokens < 0 || num_rows < 0 || W <= 0 || (dtype != 0 && dtype != 1)) return B200_ERR_ARG;
  if ((y != nullptr) == (ids_i64 != nullptr) || (ids_i64 && (!embed || extra)) || (scatter_index_i32 && (!y || topk < 1)))
    return B200_ERR_ARG;
  if (post_bias_f32 && (!post_f32 || (norm_w_f32 && !norm_bias_f32))) return B200_ERR_ARG;
  if ((gate && (post_f32 || !y)) || (gate_bias_f32 && !gate)) return B200_ERR_ARG;
  if ((norm_w_f32 && (!xn || xn_cols < W)) || (rows_i32 && write_back)) return B200_ERR_ARG;
  if (num_rows > 0x7fffffffLL) return B200_ERR_SHAPE;
  if (num_rows == 0) return B200_OK;
  if (W % 4 == 0 && (y_row_stride % 4 || xn_row_stride % 4 || extra_row_stride % 4 || gate_row_stride % 4)) return B200_ERR_SHAPE;
  ResidualParams p{(float*)x_f32, y, y_row_stride, y_rows, (const int*)scatter_index_i32, topk, extra, extra_row_stride,
                   embed, (const long long*)ids_i64, vocab, (const int*)rows_i32, num_tokens, (const float*)post_f32,
                   (const float*)add_f32, (const float*)norm_w_f32, eps, xn, xn_row_stride, xn_cols, W, write_back,
                   num_rows, embed_scale, (const float*)post_bias_f32, (const float*)norm_bias_f32, post_alpha, norm_alpha, gate,
                   gate_row_stride, (const float*)gate_bias_f32};
  const cudaStream_t st = (cudaStream_t)stream;
  if (scatter_index_i32)
    return dtype == 0 ? residual_launch<__nv_bfloat16, true>(p, num_rows, st) : residual_launch<float, true>(p, num_rows, st);
  return dtype == 0 ? residual_launch<__nv_bfloat16, false>(p, num_rows, st) : residual_launch<float, false>(p, num_rows, st);
}
