// Hyper-connections: a residual made of NS parallel fp32 streams per token, with the pre-norm of the next sublayer.
//
// Between two sublayers, for every token (streams x_s, output y of the sublayer just done):
//     x_t <- sum_s mix[s, t] x_s + m * out[t] * y              (skipped when there is no y: start of the model)
//     u    = sum_s in[s] x_s                                   (the next sublayer's input; in = 1 at the end)
//     xn   = u / sqrt(mean(u^2) + eps) * (1 + w)               (norm weight stored around zero)
// One CTA per token does all of it in fp32: the streams are read and written once, y read once, xn written once.
// NS = 1 with mix = in = out = 1 is the ordinary residual x + m * y.
//
// Start of the model: the streams are NS copies of the token's embedding row (ids given, no y).
// End of the model: `rows` picks the tokens whose final norm is wanted; nothing is written back to the streams.
//
// Algorithmic bytes per token: 8 NS W (streams) + b W (y) + b W (xn), b = 2 or 4: the roofline is HBM bandwidth.
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int HYPER_CHUNKS = 8;   // register chunks per thread: W <= threads * HYPER_CHUNKS * 4

struct HyperParams {
  float* streams;             // [T, NS, W]
  const void* y;              // [T, y_stride] or null
  long long y_stride;
  const void* embed;          // [vocab, W] or null
  const long long* ids;       // [T]
  long long vocab;
  const int* rows;            // [R] source token of each output row, or null (row r is token r)
  long long num_tokens;       // bound of the rows / of the grid
  const float* mix;           // [NS, NS], [from, to]
  const float* out_w;         // [NS]
  float m;
  const float* in_w;          // [NS] or null (ones)
  const float* norm_w;        // [W] around zero, or null (no xn)
  float eps;
  void* xn;                   // [R, xn_stride]; columns W .. xn_cols are zeroed
  long long xn_stride;
  int xn_cols;
  int W;
  int write_back;
};

template <typename T>
__device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <>
__device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
template <>
__device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  unpack_bf2(t.x, v[0], v[1]);
  unpack_bf2(t.y, v[2], v[3]);
}
template <typename T>
__device__ __forceinline__ void store4(T* p, const float (&v)[4]);
template <>
__device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]));
}
template <typename T>
__device__ __forceinline__ float to_f32(T v) { return (float)v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v) { return (T)v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return f2bf(v); }

template <int NS, typename T>
__global__ void __launch_bounds__(1024) hyper_step_kernel(const HyperParams p) {
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
  float mix[NS][NS], outw[NS], inw[NS];
#pragma unroll
  for (int s = 0; s < NS; ++s) {
    inw[s] = p.in_w ? p.in_w[s] : 1.f;
    outw[s] = p.y ? p.m * p.out_w[s] : 0.f;
#pragma unroll
    for (int q = 0; q < NS; ++q) mix[s][q] = p.y ? p.mix[s * NS + q] : 0.f;
  }
  const T* yrow = p.y ? reinterpret_cast<const T*>(p.y) + t * p.y_stride : nullptr;
  const T* erow = nullptr;
  if (p.ids) {
    long long id = p.ids[t];
    if (id < 0 || id >= p.vocab) {
      if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, (int)id);
      id = 0;
    }
    erow = reinterpret_cast<const T*>(p.embed) + id * W;
  }
  float* srow = p.streams + t * (long long)NS * W;
  float u[HYPER_CHUNKS][4];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < HYPER_CHUNKS; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    u[c][0] = u[c][1] = u[c][2] = u[c][3] = 0.f;
    if (i >= W) continue;
    float x[NS][4];
    if (erow) {
      float e[4];
      if (W % 4 == 0) load4(erow + i, e);
      else
#pragma unroll
        for (int k = 0; k < 4; ++k) e[k] = i + k < W ? to_f32(erow[i + k]) : 0.f;
#pragma unroll
      for (int s = 0; s < NS; ++s)
#pragma unroll
        for (int k = 0; k < 4; ++k) x[s][k] = e[k];
    } else {
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        if (W % 4 == 0) load4(srow + (long long)s * W + i, x[s]);
        else
#pragma unroll
          for (int k = 0; k < 4; ++k) x[s][k] = i + k < W ? srow[(long long)s * W + i + k] : 0.f;
      }
    }
    if (yrow) {
      float y[4], n[NS][4];
      if (W % 4 == 0) load4(yrow + i, y);
      else
#pragma unroll
        for (int k = 0; k < 4; ++k) y[k] = i + k < W ? to_f32(yrow[i + k]) : 0.f;
#pragma unroll
      for (int q = 0; q < NS; ++q)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          float a = outw[q] * y[k];
#pragma unroll
          for (int s = 0; s < NS; ++s) a = fmaf(mix[s][q], x[s][k], a);
          n[q][k] = a;
        }
#pragma unroll
      for (int q = 0; q < NS; ++q)
#pragma unroll
        for (int k = 0; k < 4; ++k) x[q][k] = n[q][k];
    }
    if (p.write_back) {
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        if (W % 4 == 0) store4(srow + (long long)s * W + i, x[s]);
        else
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (i + k < W) srow[(long long)s * W + i + k] = x[s][k];
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      float a = 0.f;
#pragma unroll
      for (int s = 0; s < NS; ++s) a = fmaf(inw[s], x[s][k], a);
      u[c][k] = a;
      ss = fmaf(a, a, ss);
    }
  }
  if (!p.norm_w) return;
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)W + p.eps);
  T* xrow = reinterpret_cast<T*>(p.xn) + r * p.xn_stride;
#pragma unroll
  for (int c = 0; c < HYPER_CHUNKS; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i >= W) continue;
    float o[4];
    if (W % 4 == 0) {
      float w[4];
      load4(p.norm_w + i, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) o[k] = u[c][k] * inv * (1.f + w[k]);
      store4(xrow + i, o);
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (i + k < W) xrow[i + k] = from_f32<T>(u[c][k] * inv * (1.f + p.norm_w[i + k]));
    }
  }
  for (int i = W + threadIdx.x; i < p.xn_cols; i += blockDim.x) xrow[i] = from_f32<T>(0.f);
}

template <typename T>
inline int hyper_launch(const HyperParams& p, int ns, long long grid, int threads, cudaStream_t st) {
  const dim3 g((unsigned)grid), b((unsigned)threads);
  switch (ns) {
    case 1: launch_k(hyper_step_kernel<1, T>, g, b, 0, st, p); break;
    case 2: launch_k(hyper_step_kernel<2, T>, g, b, 0, st, p); break;
    case 3: launch_k(hyper_step_kernel<3, T>, g, b, 0, st, p); break;
    case 4: launch_k(hyper_step_kernel<4, T>, g, b, 0, st, p); break;
    case 5: launch_k(hyper_step_kernel<5, T>, g, b, 0, st, p); break;
    case 6: launch_k(hyper_step_kernel<6, T>, g, b, 0, st, p); break;
    case 7: launch_k(hyper_step_kernel<7, T>, g, b, 0, st, p); break;
    case 8: launch_k(hyper_step_kernel<8, T>, g, b, 0, st, p); break;
    default: return B200_ERR_SHAPE;
  }
  return launch_status();
}

}  // namespace b200

// dtype: 0 = bf16, 1 = fp32 (embed, y and xn; streams, coefficients and norm weights are always fp32).
extern "C" int b200_hyper_step(void* streams_f32, const void* y, long long y_row_stride, const void* embed,
                               const void* ids_i64, long long vocab, const void* rows_i32, long long num_tokens,
                               long long num_rows, int num_streams, int W, const void* mix_f32, const void* out_f32,
                               float m, const void* in_f32, const void* norm_w_f32, float eps, void* xn,
                               long long xn_row_stride, int xn_cols, int write_back, int dtype,
                               void* stream) {
  using namespace b200;
  if (!streams_f32 || num_tokens < 0 || num_rows < 0 || W <= 0 || num_streams <= 0 || (dtype != 0 && dtype != 1))
    return B200_ERR_ARG;
  if ((y != nullptr) == (ids_i64 != nullptr) || (ids_i64 && !embed) || (y && (!mix_f32 || !out_f32))) return B200_ERR_ARG;
  if (norm_w_f32 && (!xn || xn_cols < W)) return B200_ERR_ARG;
  if (rows_i32 && write_back) return B200_ERR_ARG;
  if (num_streams > 8 || num_rows > 0x7fffffffLL) return B200_ERR_SHAPE;
  if (num_rows == 0) return B200_OK;
  if (W % 4 == 0 && (y_row_stride % 4 != 0 || xn_row_stride % 4 != 0)) return B200_ERR_SHAPE;
  const int chunks = (W + 3) / 4;
  int threads = 64;
  while (threads < 256 && chunks > threads) threads <<= 1;
  while (threads < 1024 && chunks > threads * HYPER_CHUNKS) threads <<= 1;
  if (chunks > threads * HYPER_CHUNKS) return B200_ERR_SHAPE;
  HyperParams p{(float*)streams_f32, y, y_row_stride, embed, (const long long*)ids_i64, vocab, (const int*)rows_i32,
                num_tokens, (const float*)mix_f32, (const float*)out_f32, m, (const float*)in_f32,
                (const float*)norm_w_f32, eps, xn, xn_row_stride, xn_cols, W, write_back};
  return dtype == 0 ? hyper_launch<__nv_bfloat16>(p, num_streams, num_rows, threads, (cudaStream_t)stream)
                    : hyper_launch<float>(p, num_streams, num_rows, threads, (cudaStream_t)stream);
}
