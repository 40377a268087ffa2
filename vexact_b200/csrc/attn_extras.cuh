// What an attention layer may add around softmax(q k^T) v, as every kernel that offers it reads it:
//
//   mask      window of w tokens: position i sees the keys i - w + 1 .. i;  chunks of c tokens: position i sees the keys
//             j <= i of its own chunk, floor(j / c) = floor(i / c), counted from the sequence's first token (0: no limit)
//   cap       a score s becomes cap * tanh(s / cap)
//   sink      exp(sink[head]) is added to the denominator: a key without a value
//   gate      the head's output is multiplied by the sigmoid of one number per head, or of one per column
//
// All of it is fp32.  In the kernels that keep scores in units of log2, the caller passes scale / cap as the score's factor
// and cap * log2(e) as `cap` (without a cap scale * log2(e) and 0).
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int GATE_NONE = 0, GATE_HEAD = 1, GATE_COLUMN = 2;

struct AttnExtras {
  float cap;               // 0: none
  const float* sink;       // [heads] or null
  const void* gate;        // rows of the model dtype, gate_stride apart: [heads] or [heads * DV]; null with GATE_NONE
  long long gate_stride;
  int gate_mode;
};

// Keys that the query at `pos` sees, its own included, and the first of them.
__device__ __forceinline__ uint32_t visible_keys(int window, int chunk, int pos) {
  uint32_t n = window > 0 ? (uint32_t)window : 0x80000000u;
  if (chunk > 0) n = min(n, (uint32_t)(pos % chunk) + 1u);
  return n;
}
__device__ __forceinline__ int first_visible(int window, int chunk, int pos) {
  const int a = window > 0 ? max(0, pos - window + 1) : 0;
  return chunk > 0 ? max(a, pos - pos % chunk) : a;
}

// tanh in fp32.  Below 1/4 the odd Taylor polynomial through x^9 (the next term is below 3e-9), above it
// 1 - 2 / (e^(2 |x|) + 1) on the special-function unit (absolute error below 4e-7).
constexpr float TANH_SERIES_MAX = 0.25f;
__device__ __forceinline__ float tanh_series(float x) {
  const float s = x * x;
  float c = 62.f / 2835.f;
  c = fmaf(c, s, -17.f / 315.f);
  c = fmaf(c, s, 2.f / 15.f);
  c = fmaf(c, s, -1.f / 3.f);
  return fmaf(c * s, x, x);
}
__device__ __forceinline__ float tanh_exponential(float x) {
  return copysignf(1.f - __fdividef(2.f, __expf(2.f * fabsf(x)) + 1.f), x);
}
__device__ __forceinline__ float tanh_either(float x) {     // both, and a selection: no branch
  const float a = tanh_series(x), b = tanh_exponential(x);
  return fabsf(x) < TANH_SERIES_MAX ? a : b;
}
// tanh in a model that stores T.
template <typename T>
__device__ __forceinline__ float tanh_as(float x) {
  return sizeof(T) == 4 ? tanhf(x) : tanh_either(x);
}

// v[i] <- cap * tanh(v[i]), the exponential form only for groups of eight that need it.  Which form an element gets depends
// on that element alone.
template <int N>
__device__ __forceinline__ void cap_scores(float (&v)[N], float cap) {
  constexpr int G = N < 8 ? N : 8;
#pragma unroll
  for (int g = 0; g < N; g += G) {
    float most = 0.f;
#pragma unroll
    for (int i = 0; i < G; ++i) most = fmaxf(most, fabsf(v[g + i]));
    if (most < TANH_SERIES_MAX) {
#pragma unroll
      for (int i = 0; i < G; ++i) v[g + i] = cap * tanh_series(v[g + i]);
    } else {
#pragma unroll
      for (int i = 0; i < G; ++i) v[g + i] = cap * tanh_either(v[g + i]);
    }
  }
}

// What exp(sink) adds to a denominator that is kept relative to 2^m.
__device__ __forceinline__ float sink_term(const AttnExtras& x, int head, float m) {
  return x.sink ? exp2f(x.sink[head] * 1.4426950408889634f - m) : 0.f;
}

// Sigmoid of a gate that is stored in T.
__device__ __forceinline__ float sigmoid_fast(float g) { return __fdividef(1.f, 1.f + __expf(-g)); }
template <typename T>
__device__ __forceinline__ float gate_sigmoid(T g) {
  if constexpr (sizeof(T) == 2) return sigmoid_fast(bf2f(g));
  else return 1.f / (1.f + expf(-g));
}

inline bool attn_extras_ok(const AttnExtras& x) {
  return x.cap >= 0.f && x.gate_mode >= GATE_NONE && x.gate_mode <= GATE_COLUMN && (x.gate != nullptr) == (x.gate_mode != GATE_NONE);
}

}  // namespace b200
