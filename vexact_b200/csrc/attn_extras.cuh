// What an attention layer may add around softmax(q k^T) v, as every kernel that offers it reads it:
//
//   mask      window of w tokens: position i sees the keys i - w + 1 .. i;  chunks of c tokens: position i sees the keys
//             j <= i of its own chunk, floor(j / c) = floor(i / c), counted from the sequence's first token (0: no limit)
//   cap       a score s becomes cap * tanh(s / cap)
//   sink      exp(sink[head]) is added to the denominator: a key without a value
//   gate      the head's output is multiplied by the sigmoid of one number per head, or of one per column
//
// All of it is fp32.  Kernels that keep scores in units of log2 get the cap in those units, cap * log2(e).
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int GATE_NONE = 0, GATE_HEAD = 1, GATE_COLUMN = 2;

// A cap and the coefficients of cap * tanh(s / cap) = s + c3 s^3 + c5 s^5 + c7 s^7 .. in the scores' units.
struct ScoreCap {
  float cap;               // 0: none
  float inv, small, c3, c5, c7;
};
inline ScoreCap score_cap(float cap) {
  if (!(cap > 0.f)) return {};
  const double q = 1.0 / ((double)cap * cap);
  return {cap, 1.f / cap, 0.2f * cap, (float)(-q / 3), (float)(2 * q * q / 15), (float)(-17 * q * q * q / 315)};
}

struct AttnExtras {
  ScoreCap cap;
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

// tanh in fp32.  Below 0.2 the odd Taylor polynomial through x^7 (the next term is below 1.2e-8), above it
// 1 - 2 / (e^(2 |x|) + 1) on the special-function unit (absolute error below 4e-7).
constexpr float TANH_SERIES_MAX = 0.2f;
__device__ __forceinline__ float tanh_series(float x, float c3 = -1.f / 3.f, float c5 = 2.f / 15.f, float c7 = -17.f / 315.f) {
  const float s = x * x;
  return fmaf(fmaf(fmaf(c7, s, c5), s, c3) * s, x, x);
}
__device__ __forceinline__ float tanh_exponential(float x) {
  return copysignf(1.f - __fdividef(2.f, __expf(2.f * fabsf(x)) + 1.f), x);
}
// tanh in a model that stores T (both forms and a selection: no branch).
template <typename T>
__device__ __forceinline__ float tanh_as(float x) {
  if (sizeof(T) == 4) return tanhf(x);
  const float a = tanh_series(x), b = tanh_exponential(x);
  return fabsf(x) < TANH_SERIES_MAX ? a : b;
}

// v[i] <- cap * tanh(v[i] / cap).  Which form an element gets depends on that element alone; rows of small scores, the usual
// case, pay for the polynomial only.
template <int N>
__device__ __forceinline__ void cap_scores(float (&v)[N], const ScoreCap& c) {
  float most[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < N; ++i) most[i & 3] = fmaxf(most[i & 3], fabsf(v[i]));
  if (fmaxf(fmaxf(most[0], most[1]), fmaxf(most[2], most[3])) < c.small) {
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = tanh_series(v[i], c.c3, c.c5, c.c7);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      if (fabsf(v[i]) < c.small) v[i] = tanh_series(v[i], c.c3, c.c5, c.c7);
      else v[i] = c.cap * tanh_exponential(v[i] * c.inv);
      if (i % 4 == 3) asm volatile("" : "+f"(v[i]), "+f"(v[i - 1]), "+f"(v[i - 2]), "+f"(v[i - 3]));   // few at a time
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

// Whether a layer needs the kernels' form with extras (EXTRAS); without it they know a window and nothing else.
inline bool attn_has_extras(const AttnExtras& x, int chunk) {
  return chunk > 0 || x.cap.cap > 0.f || x.sink || x.gate_mode != GATE_NONE;
}

inline bool attn_extras_ok(const AttnExtras& x) {
  return x.gate_mode >= GATE_NONE && x.gate_mode <= GATE_COLUMN && (x.gate != nullptr) == (x.gate_mode != GATE_NONE);
}

}  // namespace b200
