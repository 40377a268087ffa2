// What an attention layer may add around softmax(q k^T) v, as every kernel that offers it reads it:
//
//   mask      window of w tokens: position i sees the keys i - w + 1 .. i;  chunks of c tokens: position i sees the keys
//             j <= i of its own chunk, floor(j / c) = floor(i / c), counted from the sequence's first token (0: no limit);
//             beside either, the sequence's first `keep` tokens are seen from everywhere behind them
//   cap       a score s becomes cap * tanh(s / cap)
//   sink      exp(sink[head]) is added to the denominator: a key without a value
//   sigmoid   a key's weight is sigmoid(score + bias[head]) and nothing is divided by a sum of weights
//   scale     the head's output times a constant
//   gate      the head's output is multiplied by the sigmoid of one number per head, or of one per column
//
// All of it is fp32.  Kernels that keep scores in units of log2 get the cap in those units, cap * log2(e).
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int GATE_NONE = 0, GATE_HEAD = 1, GATE_COLUMN = 2;
// Forms of an attention kernel: softmax inside a window and nothing else, softmax with all of the above, sigmoid weights.
constexpr int ATTN_PLAIN = 0, ATTN_EXTRAS = 1, ATTN_SIGMOID = 2;

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
  const float* sigmoid_bias;   // [heads]: sigmoid weights; null: softmax
  float out_scale;
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

// Key j (of a causal walk) is seen from `pos`: n = visible_keys(window, chunk, pos).
__device__ __forceinline__ bool key_visible(uint32_t n, int keep, int pos, int j) {
  return (uint32_t)(pos - j) < (keep > 0 && j < keep ? 0x80000000u : n);
}

// Blocks of BN keys that some query of first .. last sees: `head` blocks from key 0 that hold kept tokens and lie before
// the window, then those from block `from`.
struct KeyBlocks {
  int head, from, count;
  __device__ __forceinline__ int at(int i) const { return i < head ? i : from + (i - head); }
};
template <int BN>
__device__ __forceinline__ KeyBlocks key_blocks(int window, int chunk, int keep, int first, int last) {
  KeyBlocks k;
  k.from = first_visible(window, chunk, first) / BN;
  k.head = keep > 0 ? min((keep + BN - 1) / BN, k.from) : 0;
  k.count = last / BN + 1 - k.from + k.head;
  return k;
}

// Sigmoid weights of scores in units of log2 (bias included), w[i] = 1 / (1 + 2^-v[i]); two share a reciprocal.  2^-v is
// kept below 2^60, so that a product of two stays in range; weights below 2^-60 come out as 2^-60.  Keys that are not seen
// (va, vb) weigh nothing, and what their scores hold does not reach the other key's rounding.
__device__ __forceinline__ void sigmoid_pair(float& a, float& b, bool va = true, bool vb = true) {
  a = va ? a : -INFINITY;
  b = vb ? b : -INFINITY;
  float ea, eb;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(ea) : "f"(fminf(-a, 60.f)));
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(eb) : "f"(fminf(-b, 60.f)));
  const float da = 1.f + ea, db = 1.f + eb;
  float inv;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(inv) : "f"(da * db));
  a = va ? db * inv : 0.f;
  b = vb ? da * inv : 0.f;
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

// The form of the kernels that a layer needs.
inline int attn_form(const AttnExtras& x, int chunk, int keep) {
  if (x.sigmoid_bias) return ATTN_SIGMOID;
  return chunk > 0 || keep > 0 || x.cap.cap > 0.f || x.sink || x.gate_mode != GATE_NONE || x.out_scale != 1.f ? ATTN_EXTRAS
                                                                                                       : ATTN_PLAIN;
}

inline bool attn_extras_ok(const AttnExtras& x) {
  return x.gate_mode >= GATE_NONE && x.gate_mode <= GATE_COLUMN && (x.gate != nullptr) == (x.gate_mode != GATE_NONE) &&
         !(x.sink && x.sigmoid_bias);
}

}  // namespace b200
