// minGRU: a gated recurrence whose gates read the current token only, element by element over `width` channels,
//     z = sigmoid(zp + z_bias),  u = xp + x_bias,  c = u + 1/2 where u >= 0 and sigmoid(u) where u < 0,
//     S_t = (1 - z) S_(t-1) + z c,      out = S_t * silu(gp) * out_scale,
// with zp, xp and gp columns of a projection row.  The state is fp32, [slots, width]; sequences and state slots as in ssm.cuh.
//
//   gru_scan_kernel    token by token: decode, short portions, fp32 models
//   gru_maps_kernel,   long portions: the maps S -> a S + b of runs of tokens, then all runs at once, each from the state that
//   gru_walk_kernel    the maps before it give
//
// Algorithmic bytes per token: the three columns once, out once (and the state once in, once out per sequence): HBM bandwidth.
#pragma once
#include "ssm.cuh"
#include "ssm_chunk.cuh"   // cp.async

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
  long long group_rows;        // rows of the maps that belong to groups (gru_maps_kernel, gru_walk_kernel)
};

// Two neighbouring channels in one register pair: one instruction for both.
struct Two {
  unsigned long long v;
  __device__ __forceinline__ Two() {}
  __device__ __forceinline__ Two(float a, float b) { asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(a), "f"(b)); }
  __device__ __forceinline__ explicit Two(float a) : Two(a, a) {}
  __device__ __forceinline__ void get(float& a, float& b) const { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
};
__device__ __forceinline__ Two operator+(const Two& a, const Two& b) {
  Two r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
  return r;
}
__device__ __forceinline__ Two operator*(const Two& a, const Two& b) {
  Two r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
  return r;
}
__device__ __forceinline__ Two fma2(const Two& a, const Two& b, const Two& c) {
  Two r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return r;
}
// 2^min(x, 40) and 1 / x on the special-function unit, c where u >= 0 and s elsewhere.
__device__ __forceinline__ Two gru_ex2(const Two& x) {
  float a, b;
  x.get(a, b);
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(a) : "f"(fminf(a, 40.f)));
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(b) : "f"(fminf(b, 40.f)));
  return Two(a, b);
}
__device__ __forceinline__ Two gru_rcp(const Two& x) {
  float a, b;
  x.get(a, b);
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(a) : "f"(a));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(b) : "f"(b));
  return Two(a, b);
}
__device__ __forceinline__ Two gru_pick(const Two& u, const Two& c, const Two& s) {
  float ua, ub, ca, cb, sa, sb;
  u.get(ua, ub);
  c.get(ca, cb);
  s.get(sa, sb);
  return Two(ua >= 0.f ? ca : sa, ub >= 0.f ? cb : sb);
}

// a = 1 - z and b = z c of two channels and a token, and o = silu(g), in bf16 models: zp, xp and g as projected, zs = -log2(e)
// z_bias, xb = x_bias.  The sigmoids share a reciprocal; their exponentials are kept below 2^40, so that the product stays in
// range (a gate below 2^-40 comes out as 2^-40).  Without GATE a and b alone.
template <bool GATE>
__device__ __forceinline__ void gru_gates(const Two& zp, const Two& zs, const Two& xp, const Two& xb, const Two& g, Two& a, Two& b,
                                          Two& o) {
  const Two one(1.f), rate(-kLog2e);
  const Two u = xp + xb, ez = gru_ex2(fma2(zp, rate, zs)), dz = ez + one, du = gru_ex2(u * rate) + one;
  Two q;
  if constexpr (GATE) {
    const Two dg = gru_ex2(g * rate) + one, dzu = dz * du, inv = gru_rcp(dzu * dg);
    q = dg * inv;
    o = g * (dzu * inv);
  } else {
    q = gru_rcp(dz * du);
  }
  const Two z = du * q;
  a = ez * z;
  b = z * gru_pick(u, u + Two(0.5f), dz * q);
}
// The same of one channel in an fp32 model, zp and u behind their biases.
__device__ __forceinline__ void gru_gates_exact(float zp, float u, float g, float& a, float& b, float& o) {
  const float z = 1.f / (1.f + expf(-zp));
  a = 1.f / (1.f + expf(zp));
  b = z * (u >= 0.f ? u + 0.5f : 1.f / (1.f + expf(-u)));
  o = silu_f32(g);
}

// Four channels of a thread: biases as gru_gates takes them, projected values.
struct GruBias {
  Two zs[2], xb[2];
  __device__ __forceinline__ void load(const GruParams& p, int c) {
    float z[4], x[4];
    load4(p.z_bias + c, z);
    load4(p.x_bias + c, x);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      zs[k] = Two(z[2 * k], z[2 * k + 1]) * Two(-kLog2e);
      xb[k] = Two(x[2 * k], x[2 * k + 1]);
    }
  }
};
__device__ __forceinline__ void gru_unpack(const uint2& r, Two (&v)[2]) {
  float a, b;
  unpack_bf2(r.x, a, b);
  v[0] = Two(a, b);
  unpack_bf2(r.y, a, b);
  v[1] = Two(a, b);
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
  GruBias bias;
  if constexpr (sizeof(T) == 2) {
    bias.load(p, c);
  } else {
    load4(p.z_bias + c, zb);
    load4(p.x_bias + c, xb);
  }
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
      float a[4], b[4], o[4], y[4];
      if constexpr (sizeof(T) == 2) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          Two ta, tb, to;
          gru_gates<true>(Two(z[q][2 * k], z[q][2 * k + 1]), bias.zs[k], Two(x[q][2 * k], x[q][2 * k + 1]), bias.xb[k],
                          Two(g[q][2 * k], g[q][2 * k + 1]), ta, tb, to);
          ta.get(a[2 * k], a[2 * k + 1]);
          tb.get(b[2 * k], b[2 * k + 1]);
          to.get(o[2 * k], o[2 * k + 1]);
        }
      } else {
#pragma unroll
        for (int k = 0; k < 4; ++k) gru_gates_exact(z[q][k] + zb[k], x[q][k] + xb[k], g[q][k], a[k], b[k], o[k]);
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        S[k] = fmaf(a[k], S[k], b[k]);
        y[k] = S[k] * o[k] * p.out_scale;
      }
      store4(out + (long long)(j + q) * p.out_stride, y);
    }
  }
  if (st) store4(st, S);
}

// ------------------------------------------------------------------ runs of tokens
// A warp has GRU_CH neighbouring channels (a lane four of them) of a run of GRU_RUN tokens, whose columns it has copied into
// shared memory, all requested at once.  gru_maps_kernel composes the maps S -> a S + b of every run and of every group, the
// GRU_WARPS runs of a CTA; gru_walk_kernel finds the state ahead of its run by applying the maps of the groups before (a CTA's
// warps share the work) and of the runs between, and walks the tokens.  Runs and groups lie at multiples of their length in a
// sequence's step and are applied in an order that depends on their number alone.
//
// maps: rows of [width] (a, b), first those of groups, then those of runs.  Sequence s, t0 its first token of the step, has the
// group rows from t0 / GRU_GROUP + 2 s, its state at the step's start as the map to a constant and then its groups, and the run
// rows from t0 / GRU_RUN + s.
constexpr int GRU_RUN = 16, GRU_WARPS = 4, GRU_CH = 128, GRU_GROUP = GRU_WARPS * GRU_RUN;
// shared memory of a CTA that copies COLS of the columns z, x, g
constexpr int gru_smem(int cols) { return GRU_WARPS * GRU_RUN * cols * GRU_CH * 2; }

struct GruRun {
  int t0, len, slot, first;    // first: the run's first token in its sequence's step
  bool fresh, live, in;        // live: the run holds tokens; in: the lane's channels exist
  long long start, run;        // maps rows of the sequence's start and of the warp's run
  int c, cc;                   // the lane's first channel, and one to read from where it does not exist
};
// False: the CTA has nothing to do.
__device__ __forceinline__ bool gru_run(const GruParams& p, int warp, int lane, GruRun& r) {
  const int s = blockIdx.z;
  if (!ssm_seq(p.seqs, s, r.t0, r.len, r.fresh, r.slot) || r.len < p.min_len || r.len > p.max_len) return false;
  if ((int)blockIdx.y * GRU_GROUP >= r.len) return false;
  r.first = blockIdx.y * GRU_GROUP + warp * GRU_RUN;
  r.live = r.first < r.len;
  r.start = r.t0 / GRU_GROUP + 2ll * s;
  r.run = p.group_rows + r.t0 / GRU_RUN + s + blockIdx.y * GRU_WARPS + warp;
  r.c = blockIdx.x * GRU_CH + lane * 4;
  r.in = r.c < p.width;        // width is a multiple of 8
  r.cc = r.in ? r.c : 0;
  return true;
}
// Copies the first COLS of the columns z, x, g of a run of n tokens into the warp's [GRU_RUN][COLS][GRU_CH] of shared memory.
template <int COLS>
__device__ __forceinline__ void gru_fetch(const GruParams& p, const GruRun& r, int n, uint32_t smem) {
  const int lane = threadIdx.x & 31, c = blockIdx.x * GRU_CH + (lane & 15) * 8;
  const bool in = c < p.width;
  const __nv_bfloat16* src =
      reinterpret_cast<const __nv_bfloat16*>(p.proj) + (long long)(r.t0 + r.first) * p.proj_stride + (in ? c : 0);
#pragma unroll
  for (int i = 0; i < GRU_RUN * COLS / 2; ++i) {
    const int row = 2 * i + (lane >> 4), token = row / COLS, col = row - token * COLS;
    cp_async16(smem + (uint32_t)(row * GRU_CH + (lane & 15) * 8) * 2,
               src + (long long)min(token, n - 1) * p.proj_stride + (col == 0 ? p.z_off : col == 1 ? p.x_off : p.g_off), in);
  }
  cp_async_commit();
}

// Maps of four channels, and what comes out of applying one behind another.
struct GruMap {
  Two a[2], b[2];
  __device__ __forceinline__ void same() {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      a[k] = Two(1.f);
      b[k] = Two(0.f);
    }
  }
  __device__ __forceinline__ void then(const GruMap& m) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      b[k] = fma2(m.a[k], b[k], m.b[k]);
      a[k] = a[k] * m.a[k];
    }
  }
  // rows of (a, b) per channel
  __device__ __forceinline__ void load(const float2* p) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const float4 v = reinterpret_cast<const float4*>(p)[k];
      a[k] = Two(v.x, v.z);
      b[k] = Two(v.y, v.w);
    }
  }
  __device__ __forceinline__ void store(float2* p) const {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      float4 v;
      a[k].get(v.x, v.z);
      b[k].get(v.y, v.w);
      reinterpret_cast<float4*>(p)[k] = v;
    }
  }
};

__global__ void __launch_bounds__(GRU_WARPS * 32, 6) gru_maps_kernel(const GruParams p, float2* maps) {
  extern __shared__ __align__(16) uint8_t gru_raw[];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  GruRun r;
  if (!gru_run(p, warp, lane, r)) return;
  const int n = min(GRU_RUN, r.len - r.first);
  uint8_t* raw = gru_raw + warp * (GRU_RUN * 2 * GRU_CH * 2);
  const uint2* mine = reinterpret_cast<const uint2*>(raw) + lane;
  if (r.live) gru_fetch<2>(p, r, n, ptx::smem_u32(raw));
  GruBias bias;
  GruMap m, one;
  bias.load(p, r.cc);
  m.same();
  cp_async_wait<0>();
  __syncwarp();
#pragma unroll 4
  for (int j = 0; j < n; ++j) {
    Two z[2], x[2], unused;
    gru_unpack(mine[(2 * j) * (GRU_CH / 4)], z);
    gru_unpack(mine[(2 * j + 1) * (GRU_CH / 4)], x);
#pragma unroll
    for (int k = 0; k < 2; ++k) gru_gates<false>(z[k], bias.zs[k], x[k], bias.xb[k], unused, one.a[k], one.b[k], unused);
    m.then(one);
  }
  __syncwarp();
  if (r.live && r.in) m.store(maps + r.run * p.width + r.c);
  m.store(reinterpret_cast<float2*>(raw) + lane * 4);     // over the warp's copies
  __syncthreads();
  if (warp != 0 || !r.in) return;
  for (int w = 1; w < GRU_WARPS; ++w) {
    one.load(reinterpret_cast<const float2*>(gru_raw + w * (GRU_RUN * 2 * GRU_CH * 2)) + lane * 4);
    m.then(one);
  }
  float2* row = maps + r.start * p.width + r.c;
  m.store(row + (1ll + blockIdx.y) * p.width);
  if (blockIdx.y == 0) {
    float S[4] = {0.f, 0.f, 0.f, 0.f};
    if (r.slot >= 0 && !r.fresh) load4(p.state + (long long)r.slot * p.width + r.c, S);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      m.a[k] = Two(0.f);
      m.b[k] = Two(S[2 * k], S[2 * k + 1]);
    }
    m.store(row);
  }
}

__global__ void __launch_bounds__(GRU_WARPS * 32, 4) gru_walk_kernel(const GruParams p, const float2* maps) {
  extern __shared__ __align__(16) uint8_t gru_raw[];
  __shared__ __align__(16) float2 s_map[GRU_WARPS][GRU_CH];      // what the rows of a warp's share of the past compose to
  __shared__ __align__(16) float2 s_own[GRU_WARPS][GRU_CH];      // the maps of this CTA's runs
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  GruRun r;
  if (!gru_run(p, warp, lane, r)) return;
  const int n = min(GRU_RUN, r.len - r.first);
  const uint2* mine = reinterpret_cast<const uint2*>(gru_raw + warp * (GRU_RUN * 3 * GRU_CH * 2)) + lane;
  if (r.live) gru_fetch<3>(p, r, n, ptx::smem_u32(gru_raw) + warp * (GRU_RUN * 3 * GRU_CH * 2));   // while the state is found
  GruBias bias;
  bias.load(p, r.cc);
  const float2* row = maps + r.start * p.width + r.cc;
  // the start and the groups before this one, a share for each warp
  const int past = 1 + (int)blockIdx.y, share = (past + GRU_WARPS - 1) / GRU_WARPS;
  GruMap m, one;
  m.same();
#pragma unroll 8
  for (int i = warp * share; i < min(past, (warp + 1) * share); ++i) {
    one.load(row + (long long)i * p.width);
    m.then(one);
  }
  m.store(&s_map[warp][lane * 4]);
  if (r.live) {
    one.load(maps + r.run * p.width + r.cc);
    one.store(&s_own[warp][lane * 4]);
  }
  __syncthreads();
  if (!r.live) return;
  m.same();                            // the first row maps to a constant, whatever it is applied to
#pragma unroll
  for (int w = 0; w < GRU_WARPS; ++w) {
    one.load(&s_map[w][lane * 4]);
    m.then(one);
  }
  for (int w = 0; w < warp; ++w) {
    one.load(&s_own[w][lane * 4]);
    m.then(one);
  }
  cp_async_wait<0>();
  __syncwarp();
  if (!r.in) return;
  const Two scale(p.out_scale);
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (long long)(r.t0 + r.first) * p.out_stride + r.c;
#pragma unroll 4
  for (int j = 0; j < n; ++j) {
    Two z[2], x[2], g[2];
    gru_unpack(mine[(3 * j) * (GRU_CH / 4)], z);
    gru_unpack(mine[(3 * j + 1) * (GRU_CH / 4)], x);
    gru_unpack(mine[(3 * j + 2) * (GRU_CH / 4)], g);
    float y[4];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      Two a, b, o;
      gru_gates<true>(z[k], bias.zs[k], x[k], bias.xb[k], g[k], a, b, o);
      m.b[k] = fma2(a, m.b[k], b);
      (m.b[k] * (o * scale)).get(y[2 * k], y[2 * k + 1]);
    }
    store4(out + (long long)j * p.out_stride, y);
  }
  if (r.first + n == r.len && r.slot >= 0) {
    float S[4];
    m.b[0].get(S[0], S[1]);
    m.b[1].get(S[2], S[3]);
    store4(p.state + (long long)r.slot * p.width + r.c, S);
  }
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

// The same recurrence in runs of 16 tokens (bf16), for the sequences that bring at least min_len tokens (max_new: the most any
// brings).  maps: scratch, rows of 2 width floats, num_tokens / 64 + 2 num_seqs of them and then num_tokens / 16 + num_seqs,
// num_tokens those of the step.
extern "C" int b200_gru_chunk_scan(const void* proj, long long proj_row_stride, int z_off, int x_off, int g_off,
                                   const void* z_bias_f32, const void* x_bias_f32, void* state_f32, void* out,
                                   long long out_row_stride, const void* query_start_loc, const void* context_lens,
                                   const void* state_slots, int num_seqs, int num_slots, int width, float out_scale,
                                   int min_len, int max_new, long long num_tokens, void* maps, void* stream) {
  using namespace b200;
  GruParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)state_slots, num_seqs, num_slots},
              proj, proj_row_stride, z_off, x_off, g_off, (const float*)z_bias_f32, (const float*)x_bias_f32,
              (float*)state_f32, out, out_row_stride, width, out_scale, min_len, max_new,
              num_tokens / GRU_GROUP + 2ll * num_seqs};
  if (int rc = gru_check(p)) return rc;
  if (max_new <= 0 || num_tokens < max_new || !maps || (reinterpret_cast<uintptr_t>(maps) & 15)) return B200_ERR_ARG;
  const long long groups = ((long long)max_new + GRU_GROUP - 1) / GRU_GROUP;
  if (groups > 65535) return B200_ERR_SHAPE;
  const dim3 grid((unsigned)((width + GRU_CH - 1) / GRU_CH), (unsigned)groups, (unsigned)num_seqs), block(GRU_WARPS * 32);
  static PerDeviceFlags maps_set, walk_set;
  if (int rc = set_max_dyn_smem_once(maps_set, gru_maps_kernel, gru_smem(2))) return rc;
  if (int rc = set_max_dyn_smem_once(walk_set, gru_walk_kernel, gru_smem(3))) return rc;
  launch_k(gru_maps_kernel, grid, block, (size_t)gru_smem(2), (cudaStream_t)stream, p, (float2*)maps);
  if (int rc = launch_status()) return rc;
  launch_k(gru_walk_kernel, grid, block, (size_t)gru_smem(3), (cudaStream_t)stream, p, (const float2*)maps);
  return launch_status();
}
