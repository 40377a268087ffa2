// Latent attention over a paged cache that holds, per token, only the normed latent c and one rotated key part shared
// by all heads: cache row = [c: R | k_rot: DR].
//
// A head's unrotated key is W_uk c and its value W_uv c, so with q' = W_uk^T q (one small product per head)
//     score = (q' . c + q_rot . k_rot) * scale,      head output = W_uv (sum_j p_j c_j),
// and attention runs as one KV head of width R + DR whose value is the first R columns of the key ("absorbed" form).
//
//   latent_prep_kernel    between the projections and attention: norms and stores c, rotates and stores k_rot, norms the
//                         latent the queries come from, rotates q in place and copies its rotated part behind q'.
//   attn_simt_kernel      attention over paged keys and values on CUDA cores, any dims, fp32 or bf16 storage: absorbed
//                         latent attention and grouped-query attention of fp32 models, and the cross-check of the
//                         tensor-core kernels.
//   latent_gather_kernel  the latents of a sequence (from the first a window reaches), gathered from their pages into
//                         packed rows (what the expanded form of long prompts projects up).
//
// A window of w tokens (0: none) means that position i sees the keys i - w + 1 .. i.  The CUDA-core kernel also takes the
// kept tokens, chunks, capped scores, sinks, gates and sigmoid weights of attn_extras.cuh.
#pragma once
#include "attn_extras.cuh"
#include "hyper.cuh"   // load4 / store4 / to_f32 / from_f32

namespace b200 {

struct LatentPrepParams {
  void* q;                   // [T, q_stride] per head DN | DR columns, rotated in place, or null
  long long q_stride;
  const void* kv;            // [T, kv_stride]: [c: R | k_rot: DR], or null
  long long kv_stride;
  void* ql;                  // [T, ql_stride]: QL columns normed in place with ql_norm, or null
  long long ql_stride;
  const float* ql_norm;
  int QL, ql_true;
  const long long* positions;
  const int* slot_mapping;   // -1 = do not store
  const float* inv_freq;     // [rot_dims / 2]
  const float* c_norm;       // [R], plain weight (zero in padding columns)
  void* cache;               // [num_slots, R + DR]
  void* q_lat;               // [T, H, R + DR]: columns R .. R + DR are written here, or null
  int heads, DN, DR, R;
  int r_true;                // columns of c that exist (the rest is padding and zero)
  int rot_dims;
  float eps;
  long long num_slots;
};

// Columns of pair i of DR / 2: the rotating pairs first, as (i, i + rot_dims / 2) with `half` and as (2i, 2i + 1) without,
// then neighbours that pass.
__device__ __forceinline__ void rot_pair(int i, int rot_dims, bool half, int& a, int& b) {
  if (half && i < (rot_dims >> 1)) {
    a = i;
    b = i + (rot_dims >> 1);
  } else {
    a = 2 * i;
    b = 2 * i + 1;
  }
}

template <typename T, bool HALF>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepParams p) {
  __shared__ float red[32];
  __shared__ float s_cos[128], s_sin[128];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int tid = threadIdx.x;
  const float pos = (float)p.positions[t];
  const int half = p.rot_dims >> 1;
  for (int i = tid; i < half; i += 128) sincosf(pos * p.inv_freq[i], &s_sin[i], &s_cos[i]);
  const int dq = p.DN + p.DR, dc = p.R + p.DR;
  if (p.ql) {
    T* x = reinterpret_cast<T*>(p.ql) + t * p.ql_stride;
    float ss = 0.f;
    for (int i = tid * 4; i < p.QL; i += 512) {
      float v[4];
      load4(x + i, v);   // padding columns hold zeros
#pragma unroll
      for (int k = 0; k < 4; ++k) ss = fmaf(v[k], v[k], ss);
    }
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)p.ql_true + p.eps);
    for (int i = tid * 4; i < p.QL; i += 512) {
      float v[4], w[4];
      load4(x + i, v);
      load4(p.ql_norm + i, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) v[k] = v[k] * inv * w[k];
      store4(x + i, v);
    }
  }
  if (p.kv) {
    const T* c = reinterpret_cast<const T*>(p.kv) + t * p.kv_stride;
    float ss = 0.f;
    for (int i = tid * 4; i < p.R; i += 512) {
      float v[4];
      load4(c + i, v);
#pragma unroll
      for (int k = 0; k < 4; ++k) ss = fmaf(v[k], v[k], ss);
    }
    ss = block_sum(ss, red);   // (its barriers also publish the sine table)
    const float inv = 1.f / sqrtf(ss / (float)p.r_true + p.eps);
    const long long slot = p.slot_mapping[t];
    if (slot >= p.num_slots && tid == 0) report_status(B200_STATUS_BAD_INDEX, (int)slot);
    if (slot >= 0 && slot < p.num_slots) {
      T* dst = reinterpret_cast<T*>(p.cache) + slot * dc;
      for (int i = tid * 4; i < p.R; i += 512) {
        float v[4], w[4];
        load4(c + i, v);
        load4(p.c_norm + i, w);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] = v[k] * inv * w[k];
        store4(dst + i, v);
      }
      const T* kr = c + p.R;
      for (int i = tid; i < (p.DR >> 1); i += 128) {
        int a, b;
        rot_pair(i, p.rot_dims, HALF, a, b);
        float u = to_f32(kr[a]), v = to_f32(kr[b]);
        if (i < half) {
          const float w = u * s_cos[i] - v * s_sin[i];
          v = v * s_cos[i] + u * s_sin[i];
          u = w;
        }
        dst[p.R + a] = from_f32<T>(u);
        dst[p.R + b] = from_f32<T>(v);
      }
    }
  } else {
    __syncthreads();           // the sine table
  }
  if (!p.q) return;
  const int pairs = p.DR >> 1;
  for (int e = tid; e < p.heads * pairs; e += 128) {
    const int h = e / pairs, i = e - h * pairs;
    int a, b;
    rot_pair(i, p.rot_dims, HALF, a, b);
    T* q = reinterpret_cast<T*>(p.q) + t * p.q_stride + h * dq + p.DN;
    float u = to_f32(q[a]), v = to_f32(q[b]);
    if (i < half) {
      const float w = u * s_cos[i] - v * s_sin[i];
      v = v * s_cos[i] + u * s_sin[i];
      u = w;
      q[a] = from_f32<T>(u);
      q[b] = from_f32<T>(v);
    }
    if (p.q_lat) {
      T* d = reinterpret_cast<T*>(p.q_lat) + (t * p.heads + h) * dc + p.R;
      d[a] = from_f32<T>(u);
      d[b] = from_f32<T>(v);
    }
  }
}

// Sequences and pages of a step, as every latent kernel reads them.
struct LatentSeqs {
  const int* query_start_loc;   // [S + 1]
  const int* context_lens;      // [S]
  const int* page_table;        // [S, page_table_stride]
  long long page_table_stride;
  int max_pages, page_size, num_blocks, num_seqs;
  int min_len, max_len;         // only sequences whose step brings min_len .. max_len tokens
  int window;                   // tokens a position sees, its own included; 0: every earlier one
  int chunk;                    // tokens of a chunk beyond which nothing is seen; 0: none
  int keep;                     // first tokens seen from everywhere behind them, whatever the window or chunk
};

// First position a query at `pos` sees.
__device__ __forceinline__ int window_first(int window, int pos) { return window > 0 ? max(0, pos - window + 1) : 0; }

// Row of key j of sequence s in the cache, or -1 (reported) for a page id out of range.
__device__ __forceinline__ long long latent_key_row(const LatentSeqs& q, int s, int j) {
  const int pg = j / q.page_size;
  const int blk = pg < q.max_pages ? q.page_table[(long long)s * q.page_table_stride + pg] : -1;
  if (blk < 0 || blk >= q.num_blocks) {
    report_status(B200_STATUS_BAD_INDEX, blk);
    return -1;
  }
  return (long long)blk * q.page_size + (j - pg * q.page_size);
}

// Index of the sequence that packed token t belongs to.
__device__ __forceinline__ int latent_seq_of(const int* query_start_loc, int num_seqs, long long t) {
  int lo = 0, hi = num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (query_start_loc[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}

struct AttnSimtParams {
  LatentSeqs seqs;
  const void* q;       // [T, H, DK]
  const void* k;       // [num_blocks * page_size, k_row]; a head's key starts at (h / group) * DK
  const void* v;       // [num_blocks * page_size, v_row]; a head's value starts at (h / group) * DV
  void* out;           // rows of [H, DV]
  long long q_row, out_row;   // elements between tokens of q, of out
  int k_row, v_row;
  int heads, group, DK, DV;
  float scale;
  AttnExtras extras;
};

constexpr int LATENT_SIMT_THREADS = 128;
constexpr int LATENT_SIMT_VPT = 8;   // value columns per thread: DV <= 1024

template <typename T>
__global__ void __launch_bounds__(LATENT_SIMT_THREADS) attn_simt_kernel(const AttnSimtParams p) {
  extern __shared__ float lat_smem[];   // q [DK]
  __shared__ float red[32];
  __shared__ float s_p[LATENT_SIMT_THREADS];
  __shared__ long long s_row[LATENT_SIMT_THREADS];
  __shared__ int s_seq;
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, tid = threadIdx.x;
  const long long t = blockIdx.x;
  if (tid == 0) s_seq = latent_seq_of(p.seqs.query_start_loc, p.seqs.num_seqs, t);
  __syncthreads();
  const int s = s_seq;
  const int t0 = p.seqs.query_start_loc[s], len = p.seqs.query_start_loc[s + 1] - t0;
  if (t < t0 || t >= t0 + len || len < p.seqs.min_len || len > p.seqs.max_len) return;
  const int pos = p.seqs.context_lens[s] - len + (int)(t - t0);
  const int keys = pos + 1, kv_head = h / p.group;   // visible keys: the kept ones, and positions first .. own
  const int first = first_visible(p.seqs.window, p.seqs.chunk, pos), kept = min(p.seqs.keep, first);
  const bool sigmoid = p.extras.sigmoid_bias != nullptr;
  const float bias = sigmoid ? p.extras.sigmoid_bias[h] : 0.f;
  const T* q = reinterpret_cast<const T*>(p.q) + t * p.q_row + (long long)h * p.DK;
  for (int i = tid; i < p.DK; i += LATENT_SIMT_THREADS) lat_smem[i] = to_f32(q[i]) * p.scale;
  float acc[LATENT_SIMT_VPT];
#pragma unroll
  for (int v = 0; v < LATENT_SIMT_VPT; ++v) acc[v] = 0.f;
  float m = -INFINITY, l = 0.f;
  const T* kbase = reinterpret_cast<const T*>(p.k) + kv_head * p.DK;
  const T* vbase = reinterpret_cast<const T*>(p.v) + kv_head * p.DV;
  for (int b = kept > 0 ? 0 : first, n; b < keys; b = b < kept && b + n == kept ? first : b + n) {
    n = min(LATENT_SIMT_THREADS, (b < kept ? kept : keys) - b);
    __syncthreads();
    long long row = tid < n ? latent_key_row(p.seqs, s, b + tid) : -1;
    s_row[tid] = row;
    float sc = -INFINITY;
    if (row >= 0) {
      const T* k = kbase + row * p.k_row;
      float a = 0.f;
      for (int i = 0; i < p.DK; i += 4) {
        float v[4];
        load4(k + i, v);
#pragma unroll
        for (int u = 0; u < 4; ++u) a = fmaf(lat_smem[i + u], v[u], a);
      }
      sc = p.extras.cap.cap > 0.f ? p.extras.cap.cap * tanhf(a / p.extras.cap.cap) : a;
    }
    float alpha = 1.f;
    if (sigmoid) {
      s_p[tid] = sc == -INFINITY ? 0.f : 1.f / (1.f + expf(-(sc + bias)));
    } else {
      const float bm = fmaxf(m, block_max(sc, red));
      const float e = sc == -INFINITY ? 0.f : expf(sc - bm);
      s_p[tid] = e;
      alpha = m == -INFINITY ? 0.f : expf(m - bm);
      l = l * alpha + block_sum(e, red);
      m = bm;
    }
    __syncthreads();
#pragma unroll
    for (int v = 0; v < LATENT_SIMT_VPT; ++v) {
      const int c = v * LATENT_SIMT_THREADS + tid;
      if (c < p.DV) {
        float a = acc[v] * alpha;
        for (int j = 0; j < n; ++j)
          if (s_row[j] >= 0) a = fmaf(s_p[j], to_f32(vbase[s_row[j] * p.v_row + c]), a);
        acc[v] = a;
      }
    }
  }
  if (p.extras.sink) l += expf(p.extras.sink[h] - m);
  const T* gate = p.extras.gate ? reinterpret_cast<const T*>(p.extras.gate) + t * p.extras.gate_stride : nullptr;
  T* out = reinterpret_cast<T*>(p.out) + t * p.out_row + (long long)h * p.DV;
#pragma unroll
  for (int v = 0; v < LATENT_SIMT_VPT; ++v) {
    const int c = v * LATENT_SIMT_THREADS + tid;
    if (c >= p.DV) continue;
    float o = sigmoid ? acc[v] : l > 0.f ? acc[v] / l : 0.f;
    o *= p.extras.out_scale;
    if (gate) o *= gate_sigmoid<T>(gate[p.extras.gate_mode == GATE_HEAD ? h : h * p.DV + c]);
    out[c] = from_f32<T>(o);
  }
}

// dst row r = cache row of key key_base[i] + (r - key_start[i]) of sequence seq_ids[i], for the i that key_start brackets.
struct LatentGatherParams {
  LatentSeqs seqs;
  const uint4* cache;
  uint4* dst;
  const int* seq_ids;     // [n]
  const int* key_start;   // [n + 1] packed start of each gathered sequence
  const int* key_base;    // [n] position of each one's first gathered key
  int n, vecs;            // 16-byte vectors per row
};

__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherParams p) {
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long r = (long long)blockIdx.x * 8 + warp;
  if (r >= p.key_start[p.n]) return;
  const int i = latent_seq_of(p.key_start, p.n, r);
  const long long row = latent_key_row(p.seqs, p.seq_ids[i], p.key_base[i] + (int)(r - p.key_start[i]));
  for (int v = lane; v < p.vecs; v += 32)
    p.dst[r * p.vecs + v] = row >= 0 ? p.cache[row * p.vecs + v] : make_uint4(0, 0, 0, 0);
}

}  // namespace b200

extern "C" int b200_latent_prep(void* q, long long q_row_stride, const void* kv, long long kv_row_stride, void* q_latent,
                                long long q_latent_row_stride, const void* q_norm_f32, int QL, int ql_true,
                                const void* positions_i64, const void* slot_mapping_i32, const void* inv_freq_f32,
                                const void* c_norm_f32, void* cache, void* q_lat, long long T, int heads, int DN, int DR,
                                int R, int r_true, int rot_dims, int rot_half, float eps, long long num_slots, int dtype,
                                void* stream) {
  using namespace b200;
  if ((!q && !kv && !q_latent) || !positions_i64 || !slot_mapping_i32 || (rot_dims > 0 && !inv_freq_f32) || (kv && (!c_norm_f32 || !cache)) ||
      (q_latent && (!q_norm_f32 || QL <= 0 || ql_true <= 0 || ql_true > QL)) || (q_lat && !q) || T < 0 || heads <= 0 ||
      DN < 0 || DR < 0 || R <= 0 || r_true <= 0 || r_true > R || rot_dims < 0 || rot_dims > DR || (dtype != 0 && dtype != 1))
    return B200_ERR_ARG;
  if (DN % 8 || DR % 8 || R % 8 || QL % 8 || q_row_stride % 8 || kv_row_stride % 8 || q_latent_row_stride % 8 ||
      rot_dims % 2 || rot_dims > 256 || T > 0x7fffffffLL)
    return B200_ERR_SHAPE;
  if (T == 0) return B200_OK;
  LatentPrepParams p{q, q_row_stride, kv, kv_row_stride, q_latent, q_latent_row_stride, (const float*)q_norm_f32, QL, ql_true,
                     (const long long*)positions_i64, (const int*)slot_mapping_i32, (const float*)inv_freq_f32,
                     (const float*)c_norm_f32, cache, q_lat, heads, DN, DR, R, r_true, rot_dims, eps, num_slots};
  const dim3 g((unsigned)T), b(128);
  const cudaStream_t st = (cudaStream_t)stream;
  if (dtype == 0) launch_k(rot_half ? latent_prep_kernel<__nv_bfloat16, true> : latent_prep_kernel<__nv_bfloat16, false>, g, b, 0, st, p);
  else launch_k(rot_half ? latent_prep_kernel<float, true> : latent_prep_kernel<float, false>, g, b, 0, st, p);
  return launch_status();
}

namespace b200 {
inline bool latent_seqs_ok(const LatentSeqs& q) {
  return q.query_start_loc && q.context_lens && q.page_table && q.num_seqs > 0 && q.page_size > 0 && q.max_pages > 0 &&
         q.num_blocks > 0;
}
}  // namespace b200

namespace b200 {
inline int attn_simt_launch(AttnSimtParams& p, long long T, int dtype, cudaStream_t st) {
  if (!latent_seqs_ok(p.seqs) || !p.q || !p.k || !p.v || !p.out || T < 0 || p.heads <= 0 || p.group <= 0 || p.DK <= 0 ||
      p.DV <= 0 || p.seqs.window < 0 || p.seqs.chunk < 0 || p.seqs.keep < 0 || !attn_extras_ok(p.extras) || (dtype != 0 && dtype != 1))
    return B200_ERR_ARG;
  if (p.heads % p.group || p.DK % 8 || p.DV % 8 || p.k_row % 8 || p.v_row % 8 || p.heads > 65535 ||
      p.DV > LATENT_SIMT_THREADS * LATENT_SIMT_VPT || p.DK > 8192 || T > 0x7fffffffLL)
    return B200_ERR_SHAPE;
  if (T == 0) return B200_OK;
  const size_t smem = (size_t)p.DK * sizeof(float);
  const dim3 grid((unsigned)T, (unsigned)p.heads);
  if (dtype == 0) launch_k(attn_simt_kernel<__nv_bfloat16>, grid, dim3(LATENT_SIMT_THREADS), smem, st, p);
  else launch_k(attn_simt_kernel<float>, grid, dim3(LATENT_SIMT_THREADS), smem, st, p);
  return launch_status();
}
}  // namespace b200

extern "C" int b200_latent_attn_simt(const void* q_lat, const void* cache, void* out, const void* query_start_loc,
                                     const void* context_lens, const void* page_table, long long page_table_stride,
                                     int max_pages, int page_size, int num_blocks, int num_seqs, int min_len,
                                     int max_len, int window, long long T, int heads, int R, int DR, float scale,
                                     int dtype, void* stream) {
  using namespace b200;
  if (R <= 0 || DR < 0 || R % 8 || DR % 8) return B200_ERR_ARG;
  AttnSimtParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)page_table, page_table_stride,
                    max_pages, page_size, num_blocks, num_seqs, min_len, max_len, window},
                   q_lat, cache, cache, out, (long long)heads * (R + DR), (long long)heads * R, R + DR, R + DR, heads, heads,
                   R + DR, R, scale, {{}, nullptr, nullptr, 0, GATE_NONE, nullptr, 1.f}};
  return attn_simt_launch(p, T, dtype, (cudaStream_t)stream);
}

// Grouped-query attention over paged per-head keys and values (the window_attn kernels' cross-check and fp32 form).
extern "C" int b200_window_attn_simt(const void* q, long long q_row_stride, const void* k_cache, const void* v_cache,
                                     void* out, long long out_row_stride, const void* query_start_loc,
                                     const void* context_lens, const void* page_table, long long page_table_stride,
                                     int max_pages, int page_size, int num_blocks, int num_seqs, int min_len, int max_len,
                                     int window, int chunk, int keep, float cap, const void* sink_f32,
                                     const void* sigmoid_bias_f32, float out_scale, const void* gate,
                                     long long gate_row_stride, int gate_mode, long long T, int heads, int kv_heads, int DK, int DV, float scale,
                                     int dtype, void* stream) {
  using namespace b200;
  if (kv_heads <= 0 || heads % kv_heads) return B200_ERR_ARG;
  AttnSimtParams p{{(const int*)query_start_loc, (const int*)context_lens, (const int*)page_table, page_table_stride,
                    max_pages, page_size, num_blocks, num_seqs, min_len, max_len, window, chunk, keep},
                   q, k_cache, v_cache, out, q_row_stride, out_row_stride, kv_heads * DK, kv_heads * DV, heads, heads / kv_heads, DK, DV,
                   scale,
                   {score_cap(cap), (const float*)sink_f32, gate, gate_row_stride, gate_mode, (const float*)sigmoid_bias_f32,
                    out_scale}};
  return attn_simt_launch(p, T, dtype, (cudaStream_t)stream);
}

extern "C" int b200_latent_gather(const void* cache, void* dst, const void* seq_ids_i32, const void* key_start_i32,
                                  const void* key_base_i32, int n, long long rows, int row_bytes, const void* page_table, long long page_table_stride,
                                  int max_pages, int page_size, int num_blocks, int num_seqs, void* stream) {
  using namespace b200;
  if (!cache || !dst || !seq_ids_i32 || !key_start_i32 || !key_base_i32 || !page_table || n <= 0 || rows < 0 || page_size <= 0 ||
      max_pages <= 0 || num_blocks <= 0 || num_seqs <= 0)
    return B200_ERR_ARG;
  if (row_bytes % 16 || row_bytes <= 0 || rows > 0x7fffffffLL) return B200_ERR_SHAPE;
  if (rows == 0) return B200_OK;
  LatentGatherParams p{{nullptr, nullptr, (const int*)page_table, page_table_stride, max_pages, page_size, num_blocks,
                        num_seqs, 0, 0, 0},
                       (const uint4*)cache, (uint4*)dst, (const int*)seq_ids_i32, (const int*)key_start_i32,
                       (const int*)key_base_i32, n, row_bytes / 16};
  launch_k(latent_gather_kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, (cudaStream_t)stream, p);
  return launch_status();
}
