// Grouped-query attention of decoded tokens and short portions over paged per-head keys and values (bf16), optionally
// inside a window or chunk, with capped scores, a sink in the denominator, an output gate or sigmoid weights
// (attn_extras.cuh).  Scores and weights are fp32: a weight enters the value product as a bf16 pair hi + lo, whose two
// products are summed in fp32, and the denominator sums the fp32 weights.  (attn.cuh and its kin round the weights to bf16, as
// the models they serve do.)
//
// One CTA of WARPS warps owns up to 8 columns of one KV head of one sequence, a column being one (token, query head)
// pair.  Warp w walks every WARPS-th block of 32 keys that some column sees (key_blocks), through a
// ring of stages of its own (TMA boxes of 64 columns, 128-byte swizzle; columns past the head dim arrive as zeros), with
//     S^T[key, col] = K[key, :] . Q[col, :],      O^T[d, col] += V[key, d]^T . P^T[key, col]          (mma.sync)
// so no MMA row is padding in decode.  The warps' results meet in shared memory in a fixed order.
//
// Algorithmic bytes: the keys and values each sequence's window holds, once per KV head: HBM bandwidth.
#pragma once
#include "attn_rows.cuh"       // the exact rows-on-lanes kernel, and through it fast_exp2, ldmatrix, mma, tensor maps
#include "latent_expand.cuh"   // the mma.sync kernel of long portions; LatentSeqs

namespace b200 {

constexpr int WAT_BN = 32;   // keys per block

struct WindowAttnParams {
  LatentSeqs seqs;
  const __nv_bfloat16* q;    // [T, q_stride]: heads of dk columns
  __nv_bfloat16* out;        // [T, out_stride]: heads of dv columns
  long long q_stride, out_stride;
  int group, head_chunks, pos_per_tile, box_tokens;
  int dk, dv;
  float scale_log2;
  AttnExtras extras;
};

template <int DK, int DV, int WARPS, int STAGES>
struct WatLayout {
  static constexpr int K = WAT_BN * DK * 2, V = WAT_BN * DV * 2, STAGE = K + V;
  static constexpr int BYTES = WARPS * STAGES * STAGE + 1024;
  static_assert(STAGES * STAGE >= DV * 8 * 4 + 64, "a warp's ring holds its partial result");
};

template <int DK, int DV, int WARPS, int STAGES, int FORM>
__global__ void __launch_bounds__(WARPS * 32)
window_attn_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                   const WindowAttnParams p) {
  using L = WatLayout<DK, DV, WARPS, STAGES>;
  constexpr int KH = DK / 64, VH = DV / 64, MT = WAT_BN / 16;
  constexpr bool EXTRAS = FORM != ATTN_PLAIN, SIGMOID = FORM == ATTN_SIGMOID;
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full_bar[WARPS][STAGES];
  __shared__ int abort_mem;
  volatile int* abort_flag = &abort_mem;
  const uint32_t base = (ptx::smem_u32(smem_raw) + 1023) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - ptx::smem_u32(smem_raw));
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int seq = blockIdx.z, kvh = blockIdx.y / p.head_chunks, hchunk = blockIdx.y % p.head_chunks;
  const int heads_here = min(8, p.group - hchunk * 8);
  const int q_start = p.seqs.query_start_loc[seq], q_len = p.seqs.query_start_loc[seq + 1] - q_start;
  const int kv_len = p.seqs.context_lens[seq], pos0 = blockIdx.x * p.pos_per_tile;
  if (q_len < p.seqs.min_len || q_len > p.seqs.max_len || pos0 >= q_len) return;
  if (kv_len < q_len) {
    if (threadIdx.x == 0) report_status(B200_STATUS_BAD_INDEX, seq);
    return;
  }
  const int q_abs0 = kv_len - q_len;
  auto col_valid = [&](int c) {
    const int pi = c / heads_here;
    return pi < p.pos_per_tile && pos0 + pi < q_len;
  };
  auto col_q = [&](int c) { return pos0 + (col_valid(c) ? c / heads_here : 0); };   // a spare column repeats the first position
  auto col_head = [&](int c) { return kvh * p.group + hchunk * 8 + c % heads_here; };
  const int last_pos = q_abs0 + min(pos0 + p.pos_per_tile, q_len) - 1;
  const int chunk = EXTRAS ? p.seqs.chunk : 0, keep = EXTRAS ? p.seqs.keep : 0;
  const KeyBlocks walk = key_blocks<WAT_BN>(p.seqs.window, chunk, keep, q_abs0 + pos0, last_pos);
  const int mine = (walk.count - warp + WARPS - 1) / WARPS;      // blocks of this warp: number warp + i * WARPS of the walk

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int w = 0; w < WARPS; ++w)
      for (int s = 0; s < STAGES; ++s) ptx::mbar_init(ptx::smem_u32(&full_bar[w][s]), 1);
    ptx::fence_barrier_init();
    ptx::prefetch_tensormap(&tm_k);
    ptx::prefetch_tensormap(&tm_v);
  }
  __syncthreads();
  const uint32_t ring = base + (uint32_t)warp * STAGES * L::STAGE;
  uint8_t* ring_ptr = base_ptr + (size_t)warp * STAGES * L::STAGE;
  const int boxes = WAT_BN / p.box_tokens;

  auto issue = [&](int i) {        // block i of this warp into its stage; the whole warp
    const int s = i % STAGES;
    const uint32_t bar = ptx::smem_u32(&full_bar[warp][s]), sk = ring + (uint32_t)s * L::STAGE, sv = sk + L::K;
    ptx::fence_proxy_async_smem();  // this lane's reads of the stage come before the refill
    __syncwarp();
    if (lane == 0) ptx::mbar_expect_tx(bar, L::STAGE);
    __syncwarp();
    if (lane < boxes) {
      const int tok = walk.at(warp + i * WARPS) * WAT_BN + lane * p.box_tokens;
      const int page = tok / p.seqs.page_size, in_page = tok - page * p.seqs.page_size;
      int phys = -1;                // out of range: zeros arrive
      if (tok < kv_len && page < p.seqs.max_pages) phys = p.seqs.page_table[(long long)seq * p.seqs.page_table_stride + page];
      if (phys >= p.seqs.num_blocks) phys = -1;
      const uint32_t off = (uint32_t)(lane * p.box_tokens) * 128;
#pragma unroll
      for (int h = 0; h < KH; ++h)
        ptx::tma_load_4d(sk + h * (WAT_BN * 128) + off, &tm_k, bar, h * 64, kvh, in_page, phys, ptx::kEvictFirst);
#pragma unroll
      for (int h = 0; h < VH; ++h)
        ptx::tma_load_4d(sv + h * (WAT_BN * 128) + off, &tm_v, bar, h * 64, kvh, in_page, phys, ptx::kEvictFirst);
    }
  };
  for (int i = 0; i < STAGES && i < mine; ++i) issue(i);

  uint32_t qb[DK / 16][2];          // Q^T as the B operand: column g, d = 16 kk + 2 t (+ 8)
  {
    const bool v = col_valid(g);
    const __nv_bfloat16* qrow = p.q + (long long)(q_start + col_q(g)) * p.q_stride + (long long)col_head(g) * p.dk;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = kk * 16 + e * 8 + 2 * t;
        qb[kk][e] = v && d < p.dk ? *reinterpret_cast<const uint32_t*>(qrow + d) : 0u;
      }
  }
  int cpos[2];
  uint32_t reach[2];                // visible: 0 <= cpos - key < reach
  float bias[2];                    // of sigmoid weights, in units of log2
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    cpos[j] = q_abs0 + col_q(2 * t + j);
    reach[j] = visible_keys(p.seqs.window, chunk, cpos[j]);
    bias[j] = SIGMOID ? p.extras.sigmoid_bias[col_head(2 * t + j)] * kLog2e : 0.f;
  }

  float o[DV / 16][4];
#pragma unroll
  for (int i = 0; i < DV / 16; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-3.0e38f, -3.0e38f}, l_run[2] = {0.f, 0.f};
  const int mi = lane >> 3, dk16 = (p.dk + 15) / 16, dv16 = (p.dv + 15) / 16;
  bool ok = true;
  for (int i = 0; i < mine; ++i) {
    const int s = i % STAGES;
    ok = ptx::mbar_wait(ptx::smem_u32(&full_bar[warp][s]), (i / STAGES) & 1, abort_flag, 800 + s);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) break;
    const uint32_t sk = ring + (uint32_t)s * L::STAGE, sv = sk + L::K;
    const int key0 = walk.at(warp + i * WARPS) * WAT_BN;
    if (key0 + WAT_BN > kv_len) {   // rows past the context may hold anything: 0 * value has to stay 0
      uint8_t* vt = ring_ptr + (size_t)s * L::STAGE + L::K;
      for (int r = kv_len - key0; r < WAT_BN; ++r)
#pragma unroll
        for (int h = 0; h < VH; ++h) reinterpret_cast<uint32_t*>(vt + h * (WAT_BN * 128) + r * 128)[lane] = 0u;
      __syncwarp();
    }
    float sc[MT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      sc[mt][0] = sc[mt][1] = sc[mt][2] = sc[mt][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        if (kk >= dk16) break;
        const int key = mt * 16 + (mi & 1) * 8 + (lane & 7), ch = kk * 2 + (mi >> 1);
        uint32_t a0, a1, a2, a3;
        ldmatrix_x4(sk + (ch >> 3) * (WAT_BN * 128) + sw128(key, ch & 7), a0, a1, a2, a3);
        mma_bf16_16816(sc[mt], a0, a1, a2, a3, qb[kk][0], qb[kk][1]);
      }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[mt][e] *= p.scale_log2;
      if (EXTRAS && p.extras.cap.cap > 0.f) cap_scores(sc[mt], p.extras.cap);
    }
    if constexpr (SIGMOID) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int key = key0 + mt * 16 + g;
          float a = sc[mt][j] + bias[j], b = sc[mt][2 + j] + bias[j];
          sigmoid_pair(a, b, key_visible(reach[j], keep, cpos[j], key), key_visible(reach[j], keep, cpos[j], key + 8));
          sc[mt][j] = a;
          sc[mt][2 + j] = b;
        }
    } else {
      float alpha[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        float mx = m_run[j];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int hh = 0; hh < 2; ++hh) {
            const int key = key0 + mt * 16 + g + hh * 8;
            float v = sc[mt][hh * 2 + j];
            if (!key_visible(reach[j], keep, cpos[j], key)) v = -INFINITY;
            sc[mt][hh * 2 + j] = v;
            mx = fmaxf(mx, v);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
        alpha[j] = fast_exp2(m_run[j] - mx);
        m_run[j] = mx;
        float sum = 0.f;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int hh = 0; hh < 2; ++hh) {
            const float e = fast_exp2(sc[mt][hh * 2 + j] - mx);
            sc[mt][hh * 2 + j] = e;
            sum += e;
          }
        l_run[j] = l_run[j] * alpha[j] + sum;      // this lane's keys; the lanes' shares meet at the end
      }
      if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
        for (int d = 0; d < DV / 16; ++d) {
          o[d][0] *= alpha[0];
          o[d][1] *= alpha[1];
          o[d][2] *= alpha[0];
          o[d][3] *= alpha[1];
        }
      }
    }
    uint32_t hi[MT][2], lo[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const float a = sc[mt][hh * 2], b = sc[mt][hh * 2 + 1];
        const uint32_t top = pack_bf2(a, b);
        float ta, tb;
        unpack_bf2(top, ta, tb);
        hi[mt][hh] = movmatrix_trans(top);
        lo[mt][hh] = movmatrix_trans(pack_bf2(a - ta, b - tb));
      }
#pragma unroll
    for (int dm = 0; dm < DV / 16; ++dm) {
      if (dm >= dv16) break;
#pragma unroll
      for (int kk = 0; kk < MT; ++kk) {
        const int key = kk * 16 + (mi >> 1) * 8 + (lane & 7), ch = dm * 2 + (mi & 1);
        uint32_t a0, a1, a2, a3;
        ldmatrix_x4_trans(sv + (ch >> 3) * (WAT_BN * 128) + sw128(key, ch & 7), a0, a1, a2, a3);
        mma_bf16_16816(o[dm], a0, a1, a2, a3, hi[kk][0], hi[kk][1]);
        mma_bf16_16816(o[dm], a0, a1, a2, a3, lo[kk][0], lo[kk][1]);
      }
    }
    __syncwarp();
    if (i + STAGES < mine) issue(i + STAGES);
  }

  // this warp's partial result into its own ring: [DV][8] sums, then 8 maxima and 8 denominators
  float* part = reinterpret_cast<float*>(ring_ptr);
  if (ok) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      float l = l_run[j];
      l += __shfl_xor_sync(0xffffffffu, l, 4);
      l += __shfl_xor_sync(0xffffffffu, l, 8);
      l += __shfl_xor_sync(0xffffffffu, l, 16);
      const int c = 2 * t + j;
      if (g == 0) {
        part[DV * 8 + c] = m_run[j];
        part[DV * 8 + 8 + c] = l;
      }
#pragma unroll
      for (int dm = 0; dm < DV / 16; ++dm) {
        part[(dm * 16 + g) * 8 + c] = o[dm][j];
        part[(dm * 16 + g + 8) * 8 + c] = o[dm][2 + j];
      }
    }
  }
  __syncthreads();
  if (*abort_flag) {               // let copies in flight land before the CTA exits
    const uint64_t w0 = global_timer_ns();
    while (global_timer_ns() - w0 < 200000ull) {
    }
    return;
  }
  const float* parts = reinterpret_cast<const float*>(base_ptr);
  constexpr int PITCH = STAGES * L::STAGE / 4;
  for (int e = threadIdx.x; e < 8 * (DV / 2); e += WARPS * 32) {
    const int c = e / (DV / 2), d = (e % (DV / 2)) * 2;
    if (!col_valid(c) || c >= heads_here * p.pos_per_tile || d >= p.dv) continue;
    float m = -3.0e38f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) m = fmaxf(m, parts[w * PITCH + DV * 8 + c]);
    float l = 0.f, a = 0.f, b = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float* q = parts + w * PITCH;
      const float f = SIGMOID ? 1.f : fast_exp2(q[DV * 8 + c] - m);
      l = fmaf(f, q[DV * 8 + 8 + c], l);
      a = fmaf(f, q[d * 8 + c], a);
      b = fmaf(f, q[(d + 1) * 8 + c], b);
    }
    const int head = col_head(c);
    const long long row = q_start + col_q(c);
    if (EXTRAS) l += sink_term(p.extras, head, m);
    const float inv = SIGMOID ? p.extras.out_scale : EXTRAS ? p.extras.out_scale / l : 1.f / l;
    a *= inv;
    b *= inv;
    if (EXTRAS && p.extras.gate_mode != GATE_NONE) {
      const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(p.extras.gate) + row * p.extras.gate_stride;
      const bool per_head = p.extras.gate_mode == GATE_HEAD;
      a *= gate_sigmoid(gate[per_head ? head : head * p.dv + d]);
      b *= gate_sigmoid(gate[per_head ? head : head * p.dv + d + 1]);
    }
    *reinterpret_cast<uint32_t*>(p.out + row * p.out_stride + (long long)head * p.dv + d) = pack_bf2(a, b);
  }
}

template <int DK, int DV, int WARPS, int STAGES, int FORM>
inline int window_attn_launch(const CUtensorMap& tk, const CUtensorMap& tv, const WindowAttnParams& p, dim3 grid,
                              cudaStream_t st) {
  constexpr int smem = WatLayout<DK, DV, WARPS, STAGES>::BYTES;
  static_assert(smem <= 226 * 1024, "shared memory budget");
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, window_attn_kernel<DK, DV, WARPS, STAGES, FORM>, smem)) return rc;
  launch_k(window_attn_kernel<DK, DV, WARPS, STAGES, FORM>, grid, dim3(WARPS * 32), (size_t)smem, st, tk, tv, p);
  return launch_status();
}

template <int FORM>
inline int window_attn_dispatch(const CUtensorMap& tk, const CUtensorMap& tv, const WindowAttnParams& p, dim3 grid,
                                cudaStream_t st) {
  if (p.dk <= 64 && p.dv <= 64) return window_attn_launch<64, 64, 2, 4, FORM>(tk, tv, p, grid, st);
  if (p.dk <= 128 && p.dv <= 128) return window_attn_launch<128, 128, 2, 3, FORM>(tk, tv, p, grid, st);
  if (p.dk <= 192 && p.dv <= 128) return window_attn_launch<192, 128, 2, 2, FORM>(tk, tv, p, grid, st);
  return window_attn_launch<256, 256, 2, 2, FORM>(tk, tv, p, grid, st);
}

}  // namespace b200

// Attention of the sequences that bring min_len .. max_len tokens.  q rows hold heads * DK columns, k_cache [blocks, page,
// kv_heads, DK] and v_cache [.., DV] are contiguous.  DK, DV multiples of 8 up to 256; page_size a multiple of 8 that
// divides 32 or is a multiple of it.
extern "C" int b200_window_attn_decode(const void* q, long long q_row_stride, const void* k_cache, const void* v_cache,
                                       void* out, long long out_row_stride, const void* query_start_loc,
                                       const void* context_lens, const void* page_table, long long page_table_stride,
                                       int max_pages, int page_size, int num_blocks, int num_seqs, int min_len, int max_len,
                                       int most_new, int window, int chunk, int keep, float cap, const void* sink_f32,
                                       const void* sigmoid_bias_f32, float out_scale, const void* gate,
                                       long long gate_row_stride, int gate_mode, int heads, int kv_heads, int DK, int DV,
                                       float scale, void* stream) {
  using namespace b200;
  WindowAttnParams p{};
  p.seqs = {(const int*)query_start_loc, (const int*)context_lens, (const int*)page_table, page_table_stride, max_pages,
            page_size, num_blocks, num_seqs, min_len < 1 ? 1 : min_len, max_len, window, chunk, keep};
  p.extras = {score_cap(cap * kLog2e), (const float*)sink_f32, gate, gate_row_stride, gate_mode,
              (const float*)sigmoid_bias_f32, out_scale};
  if (!latent_seqs_ok(p.seqs) || !q || !k_cache || !v_cache || !out || heads <= 0 || kv_heads <= 0 || heads % kv_heads ||
      DK <= 0 || DV <= 0 || window < 0 || chunk < 0 || keep < 0 || max_len < 1 || most_new < 0 || !attn_extras_ok(p.extras))
    return B200_ERR_ARG;
  const bool pages_ok = page_size % 8 == 0 && (page_size % WAT_BN == 0 || WAT_BN % page_size == 0);
  if (DK % 8 || DV % 8 || DK > 256 || DV > 256 || !pages_ok || q_row_stride % 2 || out_row_stride % 2 ||
      (reinterpret_cast<uintptr_t>(q) & 3) || (reinterpret_cast<uintptr_t>(out) & 3) || num_seqs > 65535)
    return B200_ERR_SHAPE;
  const int most = most_new < max_len ? most_new : max_len;
  if (most == 0) return B200_OK;
  p.q = (const __nv_bfloat16*)q;
  p.out = (__nv_bfloat16*)out;
  p.q_stride = q_row_stride;
  p.out_stride = out_row_stride;
  p.group = heads / kv_heads;
  p.head_chunks = (p.group + 7) / 8;
  p.pos_per_tile = p.group >= 8 ? 1 : 8 / p.group;
  p.box_tokens = page_size < WAT_BN ? page_size : WAT_BN;
  p.dk = DK;
  p.dv = DV;
  p.scale_log2 = scale * kLog2e;
  CUtensorMap tk, tv;
  int rc = make_tmap_cache(&tk, k_cache, num_blocks, page_size, kv_heads, DK, (long long)page_size * kv_heads * DK,
                           (long long)kv_heads * DK, DK, p.box_tokens);
  if (rc) return rc;
  rc = make_tmap_cache(&tv, v_cache, num_blocks, page_size, kv_heads, DV, (long long)page_size * kv_heads * DV,
                       (long long)kv_heads * DV, DV, p.box_tokens);
  if (rc) return rc;
  if ((long long)kv_heads * p.head_chunks > 65535) return B200_ERR_SHAPE;
  const dim3 grid((unsigned)((most + p.pos_per_tile - 1) / p.pos_per_tile), (unsigned)(kv_heads * p.head_chunks),
                  (unsigned)num_seqs);
  const cudaStream_t st = (cudaStream_t)stream;
  switch (attn_form(p.extras, chunk, keep)) {
    case ATTN_PLAIN: return window_attn_dispatch<ATTN_PLAIN>(tk, tv, p, grid, st);
    case ATTN_EXTRAS: return window_attn_dispatch<ATTN_EXTRAS>(tk, tv, p, grid, st);
    default: return window_attn_dispatch<ATTN_SIGMOID>(tk, tv, p, grid, st);
  }
}

// Long portions: the n sequences named, which are those that bring at least min_len tokens.  Heads of 65 .. 128 columns go
// to the tcgen05 kernel (exact form of attn_rows.cuh) when the query layout suits its copies, others to the mma.sync kernel
// of latent_expand.cuh; form: 0 = this choice, 1 = mma.sync (cross-checks).
extern "C" int b200_window_attn_prefill(const void* q, long long q_row_stride, const void* k_cache, const void* v_cache,
                                        void* out, long long out_row_stride, const void* query_start_loc,
                                        const void* context_lens, const void* page_table, long long page_table_stride,
                                        int max_pages, int page_size, int num_blocks, int num_seqs, const void* seq_ids_i32,
                                        int n, int max_len, int min_len, int window, int chunk, int keep,
                                        float cap, const void* sink_f32, const void* sigmoid_bias_f32, float out_scale,
                                        const void* gate, long long gate_row_stride, int gate_mode, long long T,
                                        int heads, int kv_heads, int DK, int DV, float scale, int form, void* stream) {
  using namespace b200;
  LatentExpandParams p{};
  p.seqs = {(const int*)query_start_loc, (const int*)context_lens, (const int*)page_table, page_table_stride, max_pages,
            page_size, num_blocks, num_seqs, 0, 0, window, chunk, keep};
  p.extras = {score_cap(cap * kLog2e), (const float*)sink_f32, gate, gate_row_stride, gate_mode,
              (const float*)sigmoid_bias_f32, out_scale};
  if (!latent_seqs_ok(p.seqs) || !q || !k_cache || !v_cache || !out || !seq_ids_i32 || n <= 0 || max_len <= 0 || T <= 0 ||
      heads <= 0 || kv_heads <= 0 || heads % kv_heads || DK <= 0 || DV <= 0 || window < 0 || chunk < 0 || keep < 0 ||
      !attn_extras_ok(p.extras))
    return B200_ERR_ARG;
  if (gate_mode == GATE_COLUMN && (gate_row_stride % 8 || (reinterpret_cast<uintptr_t>(gate) & 15))) return B200_ERR_SHAPE;
  if (DK % 8 || DV % 8 || q_row_stride % 8 || out_row_stride % 8 || DK > 256 || DV > 256 || heads > 65535 || n > 65535)
    return B200_ERR_SHAPE;
  const cudaStream_t st = (cudaStream_t)stream;
  const int group = heads / kv_heads, hh = group < 8 ? group : 8;
  const bool pages_ok = page_size % 8 == 0 && (page_size < ATT_BN ? ATT_BN % page_size == 0 : page_size % ATT_BN == 0);
  if (form == 0 && DK <= 128 && DV <= 128 && (DK > 64 || DV > 64) && (group <= 8 || group % 8 == 0) && pages_ok &&
      num_seqs <= 65535) {
    AttnParams a{};
    a.q = (const __nv_bfloat16*)q;
    a.out = (__nv_bfloat16*)out;
    a.q_tok_stride = q_row_stride;
    a.q_head_stride = DK;
    a.o_tok_stride = out_row_stride;
    a.o_head_stride = DV;
    a.cu_seqlens_q = p.seqs.query_start_loc;
    a.seqused_k = p.seqs.context_lens;
    a.page_table = p.seqs.page_table;
    a.page_table_stride = page_table_stride;
    a.max_pages = max_pages;
    a.page_size = page_size;
    a.box_tokens = page_size < ATT_BN ? page_size : ATT_BN;
    a.num_q_heads = heads;
    a.num_kv_heads = kv_heads;
    a.group = group;
    a.head_chunks = (group + 7) / 8;
    a.pos_per_tile = ATR_ROWS / hh;
    a.qk_scale = scale * kLog2e;
    a.extras = p.extras;
    a.chunk = chunk;
    a.keep = keep;
    a.num_blocks = num_blocks;
    a.num_seqs = num_seqs;
    a.max_seqlen_q = max_len;
    a.min_q = min_len;
    a.window = window;
    a.dv = DV;
    a.tc_q_tiles = (max_len + a.pos_per_tile - 1) / a.pos_per_tile;
    a.tc_hy = kv_heads * a.head_chunks;
    const long long tiles = (long long)a.tc_q_tiles * a.tc_hy * num_seqs;
    if (tiles > 0x3fffffffLL) return B200_ERR_SHAPE;
    a.tc_tiles = (int)tiles;
    const int ctas = a.tc_tiles < sm_count() ? a.tc_tiles : sm_count();
    a.tc_slots = (a.tc_tiles + ctas - 1) / ctas * ctas;
    CUtensorMap tk, tv, tq, to;
    const long long kr = (long long)kv_heads * DK, vr = (long long)kv_heads * DV;
    int rc = make_tmap_cache(&tk, k_cache, num_blocks, page_size, kv_heads, DK, page_size * kr, kr, DK, a.box_tokens);
    if (!rc) rc = make_tmap_cache(&tv, v_cache, num_blocks, page_size, kv_heads, DV, page_size * vr, vr, DV, a.box_tokens);
    if (rc) return rc;
    to = tk;
    if (make_tmap_q(&tq, q, T, heads, DK, q_row_stride, DK, hh, a.pos_per_tile) == B200_OK) {
      a.q_tma = 1;
      a.o_tma = 32 % hh == 0 && make_tmap_q(&to, out, T, heads, DV, out_row_stride, DV, hh, 32 / hh, true) == B200_OK;
      CUtensorMap tg = tk;
      a.g_tma = gate_mode == GATE_COLUMN && 32 % hh == 0 &&
                make_tmap_q(&tg, gate, T, heads, DV, gate_row_stride, DV, hh, 32 / hh, true) == B200_OK;
      switch (attn_form(a.extras, chunk, keep)) {
        case ATTN_PLAIN: return attn_rows_launch<128, true, ATTN_PLAIN>(tk, tv, tq, to, tg, a, st);
        case ATTN_EXTRAS: return attn_rows_launch<128, true, ATTN_EXTRAS>(tk, tv, tq, to, tg, a, st);
        default: return attn_rows_launch<128, true, ATTN_SIGMOID>(tk, tv, tq, to, tg, a, st);
      }
    }
  }
  p.seq_ids = (const int*)seq_ids_i32;
  p.q = (const __nv_bfloat16*)q;
  p.k = (const __nv_bfloat16*)k_cache;
  p.v = (const __nv_bfloat16*)v_cache;
  p.out = (__nv_bfloat16*)out;
  p.q_stride = q_row_stride;
  p.k_stride = (long long)kv_heads * DK;
  p.v_stride = (long long)kv_heads * DV;
  p.out_stride = out_row_stride;
  p.heads = heads;
  p.group = group;
  p.DN = DK;
  p.DV = DV;
  p.scale_log2 = scale * kLog2e;
  switch (attn_form(p.extras, chunk, keep)) {
    case ATTN_PLAIN: return latent_expand_dispatch<true, ATTN_PLAIN>(p, max_len, n, st);
    case ATTN_EXTRAS: return latent_expand_dispatch<true, ATTN_EXTRAS>(p, max_len, n, st);
    default: return latent_expand_dispatch<true, ATTN_SIGMOID>(p, max_len, n, st);
  }
}
