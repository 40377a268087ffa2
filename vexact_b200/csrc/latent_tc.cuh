// Absorbed latent attention on tcgen05 tensor cores (bf16): decode and short portions.
//
// The paged latent cache is one KV head whose row is [c: R | k_rot: DR] and whose value is c.  A tile is 16 columns, a
// column being one (token, head) row of a sequence; its keys are cut into splits of LTC_SPLIT (so that a long context
// is shared by many SMs, always at the same keys) and walked in blocks of 128:
//
//   S^T[key, col] = row[key, :] . q'[col, :]          UMMA M = 128 keys, N = 16                     -> TMEM
//   softmax over the split's keys, per column, fp32   256 compute threads
//   O^T[dim, col] = c[key, dim]^T . P^T[key, col]     UMMA M = 128 dims (ceil(R / 128) times), N = 32 -> TMEM
//
// The key tile is read from memory once for both products: TMA writes 128-byte-swizzled 128 x 64 boxes, which QK^T reads
// K-major and the value product MN-major, in place.  N is 32 in the value product because a weight enters as the bf16
// pair hi + lo in two columns (the sum of the two results keeps 16 bits of its mantissa).
//
// Boxes of c travel in pairs (128 dims, one UMMA M block) through a ring of slots that are given back one by one as the
// value product has read them; the boxes of k_rot have slots of their own, free again after QK^T.
//
// O^T stays in tensor memory across blocks.  A column's reference maximum moves only when a block's maximum exceeds it by
// more than 2^8 (weights up to 2^8 are as exact as weights up to 1); then the sums so far are taken into registers and
// rescaled, and O^T starts anew.
//
// With a window the walk starts at the block (of 128) that holds the first key any of the sequence's new tokens sees, and
// the splits before it do not exist; blocks and splits lie at the same keys either way.
//
// Persistent CTAs take items (sequence, column tile, split) from a list made once per step (latent_plan_kernel).
// Warps: 0 = TMA producer, 1 = UMMA issuer and TMEM owner, 2..9 = softmax and accumulation (thread = TMEM lane, half of
// the columns), 10 = query loader.  A row whose sequence has one split is finished here, otherwise
// latent_combine_kernel joins the splits.  All waits are bounded.
#pragma once
#include <cuda.h>

#include "attn_tc.cuh"     // descriptors, fast_exp2, halving_warp_sum
#include "latent.cuh"
#include "ssm_chunk.cuh"   // split_bf2

namespace b200 {

constexpr int LTC_BN = 128, LTC_NC = 16, LTC_SPLIT = 512, LTC_THREADS = 352;
constexpr int LTC_BOX = LTC_BN * 128;             // bytes of a 128-key x 64-column box
constexpr int LTC_MAX_PAIRS = 6;
constexpr float LTC_SLACK = 8.f;                  // log2 of how far a weight may exceed 1 before the rescale
constexpr int LTC_SMEM = 225 * 1024;          // always this much: one CTA per SM (the static arrays are beside it)

struct LatentTcParams {
  LatentSeqs seqs;
  const __nv_bfloat16* q_lat;   // [T, H, R + DR]
  __nv_bfloat16* out;           // [T, H, R]
  const int4* items;            // pairs {sequence, first token, new tokens, context}, {column tile, split, splits, first key}
  const int* item_count;
  int max_items;
  float* part_o;                // [items, 16, R]
  float2* part_ml;              // [items, 16]: running maximum (base 2) and sum
  int heads, R, DR, box_tokens;
  int pair_slots, rot_slots;    // ring sizes
  float scale_log2;
};

// Items of a step: for every sequence with min_len .. max_len new tokens, column tiles x splits.  One CTA.
struct LatentPlanParams {
  LatentSeqs seqs;
  int heads, max_items;
  int4* items;
  int* item_count;
  int* first_item;   // [S]
};

// First key walked for a sequence, and how many splits there are from the one that holds it.
__device__ __forceinline__ int ltc_first_key(int window, int ctx, int len) {
  return window_first(window, ctx - len) / LTC_BN * LTC_BN;
}
__device__ __forceinline__ int ltc_splits(int first_key, int ctx) {
  return (ctx + LTC_SPLIT - 1) / LTC_SPLIT - first_key / LTC_SPLIT;
}

__global__ void __launch_bounds__(1024) latent_plan_kernel(const LatentPlanParams p) {
  __shared__ int s_warp[32];
  __shared__ int s_base;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) s_base = 0;
  __syncthreads();
  for (int s0 = 0; s0 < p.seqs.num_seqs; s0 += 1024) {
    const int s = s0 + tid;
    int tiles = 0, splits = 0, t0 = 0, len = 0, ctx = 0, key = 0;
    if (s < p.seqs.num_seqs) {
      t0 = p.seqs.query_start_loc[s];
      len = p.seqs.query_start_loc[s + 1] - t0;
      ctx = p.seqs.context_lens[s];
      if (len >= p.seqs.min_len && len <= p.seqs.max_len && len > 0) {
        tiles = (len * p.heads + LTC_NC - 1) / LTC_NC;
        key = ltc_first_key(p.seqs.window, ctx, len);
        splits = ltc_splits(key, ctx);
      }
    }
    const int n = tiles * splits;
    int inc = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    if (lane == 31) s_warp[warp] = inc;
    __syncthreads();
    int before = s_base;
    for (int w = 0; w < warp; ++w) before += s_warp[w];
    const int first = before + inc - n;
    if (s < p.seqs.num_seqs) p.first_item[s] = first;
    for (int i = 0; i < n; ++i) {
      if (first + i < p.max_items) {
        p.items[2 * (first + i)] = make_int4(s, t0, len, ctx);
        p.items[2 * (first + i) + 1] = make_int4(i / splits, key / LTC_SPLIT + i % splits, splits, key);
      } else report_status(B200_STATUS_BAD_INDEX, first + i);
    }
    __syncthreads();
    if (tid == 1023) s_base = before + inc;
    __syncthreads();
  }
  if (tid == 0) *p.item_count = min(s_base, p.max_items);
}

// Rows of sequences with several splits: out = sum_i 2^(m_i - m) o_i / sum_i 2^(m_i - m) l_i.
struct LatentCombineParams {
  LatentSeqs seqs;
  const int* first_item;
  int max_items;
  const float* part_o;
  const float2* part_ml;
  __nv_bfloat16* out;
  int heads, R;
};

__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentCombineParams p) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int h = blockIdx.y;
  const int s = latent_seq_of(p.seqs.query_start_loc, p.seqs.num_seqs, t);
  const int t0 = p.seqs.query_start_loc[s], len = p.seqs.query_start_loc[s + 1] - t0;
  if (t < t0 || t >= t0 + len || len < p.seqs.min_len || len > p.seqs.max_len) return;
  const int ctx = p.seqs.context_lens[s];
  const int splits = ltc_splits(ltc_first_key(p.seqs.window, ctx, len), ctx);
  if (splits <= 1) return;
  const int row = (int)(t - t0) * p.heads + h;
  const long long item = p.first_item[s] + (long long)(row / LTC_NC) * splits;
  if (item + splits > p.max_items) return;   // reported by the plan
  const int c = row % LTC_NC;
  float m = -INFINITY, l = 0.f;
  for (int i = 0; i < splits; ++i) m = fmaxf(m, p.part_ml[(item + i) * LTC_NC + c].x);
  for (int i = 0; i < splits; ++i) {
    const float2 v = p.part_ml[(item + i) * LTC_NC + c];
    l += fast_exp2(v.x - m) * v.y;
  }
  const float inv = 1.f / l;
  for (int d = threadIdx.x * 4; d < p.R; d += 512) {
    float a[4] = {0.f, 0.f, 0.f, 0.f};
    for (int i = 0; i < splits; ++i) {
      const float f = fast_exp2(p.part_ml[(item + i) * LTC_NC + c].x - m);
      float v[4];
      load4(p.part_o + ((item + i) * LTC_NC + c) * p.R + d, v);
#pragma unroll
      for (int k = 0; k < 4; ++k) a[k] = fmaf(f, v[k], a[k]);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) a[k] *= inv;
    store4(p.out + (t * p.heads + h) * (long long)p.R + d, a);
  }
}

// One item's extent.  The two words of its description are read an item ahead (LtcRaw), so that nobody waits for them.
struct LtcRaw {
  int4 a, b;
};
struct LtcItem {
  int seq, tile, splits, t0, len, ctx, key0, nblk, rows;
};

__device__ __forceinline__ LtcRaw ltc_raw(const LatentTcParams& p, int idx, int count) {
  const int i = min(idx, count - 1);
  return LtcRaw{p.items[2 * i], p.items[2 * i + 1]};
}
__device__ __forceinline__ LtcItem ltc_item(const LatentTcParams& p, const LtcRaw& r) {
  LtcItem t;
  t.seq = r.a.x;
  t.t0 = r.a.y;
  t.len = r.a.z;
  t.ctx = r.a.w;
  t.tile = r.b.x;
  t.splits = r.b.z;
  t.key0 = max(r.b.y * LTC_SPLIT, r.b.w);
  t.nblk = (min(t.ctx, (r.b.y + 1) * LTC_SPLIT) - t.key0 + LTC_BN - 1) / LTC_BN;
  t.rows = min(LTC_NC, t.len * p.heads - t.tile * LTC_NC);
  return t;
}

// Named barrier 3 of the compute warps with a vote: true when any of the n threads brings true.
__device__ __forceinline__ bool barrier_any(bool mine, int n) {
  uint32_t any;
  asm volatile(
      "{\n"
      ".reg .pred p, q;\n"
      "setp.ne.u32 q, %1, 0;\n"
      "barrier.cta.red.or.pred p, 3, %2, q;\n"
      "selp.u32 %0, 1, 0, p;\n"
      "}\n"
      : "=r"(any)
      : "r"((uint32_t)mine), "r"(n)
      : "memory");
  return any != 0;
}

__device__ __forceinline__ void tmem_ld8(uint32_t taddr, uint32_t* r) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
               : "r"(taddr)
               : "memory");
}

template <int CP>   // pairs of 64-column boxes of c: R <= 128 CP
__global__ void __launch_bounds__(LTC_THREADS, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap tm, const LatentTcParams p) {
  constexpr int NC = LTC_NC, NH = NC / 2;
  constexpr int TMEM_COLS = 2 * NC + CP * 2 * NC <= 64 ? 64 : 2 * NC + CP * 2 * NC <= 128 ? 128 : 256;
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t bars[2 * LTC_MAX_PAIRS + 4 + 4 + 3 + 4];
  __shared__ int abort_mem, s_fresh;
  __shared__ uint32_t tmem_slot;
  __shared__ __align__(16) float s_wmax[2][NC][4];
  __shared__ __align__(16) float s_lred[NC][4];
  volatile int* abort_flag = &abort_mem;
  const int R = p.R, DR = p.DR, CB = (R + 63) / 64, RB = (DR + 63) / 64, NBX = CB + RB;
  const int NP = p.pair_slots, NR = p.rot_slots;
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - raw);
  const uint32_t rot_off = (uint32_t)NP * 2 * LTC_BOX, q_off = rot_off + (uint32_t)NR * RB * LTC_BOX;
  const uint32_t q_bytes = (uint32_t)NBX * NC * 128, p_off = q_off + 2 * q_bytes;
  auto bar = [&](int i) { return ptx::smem_u32(&bars[i]); };
  auto pfull = [&](int s) { return bar(s); };
  auto pempty = [&](int s) { return bar(LTC_MAX_PAIRS + s); };
  auto rfull = [&](int s) { return bar(2 * LTC_MAX_PAIRS + s); };
  auto rempty = [&](int s) { return bar(2 * LTC_MAX_PAIRS + 2 + s); };
  auto sfull = [&](int b) { return bar(2 * LTC_MAX_PAIRS + 4 + b); };
  auto sfree = [&](int b) { return bar(2 * LTC_MAX_PAIRS + 6 + b); };
  const uint32_t pready = bar(2 * LTC_MAX_PAIRS + 8), ofull = bar(2 * LTC_MAX_PAIRS + 9);
  auto qfull = [&](int b) { return bar(2 * LTC_MAX_PAIRS + 11 + b); };
  auto qfree = [&](int b) { return bar(2 * LTC_MAX_PAIRS + 13 + b); };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int s = 0; s < LTC_MAX_PAIRS; ++s) {
      ptx::mbar_init(pfull(s), 1);
      ptx::mbar_init(pempty(s), 1);
    }
    for (int b = 0; b < 2; ++b) {
      ptx::mbar_init(rfull(b), 1);
      ptx::mbar_init(rempty(b), 1);
      ptx::mbar_init(sfull(b), 1);
      ptx::mbar_init(sfree(b), 8);
      ptx::mbar_init(qfull(b), 1);
      ptx::mbar_init(qfree(b), 1);
    }
    ptx::mbar_init(pready, 8);
    ptx::mbar_init(ofull, 1);
    ptx::fence_barrier_init();
    ptx::prefetch_tensormap(&tm);
  }
  if (warp == 1) {
    ptx::tmem_alloc(ptx::smem_u32(&tmem_slot), TMEM_COLS);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tm_s = tmem_slot, tm_o = tm_s + 2 * NC;
  pdl_trigger();
  pdl_wait();
  const int count = *p.item_count;

  if (count == 0) {
    // nothing to do: straight to the teardown
  } else if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer (whole warp)
    const int subs = LTC_BN / p.box_tokens;      // boxes of one page's tokens per 128 keys
    const long long none = (long long)p.seqs.num_blocks * p.seqs.page_size;   // past the tensor: zeros arrive
    auto row_of = [&](const LtcItem& t, int j) -> int {      // first cache row of this lane's box of block j
      const int key = t.key0 + j * LTC_BN + lane * p.box_tokens;
      if (lane >= subs || key >= t.ctx) return (int)none;
      const long long row = latent_key_row(p.seqs, t.seq, key);
      return row < 0 ? (int)none : (int)row;
    };
    uint32_t pc = 0, rc = 0;
    bool ok = true;
    LtcItem t = ltc_item(p, ltc_raw(p, blockIdx.x, count));
    int row_next = (int)blockIdx.x < count ? row_of(t, 0) : (int)none;
    for (int idx = blockIdx.x; idx < count && ok; idx += gridDim.x) {
      const LtcRaw raw_next = ltc_raw(p, idx + gridDim.x, count);
      const int nblk = t.nblk;
      for (int j = 0; j < nblk && ok; ++j) {
        const int row = row_next;       // the look-up of the next block runs under this block's waits
        if (j + 1 < nblk) {
          row_next = row_of(t, j + 1);
        } else {
          t = ltc_item(p, raw_next);
          row_next = row_of(t, 0);
        }
        if (RB > 0) {
          const int s = rc % NR;
          ok = ptx::mbar_wait_warp(rempty(s), ((rc / NR) & 1) ^ 1, abort_flag, 700 + s);
          if (!ok) break;
          if (lane == 0) ptx::mbar_expect_tx(rfull(s), (uint32_t)RB * LTC_BOX);
          __syncwarp();
          if (lane < subs)
            for (int b = 0; b < RB; ++b)
              ptx::tma_load_2d(base + rot_off + (uint32_t)(s * RB + b) * LTC_BOX + (uint32_t)(lane * p.box_tokens) * 128,
                               &tm, rfull(s), R + b * 64, row, ptx::kEvictFirst);
          ++rc;
        }
        for (int i = 0; i < CP; ++i, ++pc) {
          const int s = pc % NP, nb = min(2, CB - 2 * i);
          ok = ptx::mbar_wait_warp(pempty(s), ((pc / NP) & 1) ^ 1, abort_flag, 710 + s);
          if (!ok) break;
          if (lane == 0) ptx::mbar_expect_tx(pfull(s), (uint32_t)nb * LTC_BOX);
          __syncwarp();
          if (lane < subs)
            for (int b = 0; b < nb; ++b)
              ptx::tma_load_2d(base + (uint32_t)(2 * s + b) * LTC_BOX + (uint32_t)(lane * p.box_tokens) * 128, &tm,
                               pfull(s), (2 * i + b) * 64, row, ptx::kEvictFirst);
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ UMMA issuer
    if (ptx::elect_one()) {
      const uint32_t idesc_s = umma_idesc_bf16(NC, false), idesc_o = umma_idesc_bf16(2 * NC, true);
      const uint64_t hi_k = ptx::umma_desc_k_sw128(0) & 0xFFFFFFFF00000000ull;
      auto kdesc = [&](uint32_t a) { return hi_k | (uint64_t)(((a & 0x3FFFFu) >> 4) | (1u << 16)); };
      const bool ahead = NP >= 2 * CP;   // QK^T of the next block may be issued before this block's value product
      uint32_t gs = 0, gp = 0, it = 0, sph = 0;
      int ss = 0, sp = 0;                // ring slot of the next pair of QK^T (sph: parity of its use) / of the value product
      int idx = blockIdx.x, j = 0, nblk = 0;
      LtcRaw raw_next = ltc_raw(p, idx, count);
      if (idx < count) {
        nblk = ltc_item(p, raw_next).nblk;
        raw_next = ltc_raw(p, idx + gridDim.x, count);
      }
      auto issue_s = [&]() {
        const int qb = it & 1, b = gs & 1, rs = NR == 2 ? gs & 1 : 0;
        if (j == 0 && !ptx::mbar_wait(qfull(qb), (it >> 1) & 1, abort_flag, 720 + qb)) return false;
        if (!ptx::mbar_wait(sfree(b), ((gs >> 1) & 1) ^ 1, abort_flag, 722 + b)) return false;
        if (RB > 0 && !ptx::mbar_wait(rfull(rs), (NR == 2 ? gs >> 1 : gs) & 1, abort_flag, 724 + rs)) return false;
        ptx::tc_fence_after();
        const uint32_t q0 = base + q_off + qb * q_bytes, d = tm_s + b * NC;
        // one 64-column box of the contraction; descriptors step by 32 bytes (2 units) per 16 columns
        auto box = [&](uint32_t a, int bx, int cols, uint32_t acc) {
          const uint64_t da = kdesc(a), db = kdesc(q0 + bx * (NC * 128));
          ptx::umma_bf16(d, da, db, idesc_s, acc);
          if (cols > 48) {
            ptx::umma_bf16_acc(d, da + 2, db + 2, idesc_s);
            ptx::umma_bf16_acc(d, da + 4, db + 4, idesc_s);
            ptx::umma_bf16_acc(d, da + 6, db + 6, idesc_s);
          } else {
            if (cols > 16) ptx::umma_bf16_acc(d, da + 2, db + 2, idesc_s);
            if (cols > 32) ptx::umma_bf16_acc(d, da + 4, db + 4, idesc_s);
          }
        };
        for (int r = 0; r < RB; ++r)
          box(base + rot_off + (uint32_t)(rs * RB + r) * LTC_BOX, r, min(64, DR - 64 * r), r != 0 ? 1u : 0u);
        if (RB > 0) ptx::umma_commit(rempty(rs));
#pragma unroll
        for (int i = 0; i < CP; ++i) {
          if (!ptx::mbar_wait(pfull(ss), sph, abort_flag, 730 + ss)) return false;
          ptx::tc_fence_after();
          const uint32_t a = base + (uint32_t)(2 * ss) * LTC_BOX;
          box(a, RB + 2 * i, min(64, R - 128 * i), i != 0 || RB > 0 ? 1u : 0u);
          if (2 * i + 1 < CB) box(a + LTC_BOX, RB + 2 * i + 1, min(64, R - 128 * i - 64), 1u);
          if (++ss == NP) {
            ss = 0;
            sph ^= 1;
          }
        }
        ptx::umma_commit(sfull(b));
        ++gs;
        if (++j == nblk) {
          ptx::umma_commit(qfree(qb));
          j = 0;
          ++it;
          idx += gridDim.x;
          nblk = ltc_item(p, raw_next).nblk;
          raw_next = ltc_raw(p, idx + gridDim.x, count);
        }
        return true;
      };
      bool ok = idx < count && issue_s();
      while (ok && gp < gs) {
        if (ahead && idx < count && !issue_s()) break;
        if (!ptx::mbar_wait(pready, gp & 1, abort_flag, 740)) break;
        ptx::tc_fence_after();
        const uint32_t keep = *(volatile int*)&s_fresh ? 0u : 1u;
        const uint64_t db = kdesc(base + p_off);
#pragma unroll
        for (int i = 0; i < CP; ++i) {
          const uint64_t da = umma_desc_mn_sw128(base + (uint32_t)(2 * sp) * LTC_BOX, LTC_BOX);   // + 16 keys: 2 KB
          const uint32_t d = tm_o + i * 2 * NC;
          ptx::umma_bf16(d, da, db, idesc_o, keep);
#pragma unroll
          for (int kk = 1; kk < LTC_BN / 16; ++kk)
            ptx::umma_bf16_acc(d, da + 128 * kk, db + (kk >> 2) * (2 * NC * 128 >> 4) + (kk & 3) * 2, idesc_o);
          ptx::umma_commit(pempty(sp));
          if (++sp == NP) sp = 0;
        }
        ptx::umma_commit(ofull);
        ++gp;
        if (!ahead && idx < count && !issue_s()) break;
      }
    }
  } else if (warp == 10) {
    // ------------------------------------------------------------------ query loader (whole warp), one item ahead
    uint32_t it = 0;
    LtcRaw raw_next = ltc_raw(p, blockIdx.x, count);
    for (int idx = blockIdx.x; idx < count; idx += gridDim.x, ++it) {
      const LtcItem t = ltc_item(p, raw_next);
      raw_next = ltc_raw(p, idx + gridDim.x, count);
      const int qb = it & 1;
      if (!ptx::mbar_wait_warp(qfree(qb), ((it >> 1) & 1) ^ 1, abort_flag, 760 + qb)) break;
      uint8_t* qd = base_ptr + q_off + qb * q_bytes;
      const __nv_bfloat16* q = p.q_lat + ((long long)t.t0 * p.heads + t.tile * NC) * (R + DR);
#pragma unroll 4
      for (int i = lane; i < NC * NBX * 8; i += 32) {
        const int c = i / (NBX * 8), ch = i % (NBX * 8), bx = ch >> 3;
        const int col = bx < RB ? ch * 8 : (ch - RB * 8) * 8;           // column of k_rot or of c
        const bool in = c < t.rows && col < (bx < RB ? DR : R);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (in) v = *reinterpret_cast<const uint4*>(q + (long long)c * (R + DR) + (bx < RB ? R + col : col));
        *reinterpret_cast<uint4*>(qd + bx * (NC * 128) + sw128(c, ch & 7)) = v;
      }
      ptx::fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(qfull(qb));
    }
  } else {
    // ------------------------------------------------------------------ softmax and accumulation (warps 2..9)
    // A thread is TMEM lane tl (key tl of the block for S^T, dim tl of every 128 for O^T) for columns c0 .. c0 + 7.
    constexpr int NCT = 256;
    const int ct = threadIdx.x - 64, q4 = warp & 3, hs = (warp - 2) >> 2, tl = q4 * 32 + lane, c0 = hs * NH;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    const int mycol = halving_col<NH>(lane);
    uint8_t* p_mine = base_ptr + p_off + (tl >> 6) * (2 * NC * 128) + (tl & 7) * 2;
    const int p_ch = (tl & 63) >> 3;
    const uint32_t reach = p.seqs.window > 0 ? (uint32_t)p.seqs.window : 0x80000000u;   // keys a column sees: 0 <= cpos - key < reach
    uint32_t g = 0;
    LtcRaw raw_next = ltc_raw(p, blockIdx.x, count);
    for (int idx = blockIdx.x; idx < count; idx += gridDim.x) {
      const LtcItem t = ltc_item(p, raw_next);
      raw_next = ltc_raw(p, idx + gridDim.x, count);
      int cpos[NH];
#pragma unroll
      for (int i = 0; i < NH; ++i)
        cpos[i] = c0 + i < t.rows ? t.ctx - t.len + (t.tile * NC + c0 + i) / p.heads : t.ctx - 1;
      float o[CP][NH], m[NH], l_w = 0.f;
#pragma unroll
      for (int i = 0; i < NH; ++i) {
        m[i] = -3.0e38f;     // a column that has seen no key yet: its weights come out as exact zeros
#pragma unroll
        for (int k = 0; k < CP; ++k) o[k][i] = 0.f;
      }
      auto fold = [&](const float (&f)[NH]) {   // o = (o + O^T) * f
#pragma unroll
        for (int k = 0; k < CP; ++k) {
          uint32_t hi[NH], lo[NH];
          tmem_ld8(tm_o + lane_addr + k * 2 * NC + c0, hi);
          tmem_ld8(tm_o + lane_addr + k * 2 * NC + NC + c0, lo);
          ptx::tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < NH; ++i)
            o[k][i] = (o[k][i] + (__uint_as_float(hi[i]) + __uint_as_float(lo[i]))) * f[i];
        }
      };
      for (int j = 0; j < t.nblk; ++j, ++g) {
        const int b = g & 1, key = t.key0 + j * LTC_BN + tl;
        float v[NH];
        bool over = j == 0;            // some weight would exceed the slack: the reference maxima have to move
        if (__all_sync(0xffffffffu, ptx::mbar_wait(sfull(b), (g >> 1) & 1, abort_flag, 770 + b))) {
          ptx::tc_fence_after();
          uint32_t r[NH];
          tmem_ld8(tm_s + lane_addr + b * NC + c0, r);
          ptx::tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < NH; ++i) {
            v[i] = (uint32_t)(cpos[i] - key) >= reach ? -INFINITY : __uint_as_float(r[i]) * p.scale_log2;
            over |= v[i] > m[i] + LTC_SLACK;
          }
          // keys past the context may hold anything: clear their rows of c so that 0 * value stays 0
          const int kb = t.key0 + j * LTC_BN;
          if (kb + LTC_BN > t.ctx) {
            for (int k = 0; k < CP; ++k) {
              uint8_t* slot = base_ptr + (size_t)(2 * ((g * CP + k) % NP)) * LTC_BOX;
              for (int r2 = t.ctx - kb + (ct >> 5); r2 < LTC_BN; r2 += NCT / 32) {
                reinterpret_cast<uint32_t*>(slot + r2 * 128)[lane] = 0u;
                if (2 * k + 1 < CB) reinterpret_cast<uint32_t*>(slot + LTC_BOX + r2 * 128)[lane] = 0u;
              }
            }
          }
        }
        const bool rescale = barrier_any(over, NCT);
        if (*abort_flag) break;
        float alpha[NH];
#pragma unroll
        for (int i = 0; i < NH; ++i) alpha[i] = 1.f;
        if (rescale) {                 // uniform over the compute threads
          float mine = -INFINITY;
#pragma unroll
          for (int i = 0; i < NH; ++i) {
            float w;
            asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(w) : "f"(v[i]));
            if ((lane & 7) == i) mine = w;
          }
          if (lane < 8) s_wmax[b][c0 + lane][q4] = mine;
          ptx::named_barrier_sync(3, NCT);
          if (*abort_flag) break;
#pragma unroll
          for (int i = 0; i < NH; ++i) {
            const float4 w = *reinterpret_cast<const float4*>(s_wmax[b][c0 + i]);
            const float cand = fmaxf(fmaxf(w.x, w.y), fmaxf(w.z, w.w));
            if (cand > m[i] + LTC_SLACK) {
              alpha[i] = fast_exp2(m[i] - cand);
              m[i] = cand;
            }
          }
        }
        float e[NH], a_mine = 1.f;
#pragma unroll
        for (int i = 0; i < NH; ++i) {
          e[i] = fast_exp2(v[i] - m[i]);
          if (i == mycol) a_mine = alpha[i];
        }
        // every value product so far has read its P^T tile and left its sums in tensor memory
        bool go = true;
        if (g > 0) go = __all_sync(0xffffffffu, ptx::mbar_wait(ofull, (g - 1) & 1, abort_flag, 772));
        if (go) {
          if (rescale && j > 0) {
            ptx::tc_fence_after();
            fold(alpha);
          }
          if (ct == 0) s_fresh = rescale;
#pragma unroll
          for (int i = 0; i < NH; ++i) {
            const int c = c0 + i;
            const __nv_bfloat16 hi = f2bf(e[i]);
            uint8_t* d = p_mine + c * 128 + ((p_ch ^ (c & 7)) << 4);
            *reinterpret_cast<__nv_bfloat16*>(d) = hi;
            *reinterpret_cast<__nv_bfloat16*>(d + NC * 128) = f2bf(e[i] - bf2f(hi));   // row 16 + c swizzles as row c
          }
          ptx::tc_fence_before();
          ptx::fence_proxy_async_smem();
          __syncwarp();
          if (lane == 0) {
            ptx::mbar_arrive(sfree(b));
            ptx::mbar_arrive(pready);
          }
          // the row sums, while the value product runs
          halving_warp_sum<NH>(e, lane);
          l_w = l_w * a_mine + e[0];
        }
      }
      bool go = !*abort_flag;
      if (go) go = __all_sync(0xffffffffu, ptx::mbar_wait(ofull, (g - 1) & 1, abort_flag, 773));
      if (go) {
        ptx::tc_fence_after();
        float one[NH];
#pragma unroll
        for (int i = 0; i < NH; ++i) one[i] = 1.f;
        fold(one);
        ptx::tc_fence_before();
        s_lred[c0 + mycol][q4] = l_w;
      }
      ptx::named_barrier_sync(3, NCT);
      if (*abort_flag) break;
#pragma unroll
      for (int i = 0; i < NH; ++i) {
        const int c = c0 + i;
        if (c >= t.rows) break;
        const float4 l4 = *reinterpret_cast<const float4*>(s_lred[c]);
        const float l = (l4.x + l4.y) + (l4.z + l4.w);
        if (t.splits == 1) {
          const float inv = 1.f / l;
          __nv_bfloat16* orow = p.out + ((long long)t.t0 * p.heads + t.tile * NC + c) * R;
#pragma unroll
          for (int k = 0; k < CP; ++k)
            if (k * 128 + tl < R) orow[k * 128 + tl] = f2bf(o[k][i] * inv);
        } else {
          float* orow = p.part_o + ((long long)idx * NC + c) * R;
#pragma unroll
          for (int k = 0; k < CP; ++k)
            if (k * 128 + tl < R) orow[k * 128 + tl] = o[k][i];
          if (tl == 0) p.part_ml[(long long)idx * NC + c] = make_float2(m[i], l);
        }
      }
    }
  }

  __syncthreads();
  if (*abort_flag) {   // let copies in flight land before the CTA exits
    const uint64_t w0 = global_timer_ns();
    while (global_timer_ns() - w0 < 200000ull) {
    }
  }
  ptx::tc_fence_after();
  if (warp == 1) {
    __syncwarp();
    ptx::tmem_dealloc(tm_s, TMEM_COLS);
  }
}

template <int CP>
inline int latent_tc_launch(const CUtensorMap& tm, const LatentTcParams& p, int grid, cudaStream_t st) {
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, latent_tc_kernel<CP>, LTC_SMEM)) return rc;
  launch_k(latent_tc_kernel<CP>, dim3((unsigned)grid), dim3(LTC_THREADS), (size_t)LTC_SMEM, st, tm, p);
  return launch_status();
}

}  // namespace b200

// Work items of a step for b200_latent_attn_tc: items [max_items] pairs of int4, item_count [1], first_item [num_seqs] (i32).
// The list depends on the sequences, the head count and the window only, so one list serves every layer that shares them.
extern "C" int b200_latent_plan(const void* query_start_loc, const void* context_lens, int num_seqs, int min_len,
                                int max_len, int window, int heads, int max_items, void* items, void* item_count, void* first_item,
                                void* stream) {
  using namespace b200;
  if (!query_start_loc || !context_lens || !items || !item_count || !first_item || num_seqs <= 0 || heads <= 0 ||
      max_items <= 0 || window < 0)
    return B200_ERR_ARG;
  LatentPlanParams p{{(const int*)query_start_loc, (const int*)context_lens, nullptr, 0, 0, 0, 0, num_seqs, min_len, max_len,
                      window},
                     heads, max_items, (int4*)items, (int*)item_count, (int*)first_item};
  launch_k(latent_plan_kernel, dim3(1), dim3(1024), 0, (cudaStream_t)stream, p);
  return launch_status();
}

// b200_latent_attn_simt on tensor cores (bf16) for the sequences of a plan; min_len / max_len as the plan was made with.
// R <= 512, DR <= 128 (0: no rotated part), multiples of 8; page_size a power of two of at least 8, or a multiple of 128.
// part_o [max_items, 16, R] and part_ml [max_items, 16, 2] fp32: scratch, NULL when no sequence has several splits (of 512
// keys, at multiples of 512).
extern "C" int b200_latent_attn_tc(const void* q_lat, const void* cache, void* out, const void* query_start_loc,
                                   const void* context_lens, const void* page_table, long long page_table_stride,
                                   int max_pages, int page_size, int num_blocks, int num_seqs, int min_len, int max_len,
                                   int window, long long T, int heads, int R, int DR, float scale, const void* items,
                                   const void* item_count, const void* first_item, int max_items, void* part_o,
                                   void* part_ml, void* stream) {
  using namespace b200;
  LatentTcParams p{};
  p.seqs = {(const int*)query_start_loc, (const int*)context_lens, (const int*)page_table, page_table_stride, max_pages,
            page_size, num_blocks, num_seqs, min_len, max_len, window};
  if (!latent_seqs_ok(p.seqs) || window < 0 || !q_lat || !cache || !out || !items || !item_count || !first_item || T < 0 || heads <= 0 ||
      R <= 0 || DR < 0 || max_items <= 0 || (part_o != nullptr) != (part_ml != nullptr))
    return B200_ERR_ARG;
  const bool pages_ok = page_size % LTC_BN == 0 || (page_size >= 8 && LTC_BN % page_size == 0);
  if (R % 8 || DR % 8 || R > 512 || DR > 128 || !pages_ok || T > 0x7fffffffLL || heads > 65535) return B200_ERR_SHAPE;
  if (T == 0) return B200_OK;
  p.q_lat = (const __nv_bfloat16*)q_lat;
  p.out = (__nv_bfloat16*)out;
  p.items = (const int4*)items;
  p.item_count = (const int*)item_count;
  p.max_items = max_items;
  p.part_o = (float*)part_o;
  p.part_ml = (float2*)part_ml;
  p.heads = heads;
  p.R = R;
  p.DR = DR;
  p.box_tokens = page_size < LTC_BN ? page_size : LTC_BN;
  p.scale_log2 = scale * kLog2e;
  const int cp = (R + 127) / 128, rb = (DR + 63) / 64, nbx = (R + 63) / 64 + rb;
  p.rot_slots = cp <= 3 ? 2 : 1;
  const int room = LTC_SMEM - 1024 - 2 * nbx * LTC_NC * 128 - 4 * LTC_NC * 128 - p.rot_slots * rb * LTC_BOX;
  p.pair_slots = room / (2 * LTC_BOX) < LTC_MAX_PAIRS ? room / (2 * LTC_BOX) : LTC_MAX_PAIRS;
  if (p.pair_slots < cp) return B200_ERR_SHAPE;
  CUtensorMap tm;
  if (int rc = make_tmap_2d(&tm, cache, (uint64_t)num_blocks * page_size, (uint64_t)(R + DR), (uint64_t)(R + DR),
                            (uint32_t)p.box_tokens))
    return rc;
  const cudaStream_t st = (cudaStream_t)stream;
  const int grid = max_items < sm_count() ? max_items : sm_count();
  int rc = B200_ERR_SHAPE;
  if (cp == 1) rc = latent_tc_launch<1>(tm, p, grid, st);
  else if (cp == 2) rc = latent_tc_launch<2>(tm, p, grid, st);
  else if (cp == 3) rc = latent_tc_launch<3>(tm, p, grid, st);
  else if (cp == 4) rc = latent_tc_launch<4>(tm, p, grid, st);
  if (rc || !part_o) return rc;
  LatentCombineParams c{p.seqs, (const int*)first_item, max_items, (const float*)part_o, (const float2*)part_ml, p.out,
                        heads, R};
  launch_k(latent_combine_kernel, dim3((unsigned)T, (unsigned)heads), dim3(128), 0, st, c);
  return launch_status();
}
