// Causal attention of long portions of prompts over per-head keys and values (bf16), optionally inside a window or chunk.
// Two sources of keys:
//
//   expanded latents   the latents of a sequence's context (from the first key the window reaches) have been gathered from
//                      their pages and projected up: packed kv rows [keys: G * DN | values: G * DV], and lat rows
//                      [c: R | k_rot: DR] from which the rotated key part shared by the heads is read
//   paged heads        k and v rows of a paged cache, [G * DN] and [G * DV] (DR = 0)
//
//   q         [T, q_stride]: per head DN unrotated, then DR rotated columns; head h uses key / value head h / group
//   out[t, h] = sum_j softmax(scale q.k_j) v_j, times the sigmoid of a gate per column, if any; FORM: with
//               the kept tokens, chunks, cap, sink, gate or sigmoid weights of attn_extras.cuh
//
// One CTA per (128 MT queries, head, sequence); warp w of 8 owns query rows 16 MT w .. 16 MT (w + 1) - 1 (MT = 2 for long
// portions: every key and value fragment read from shared memory then serves two products); 64 keys per block, double
// buffered with cp.async, 32 per softmax step.  Scores and weights stay fp32: a weight enters the value product as a bf16
// pair hi + lo.  Query tiles are dealt from a sequence's last (longest) to its first.
#pragma once
#include "attn_tc.cuh"     // fast_exp2
#include "latent.cuh"
#include "ssm_chunk.cuh"   // cp.async, split_bf2, fragment loads

namespace b200 {

constexpr int LEX_BN = 64, LEX_SUB = 32, LEX_THREADS = 256;

struct LatentExpandParams {
  LatentSeqs seqs;
  const int* seq_ids;      // [n] sequences with long portions
  const int* key_start;    // [n + 1] first packed row of each (packed sources)
  const int* key_base;     // [n] position of that row's key (packed sources)
  const __nv_bfloat16* q;
  const __nv_bfloat16* k;      // rows k_stride apart, head g at column g * DN
  const __nv_bfloat16* v;      // rows v_stride apart, head g at column g * DV
  const __nv_bfloat16* rot;    // rows rot_stride apart: the shared rotated part (DR > 0)
  __nv_bfloat16* out;
  long long q_stride, k_stride, v_stride, rot_stride, out_stride;
  int heads, group, DN, DR, DV;
  float scale_log2;
  AttnExtras extras;
};

template <int DK, int DV, int MT>
struct LexLayout {
  static constexpr int BM = 128 * MT;
  static constexpr int LDK = DK + 8, LDV = DV + 8;
  static constexpr int Q = BM * LDK * 2, K = LEX_BN * LDK * 2, V = LEX_BN * LDV * 2;
  static constexpr int BYTES = Q + 2 * (K + V);
};

template <int DK, int DV, int MT, bool PAGED, int FORM>
__global__ void __launch_bounds__(LEX_THREADS, 1) latent_expand_kernel(const LatentExpandParams p) {
  using L = LexLayout<DK, DV, MT>;
  constexpr int LEX_BM = L::BM, NS = LEX_SUB / 8;
  constexpr bool EXTRAS = FORM != ATTN_PLAIN, SIGMOID = FORM == ATTN_SIGMOID;
  extern __shared__ __align__(16) uint8_t lex_smem[];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.z, h = blockIdx.y, kvh = h / p.group, seq = p.seq_ids[i];
  const int t0 = p.seqs.query_start_loc[seq], len = p.seqs.query_start_loc[seq + 1] - t0;
  const int tiles = (len + LEX_BM - 1) / LEX_BM;
  if ((int)blockIdx.x >= tiles) return;
  const int row_base = (tiles - 1 - (int)blockIdx.x) * LEX_BM;
  const int keys = p.seqs.context_lens[seq], past = keys - len;
  const int window = p.seqs.window > 0 ? p.seqs.window : 0x3fffffff, chunk = EXTRAS ? p.seqs.chunk : 0;
  const int keep = EXTRAS ? p.seqs.keep : 0;
  const int key_base = PAGED ? 0 : p.key_base[i];
  const long long key0 = PAGED ? 0 : p.key_start[i] - key_base;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const uint32_t smem = ptx::smem_u32(lex_smem);
  const int dk16 = (p.DN + p.DR + 15) / 16;
  const int rows = min(LEX_BM, len - row_base);
  const int last_key = min(keys, past + row_base + rows);       // keys any row of the tile sees
  const int first_key = first_visible(window, chunk, past + row_base);
  const KeyBlocks walk = key_blocks<LEX_BN>(window, chunk, keep, past + row_base, last_key - 1);

  for (int e = tid; e < LEX_BM * (DK / 8); e += LEX_THREADS) {
    const int r = e / (DK / 8), v = e % (DK / 8);
    const bool in = r < rows && v * 8 < p.DN + p.DR;
    cp_async16(smem + (uint32_t)(r * L::LDK + v * 8) * 2,
               p.q + (long long)(t0 + row_base + (in ? r : 0)) * p.q_stride + (long long)h * (p.DN + p.DR) + (in ? v * 8 : 0),
               in);
  }
  auto seen = [&](int j) {      // by some row of the tile
    return (uint32_t)(j - first_key) < (uint32_t)(last_key - first_key) || (EXTRAS && j < min(keep, last_key));
  };
  // source row of key j; a key that is not wanted (or whose page is bad) names some readable row
  auto row_of = [&](int j, bool& in) -> long long {
    if constexpr (PAGED) {
      const long long row = in ? latent_key_row(p.seqs, seq, j) : -1;
      in = row >= 0;
      return in ? row : 0;
    } else {
      return key0 + (in ? j : first_key);
    }
  };
  auto load = [&](int b) {      // block b of the walk
    const uint32_t k = smem + L::Q + (b & 1) * (L::K + L::V), vt = k + L::K;
    const int base = walk.at(b) * LEX_BN;
    for (int e = tid; e < LEX_BN * (DK / 8); e += LEX_THREADS) {
      const int r = e / (DK / 8), col = (e % (DK / 8)) * 8;
      bool in = seen(base + r) && col < p.DN + p.DR;
      const long long row = row_of(base + r, in);
      const __nv_bfloat16* src = col < p.DN || !in ? p.k + row * p.k_stride + (long long)kvh * p.DN + (in ? col : 0)
                                                   : p.rot + row * p.rot_stride + (col - p.DN);
      cp_async16(k + (uint32_t)(r * L::LDK + col) * 2, src, in);
    }
    for (int e = tid; e < LEX_BN * (DV / 8); e += LEX_THREADS) {
      const int r = e / (DV / 8), col = (e % (DV / 8)) * 8;
      bool in = seen(base + r) && col < p.DV;
      const long long row = row_of(base + r, in);
      cp_async16(vt + (uint32_t)(r * L::LDV + col) * 2, p.v + row * p.v_stride + (long long)kvh * p.DV + (in ? col : 0), in);
    }
    cp_async_commit();
  };
  load(0);

  float o[MT][DV / 8][4];
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) o[t][j][0] = o[t][j][1] = o[t][j][2] = o[t][j][3] = 0.f;
  float m[MT][2], l[MT][2];
#pragma unroll
  for (int t = 0; t < MT; ++t) {
    m[t][0] = m[t][1] = -3.0e38f;
    l[t][0] = l[t][1] = 0.f;
  }
  const int r0 = 16 * MT * warp;
  const int first_pos = past + row_base + r0;                    // position of the warp's first row
  // no row of the warp sees keys before the first of these, every row sees from the second (up to itself)
  const int warp_first = EXTRAS ? first_visible(window, chunk, first_pos) : first_pos - window + 1;
  const int warp_full = EXTRAS ? first_visible(window, chunk, first_pos + 16 * MT - 1) : first_pos + 16 * MT - window;
  uint32_t reach[EXTRAS ? MT : 1][2];                            // a row sees 0 <= its position - key < reach
  if constexpr (EXTRAS) {
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
      for (int e = 0; e < 2; ++e) reach[t][e] = visible_keys(window, chunk, first_pos + 16 * t + g4 + 8 * e);
  }
  float bias = 0.f;                                              // of sigmoid weights, in units of log2
  if constexpr (SIGMOID) bias = p.extras.sigmoid_bias[h] * kLog2e;
  for (int b = 0; b < walk.count; ++b) {
    if (b + 1 < walk.count) {
      load(b + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t sk = smem + L::Q + (b & 1) * (L::K + L::V), sv = sk + L::K;
#pragma unroll 1
    for (int sub = 0; sub < LEX_BN / LEX_SUB; ++sub) {
      const int base = walk.at(b) * LEX_BN + sub * LEX_SUB;
      if (r0 >= rows || base > first_pos + 16 * MT - 1) break;   // no row of this warp sees these keys
      if (base + LEX_SUB - 1 < warp_first && base >= keep) continue;   // nor these, before every row's window or chunk
      float s[MT][NS][4];
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int j = 0; j < NS; ++j) s[t][j][0] = s[t][j][1] = s[t][j][2] = s[t][j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < dk16; ++kk) {
        uint32_t a[MT][4], kb[4];
#pragma unroll
        for (int t = 0; t < MT; ++t) abm_frag_a(smem, L::LDK, r0 + 16 * t, kk * 16, lane, a[t]);
#pragma unroll
        for (int j = 0; j < NS; j += 2) {
          abm_frag_b_rows(sk, L::LDK, sub * LEX_SUB + j * 8, kk * 16, lane, kb);
#pragma unroll
          for (int t = 0; t < MT; ++t) {
            mma_bf16_16816(s[t][j], a[t][0], a[t][1], a[t][2], a[t][3], kb[0], kb[1]);
            mma_bf16_16816(s[t][j + 1], a[t][0], a[t][1], a[t][2], a[t][3], kb[2], kb[3]);
          }
        }
      }
      // some (row, key) of these is masked
      const bool edge = base + LEX_SUB - 1 > first_pos || (base < warp_full && !(EXTRAS && base + LEX_SUB <= keep));
#pragma unroll
      for (int t = 0; t < MT; ++t) {
        const int pos0 = first_pos + 16 * t + g4;                 // position of row g4 of the tile (and + 8)
        float mb[2] = {m[t][0], m[t][1]};
#pragma unroll
        for (int j = 0; j < NS; ++j) {
#pragma unroll
          for (int e = 0; e < 4; ++e) s[t][j][e] *= p.scale_log2;
          if constexpr (EXTRAS) {
            if (p.extras.cap.cap > 0.f) cap_scores(s[t][j], p.extras.cap);
          }
        }
        if constexpr (SIGMOID) {
#pragma unroll
          for (int j = 0; j < NS; ++j) {
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
              const int key = base + 8 * j + 2 * t4, pos = pos0 + 4 * e;
              float a = s[t][j][e] + bias, b = s[t][j][e + 1] + bias;
              sigmoid_pair(a, b, !edge || key_visible(reach[t][e >> 1], keep, pos, key),
                           !edge || key_visible(reach[t][e >> 1], keep, pos, key + 1));
              s[t][j][e] = a;
              s[t][j][e + 1] = b;
            }
          }
        } else {
#pragma unroll
          for (int j = 0; j < NS; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float v = s[t][j][e];
              const uint32_t seen = EXTRAS ? reach[EXTRAS ? t : 0][e >> 1] : (uint32_t)window;   // 0 <= position - key < seen
              if (edge && !key_visible(seen, keep, pos0 + 8 * (e >> 1), base + 8 * j + 2 * t4 + (e & 1))) v = -INFINITY;
              s[t][j][e] = v;
              mb[e >> 1] = fmaxf(mb[e >> 1], v);
            }
          float alpha[2], sum[2] = {0.f, 0.f};
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mb[e] = abm_quad_max(mb[e]);
            alpha[e] = fast_exp2(m[t][e] - mb[e]);
          }
          const bool moved = mb[0] > m[t][0] || mb[1] > m[t][1];
          m[t][0] = mb[0];
          m[t][1] = mb[1];
#pragma unroll
          for (int j = 0; j < NS; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              s[t][j][e] = fast_exp2(s[t][j][e] - m[t][e >> 1]);
              sum[e >> 1] += s[t][j][e];
            }
#pragma unroll
          for (int e = 0; e < 2; ++e) l[t][e] = l[t][e] * alpha[e] + sum[e];   // the quad's four shares meet at the end
          if (__any_sync(0xffffffffu, moved)) {                     // otherwise every factor is exactly 1
#pragma unroll
            for (int j = 0; j < DV / 8; ++j) {
              o[t][j][0] *= alpha[0];
              o[t][j][1] *= alpha[0];
              o[t][j][2] *= alpha[1];
              o[t][j][3] *= alpha[1];
            }
          }
        }
      }
#pragma unroll
      for (int kt = 0; kt < LEX_SUB / 16; ++kt) {
        uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const float(&w)[4] = s[t][2 * kt + q];
            split_bf2(w[0], w[1], hi[t][2 * q], lo[t][2 * q]);
            split_bf2(w[2], w[3], hi[t][2 * q + 1], lo[t][2 * q + 1]);
          }
#pragma unroll
        for (int j = 0; j < DV / 8; j += 2) {
          if (j * 8 >= p.DV) break;
          uint32_t vb[4];
          abm_frag_b_cols(sv, L::LDV, sub * LEX_SUB + kt * 16, j * 8, lane, vb);
#pragma unroll
          for (int t = 0; t < MT; ++t) {
            mma_bf16_16816(o[t][j], hi[t][0], hi[t][1], hi[t][2], hi[t][3], vb[0], vb[1]);
            mma_bf16_16816(o[t][j + 1], hi[t][0], hi[t][1], hi[t][2], hi[t][3], vb[2], vb[3]);
          }
#pragma unroll
          for (int t = 0; t < MT; ++t) {
            mma_bf16_16816(o[t][j], lo[t][0], lo[t][1], lo[t][2], lo[t][3], vb[0], vb[1]);
            mma_bf16_16816(o[t][j + 1], lo[t][0], lo[t][1], lo[t][2], lo[t][3], vb[2], vb[3]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int tt = 0; tt < MT; ++tt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float inv = EXTRAS ? p.extras.out_scale : 1.f;
      if constexpr (!SIGMOID) {
        float sum = abm_quad_sum(l[tt][e]);
        if (EXTRAS) sum += sink_term(p.extras, h, m[tt][e]);
        inv /= sum;
      }
      const int r = r0 + 16 * tt + g4 + 8 * e;
      if (r >= rows) continue;
      const long long t = t0 + row_base + r;
      const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(p.extras.gate) + t * p.extras.gate_stride;
      if (EXTRAS && p.extras.gate_mode == GATE_HEAD) inv *= gate_sigmoid(gate[h]);
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) {
        const int c = 8 * j + 2 * t4;
        if (c < p.DV) {
          float a = o[tt][j][2 * e] * inv, b = o[tt][j][2 * e + 1] * inv;
          if (p.extras.gate_mode == GATE_COLUMN) {
            float ga, gb;
            unpack_bf2(*reinterpret_cast<const uint32_t*>(gate + h * p.DV + c), ga, gb);
            a *= sigmoid_fast(ga);
            b *= sigmoid_fast(gb);
          }
          *reinterpret_cast<uint32_t*>(p.out + t * p.out_stride + (long long)h * p.DV + c) = pack_bf2(a, b);
        }
      }
    }
}

template <int DK, int DV, int MT, bool PAGED, int FORM>
inline int latent_expand_launch(const LatentExpandParams& p, int max_len, int n, cudaStream_t st) {
  constexpr int smem = LexLayout<DK, DV, MT>::BYTES, LEX_BM = LexLayout<DK, DV, MT>::BM;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, latent_expand_kernel<DK, DV, MT, PAGED, FORM>, smem)) return rc;
  launch_k(latent_expand_kernel<DK, DV, MT, PAGED, FORM>,
           dim3((unsigned)((max_len + LEX_BM - 1) / LEX_BM), (unsigned)p.heads, (unsigned)n), dim3(LEX_THREADS), (size_t)smem,
           st, p);
  return launch_status();
}

template <bool PAGED, int FORM>
inline int latent_expand_dispatch(const LatentExpandParams& p, int max_len, int n, cudaStream_t st) {
  const int dk = p.DN + p.DR;
  const bool two = max_len > 128;
  if (dk <= 64 && p.DV <= 64)
    return two ? latent_expand_launch<64, 64, 2, PAGED, FORM>(p, max_len, n, st) : latent_expand_launch<64, 64, 1, PAGED, FORM>(p, max_len, n, st);
  if (dk <= 128 && p.DV <= 128)
    return two ? latent_expand_launch<128, 128, 2, PAGED, FORM>(p, max_len, n, st) : latent_expand_launch<128, 128, 1, PAGED, FORM>(p, max_len, n, st);
  if (dk <= 192 && p.DV <= 128)
    return two ? latent_expand_launch<192, 128, 2, PAGED, FORM>(p, max_len, n, st) : latent_expand_launch<192, 128, 1, PAGED, FORM>(p, max_len, n, st);
  return latent_expand_launch<256, 256, 1, PAGED, FORM>(p, max_len, n, st);
}

}  // namespace b200

// Causal attention of n gathered sequences (bf16; see the head of this file): packed row r of sequence i holds the key at
// position key_base[i] + r - key_start[i], up to its last.  gate NULL: no output gate.  DN, DR, DV multiples of 8,
// DN + DR and DV <= 256; max_len: the most tokens any of them brings in this step.
extern "C" int b200_latent_attn_expanded(const void* q, long long q_row_stride, const void* kv, long long kv_row_stride,
                                         const void* lat, long long lat_row_stride, int rot_off, const void* gate,
                                         long long gate_row_stride, void* out, long long out_row_stride,
                                         const void* query_start_loc, const void* context_lens, const void* seq_ids_i32,
                                         const void* key_start_i32, const void* key_base_i32, int n, int max_len, int window,
                                         int heads, int DN, int DR, int DV, float scale, void* stream) {
  using namespace b200;
  if (!q || !kv || !lat || !out || !query_start_loc || !context_lens || !seq_ids_i32 || !key_start_i32 || !key_base_i32 ||
      n <= 0 || max_len <= 0 || heads <= 0 || DN <= 0 || DR < 0 || DV <= 0 || window < 0)
    return B200_ERR_ARG;
  if (DN % 8 || DR % 8 || DV % 8 || rot_off % 8 || q_row_stride % 8 || kv_row_stride % 8 || lat_row_stride % 8 ||
      gate_row_stride % 8 || out_row_stride % 8 || DN + DR > 256 || DV > 256 || heads > 65535 || n > 65535)
    return B200_ERR_SHAPE;
  LatentExpandParams p{};
  p.seqs.query_start_loc = (const int*)query_start_loc;
  p.seqs.context_lens = (const int*)context_lens;
  p.seqs.window = window;
  p.seq_ids = (const int*)seq_ids_i32;
  p.key_start = (const int*)key_start_i32;
  p.key_base = (const int*)key_base_i32;
  p.q = (const __nv_bfloat16*)q;
  p.k = (const __nv_bfloat16*)kv;
  p.v = (const __nv_bfloat16*)kv + (long long)heads * DN;
  p.rot = (const __nv_bfloat16*)lat + rot_off;
  p.out = (__nv_bfloat16*)out;
  p.q_stride = q_row_stride;
  p.k_stride = p.v_stride = kv_row_stride;
  p.rot_stride = lat_row_stride;
  p.extras = {{}, nullptr, gate, gate_row_stride, gate ? GATE_COLUMN : GATE_NONE, nullptr, 1.f};
  p.out_stride = out_row_stride;
  p.heads = heads;
  p.group = 1;
  p.DN = DN;
  p.DR = DR;
  p.DV = DV;
  p.scale_log2 = scale * kLog2e;
  return latent_expand_dispatch<false, ATTN_PLAIN>(p, max_len, n, (cudaStream_t)stream);
}
