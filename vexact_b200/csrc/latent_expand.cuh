// Expanded form of latent attention for long portions of prompts (bf16): the latents of a sequence's whole context have
// been gathered from their pages and projected up to per-head keys and values, and this kernel runs ordinary causal
// attention over them.
//
//   kv rows   [keys: H * DN | values: H * DV]  (one row per key of the gathered sequences)
//   lat rows  [c: R | k_rot: DR]               (the rotated key part shared by the heads is read from here)
//   q         [T, q_stride]: per head DN unrotated, then DR rotated columns
//   out[t, h] = sigmoid(gate[t, h]) * sum_j softmax(scale q.k_j) v_j
//
// One CTA per (128 MT queries, head, sequence); warp w of 8 owns query rows 16 MT w .. 16 MT (w + 1) - 1 (MT = 2 for long
// portions: every key and value fragment read from shared memory then serves two products); 64 keys per block, double
// buffered with cp.async, 32 per softmax step.  Scores and weights stay fp32: a weight enters the value product as a bf16 pair hi + lo.
// Query tiles are dealt from a sequence's last (longest) to its first.
#pragma once
#include "attn_tc.cuh"     // fast_exp2
#include "latent.cuh"
#include "ssm_chunk.cuh"   // cp.async, split_bf2, fragment loads

namespace b200 {

constexpr int LEX_BN = 64, LEX_SUB = 32, LEX_THREADS = 256;

struct LatentExpandParams {
  const int* query_start_loc;
  const int* context_lens;
  const int* seq_ids;      // [n] gathered sequences
  const int* key_start;    // [n + 1] first kv / lat row of each
  const __nv_bfloat16* q;
  const __nv_bfloat16* kv;
  const __nv_bfloat16* lat;
  const __nv_bfloat16* gate;
  __nv_bfloat16* out;
  long long q_stride, kv_stride, lat_stride, gate_stride, out_stride;
  int heads, DN, DR, DV, rot_off;   // rot_off: column of k_rot in a lat row
  float scale_log2;
};

template <int DK, int DV, int MT>
struct LexLayout {
  static constexpr int BM = 128 * MT;
  static constexpr int LDK = DK + 8, LDV = DV + 8;
  static constexpr int Q = BM * LDK * 2, K = LEX_BN * LDK * 2, V = LEX_BN * LDV * 2;
  static constexpr int BYTES = Q + 2 * (K + V);
};

template <int DK, int DV, int MT>
__global__ void __launch_bounds__(LEX_THREADS, 1) latent_expand_kernel(const LatentExpandParams p) {
  using L = LexLayout<DK, DV, MT>;
  constexpr int LEX_BM = L::BM, NS = LEX_SUB / 8;
  extern __shared__ __align__(16) uint8_t lex_smem[];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.z, h = blockIdx.y, seq = p.seq_ids[i];
  const int t0 = p.query_start_loc[seq], len = p.query_start_loc[seq + 1] - t0;
  const int tiles = (len + LEX_BM - 1) / LEX_BM;
  if ((int)blockIdx.x >= tiles) return;
  const int row_base = (tiles - 1 - (int)blockIdx.x) * LEX_BM;
  const int keys = p.key_start[i + 1] - p.key_start[i], past = keys - len;
  const long long key0 = p.key_start[i];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const uint32_t smem = ptx::smem_u32(lex_smem);
  const int dk16 = (p.DN + p.DR + 15) / 16;
  const int rows = min(LEX_BM, len - row_base);
  const int last_key = min(keys, past + row_base + rows);       // keys any row of the tile sees
  const int blocks = (last_key + LEX_BN - 1) / LEX_BN;

  for (int e = tid; e < LEX_BM * (DK / 8); e += LEX_THREADS) {
    const int r = e / (DK / 8), v = e % (DK / 8);
    const bool in = r < rows && v * 8 < p.DN + p.DR;
    cp_async16(smem + (uint32_t)(r * L::LDK + v * 8) * 2,
               p.q + (long long)(t0 + row_base + (in ? r : 0)) * p.q_stride + (long long)h * (p.DN + p.DR) + (in ? v * 8 : 0),
               in);
  }
  auto load = [&](int b) {
    const uint32_t k = smem + L::Q + (b & 1) * (L::K + L::V), vt = k + L::K;
    const int base = b * LEX_BN;
    for (int e = tid; e < LEX_BN * (DK / 8); e += LEX_THREADS) {
      const int r = e / (DK / 8), col = (e % (DK / 8)) * 8;
      const bool in = base + r < last_key && col < p.DN + p.DR;
      const long long row = key0 + (in ? base + r : 0);
      const __nv_bfloat16* src = col < p.DN || !in ? p.kv + row * p.kv_stride + (long long)h * p.DN + (in ? col : 0)
                                                   : p.lat + row * p.lat_stride + p.rot_off + (col - p.DN);
      cp_async16(k + (uint32_t)(r * L::LDK + col) * 2, src, in);
    }
    for (int e = tid; e < LEX_BN * (DV / 8); e += LEX_THREADS) {
      const int r = e / (DV / 8), col = (e % (DV / 8)) * 8;
      const bool in = base + r < last_key && col < p.DV;
      cp_async16(vt + (uint32_t)(r * L::LDV + col) * 2,
                 p.kv + (key0 + (in ? base + r : 0)) * p.kv_stride + (long long)p.heads * p.DN + (long long)h * p.DV +
                     (in ? col : 0),
                 in);
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
  for (int b = 0; b < blocks; ++b) {
    if (b + 1 < blocks) {
      load(b + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t sk = smem + L::Q + (b & 1) * (L::K + L::V), sv = sk + L::K;
#pragma unroll 1
    for (int sub = 0; sub < LEX_BN / LEX_SUB; ++sub) {
      const int base = b * LEX_BN + sub * LEX_SUB;
      if (r0 >= rows || base > first_pos + 16 * MT - 1) break;   // no row of this warp sees these keys
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
      const bool edge = base + LEX_SUB - 1 > first_pos;           // some (row, key) of these is masked
#pragma unroll
      for (int t = 0; t < MT; ++t) {
        const int pos0 = first_pos + 16 * t + g4;                 // position of row g4 of the tile (and + 8)
        float mb[2] = {m[t][0], m[t][1]};
#pragma unroll
        for (int j = 0; j < NS; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float v = s[t][j][e] * p.scale_log2;
            if (edge && base + 8 * j + 2 * t4 + (e & 1) > pos0 + 8 * (e >> 1)) v = -INFINITY;
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
      const float inv = 1.f / abm_quad_sum(l[tt][e]);
      const int r = r0 + 16 * tt + g4 + 8 * e;
      if (r >= rows) continue;
      const long long t = t0 + row_base + r;
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) {
        const int c = 8 * j + 2 * t4;
        if (c < p.DV) {
          float ga, gb;
          unpack_bf2(*reinterpret_cast<const uint32_t*>(p.gate + t * p.gate_stride + (long long)h * p.DV + c), ga, gb);
          *reinterpret_cast<uint32_t*>(p.out + t * p.out_stride + (long long)h * p.DV + c) =
              pack_bf2(o[tt][j][2 * e] * inv * __fdividef(1.f, 1.f + __expf(-ga)),
                       o[tt][j][2 * e + 1] * inv * __fdividef(1.f, 1.f + __expf(-gb)));
        }
      }
    }
}

template <int DK, int DV, int MT>
inline int latent_expand_launch(const LatentExpandParams& p, int max_len, int n, cudaStream_t st) {
  constexpr int smem = LexLayout<DK, DV, MT>::BYTES, LEX_BM = LexLayout<DK, DV, MT>::BM;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  static PerDeviceFlags attr_set;
  if (int rc = set_max_dyn_smem_once(attr_set, latent_expand_kernel<DK, DV, MT>, smem)) return rc;
  launch_k(latent_expand_kernel<DK, DV, MT>, dim3((unsigned)((max_len + LEX_BM - 1) / LEX_BM), (unsigned)p.heads, (unsigned)n),
           dim3(LEX_THREADS), (size_t)smem, st, p);
  return launch_status();
}

}  // namespace b200

// Causal attention of n gathered sequences (bf16; see the head of this file).  DN, DR, DV multiples of 8,
// DN + DR and DV <= 256; max_len: the most tokens any of them brings in this step.
extern "C" int b200_latent_attn_expanded(const void* q, long long q_row_stride, const void* kv, long long kv_row_stride,
                                         const void* lat, long long lat_row_stride, int rot_off, const void* gate,
                                         long long gate_row_stride, void* out, long long out_row_stride,
                                         const void* query_start_loc, const void* context_lens, const void* seq_ids_i32,
                                         const void* key_start_i32, int n, int max_len, int heads, int DN, int DR, int DV,
                                         float scale, void* stream) {
  using namespace b200;
  if (!q || !kv || !lat || !gate || !out || !query_start_loc || !context_lens || !seq_ids_i32 || !key_start_i32 || n <= 0 ||
      max_len <= 0 || heads <= 0 || DN <= 0 || DR < 0 || DV <= 0)
    return B200_ERR_ARG;
  if (DN % 8 || DR % 8 || DV % 8 || rot_off % 8 || q_row_stride % 8 || kv_row_stride % 8 || lat_row_stride % 8 ||
      gate_row_stride % 8 || out_row_stride % 8 || DN + DR > 256 || DV > 256 || heads > 65535 || n > 65535)
    return B200_ERR_SHAPE;
  LatentExpandParams p{(const int*)query_start_loc, (const int*)context_lens, (const int*)seq_ids_i32,
                       (const int*)key_start_i32, (const __nv_bfloat16*)q, (const __nv_bfloat16*)kv,
                       (const __nv_bfloat16*)lat, (const __nv_bfloat16*)gate, (__nv_bfloat16*)out, q_row_stride,
                       kv_row_stride, lat_row_stride, gate_row_stride, out_row_stride, heads, DN, DR, DV, rot_off,
                       scale * kLog2e};
  const int dk = DN + DR;
  const cudaStream_t st = (cudaStream_t)stream;
  const bool two = max_len > 128;
  if (dk <= 64 && DV <= 64) return two ? latent_expand_launch<64, 64, 2>(p, max_len, n, st) : latent_expand_launch<64, 64, 1>(p, max_len, n, st);
  if (dk <= 128 && DV <= 128)
    return two ? latent_expand_launch<128, 128, 2>(p, max_len, n, st) : latent_expand_launch<128, 128, 1>(p, max_len, n, st);
  if (dk <= 192 && DV <= 128)
    return two ? latent_expand_launch<192, 128, 2>(p, max_len, n, st) : latent_expand_launch<192, 128, 1>(p, max_len, n, st);
  return latent_expand_launch<256, 256, 1>(p, max_len, n, st);
}
