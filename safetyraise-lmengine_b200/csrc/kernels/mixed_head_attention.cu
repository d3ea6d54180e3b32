// Paged causal attention whose heads exchange their weights behind the softmax:
//
//   s_h(i, j) = (q_i . k_j) * scale + bias[h, min(i - j, n_dist - 1)]           q: head h, k: its KV head
//   p_h = softmax over the visible j:  j <= i and (i - j < window or j < keep)   (window 0: every earlier key)
//   w_h(i, j) = sum_g mix[h, g] p_g(i, j)                                        (mix null: w_h = p_h)
//   out_h(i) = (sum_j w_h(i, j) v_j) * logistic(gate row of the element)         v: h's own KV head
//
// The mixing needs every head's finished weight, so the softmax's maximum and sum come first and the weighted sum of the
// values second; a rescaled running sum does not serve.  This file holds the kernel that writes a step's keys and values
// (with the norm of q and k over all heads at once) and the float32 form of the attention, for the float32 engine and for
// sizes the tensor-core forms of mixed_head_attention_mma.cu do not take.
#include <math_constants.h>

#include "common.cuh"
#include "mixed_head_attention.cuh"

namespace srlm {

// One block per token: q (all heads at once) and k (all heads at once) of a stacked q | k | v projection are divided by
// their root mean square over the whole projection and multiplied by a weight per element (eps <= 0: as projected); q goes
// to its own buffer (float32 or bfloat16), k and v to the pages.
template <typename TP, typename TC>
__global__ void attention_wide_norm_append_kernel(const TP* __restrict__ proj, long long ldp, float eps,
                                                  const float* __restrict__ qw, const float* __restrict__ kw,
                                                  float* __restrict__ q_out, bf16* __restrict__ q_out_bf16,
                                                  TC* __restrict__ k_cache, TC* __restrict__ v_cache,
                                                  const int* __restrict__ kv_slot, int write_kv, int nq, int nkv, int dk,
                                                  int dv, int page_size) {
  pdl_wait();
  pdl_trigger();
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const TP* p = proj + (size_t)t * ldp;
  const int nqd = nq * dk, nkd = nkv * dk, nvd = nkv * dv;
  float inv_q = 1.f, inv_k = 1.f;
  if (eps > 0.f) {
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < nqd; c += blockDim.x) {
      const float v = to_float(p[c]);
      sq += v * v;
    }
    for (int c = threadIdx.x; c < nkd; c += blockDim.x) {
      const float v = to_float(p[nqd + c]);
      sk += v * v;
    }
    inv_q = 1.f / sqrtf(block_sum(sq, scratch) / (float)nqd + eps);
    inv_k = 1.f / sqrtf(block_sum(sk, scratch) / (float)nkd + eps);
  }
  for (int c = threadIdx.x; c < nqd; c += blockDim.x) {
    const float v = to_float(p[c]) * inv_q * (qw ? qw[c] : 1.f);
    if (q_out_bf16) q_out_bf16[(size_t)t * nqd + c] = __float2bfloat16_rn(v);
    else q_out[(size_t)t * nqd + c] = v;
  }
  if (!write_kv) return;
  const int slot = kv_slot[t];
  const size_t page = slot / page_size, off = slot % page_size;
  for (int c = threadIdx.x; c < nkd; c += blockDim.x) {
    const int h = c / dk, d = c - h * dk;
    k_cache[((page * nkv + h) * page_size + off) * dk + d] = from_float<TC>(to_float(p[nqd + c]) * inv_k * (kw ? kw[c] : 1.f));
  }
  for (int c = threadIdx.x; c < nvd; c += blockDim.x) {
    const int h = c / dv, d = c - h * dv;
    v_cache[((page * nkv + h) * page_size + off) * dv + d] = from_float<TC>(to_float(p[nqd + nkd + c]));
  }
}

// Float32 arithmetic, any sizes.  A block takes one token and all its heads and walks the visible keys twice in tiles of
// 32 aligned to the start of the sequence: once for every head's maximum and sum, once for the weights, their mixture and
// the sums over the values.  A token's sums depend on its position alone.
constexpr int kMixKeys = 32;

template <typename TC, typename TO>
__global__ void __launch_bounds__(256)
mixed_head_attention_kernel(const float* __restrict__ q, const TC* __restrict__ k_cache, const TC* __restrict__ v_cache,
                            TO* __restrict__ out, const int* __restrict__ block_table, int table_stride,
                            const int* __restrict__ entry_of_token, const int* __restrict__ positions, int nq, int nkv,
                            int dk, int dv, int page_size, float scale, MixMask mask, DistanceBias bias,
                            const float* __restrict__ mix, ElementGate gate) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float mh_smem[];
  const int wide = dk + 1 > dv ? dk + 1 : dv;
  float* q_s = mh_smem;                            // [nq][dk]
  float* tile = q_s + (size_t)nq * dk;             // [32][dk + 1] keys of one KV head, or [32][dv] values
  float* p_s = tile + (size_t)kMixKeys * wide;     // [nq][32] scores, then weights
  float* w_s = p_s + (size_t)nq * kMixKeys;        // [nq][32] mixed weights
  float* m_s = w_s + (size_t)nq * kMixKeys;        // [nq]
  float* l_s = m_s + nq;                           // [nq]
  float* acc = l_s + nq;                           // [nq][dv]
  const int t = blockIdx.x, pos = positions[t];
  const int* table = block_table + (size_t)entry_of_token[t] * table_stride;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  const int G = nq / nkv, first = mask.first_key(pos);
  for (int c = tid; c < nq * dk; c += blockDim.x) q_s[c] = q[(size_t)t * nq * dk + c];
  for (int c = tid; c < nq * dv; c += blockDim.x) acc[c] = 0.f;
  for (int h = tid; h < nq; h += blockDim.x) {
    m_s[h] = -CUDART_INF_F;
    l_s[h] = 0.f;
  }
  for (int pass = 0; pass < 2; ++pass) {
    for (int jb = 0; jb <= pos; jb += kMixKeys) {
      if (jb >= mask.keep && jb + kMixKeys <= first) {      // nothing visible up to the window's first tile
        jb = first / kMixKeys * kMixKeys;
      }
      const int j = jb + lane;
      const bool seen = mask.visible(pos, j);
      for (int c = 0; c < nkv; ++c) {
        __syncthreads();
        for (int idx = tid; idx < kMixKeys * dk; idx += blockDim.x) {
          const int jj = idx / dk, d = idx - jj * dk;
          float v = 0.f;
          if (mask.visible(pos, jb + jj)) {                 // pages nobody sees any more may be given back
            const size_t row = ((size_t)table[(jb + jj) / page_size] * nkv + c) * page_size + (jb + jj) % page_size;
            v = to_float(k_cache[row * dk + d]);
          }
          tile[jj * (dk + 1) + d] = v;
        }
        __syncthreads();
        for (int h = c * G + warp; h < (c + 1) * G; h += warps) {
          float dot = 0.f;
          for (int d = 0; d < dk; ++d) dot += q_s[h * dk + d] * tile[lane * (dk + 1) + d];
          float s = -CUDART_INF_F;
          if (seen) s = dot * scale + bias.at(h, pos - j);
          if (pass == 0) {
            const float m_new = fmaxf(m_s[h], warp_max(s));
            const float sum = warp_sum(seen ? expf(s - m_new) : 0.f);
            __syncwarp();
            if (lane == 0 && m_new != -CUDART_INF_F) {
              l_s[h] = l_s[h] * expf(m_s[h] - m_new) + sum;
              m_s[h] = m_new;
            }
            __syncwarp();
          } else {
            p_s[h * kMixKeys + lane] = seen ? expf(s - m_s[h]) / l_s[h] : 0.f;
          }
        }
      }
      if (pass == 0) continue;
      __syncthreads();
      const float* w = p_s;
      if (mix) {
        for (int h = warp; h < nq; h += warps) {
          float a = 0.f;
          for (int g = 0; g < nq; ++g) a += mix[h * nq + g] * p_s[g * kMixKeys + lane];
          w_s[h * kMixKeys + lane] = a;
        }
        w = w_s;
      }
      const int n_here = min(kMixKeys, pos - jb + 1);
      for (int c = 0; c < nkv; ++c) {
        __syncthreads();
        for (int idx = tid; idx < kMixKeys * dv; idx += blockDim.x) {
          const int jj = idx / dv, d = idx - jj * dv;
          float v = 0.f;
          if (mask.visible(pos, jb + jj)) {
            const size_t row = ((size_t)table[(jb + jj) / page_size] * nkv + c) * page_size + (jb + jj) % page_size;
            v = to_float(v_cache[row * dv + d]);
          }
          tile[idx] = v;
        }
        __syncthreads();
        for (int idx = tid; idx < G * dv; idx += blockDim.x) {
          const int h = c * G + idx / dv, d = idx % dv;
          float a = acc[h * dv + d];
          for (int jj = 0; jj < n_here; ++jj) a += w[h * kMixKeys + jj] * tile[jj * dv + d];
          acc[h * dv + d] = a;
        }
      }
    }
  }
  __syncthreads();
  for (int c = tid; c < nq * dv; c += blockDim.x) out[(size_t)t * nq * dv + c] = from_float<TO>(acc[c] * gate.at(t, c));
}

}  // namespace srlm

using namespace srlm;

// proj [T, ldp]: columns q (nq dk), k (nkv dk), v (nkv dv), then whatever else the projection carries; qw float32 [nq dk],
// kw float32 [nkv dk] (null: no weight).
extern "C" int srlm_attention_wide_norm_append(const void* proj, int proj_dtype, long long ldp, float eps, const float* qw,
                                               const float* kw, void* q_out, int q_dtype, void* k_cache, void* v_cache,
                                               int cache_dtype, const int* kv_slot, int write_kv, int T, int nq, int nkv,
                                               int dk, int dv, int page_size, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (nq <= 0 || nkv <= 0 || dk <= 0 || dv <= 0 || page_size <= 0 || ldp < (long long)nq * dk + (long long)nkv * (dk + dv))
    return refuse(ST_BAD_SIZE, "attention_wide_norm_append: nq=%d nkv=%d dk=%d dv=%d ldp=%lld", nq, nkv, dk, dv, ldp);
#define SRLM_APPEND(TP, TC)                                                                                        \
  launch_pdl(attention_wide_norm_append_kernel<TP, TC>, dim3(T), dim3(256), 0, stream, (const TP*)proj, ldp, eps, qw, kw, \
             q_dtype == DT_F32 ? (float*)q_out : nullptr, q_dtype == DT_BF16 ? (bf16*)q_out : nullptr,             \
             (TC*)k_cache, (TC*)v_cache, kv_slot, write_kv, nq, nkv, dk, dv, page_size)
  if (proj_dtype == DT_F32 && cache_dtype == DT_F32) SRLM_APPEND(float, float);
  else if (proj_dtype == DT_F32 && cache_dtype == DT_BF16) SRLM_APPEND(float, bf16);
  else return refuse(ST_BAD_DTYPE, "attention_wide_norm_append: projection dtype %d with cache dtype %d", proj_dtype, cache_dtype);
#undef SRLM_APPEND
  return launched();
}

// q float32 [T, nq, dk]; k_cache [pages, nkv, page_size, dk], v_cache [pages, nkv, page_size, dv]; out [T, nq, dv];
// bias float32 [nq, n_dist] or null; mix float32 [nq, nq] or null; gate_logits float32 [T, ld_gate] (nq dv columns) or null.
extern "C" int srlm_mixed_head_attention(const float* q, const void* k_cache, const void* v_cache, void* out, int cache_dtype,
                                         int out_dtype, const int* block_table, int table_stride, const int* entry_of_token,
                                         const int* positions, int T, int nq, int nkv, int dk, int dv, int page_size,
                                         float scale, int window, int keep, const float* bias, int n_dist, const float* mix,
                                         const float* gate_logits, long long ld_gate, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (nq <= 0 || nkv <= 0 || nq % nkv || dk <= 0 || dv <= 0 || page_size <= 0 || window < 0 || keep < 0 || (bias && n_dist <= 0))
    return refuse(ST_BAD_SIZE, "mixed_head_attention: nq=%d nkv=%d dk=%d dv=%d window=%d keep=%d", nq, nkv, dk, dv, window, keep);
  const size_t wide = dk + 1 > dv ? dk + 1 : dv;
  const size_t smem = ((size_t)nq * dk + kMixKeys * wide + 2ull * nq * kMixKeys + 2ull * nq + (size_t)nq * dv) * sizeof(float);
  if (smem > 220 * 1024)
    return refuse(ST_BAD_SIZE, "mixed_head_attention: %d heads of %d and %d need %zu bytes of shared memory", nq, dk, dv, smem);
  const MixMask mask{window, window > 0 ? keep : 0};
  const DistanceBias db{bias, n_dist};
  const ElementGate gate{gate_logits, ld_gate};
#define SRLM_MIX(TC, TO)                                                                                                    \
  do {                                                                                                                      \
    auto kern = mixed_head_attention_kernel<TC, TO>;                                                                        \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);               \
    launch_pdl(kern, dim3(T), dim3(256), smem, stream, q, (const TC*)k_cache, (const TC*)v_cache, (TO*)out, block_table,    \
               table_stride, entry_of_token, positions, nq, nkv, dk, dv, page_size, scale, mask, db, mix, gate);            \
  } while (0)
  if (cache_dtype == DT_F32 && out_dtype == DT_F32) SRLM_MIX(float, float);
  else if (cache_dtype == DT_BF16 && out_dtype == DT_BF16) SRLM_MIX(bf16, bf16);
  else return refuse(ST_BAD_DTYPE, "mixed_head_attention: cache dtype %d with output dtype %d", cache_dtype, out_dtype);
#undef SRLM_MIX
  return launched();
}
