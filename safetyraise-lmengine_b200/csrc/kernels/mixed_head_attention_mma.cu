// The mixed-head attention of mixed_head_attention.cu on bfloat16 tensor cores (mma.sync m16n8k16, float32 sums).
//
// Prompts, portions and mixed steps take two kernels:
//   mixed_head_lse      every row's logarithm of the softmax's sum, L = log2 sum_j 2^(s_j), a block for 64 rows (tokens x
//                       query heads) of one KV head: the running maximum and sum of an ordinary attention, without values;
//   mixed_head_attention_mma   a block for 16 / HT tokens and ALL heads.  Per tile of 32 keys: every warp forms the scores
//                       of its 16 rows (HT heads x 16 / HT tokens) and p = 2^(s - L), finished weights; the block mixes
//                       them; every warp multiplies its rows of the mixture with its KV head's values.
// The mixture is a product of mix [H, H] with the weights of a tile [H, tokens x keys], on tensor cores with the weights as
// pairs of bfloat16 (p = hi + lo, 16 significant bits each way of the exact sum), float32 sums; mix itself is rounded to such
// a pair when its values are no bfloat16 numbers.  Keys and values have one buffer each: the next tile's keys are fetched
// while the block mixes and multiplies values, this tile's values while it forms scores.
//
// Decode steps (one token an entry) take one kernel: a thread-block cluster for an entry, a slice of its visible keys for
// each block.  A block forms the scores of all heads over its slice and keeps them in shared memory; the blocks exchange
// maxima and sums through distributed shared memory; each turns its scores into finished weights, mixes them, multiplies
// its slice's values; and the blocks add their sums, a share of the columns each, as they gate and write them.
#include <math_constants.h>

#include "common.cuh"
#include "mixed_head_attention.cuh"
#include "mma_sync.cuh"

namespace srlm {

constexpr float kLog2e = 1.4426950408889634f;
constexpr int kMhKeys = 32;                   // keys of a tile
constexpr int kMhPad = 8;
constexpr int kMhRow = kMhKeys + kMhPad;      // a token's weights of a tile in shared memory

// The tiles of `width` keys that some query at min_pos .. max_pos sees: those of the kept tokens, then those from the
// window's first key on.
struct MixTiles {
  int kept, base, count;
  __device__ __forceinline__ MixTiles(const MixMask& mask, int min_pos, int max_pos, int width) {
    base = mask.first_key(min_pos) / width;
    kept = mask.window > 0 ? min((mask.keep + width - 1) / width, base) : 0;
    count = kept + max_pos / width - base + 1;
  }
  __device__ __forceinline__ int key(int n, int width) const { return (n < kept ? n : base + n - kept) * width; }
};

// 2^x by the hardware's approximation (two units in the last place; results below 2^-126 become 0).
__device__ __forceinline__ float pow2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Pages of keys or values: the row of key j for KV head h is row(j) + h * size.  shift: log2 of the page size, or -1.
struct MixPages {
  const int* table;
  int nkv, size, shift;
  __device__ __forceinline__ int row(int j) const {
    const int page = shift >= 0 ? j >> shift : j / size;
    return __ldg(table + page) * nkv * size + (j - page * size);
  }
};

// A thread's share of a copy of rows of `vec` 16-byte pieces: piece c of rows r, r + step, ...
struct MixCopy {
  int r, c, step;
  __device__ __forceinline__ MixCopy(int vec, int threads) {
    step = threads / vec;
    r = (int)threadIdx.x / vec;
    c = (int)threadIdx.x - r * vec;
    if (r >= step) r = 1 << 30;               // threads left over copy nothing
  }
};

// ---- the softmax's sums -------------------------------------------------------------------------------------------
constexpr int kLseRows = 64, kLseKeys = 64;

// KS > 0: keys of exactly KS * 16 elements; 0: of dk_ elements.  Eight warps: warps w and w + 4 hold the same 16 rows, one the
// first half of every tile's keys, the other the second; their maxima and sums meet at the end.
template <int KS>
__global__ void __launch_bounds__(256)
mixed_head_lse_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k_cache, float* __restrict__ lse,
                      const int* __restrict__ block_table, int table_stride, const int* __restrict__ cu_q,
                      const int* __restrict__ kv_lens, int nq, int nkv, int dk_, int page_size, int page_shift, float scale,
                      MixMask mask, DistanceBias bias, int span) {
  pdl_wait();
  pdl_trigger();
  const int dk = KS > 0 ? KS * 16 : dk_;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int e = blockIdx.z, kvh = blockIdx.y, G = nq / nkv;
  const int t0 = cu_q[e], q_len = cu_q[e + 1] - t0, start = kv_lens[e] - q_len, rows = q_len * G;
  const int r0 = (gridDim.x - 1 - blockIdx.x) * kLseRows;      // the last rows see the most keys: they start first
  if (r0 >= rows) return;
  const int ks = dk + kMhPad;
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);               // [64][dk + 8]
  bf16* k_s = q_s + kLseRows * ks;                             // [2][64][dk + 8]
  float* bias_s = reinterpret_cast<float*>(k_s + 2 * kLseKeys * ks);    // [2][G][span]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const MixPages pages{block_table + (size_t)e * table_stride, nkv, page_size, page_shift};
  const MixCopy copy(dk / 8, 256);
  const int row0 = (warp & 3) * 16, half = (warp >> 2) * (kLseKeys / 2);
  for (int x = copy.r; x < kLseRows; x += copy.step) {
    const int row = r0 + x;
    const bool there = row < rows;
    const bf16* src = there ? q + ((size_t)(t0 + row / G) * nq + kvh * G + row % G) * dk + copy.c * 8 : q;
    cp_async_16(q_s + x * ks + copy.c * 8, src, there);
  }
  float m[2], l[2];
  int pos[2], head[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = r0 + row0 + (lane >> 2) + 8 * i;
    pos[i] = row < rows ? start + row / G : -1;
    head[i] = row < rows ? row % G : 0;
    m[i] = -CUDART_INF_F;
    l[i] = 0.f;
  }
  const int last_row = min(rows, r0 + kLseRows) - 1;
  const int max_pos = start + last_row / G, min_pos = start + r0 / G;
  const int first_seen = mask.first_key(min_pos);
  const MixTiles tiles(mask, min_pos, max_pos, kLseKeys);
  auto fetch = [&](int jb, int buf) {
    const bf16* pool = k_cache + (size_t)kvh * page_size * dk + copy.c * 8;
    bf16* to = k_s + buf * kLseKeys * ks + copy.c * 8;
    if (jb >= first_seen && jb + kLseKeys - 1 <= max_pos) {
#pragma unroll
      for (int x = 0; x < 4; ++x) {              // (a step of 16 rows or more: keys of up to 128 elements)
        const int jj = copy.r + x * copy.step;
        if (jj < kLseKeys) cp_async_16(to + jj * ks, pool + (size_t)pages.row(jb + jj) * dk, true);
      }
    } else {
      for (int jj = copy.r; jj < kLseKeys; jj += copy.step) {
        const int j = jb + jj;
        const bool there = j <= max_pos && (j >= first_seen || j < mask.keep);
        cp_async_16(to + jj * ks, there ? pool + (size_t)pages.row(j) * dk : k_cache, there);
      }
    }
    if (bias.table) {
      // bias_s[h][x] belongs to distance min_pos - (jb + 63) + x
      const int d0 = min_pos - jb - (kLseKeys - 1);
      for (int h = warp; h < G; h += 8)
        for (int x = lane; x < span; x += 32)
          cp_async_4(bias_s + (size_t)(buf * G + h) * span + x, bias.of(kvh * G + h, max(d0 + x, 0)));
    }
    cp_async_commit();
  };
  fetch(tiles.key(0, kLseKeys), 0);
  for (int n = 0, buf = 0; n < tiles.count; ++n, buf ^= 1) {
    const int jb = tiles.key(n, kLseKeys);
    if (n + 1 < tiles.count) {
      fetch(tiles.key(n + 1, kLseKeys), buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    float s[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) s[i][c] = 0.f;
    const bf16* qa = q_s + (row0 + (lane & 15)) * ks + (lane >> 4) * 8;
    const bf16* kb = k_s + (buf * kLseKeys + half + (lane & 7) + (lane >> 4) * 8) * ks + ((lane >> 3) & 1) * 8;
#pragma unroll(KS > 0 ? KS : 1)
    for (int k0 = 0; k0 < dk; k0 += 16) {
      uint32_t a[4];
      ldmatrix_x4(a, qa + k0);
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t b[4];
        ldmatrix_x4(b, kb + n2 * 16 * ks + k0);
        mma_bf16(s[2 * n2], a, b[0], b[1]);
        mma_bf16(s[2 * n2 + 1], a, b[2], b[3]);
      }
    }
    // every key of the tile visible to every row of the block: no masking
    const bool whole = jb + kLseKeys - 1 <= min_pos && (mask.window <= 0 || jb > max_pos - mask.window) && r0 + kLseRows <= rows;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      if (bias.table) {
        const float* bs = bias_s + (size_t)(buf * G + head[i]) * span + max(pos[i] - min_pos, 0) + (kLseKeys - 1) - half - (lane & 3) * 2;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          s[x][2 * i] = fmaf(s[x][2 * i], scale, bs[-x * 8]);
          s[x][2 * i + 1] = fmaf(s[x][2 * i + 1], scale, bs[-x * 8 - 1]);
        }
      } else {
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          s[x][2 * i] *= scale;
          s[x][2 * i + 1] *= scale;
        }
      }
      if (!whole) {
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
          for (int c = 0; c < 2; ++c)
            if (!mask.visible(pos[i], jb + half + x * 8 + (lane & 3) * 2 + c)) s[x][2 * i + c] = -CUDART_INF_F;
      }
      float mx = -CUDART_INF_F;
#pragma unroll
      for (int x = 0; x < 4; ++x) mx = fmaxf(mx, fmaxf(s[x][2 * i], s[x][2 * i + 1]));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m[i], mx);
      if (m_new != -CUDART_INF_F) {
        const float m2 = m_new * kLog2e;
        float sum[2] = {0.f, 0.f};
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          sum[0] += pow2(fmaf(s[x][2 * i], kLog2e, -m2));
          sum[1] += pow2(fmaf(s[x][2 * i + 1], kLog2e, -m2));
        }
        l[i] = l[i] * pow2(fmaf(m[i], kLog2e, -m2)) + sum[0] + sum[1];    // the lane's own share of the row's sum
        m[i] = m_new;
      }
    }
    __syncthreads();
  }
  float* other = reinterpret_cast<float*>(smem_raw);           // [64][2]: what the second half found (the queries are read)
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    const int x = row0 + (lane >> 2) + 8 * i;
    if (half && (lane & 3) == 0) {
      other[2 * x] = m[i];
      other[2 * x + 1] = l[i];
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int x = row0 + (lane >> 2) + 8 * i, row = r0 + x;
    if (half || row >= rows || (lane & 3) != 0) continue;
    const float m_new = fmaxf(m[i], other[2 * x]);             // a row sees its own key at least: finite
    const float sum = l[i] * pow2((m[i] - m_new) * kLog2e) + other[2 * x + 1] * pow2((other[2 * x] - m_new) * kLog2e);
    lse[(size_t)(t0 + row / G) * nq + kvh * G + row % G] = m_new * kLog2e + log2f(sum);
  }
}

// ---- weights, mixture, values ----------------------------------------------------------------------------------------
// KS: 16-element steps of a key, NT: 8-column tiles of the block's slab of values, HT: 16-head tiles of the mixture and heads
// of a warp's 16 rows.  EXACT: exactly so many, 16 HT heads and one slab; else at most.
template <int KS, int NT, int HT, bool EXACT>
__global__ void __launch_bounds__(512)
mixed_head_attention_mma_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k_cache,
                                const bf16* __restrict__ v_cache, const float* __restrict__ lse, bf16* __restrict__ out,
                                const int* __restrict__ block_table, int table_stride, const int* __restrict__ cu_q,
                                const int* __restrict__ kv_lens, int nq_, int nkv, int dk_, int dv_, int slab_, int page_size,
                                int page_shift, float scale, MixMask mask, DistanceBias bias, const float* __restrict__ mix, int mix_low,
                                ElementGate gate, int nsplit, float* __restrict__ part) {
  pdl_wait();
  pdl_trigger();
  const int dk = EXACT ? KS * 16 : dk_, dv = EXACT ? NT * 8 : dv_, slab = EXACT ? NT * 8 : slab_, nq = EXACT ? 16 * HT : nq_;
  constexpr int R = 16 / HT;                                   // tokens of the block
  constexpr int HP = 16 * HT;                                  // heads, padded
  constexpr int RS = R * kMhRow + kMhPad;                      // a head's weights of a tile
  constexpr int BL = R + kMhKeys;                              // distances of a tile
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int e = blockIdx.z, slabs = EXACT ? 1 : (dv + slab - 1) / slab, G = nq / nkv;
  const int c0 = EXACT ? 0 : (blockIdx.y % slabs) * slab, split = blockIdx.y / slabs;
  const int t0 = cu_q[e], q_len = cu_q[e + 1] - t0, start = kv_lens[e] - q_len;
  const int i0 = (gridDim.x - 1 - blockIdx.x) * R;
  if (i0 >= q_len) return;
  const int ks = dk + kMhPad, width = EXACT ? slab : min(slab, dv - c0), vs = slab + kMhPad;
  bf16* k_s = reinterpret_cast<bf16*>(smem_raw);               // [nkv][32][dk + 8]
  bf16* v_s = k_s + nkv * kMhKeys * ks;                        // [nkv][32][slab + 8]
  bf16* p_hi = v_s + nkv * kMhKeys * vs;                       // [HP][RS]: weights, then their mixture
  bf16* p_lo = p_hi + HP * RS;
  bf16* mix_s = p_lo + HP * RS;                                // [2][HP][HP + 8]
  float* bias_s = reinterpret_cast<float*>(mix_s + 2 * HP * (HP + kMhPad));   // [nq][BL]
  const int threads = EXACT ? 512 : blockDim.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = threads >> 5;
  const MixPages pages{block_table + (size_t)e * table_stride, nkv, page_size, page_shift};
  const int min_pos = start + i0, max_pos = start + min(q_len, i0 + R) - 1;
  const int first_seen = mask.first_key(min_pos);
  const MixTiles tiles(mask, min_pos, max_pos, kMhKeys);
  const int per = (tiles.count + nsplit - 1) / nsplit;
  const int n_first = split * per, n_last = min(tiles.count, n_first + per);

  // A thread looks a key up once and copies its piece of the key's row for every KV head.  EXACT: one key a thread, whose
  // row is looked up a tile ahead of its copies, so that no copy waits for the block table.
  auto there = [&](int j) { return j <= max_pos && (j >= first_seen || j < mask.keep); };
  auto copy = [&](const bf16* pool, int dim, int row, int c, bf16* to, int stride) {
    const bf16* src = pool + (row >= 0 ? (size_t)row * dim + c : 0);
    const int src_step = row >= 0 ? page_size * dim : 0, to_step = kMhKeys * stride;
#pragma unroll 4
    for (int h = 0; h < nkv; ++h, src += src_step, to += to_step) cp_async_16(to, src, row >= 0);
  };
  constexpr int EV = EXACT ? KS * 2 : 1;                       // EXACT: pieces of a row (keys and values alike)
  static_assert(!EXACT || (kMhKeys * EV <= 512 && KS * 16 == NT * 8), "a thread copies one piece of one key");
  const int my_key = tid / EV, my_c = (tid % EV) * 8;
  auto look_up = [&](int n) {
    const int j = my_key < kMhKeys && n < n_last ? tiles.key(n, kMhKeys) + my_key : 1 << 30;
    return there(j) ? pages.row(j) : -1;
  };
  auto fetch_rows = [&](int jb, int vec, bf16* dst, int stride, const bf16* pool, int dim) {
    for (int slot = tid; slot < kMhKeys * vec; slot += threads) {
      const int jj = slot / vec, c = (slot - jj * vec) * 8;
      copy(pool, dim, there(jb + jj) ? pages.row(jb + jj) : -1, c, dst + jj * stride + c, stride);
    }
  };
  auto fetch_k = [&](int n, int row) {                         // and the biases of its distances
    const int jb = tiles.key(n, kMhKeys);
    if (EXACT) {
      if (my_key < kMhKeys) copy(k_cache, dk, row, my_c, k_s + my_key * ks + my_c, ks);
    } else {
      fetch_rows(jb, dk / 8, k_s, ks, k_cache, dk);
    }
    if (bias.table) {                                          // bias_s[h][x]: distance min_pos - (jb + 31) + x
      const int d0 = min_pos - jb - (kMhKeys - 1);
#pragma unroll
      for (int i = 0; i < HT; ++i)
#pragma unroll
        for (int x = 0; x < (BL + 31) / 32; ++x)
          if (x * 32 + lane < BL)
            cp_async_4(bias_s + (warp * HT + i) * BL + x * 32 + lane, bias.of(warp * HT + i, max(d0 + x * 32 + lane, 0)));
    }
    cp_async_commit();
  };
  auto fetch_v = [&](int n, int row) {
    if (EXACT) {
      if (my_key < kMhKeys) copy(v_cache, dv, row, my_c, v_s + my_key * vs + my_c, vs);
    } else {
      fetch_rows(tiles.key(n, kMhKeys), width / 8, v_s, vs, v_cache + c0, dv);
    }
    cp_async_commit();
  };
  int row_now = -1, row_next = -1;                             // EXACT: of this tile's key, of the next tile's
  if (EXACT) {
    row_now = look_up(n_first);
    row_next = look_up(n_first + 1);
  }
  if (n_first < n_last) fetch_k(n_first, row_now);

  // the mixture's matrix as a pair of bfloat16 (the rounding, and what it leaves), and zero rows for heads that do not exist
  for (int idx = tid; idx < HP * (HP + kMhPad); idx += blockDim.x) {
    const int h = idx / (HP + kMhPad), g = idx % (HP + kMhPad);
    const float v = h < nq && g < nq ? (mix ? mix[h * nq + g] : h == g ? 1.f : 0.f) : 0.f;
    const bf16 hi = __float2bfloat16_rn(v);
    mix_s[idx] = hi;
    mix_s[HP * (HP + kMhPad) + idx] = __float2bfloat16_rn(v - __bfloat162float(hi));
  }
  for (int idx = tid; idx < (HP - nq) * RS; idx += blockDim.x) {
    p_hi[nq * RS + idx] = __float2bfloat16_rn(0.f);
    p_lo[nq * RS + idx] = __float2bfloat16_rn(0.f);
  }

  // a warp's rows: HT heads of one KV head x R tokens; a thread's two rows are lane / 4 and lane / 4 + 8
  const int head0 = warp * HT, kvh = head0 / G;
  uint32_t qf[KS][4];
  float L[2];
  int pos[2], at[2], bias_at[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = (lane >> 2) + 8 * i, h = head0 + r / R, tok = r % R;
    const bool live = i0 + tok < q_len;
    pos[i] = live ? min_pos + tok : -1;
    at[i] = h * RS + tok * kMhRow;
    bias_at[i] = h * BL + tok + kMhKeys - 1 - (lane & 3) * 2;
    L[i] = live ? lse[(size_t)(t0 + i0 + tok) * nq + h] : 0.f;
    const bf16* src = q + ((size_t)(t0 + i0 + (live ? tok : 0)) * nq + h) * dk + (lane & 3) * 2;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      const bool there = live && (EXACT || k * 16 < dk);
      qf[k][i] = there ? *reinterpret_cast<const uint32_t*>(src + k * 16) : 0u;
      qf[k][2 + i] = there ? *reinterpret_cast<const uint32_t*>(src + k * 16 + 8) : 0u;
    }
  }
  float o[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[n][c] = 0.f;

  for (int n = n_first; n < n_last; ++n) {
    const int jb = tiles.key(n, kMhKeys);
    cp_async_wait<0>();
    __syncthreads();                                           // the keys are here; the values and weights before are read
    fetch_v(n, row_now);

    float s[kMhKeys / 8][4];
#pragma unroll
    for (int x = 0; x < kMhKeys / 8; ++x)
#pragma unroll
      for (int c = 0; c < 4; ++c) s[x][c] = 0.f;
    const bf16* kb = k_s + (kvh * kMhKeys + (lane & 7) + (lane >> 4) * 8) * ks + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if (EXACT || k * 16 < dk) {
#pragma unroll
        for (int n2 = 0; n2 < kMhKeys / 16; ++n2) {
          uint32_t b[4];
          ldmatrix_x4(b, kb + n2 * 16 * ks + k * 16);
          mma_bf16(s[2 * n2], qf[k], b[0], b[1]);
          mma_bf16(s[2 * n2 + 1], qf[k], b[2], b[3]);
        }
      }
    }
    const bool whole = jb + kMhKeys - 1 <= min_pos && (mask.window <= 0 || jb > max_pos - mask.window) && i0 + R <= q_len;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      if (bias.table) {
        const float* bs = bias_s + bias_at[i];
#pragma unroll
        for (int x = 0; x < kMhKeys / 8; ++x) {
          s[x][2 * i] = pow2(fmaf(fmaf(s[x][2 * i], scale, bs[-x * 8]), kLog2e, -L[i]));
          s[x][2 * i + 1] = pow2(fmaf(fmaf(s[x][2 * i + 1], scale, bs[-x * 8 - 1]), kLog2e, -L[i]));
        }
      } else {
#pragma unroll
        for (int x = 0; x < kMhKeys / 8; ++x) {
          s[x][2 * i] = pow2(fmaf(s[x][2 * i], scale * kLog2e, -L[i]));
          s[x][2 * i + 1] = pow2(fmaf(s[x][2 * i + 1], scale * kLog2e, -L[i]));
        }
      }
      if (!whole) {
#pragma unroll
        for (int x = 0; x < kMhKeys / 8; ++x)
#pragma unroll
          for (int c = 0; c < 2; ++c)
            if (!mask.visible(pos[i], jb + x * 8 + (lane & 3) * 2 + c)) s[x][2 * i + c] = 0.f;
      }
#pragma unroll
      for (int x = 0; x < kMhKeys / 8; ++x) {
        const __nv_bfloat162 hi = __floats2bfloat162_rn(s[x][2 * i], s[x][2 * i + 1]);
        const float2 back = __bfloat1622float2(hi);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(s[x][2 * i] - back.x, s[x][2 * i + 1] - back.y);
        const int to = at[i] + x * 8 + (lane & 3) * 2;
        *reinterpret_cast<__nv_bfloat162*>(p_hi + to) = hi;
        *reinterpret_cast<__nv_bfloat162*>(p_lo + to) = lo;
      }
    }
    __syncthreads();                                           // all heads' weights are written; the keys are read
    if (n + 1 < n_last) fetch_k(n + 1, row_next);
    if (EXACT) {
      row_now = row_next;
      row_next = look_up(n + 2);
    }

    // the mixture, in place: a warp takes 8 keys of a token at a time, all heads
    uint32_t mix_f[4];                                         // one tile of heads: its matrix is loaded once
    if (HT == 1) ldmatrix_x4(mix_f, mix_s + (lane & 15) * (HP + kMhPad) + (lane >> 4) * 8);
#pragma unroll(EXACT ? R * (kMhKeys / 8) / 16 : 1)
    for (int ct = warp; ct < R * (kMhKeys / 8); ct += warps) {
      const int col = (ct / (kMhKeys / 8)) * kMhRow + (ct % (kMhKeys / 8)) * 8;
      uint32_t b[HT][4];
#pragma unroll
      for (int k = 0; k < HT; ++k) ldmatrix_x4_trans(b[k], ((lane >> 4) ? p_lo : p_hi) + (k * 16 + (lane & 15)) * RS + col);
      __syncwarp();
#pragma unroll
      for (int mt = 0; mt < HT; ++mt) {
        float d[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int k = 0; k < HT; ++k) {
          uint32_t a[4];
          if (HT == 1) { a[0] = mix_f[0]; a[1] = mix_f[1]; a[2] = mix_f[2]; a[3] = mix_f[3]; }
          else ldmatrix_x4(a, mix_s + (mt * 16 + (lane & 15)) * (HP + kMhPad) + k * 16 + (lane >> 4) * 8);
          mma_bf16(d, a, b[k][2], b[k][3]);
          mma_bf16(d, a, b[k][0], b[k][1]);
          if (mix_low) {
            ldmatrix_x4(a, mix_s + (HP + mt * 16 + (lane & 15)) * (HP + kMhPad) + k * 16 + (lane >> 4) * 8);
            mma_bf16(d, a, b[k][0], b[k][1]);
          }
        }
        bf16* w = p_hi + (mt * 16 + (lane >> 2)) * RS + col + (lane & 3) * 2;
        *reinterpret_cast<__nv_bfloat162*>(w) = __floats2bfloat162_rn(d[0], d[1]);
        *reinterpret_cast<__nv_bfloat162*>(w + 8 * RS) = __floats2bfloat162_rn(d[2], d[3]);
      }
    }
    if (n + 1 < n_last) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();                                           // the mixture and the values are here

    const bf16* wa = p_hi + (head0 + (lane & 15) / R) * RS + ((lane & 15) % R) * kMhRow + (lane >> 4) * 8;
    const bf16* vb = v_s + (kvh * kMhKeys + (lane & 15)) * vs + (lane >> 4) * 8;
#pragma unroll
    for (int kk = 0; kk < kMhKeys / 16; ++kk) {
      uint32_t a[4];
      ldmatrix_x4(a, wa + kk * 16);
#pragma unroll
      for (int n2 = 0; n2 < NT / 2; ++n2) {
        if (EXACT || n2 * 16 < width) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, vb + kk * 16 * vs + n2 * 16);
          mma_bf16(o[2 * n2], a, b[0], b[1]);
          mma_bf16(o[2 * n2 + 1], a, b[2], b[3]);
        }
      }
    }
  }

#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = (lane >> 2) + 8 * i, h = head0 + r / R, tok = i0 + r % R;
    if (tok >= q_len) continue;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      if (!EXACT && n * 8 >= width) continue;
      const int c = h * dv + c0 + n * 8 + (lane & 3) * 2;
      if (nsplit > 1) {
        *reinterpret_cast<float2*>(part + ((size_t)(t0 + tok) * nsplit + split) * nq * dv + c) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
      } else {
        const float a = o[n][2 * i] * gate.at(t0 + tok, c), b = o[n][2 * i + 1] * gate.at(t0 + tok, c + 1);
        *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(t0 + tok) * nq * dv + c) = __floats2bfloat162_rn(a, b);
      }
    }
  }
}

// out[t, c] = (sum over the key slices of part[t, slice, c]) * gate; the slices' weights are finished, so they just add.
__global__ void mixed_head_add_kernel(const float* __restrict__ part, bf16* __restrict__ out, int nsplit, int columns,
                                      ElementGate gate) {
  pdl_wait();
  pdl_trigger();
  const size_t t = blockIdx.x;
  for (int c = threadIdx.x; c < columns; c += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < nsplit; ++s) a += part[(t * nsplit + s) * columns + c];
    out[t * columns + c] = __float2bfloat16_rn(a * gate.at(t, c));
  }
}

// ---- decode steps ----------------------------------------------------------------------------------------------------
__device__ __forceinline__ void mh_cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// The float at `p` of this block's shared memory, in block `rank` of the cluster.
__device__ __forceinline__ float mh_remote(const float* p, int rank) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  uint32_t r;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(r));
  return v;
}

constexpr int kMdThreads = 256, kMdWarps = kMdThreads / 32;

struct MixDecodeLayout {             // offsets in bytes of a block's shared memory
  int q, tile, tile_bytes, w, s, stats, lse, mix, total, keys;      // keys: a head's row of scores
  __host__ __device__ MixDecodeLayout(int nq, int nkv, int row_tiles, int dk, int dv, int tiles_here, int nbuf) {
    const int rows = nkv * row_tiles * 16, wide = (dk > dv ? dk : dv) + kMhPad;
    keys = tiles_here * kMhKeys + 4;
    q = 0;
    tile = q + rows * (dk + kMhPad) * 2;
    tile_bytes = nkv * kMhKeys * wide * 2;
    int buffers = nbuf * tile_bytes;
    if (buffers < nq * dv * 4) buffers = nq * dv * 4;                // the block's sums lie there at the end
    w = tile + buffers;
    s = w + rows * kMhRow * 2;
    stats = s + nq * keys * 4;
    lse = stats + nq * 8;
    mix = (lse + nq * 4 + 15) / 16 * 16;
    total = mix + nq * (nq + 1) * 4;
  }
};

// UN: units of 32 value columns of 16 rows that a warp holds; D > 0: keys and values of exactly D elements (0: of dk_ and
// dv_).  grid (cluster, entries).
template <int UN, int D>
__global__ void __launch_bounds__(kMdThreads)
mixed_head_attention_decode_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k_cache,
                                   const bf16* __restrict__ v_cache, bf16* __restrict__ out,
                                   const int* __restrict__ block_table, int table_stride, const int* __restrict__ cu_q,
                                   const int* __restrict__ kv_lens, int nq, int nkv, int row_tiles, int dk_, int dv_,
                                   int page_size, int page_shift, float scale2, MixMask mask, DistanceBias bias,
                                   const float* __restrict__ mix, ElementGate gate, int tiles_cap, int nbuf) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int dk = D > 0 ? D : dk_, dv = D > 0 ? D : dv_;
  const MixDecodeLayout at(nq, nkv, row_tiles, dk, dv, tiles_cap, nbuf);
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw + at.q);        // [nkv][row_tiles * 16][dk + 8]
  bf16* w_s = reinterpret_cast<bf16*>(smem_raw + at.w);        // [nkv][row_tiles * 16][40]
  float* s_s = reinterpret_cast<float*>(smem_raw + at.s);      // [nq][keys]
  float* stats = reinterpret_cast<float*>(smem_raw + at.stats);     // [nq][2]: maximum and sum of the slice
  float* lse = reinterpret_cast<float*>(smem_raw + at.lse);    // [nq]
  float* mix_s = reinterpret_cast<float*>(smem_raw + at.mix);  // [nq][nq + 1]
  float* o_s = reinterpret_cast<float*>(smem_raw + at.tile);   // [nq][dv], at the end
  const int rank = blockIdx.x, cluster = gridDim.x, e = blockIdx.y;
  const int G = nq / nkv, rows_c = row_tiles * 16, ks = dk + kMhPad, vs = dv + kMhPad;
  const int t = cu_q[e], pos = kv_lens[e] - 1;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const MixPages pages{block_table + (size_t)e * table_stride, nkv, page_size, page_shift};
  const MixTiles tiles(mask, pos, pos, kMhKeys);
  int per = (tiles.count + cluster - 1) / cluster;             // (never above tiles_cap: the host planned for the longest)
  if (per > tiles_cap) per = tiles_cap;
  const int n0 = min(tiles.count, rank * per), n_here = min(tiles.count - n0, per);
  const int kvec = dk / 8;

  // stage x: 0 .. n_here - 1 fetch keys, n_here .. 2 n_here - 1 values, buffer x % nbuf
  auto fetch = [&](int x) {
    const bool values = x >= n_here;
    const int jb = tiles.key(n0 + (values ? x - n_here : x), kMhKeys);
    bf16* dst = reinterpret_cast<bf16*>(smem_raw + at.tile + (x % nbuf) * at.tile_bytes);
    const int vec = (values ? dv : dk) / 8, stride = values ? vs : ks, dim = values ? dv : dk;
    const bf16* pool = values ? v_cache : k_cache;
    for (int slot = tid; slot < kMhKeys * vec; slot += kMdThreads) {
      const int jj = slot / vec, c = (slot - jj * vec) * 8, j = jb + jj;
      const bool there = mask.visible(pos, j);
      const bf16* src = pool + (there ? (size_t)pages.row(j) * dim + c : 0);
      bf16* to = dst + jj * stride + c;
      const int src_step = there ? page_size * dim : 0, to_step = kMhKeys * stride;
#pragma unroll 4
      for (int h = 0; h < nkv; ++h, src += src_step, to += to_step) cp_async_16(to, src, there);
    }
    cp_async_commit();
  };
  const int stages = 2 * n_here;
  if (stages) fetch(0);
  for (int idx = tid; idx < nkv * rows_c * kvec; idx += blockDim.x) {
    const int row = idx / kvec, c = idx - row * kvec, h = row / rows_c, r = row % rows_c;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < G) v = *reinterpret_cast<const uint4*>(q + ((size_t)t * nq + h * G + r) * dk + c * 8);
    *reinterpret_cast<uint4*>(q_s + row * ks + c * 8) = v;
  }
  for (int idx = tid; idx < nkv * rows_c * kMhRow; idx += blockDim.x) w_s[idx] = __float2bfloat16_rn(0.f);
  for (int idx = tid; idx < nq * nq; idx += blockDim.x)
    mix_s[idx / nq * (nq + 1) + idx % nq] = mix ? mix[idx] : idx / nq == idx % nq ? 1.f : 0.f;

  float o[UN][4][4];
#pragma unroll
  for (int u = 0; u < UN; ++u)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) o[u][n][c] = 0.f;
  const int col_units = (dv + 31) / 32, units = nkv * row_tiles * col_units;

  for (int x = 0; x < stages; ++x) {
    if (nbuf > 1 && x + 1 < stages) {
      fetch(x + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bf16* buf = reinterpret_cast<const bf16*>(smem_raw + at.tile + (x % nbuf) * at.tile_bytes);
    if (x < n_here) {
      // scores of 16 rows x 16 keys a job
      const int jb = tiles.key(n0 + x, kMhKeys);
      for (int job = warp; job < nkv * row_tiles * (kMhKeys / 16); job += kMdWarps) {
        const int n2 = job % (kMhKeys / 16), rt = job / (kMhKeys / 16), h = rt / row_tiles, r0 = (rt % row_tiles) * 16;
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        const bf16* qa = q_s + (rt * 16 + (lane & 15)) * ks + (lane >> 4) * 8;
        const bf16* kb = buf + (h * kMhKeys + n2 * 16 + (lane & 7) + (lane >> 4) * 8) * ks + ((lane >> 3) & 1) * 8;
#pragma unroll(D > 0 ? D / 16 : 1)
        for (int k0 = 0; k0 < dk; k0 += 16) {
          uint32_t a[4], b[4];
          ldmatrix_x4(a, qa + k0);
          ldmatrix_x4(b, kb + k0);
          mma_bf16(s[0], a, b[0], b[1]);
          mma_bf16(s[1], a, b[2], b[3]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int r = r0 + (lane >> 2) + 8 * i;
          if (r >= G) continue;
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
              const int jj = n2 * 16 + n * 8 + (lane & 3) * 2 + c;
              float v = -CUDART_INF_F;
              if (mask.visible(pos, jb + jj)) v = fmaf(s[n][2 * i + c], scale2, bias.at(h * G + r, pos - jb - jj) * kLog2e);
              s_s[(size_t)(h * G + r) * at.keys + x * kMhKeys + jj] = v;
            }
        }
      }
      if (x == n_here - 1) {
        // the slice's maximum and sum of every head, exchanged; then the scores become finished weights
        __syncthreads();
        for (int h = warp; h < nq; h += kMdWarps) {
          float m = -CUDART_INF_F, l = 0.f;
          for (int j = lane; j < n_here * kMhKeys; j += 32) m = fmaxf(m, s_s[(size_t)h * at.keys + j]);
          m = warp_max(m);
          if (m != -CUDART_INF_F)
            for (int j = lane; j < n_here * kMhKeys; j += 32) l += pow2(s_s[(size_t)h * at.keys + j] - m);
          l = warp_sum(l);
          if (lane == 0) { stats[2 * h] = m; stats[2 * h + 1] = l; }
        }
      }
    }
    if (x == n_here - 1) {
      mh_cluster_sync();
      for (int h = warp; h < nq; h += kMdWarps) {              // a lane a block of the cluster
        const float mr = lane < cluster ? mh_remote(stats + 2 * h, lane) : -CUDART_INF_F;
        const float lr = lane < cluster ? mh_remote(stats + 2 * h + 1, lane) : 0.f;
        const float m = warp_max(mr);
        const float l = warp_sum(mr != -CUDART_INF_F ? lr * pow2(mr - m) : 0.f);
        if (lane == 0) lse[h] = m + log2f(l);
      }
      __syncthreads();
      for (int h = warp; h < nq; h += kMdWarps)
        for (int j = lane; j < n_here * kMhKeys; j += 32) s_s[(size_t)h * at.keys + j] = pow2(s_s[(size_t)h * at.keys + j] - lse[h]);
    }
    if (x >= n_here) {
      const int j0 = (x - n_here) * kMhKeys;
      for (int h = warp; h < nq; h += kMdWarps) {
        float a = 0.f;
        for (int g = 0; g < nq; ++g) a += mix_s[h * (nq + 1) + g] * s_s[(size_t)g * at.keys + j0 + lane];
        w_s[((h / G) * rows_c + h % G) * kMhRow + lane] = __float2bfloat16_rn(a);
      }
      __syncthreads();
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int unit = warp + u * kMdWarps;
        if (unit < units) {
          const int rt = unit / col_units, cu = (unit % col_units) * 32, h = rt / row_tiles;
#pragma unroll
          for (int kk = 0; kk < kMhKeys / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4(a, w_s + (rt * 16 + (lane & 15)) * kMhRow + kk * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int n2 = 0; n2 < 2; ++n2) {
              if (cu + n2 * 16 < dv) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, buf + (h * kMhKeys + kk * 16 + (lane & 15)) * vs + cu + n2 * 16 + (lane >> 4) * 8);
                mma_bf16(o[u][2 * n2], a, b[0], b[1]);
                mma_bf16(o[u][2 * n2 + 1], a, b[2], b[3]);
              }
            }
          }
        }
      }
    }
    __syncthreads();                                           // the buffer and the weights are read
    if (nbuf == 1 && x + 1 < stages) fetch(x + 1);
  }
  if (n_here == 0) {                                           // a block without keys still takes part in the exchange
    for (int h = tid; h < nq; h += blockDim.x) { stats[2 * h] = -CUDART_INF_F; stats[2 * h + 1] = 0.f; }
    mh_cluster_sync();
  }

  // the block's sums, then every block adds a share of the columns over the cluster
#pragma unroll
  for (int u = 0; u < UN; ++u) {
    const int unit = warp + u * kMdWarps;
    if (unit < units) {
      const int rt = unit / col_units, cu = (unit % col_units) * 32, h = rt / row_tiles, r0 = (rt % row_tiles) * 16;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = r0 + (lane >> 2) + 8 * i;
        if (r >= G) continue;
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int c = cu + n * 8 + (lane & 3) * 2;
          if (c < dv) {
            o_s[(size_t)(h * G + r) * dv + c] = o[u][n][2 * i];
            o_s[(size_t)(h * G + r) * dv + c + 1] = o[u][n][2 * i + 1];
          }
        }
      }
    }
  }
  mh_cluster_sync();
  for (int c = rank * kMdThreads + tid; c < nq * dv; c += cluster * kMdThreads) {
    float a = 0.f;
    for (int r = 0; r < cluster; r += 4) {                     // four loads on their way at a time
      float v[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) v[x] = r + x < cluster ? mh_remote(o_s + c, r + x) : 0.f;
      a += (v[0] + v[1]) + (v[2] + v[3]);
    }
    out[(size_t)t * nq * dv + c] = __float2bfloat16_rn(a * gate.at(t, c));
  }
  mh_cluster_sync();                                           // nobody leaves while its sums are read
}

}  // namespace srlm

using namespace srlm;

static int mh_heads_tiles(int nq, int nkv) {      // 16-head tiles of the rows form, 0: not taken
  if (nq <= 16) return 1;
  if (nq <= 32 && nq % 2 == 0 && (nq / nkv) % 2 == 0) return 2;
  return 0;
}
static int mh_page_shift(int page_size) {
  int s = 0;
  while ((1 << s) < page_size) ++s;
  return (1 << s) == page_size ? s : -1;
}
static int mh_slab(int dv) { return dv <= 128 ? dv : 128; }
static size_t mh_rows_smem(int nq, int nkv, int dk, int dv) {
  const int ht = mh_heads_tiles(nq, nkv), hp = 16 * ht, R = 16 / ht, rs = R * kMhRow + kMhPad, slab = mh_slab(dv);
  return (size_t)nkv * kMhKeys * (dk + kMhPad) * 2 + (size_t)nkv * kMhKeys * (slab + kMhPad) * 2 + 2ull * hp * rs * 2 +
         2ull * hp * (hp + kMhPad) * 2 + (size_t)nq * (R + kMhKeys) * 4;
}
static int mh_lse_span(int G) { return kLseKeys + kLseRows / G + 1; }
static size_t mh_lse_smem(int G, int dk) {
  return (size_t)(kLseRows + 2 * kLseKeys) * (dk + kMhPad) * 2 + 2ull * G * mh_lse_span(G) * 4;
}

// Whether the tensor-core forms take these sizes (bfloat16 cache): up to 16 heads, or an even number up to 32 with an even
// number a KV head; key size a multiple of 16 up to 128, value size a multiple of 16.
extern "C" int srlm_mixed_head_attention_mma_takes(int nq, int nkv, int dk, int dv) {
  if (nq <= 0 || nkv <= 0 || nq % nkv || !mh_heads_tiles(nq, nkv) || dk <= 0 || dk % 16 || dk > 128 || dv <= 0 || dv % 16) return 0;
  return mh_rows_smem(nq, nkv, dk, dv) <= 220 * 1024 && mh_lse_smem(nq / nkv, dk) <= 220 * 1024;
}

extern "C" int srlm_mixed_head_tokens(int nq, int nkv) { const int ht = mh_heads_tiles(nq, nkv); return ht ? 16 / ht : 0; }

// q bfloat16 [T, nq, dk]; lse float32 [T, nq] (written by the first kernel, read by the second); part float32
// [T, nsplit, nq dv] when nsplit > 1 (the visible keys in nsplit slices, added by a third kernel).
extern "C" int srlm_mixed_head_attention_mma(const void* q, const void* k_cache, const void* v_cache, void* out, float* lse,
                                             const int* block_table, int table_stride, const int* cu_q, const int* kv_lens,
                                             int n_entries, int max_q_len, int T, int nq, int nkv, int dk, int dv,
                                             int page_size, float scale, int window, int keep, const float* bias, int n_dist,
                                             const float* mix, int mix_low, const float* gate_logits, long long ld_gate,
                                             int nsplit, float* part, cudaStream_t stream) {
  if (n_entries <= 0 || max_q_len <= 0 || T <= 0) return ST_OK;
  if (!srlm_mixed_head_attention_mma_takes(nq, nkv, dk, dv) || page_size <= 0 || window < 0 || keep < 0 || (bias && n_dist <= 0) || !lse)
    return refuse(ST_BAD_SIZE, "mixed_head_attention_mma: nq=%d nkv=%d dk=%d dv=%d", nq, nkv, dk, dv);
  if ((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) != 0)
    return refuse(ST_BAD_ALIGN, "mixed_head_attention_mma: queries and pools must be 16-byte aligned");
  if (nsplit < 1) nsplit = 1;
  if (nsplit > 1 && !part) return refuse(ST_BAD_SIZE, "mixed_head_attention_mma: %d key slices need a workspace", nsplit);
  const int G = nq / nkv, ht = mh_heads_tiles(nq, nkv), R = 16 / ht, slab = mh_slab(dv), slabs = (dv + slab - 1) / slab;
  if (n_entries > 65535 || nkv > 65535 || (long long)slabs * nsplit > 65535)
    return refuse(ST_BAD_SIZE, "mixed_head_attention_mma: %d entries", n_entries);
  const MixMask mask{window, window > 0 ? keep : 0};
  const DistanceBias db{bias, n_dist};
  const ElementGate gate{gate_logits, ld_gate};
  {
    const size_t smem = mh_lse_smem(G, dk);
    auto kern = dk == 64 ? mixed_head_lse_kernel<4> : dk == 128 ? mixed_head_lse_kernel<8> : mixed_head_lse_kernel<0>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_pdl(kern, dim3((unsigned)(((long long)max_q_len * G + kLseRows - 1) / kLseRows), nkv, n_entries), dim3(256),
               smem, stream, (const bf16*)q, (const bf16*)k_cache, lse, block_table, table_stride, cu_q, kv_lens, nq, nkv, dk,
               page_size, mh_page_shift(page_size), scale, mask, db, mh_lse_span(G));
  }
  const size_t smem = mh_rows_smem(nq, nkv, dk, dv);
  const dim3 grid((unsigned)((max_q_len + R - 1) / R), (unsigned)(slabs * nsplit), (unsigned)n_entries);
  const int threads = nq / ht * 32;
#define SRLM_MH(KS, NT, HT, EX)                                                                                           \
  do {                                                                                                                  \
    auto kern = mixed_head_attention_mma_kernel<KS, NT, HT, EX>;                                                            \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
    launch_pdl(kern, grid, dim3(threads), smem, stream, (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, lse, \
               (bf16*)out, block_table, table_stride, cu_q, kv_lens, nq, nkv, dk, dv, slab, page_size, mh_page_shift(page_size), scale, mask, db, \
               mix, mix_low, gate, nsplit, part);                                                                       \
  } while (0)
#define SRLM_MH_SIZES(HT)                               \
  do {                                                  \
    if (dk == 64 && dv == 64 && nq == 16 * HT) SRLM_MH(4, 8, HT, true);          \
    else if (dk == 128 && dv == 128 && nq == 16 * HT) SRLM_MH(8, 16, HT, true);  \
    else if (dk <= 64 && slab <= 64) SRLM_MH(4, 8, HT, false); \
    else SRLM_MH(8, 16, HT, false);                     \
  } while (0)
  if (ht == 1) SRLM_MH_SIZES(1);
  else SRLM_MH_SIZES(2);
#undef SRLM_MH_SIZES
#undef SRLM_MH
  if (nsplit > 1)
    launch_pdl(mixed_head_add_kernel, dim3(T), dim3(256), 0, stream, part, (bf16*)out, nsplit, nq * dv, gate);
  return launched();
}

// Bytes of shared memory of a block of the decode form whose slice has tiles_here tiles of 32 keys; 0: sizes not taken.
extern "C" int srlm_mixed_head_decode_smem(int nq, int nkv, int dk, int dv, int tiles_here, int nbuf) {
  if (nq <= 0 || nkv <= 0 || nq % nkv || nq > 128 || dk <= 0 || dk % 16 || dv <= 0 || dv % 16) return 0;
  const int row_tiles = (nq / nkv + 15) / 16, units = nkv * row_tiles * ((dv + 31) / 32);
  if (units > 8 * kMdWarps) return 0;
  const MixDecodeLayout at(nq, nkv, row_tiles, dk, dv, tiles_here, nbuf);
  return at.total <= 225 * 1024 ? at.total : 0;
}

// One token an entry; the visible keys of an entry, at most 32 * tiles_here * cluster of them, in `cluster` (1, 2, 4, 8 or 16)
// slices of whole tiles.
extern "C" int srlm_mixed_head_attention_decode(const void* q, const void* k_cache, const void* v_cache, void* out,
                                                const int* block_table, int table_stride, const int* cu_q,
                                                const int* kv_lens, int n_entries, int nq, int nkv, int dk, int dv,
                                                int page_size, float scale, int window, int keep, const float* bias, int n_dist,
                                                const float* mix, const float* gate_logits, long long ld_gate, int cluster,
                                                int tiles_here, int nbuf, cudaStream_t stream) {
  if (n_entries <= 0) return ST_OK;
  const int smem = srlm_mixed_head_decode_smem(nq, nkv, dk, dv, tiles_here, nbuf);
  if (!smem || page_size <= 0 || window < 0 || keep < 0 || (bias && n_dist <= 0) || tiles_here <= 0 || nbuf < 1 || nbuf > 2 ||
      n_entries > 65535 || (cluster != 1 && cluster != 2 && cluster != 4 && cluster != 8 && cluster != 16))
    return refuse(ST_BAD_SIZE, "mixed_head_attention_decode: nq=%d nkv=%d dk=%d dv=%d cluster=%d of %d tiles", nq, nkv, dk, dv,
                  cluster, tiles_here);
  if ((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) != 0)
    return refuse(ST_BAD_ALIGN, "mixed_head_attention_decode: queries and pools must be 16-byte aligned");
  const int row_tiles = (nq / nkv + 15) / 16, units = nkv * row_tiles * ((dv + 31) / 32);
  const MixMask mask{window, window > 0 ? keep : 0};
  const DistanceBias db{bias, n_dist};
  const ElementGate gate{gate_logits, ld_gate};
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cluster, n_entries, 1);
  cfg.blockDim = dim3(kMdThreads, 1, 1);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
#define SRLM_MD(UN, D)                                                                                                 \
  do {                                                                                                                \
    auto kern = mixed_head_attention_decode_kernel<UN, D>;                                                              \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);              \
    if (cluster > 8) cudaFuncSetAttribute(kern, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);                   \
    cudaLaunchKernelEx(&cfg, kern, (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, block_table, \
                       table_stride, cu_q, kv_lens, nq, nkv, row_tiles, dk, dv, page_size, mh_page_shift(page_size), scale * kLog2e, mask, db, mix, \
                       gate, tiles_here, nbuf);                                                                       \
  } while (0)
#define SRLM_MD_UNITS(D)                             \
  do {                                              \
    if (units <= 2 * kMdWarps) SRLM_MD(2, D);       \
    else if (units <= 4 * kMdWarps) SRLM_MD(4, D);  \
    else SRLM_MD(8, D);                             \
  } while (0)
  if (dk == 128 && dv == 128) SRLM_MD_UNITS(128);
  else SRLM_MD_UNITS(0);
#undef SRLM_MD_UNITS
#undef SRLM_MD
  return launched();
}
