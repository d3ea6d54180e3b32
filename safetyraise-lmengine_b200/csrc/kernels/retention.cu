// Retention: a linear attention whose state fades at a fixed rate per head, in float32.
//
//   q = R(q), k = R(k) / sqrt(d)      R: pairs (i, i + pairs) of the head's leading 2 pairs elements turned by the token's angle
//   S <- decay_h S + k v^T;   o = S^T q;   out = o / sqrt(mean(o^2) + eps) * silu(gate)
//
// proj float32 [T, ldp]: columns q (H d) | k (H d) | v (H dv) | gate (H dv).  A request's state row: S [H][d][dv], zeros for
// a new request.
//
// retention_walk: token by token.  A block takes one entry, one head and a tile of up to 128 value columns; the state of
// the tile stays in registers: a thread holds VEC neighbouring columns of RPT rows (rows g, g + RG, ... of row group g), so
// the read-out is a sum in registers and one exchange through shared memory a token.  Where one tile holds the whole head
// the norm, the gate and the rounding happen in the same kernel; else o goes to a buffer and retention_output follows.
//
// Entries of more than walk_max tokens take three kernels over chunks of 64 tokens instead (the walk leaves them alone):
//   retention_chunks   U_c = sum_s decay^(n - 1 - s) k_s v_s^T for every chunk of n tokens, all chunks at once;
//   retention_fold     the state ahead of every chunk, in U's place: S_c, then S_(c + 1) = decay^n S_c + U_c; the slot's state
//   retention_read     o_t = decay^(t + 1) S_c^T q_t + sum_(s <= t) decay^(t - s) (q_t . k_s) v_s, norm and gate
// The decays are known ahead, so nothing but the fold runs along the tokens.  All sums are float32 FMAs: what enters the
// recurrence is 32-bit by design.  Two FMAs of neighbouring columns are one packed instruction (fma.rn.f32x2).
#include "state_walk.cuh"

namespace srlm {

constexpr int kRetThreads = 512;

template <int VEC, int RPT, typename TO>
__global__ void __launch_bounds__(kRetThreads)
retention_walk_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ cos_t,
                      const float* __restrict__ sin_t, int pairs, const float* __restrict__ decay, float eps,
                      float* __restrict__ state, long long state_stride, const int* __restrict__ cu_q,
                      const int* __restrict__ slots, float* __restrict__ o_out, TO* __restrict__ out, int H, int d, int dv,
                      int cols, int col_threads, int row_groups, int walk_max) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float ret_smem[];
  float* q_s = ret_smem;                               // [d]
  float* k_s = q_s + d;                                // [d]
  float* part = k_s + d;                               // [row_groups][cols]
  float* o_s = part + (size_t)row_groups * cols;       // [cols]
  __shared__ float scratch[32];
  const int e = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * cols;
  const int t0 = cu_q[e], n = cu_q[e + 1] - t0;
  if (n > walk_max) return;                            // in chunks
  const int tid = threadIdx.x, ct = tid % col_threads, rg = tid / col_threads;
  const int col = c0 + ct * VEC;
  const bool live = rg < row_groups && ct * VEC < cols && col < dv;
  float* S = state + (size_t)slots[e] * state_stride + (size_t)h * d * dv;
  const float keep = decay[h], k_scale = 1.f / sqrtf((float)d);
  float s[RPT][VEC];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = rg + i * row_groups;
#pragma unroll
    for (int c = 0; c < VEC; ++c) s[i][c] = 0.f;
    if (live && r < d) {
      if (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(S + (size_t)r * dv + col);
        s[i][0] = v.x; s[i][VEC > 1 ? 1 : 0] = v.y; s[i][VEC > 2 ? 2 : 0] = v.z; s[i][VEC > 3 ? 3 : 0] = v.w;
      } else {
        s[i][0] = S[(size_t)r * dv + col];
      }
    }
  }
  for (int t = t0; t < t0 + n; ++t) {
    const float* p = proj + (size_t)t * ldp;
    __syncthreads();                                   // the token before is no longer read
    for (int idx = tid; idx < 2 * d; idx += blockDim.x) {
      const bool is_k = idx >= d;
      const int i = is_k ? idx - d : idx;
      const float* x = p + (is_k ? (size_t)H * d : 0) + (size_t)h * d;
      float v = x[i];
      if (i < 2 * pairs) {
        const int a = i < pairs ? i : i - pairs;
        const float cs = cos_t[(size_t)t * pairs + a], sn = sin_t[(size_t)t * pairs + a];
        v = i < pairs ? v * cs - x[i + pairs] * sn : v * cs + x[i - pairs] * sn;
      }
      (is_k ? k_s : q_s)[i] = is_k ? v * k_scale : v;
    }
    float v[VEC], o[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      v[c] = live && col + c < dv ? p[2 * (size_t)H * d + (size_t)h * dv + col + c] : 0.f;
      o[c] = 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * row_groups;
      if (r < d) {
        const float kr = k_s[r], qr = q_s[r];
#pragma unroll
        for (int c = 0; c < VEC; ++c) {
          s[i][c] = keep * s[i][c] + kr * v[c];
          o[c] += qr * s[i][c];
        }
      }
    }
    if (live) {
#pragma unroll
      for (int c = 0; c < VEC; ++c) part[(size_t)rg * cols + ct * VEC + c] = o[c];
    }
    __syncthreads();
    float ss = 0.f;
    const int width = min(cols, dv - c0);
    for (int c = tid; c < width; c += blockDim.x) {
      float a = 0.f;
      for (int g = 0; g < row_groups; ++g) a += part[(size_t)g * cols + c];
      if (o_out) o_out[((size_t)t * H + h) * dv + c0 + c] = a;
      else o_s[c] = a;
      ss += a * a;
    }
    if (!o_out) {
      const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)dv + eps);
      const float* g = p + 2 * (size_t)H * d + (size_t)H * dv + (size_t)h * dv;
      for (int c = tid; c < width; c += blockDim.x) {
        const float z = g[c];
        out[((size_t)t * H + h) * dv + c] = from_float<TO>(o_s[c] * inv * (z / (1.f + expf(-z))));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = rg + i * row_groups;
    if (live && r < d) {
      if (VEC == 4)
        *reinterpret_cast<float4*>(S + (size_t)r * dv + col) =
            make_float4(s[i][0], s[i][VEC > 1 ? 1 : 0], s[i][VEC > 2 ? 2 : 0], s[i][VEC > 3 ? 3 : 0]);
      else
        S[(size_t)r * dv + col] = s[i][0];
    }
  }
}

// ---- chunks ------------------------------------------------------------------------------------------------------------
constexpr int kRetChunk = 64;

// decay^n, formed in double precision and rounded once.
__device__ __forceinline__ float decay_power(float decay, int n) {
  double p = 1.0, b = decay;
  for (; n; n >>= 1, b *= b)
    if (n & 1) p *= b;
  return (float)p;
}

// Where chunk `index` of the step lies: chunks number the entries of more than walk_max tokens in order.
struct ChunkHome {
  int entry, t0, n, first;        // entry; first token (of the step); tokens; the entry's first chunk
};
__device__ __forceinline__ ChunkHome chunk_home(const int* __restrict__ cu_q, int n_entries, int walk_max, int index) {
  int base = 0;
  for (int e = 0; e < n_entries; ++e) {
    const int a = cu_q[e], len = cu_q[e + 1] - a;
    if (len <= walk_max) continue;
    const int chunks = (len + kRetChunk - 1) / kRetChunk;
    if (index < base + chunks) {
      const int at = (index - base) * kRetChunk;
      return ChunkHome{e, a + at, min(kRetChunk, len - at), base};
    }
    base += chunks;
  }
  return ChunkHome{-1, 0, 0, 0};
}

__device__ __forceinline__ void ret_copy_16(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src));
}
__device__ __forceinline__ void ret_copy_4(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src));
}
__device__ __forceinline__ void ret_commit() { asm volatile("cp.async.commit_group;" ::); }
template <int N> __device__ __forceinline__ void ret_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }

// dst[x][c] (row stride `stride`, a multiple of 4) = src[x * ld + c] for x < n and c < width, zeros up to `rows` rows and
// `padded` columns; asynchronous, in 16-byte pieces when `vec` says that every row of src starts on 16 bytes and width and
// padded are multiples of 4.
__device__ __forceinline__ void ret_copy_rows(float* dst, int stride, const float* src, long long ld, int n, int rows, int width,
                                              int padded, bool vec) {
  if (vec) {
    const int pieces = padded / 4, step = (int)blockDim.x / pieces, c = ((int)threadIdx.x % pieces) * 4;
    if (step == 0) {                                   // rows of more pieces than the block has threads
      for (int idx = threadIdx.x; idx < rows * pieces; idx += blockDim.x) {
        const int x = idx / pieces, cc = (idx - x * pieces) * 4;
        if (x < n && cc < width) ret_copy_16(dst + x * stride + cc, src + (size_t)x * ld + cc);
        else *reinterpret_cast<float4*>(dst + x * stride + cc) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
      return;
    }
    if ((int)threadIdx.x >= step * pieces) return;
#pragma unroll 4
    for (int x = (int)threadIdx.x / pieces; x < rows; x += step) {
      if (x < n && c < width) ret_copy_16(dst + x * stride + c, src + (size_t)x * ld + c);
      else *reinterpret_cast<float4*>(dst + x * stride + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int idx = threadIdx.x; idx < rows * padded; idx += blockDim.x) {
      const int x = idx / padded, c = idx - x * padded;
      if (x < n && c < width) ret_copy_4(dst + x * stride + c, src + (size_t)x * ld + c);
      else dst[x * stride + c] = 0.f;
    }
  }
}

// Turns the leading 2 pairs elements of rows of shared memory: row x by the angles of token t0 + x; then multiplies the
// whole row by scale[x] (null: leaves it).
__device__ __forceinline__ void ret_rotate_rows(float* rows_s, int stride, int n, int d, const float* __restrict__ cos_t,
                                                const float* __restrict__ sin_t, int t0, int pairs, const float* scale) {
  if (pairs) {
#pragma unroll 4
    for (int idx = threadIdx.x; idx < n * pairs; idx += blockDim.x) {
      const int x = idx / pairs, i = idx - x * pairs;
      const float c = __ldg(cos_t + (size_t)t0 * pairs + idx), sn = __ldg(sin_t + (size_t)t0 * pairs + idx);
      float* row = rows_s + x * stride;
      const float u = row[i], v = row[i + pairs], f = scale ? scale[x] : 1.f;
      row[i] = (u * c - v * sn) * f;
      row[i + pairs] = (v * c + u * sn) * f;
    }
  }
  const int rest = d - 2 * pairs;
  if (scale && rest > 0)
    for (int idx = threadIdx.x; idx < n * rest; idx += blockDim.x) rows_s[(idx / rest) * stride + 2 * pairs + idx % rest] *= scale[idx / rest];
}

// U of a chunk and head: a tile of 16 TM rows (of d) x 16 TN columns (of dv) a block, TM x TN of it a thread.
template <int TM, int TN>
__global__ void __launch_bounds__(256)
retention_chunks_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ cos_t,
                        const float* __restrict__ sin_t, int pairs, const float* __restrict__ decay,
                        const int* __restrict__ cu_q, int n_entries, int walk_max, float* __restrict__ U, int H, int d, int dv,
                        int dp, int vec) {
  pdl_wait();
  pdl_trigger();
  constexpr int BM = 16 * TM, BN = 16 * TN;
  extern __shared__ __align__(16) float ret_chunk_smem[];
  const int ks = dp + 4;                             // dp: d rounded up to whole row tiles
  float* k_s = ret_chunk_smem;                       // [64][dp + 4]
  float* v_s = k_s + kRetChunk * ks;                 // [64][BN + 4]
  __shared__ float fade[kRetChunk];
  const int h = blockIdx.y, c0 = blockIdx.z * BN;
  const ChunkHome home = chunk_home(cu_q, n_entries, walk_max, blockIdx.x);
  if (home.entry < 0) return;
  const int tid = threadIdx.x;
  const float* first = proj + (size_t)home.t0 * ldp;
  ret_copy_rows(k_s, ks, first + (size_t)(H + h) * d, ldp, home.n, kRetChunk, d, dp, vec);
  ret_copy_rows(v_s, BN + 4, first + 2 * (size_t)H * d + (size_t)h * dv + c0, ldp, home.n, kRetChunk, min(BN, dv - c0), BN, vec);
  ret_commit();
  if (tid < home.n) fade[tid] = decay_power(decay[h], home.n - 1 - tid) / sqrtf((float)d);
  ret_wait<0>();
  __syncthreads();
  ret_rotate_rows(k_s, ks, home.n, d, cos_t, sin_t, home.t0, pairs, fade);
  __syncthreads();
  const int tn = (tid % 16) * 2;                     // a thread's columns: tn, tn + 1 of every 32
  float* dst = U + ((size_t)blockIdx.x * H + h) * d * dv;
  for (int m0 = 0; m0 < d; m0 += BM) {
    const int tm = m0 + (tid / 16) * TM;
    float2 acc[TM][TN / 2];
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) acc[i][j] = make_float2(0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < kRetChunk; ++s) {
      float a[TM];
      float2 b[TN / 2];
#pragma unroll
      for (int i = 0; i < TM; ++i) a[i] = k_s[s * ks + tm + i];
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) b[j] = *reinterpret_cast<const float2*>(v_s + s * (BN + 4) + tn + 32 * j);
#pragma unroll
      for (int i = 0; i < TM; ++i)
#pragma unroll
        for (int j = 0; j < TN / 2; ++j) acc[i][j] = fma2(make_float2(a[i], a[i]), b[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < TM; ++i) {
      const int r = tm + i;
      if (r >= d) continue;
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) {
        const int c = c0 + tn + 32 * j;
        if (vec) {
          if (c < dv) *reinterpret_cast<float2*>(dst + (size_t)r * dv + c) = acc[i][j];
        } else {
          if (c < dv) dst[(size_t)r * dv + c] = acc[i][j].x;
          if (c + 1 < dv) dst[(size_t)r * dv + c + 1] = acc[i][j].y;
        }
      }
    }
  }
}

// grid (elements of a state / (256 V), entries): S of the slot through the entry's chunks; U_c <- the state ahead of chunk
// c.  V neighbouring elements a thread (4 when the rows of U and of the state allow 16-byte accesses).
template <int V>
__global__ void __launch_bounds__(256)
retention_fold_kernel(float* __restrict__ U, const float* __restrict__ decay, float* __restrict__ state, long long state_stride,
                      const int* __restrict__ cu_q, const int* __restrict__ slots, int walk_max, int H, int d, int dv) {
  pdl_wait();
  pdl_trigger();
  const int e = blockIdx.y;
  const int len = cu_q[e + 1] - cu_q[e];
  if (len <= walk_max) return;
  int base = 0;
  for (int x = 0; x < e; ++x) {
    const int l = cu_q[x + 1] - cu_q[x];
    if (l > walk_max) base += (l + kRetChunk - 1) / kRetChunk;
  }
  const size_t per = (size_t)H * d * dv, i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= per) return;
  const int h = (int)(i / ((size_t)d * dv)), chunks = (len + kRetChunk - 1) / kRetChunk;
  const float whole = decay_power(decay[h], kRetChunk), rest = decay_power(decay[h], len - (chunks - 1) * kRetChunk);
  float* u = U + (size_t)base * per + i;
  float* slot = state + (size_t)slots[e] * state_stride + i;
  auto get = [](const float* p, float (&v)[V]) {
    if (V == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    else v[0] = p[0];
  };
  auto put = [](float* p, const float (&v)[V]) {
    if (V == 4) *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(v);
    else p[0] = v[0];
  };
  alignas(16) float S[V];
  get(slot, S);
  constexpr int kAhead = 8;
  for (int c = 0; c < chunks; c += kAhead) {
    alignas(16) float next[kAhead][V];
#pragma unroll
    for (int x = 0; x < kAhead; ++x)
      if (c + x < chunks) get(u + (size_t)(c + x) * per, next[x]);
#pragma unroll
    for (int x = 0; x < kAhead; ++x) {
      if (c + x < chunks) {
        put(u + (size_t)(c + x) * per, S);
        const float f = c + x + 1 < chunks ? whole : rest;
#pragma unroll
        for (int y = 0; y < V; ++y) S[y] = fmaf(f, S[y], next[x][y]);
      }
    }
  }
  put(slot, S);
}

// A chunk of 64 tokens, one head, a tile of 16 TN value columns a block: thread (ty, tx) holds rows 4 ty .. 4 ty + 3 and
// the column pairs 2 tx + 32 j.  Where one tile holds the head it norms and gates; else o_out.
constexpr int kRetSlab = 16;                          // rows of the state that are multiplied at a time

template <int TN, typename TO>
__global__ void __launch_bounds__(256)
retention_read_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ cos_t,
                      const float* __restrict__ sin_t, int pairs, const float* __restrict__ decay, float eps,
                      const int* __restrict__ cu_q, int n_entries, int walk_max, const float* __restrict__ U,
                      float* __restrict__ o_out, TO* __restrict__ out, int H, int d, int dv, int dp, int vec) {
  pdl_wait();
  pdl_trigger();
  constexpr int BN = 16 * TN, BS = BN + 4;
  extern __shared__ __align__(16) float ret_chunk_smem[];
  const int qs = dp + 4;                              // dp: d rounded up to a multiple of 4 (zeros behind it)
  float* q_s = ret_chunk_smem;                        // [64][dp + 4]
  float* v_s = q_s + kRetChunk * qs;                  // [64][BN + 4]
  float* k_s = v_s + kRetChunk * BS;                  // [64][dp + 4]; then a_t and two slabs of the state
  float* a_t = k_s;                                   // [64][64]: (s, t): what token t takes of v_s
  float* s_s = a_t + kRetChunk * kRetChunk;           // [2][16][BN + 4]
  __shared__ float pw[kRetChunk + 1];
  const int h = blockIdx.y, c0 = blockIdx.z * BN, width = min(BN, dv - c0);
  const ChunkHome home = chunk_home(cu_q, n_entries, walk_max, blockIdx.x);
  if (home.entry < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5;
  const float* first = proj + (size_t)home.t0 * ldp + (size_t)h * d;
  ret_copy_rows(q_s, qs, first, ldp, home.n, kRetChunk, d, dp, vec);
  ret_copy_rows(k_s, qs, first + (size_t)H * d, ldp, home.n, kRetChunk, d, dp, vec);
  ret_commit();
  ret_copy_rows(v_s, BS, proj + (size_t)home.t0 * ldp + 2 * (size_t)H * d + (size_t)h * dv + c0, ldp, home.n, kRetChunk, width, BN, vec);
  ret_commit();
  if (tid <= kRetChunk) pw[tid] = decay_power(decay[h], tid);
  ret_wait<1>();
  __syncthreads();
  ret_rotate_rows(q_s, qs, home.n, d, cos_t, sin_t, home.t0, pairs, nullptr);
  ret_rotate_rows(k_s, qs, home.n, d, cos_t, sin_t, home.t0, pairs, nullptr);
  __syncthreads();

  const int ty = tid / 16, tx = tid % 16, tm = ty * 4, tn = tx * 2;
  const float k_scale = 1.f / sqrtf((float)d);
  float dot[4][4];                                    // [t][s]: 4 tokens t = tm + i, 4 tokens s = tx + 16 j
  {
    float2 sum[4][4];                                 // even and odd elements apart
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) sum[i][j] = make_float2(0.f, 0.f);
#pragma unroll 2
    for (int x = 0; x < dp; x += 4) {
      float4 a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(q_s + (tm + i) * qs + x);
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = *reinterpret_cast<const float4*>(k_s + (tx + 16 * j) * qs + x);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          sum[i][j] = fma2(make_float2(a[i].x, a[i].y), make_float2(b[j].x, b[j].y), sum[i][j]);
          sum[i][j] = fma2(make_float2(a[i].z, a[i].w), make_float2(b[j].z, b[j].w), sum[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) dot[i][j] = (sum[i][j].x + sum[i][j].y) * k_scale;
  }
  __syncthreads();                                    // k_s is read: a_t and the slabs take its place
  const float* S = U + ((size_t)blockIdx.x * H + h) * d * dv + c0;
  auto fetch = [&](int slab) {
    const int r0 = slab * kRetSlab;
    ret_copy_rows(s_s + (slab & 1) * kRetSlab * BS, BS, S + (size_t)r0 * dv, dv, min(kRetSlab, d - r0), kRetSlab, width, BN, vec);
    ret_commit();
  };
  fetch(0);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int s = tx + 16 * j;
#pragma unroll
    for (int i = 0; i < 4; ++i) dot[i][j] = s <= tm + i ? dot[i][j] * pw[max(tm + i - s, 0)] : 0.f;
    *reinterpret_cast<float4*>(a_t + s * kRetChunk + tm) = make_float4(dot[0][j], dot[1][j], dot[2][j], dot[3][j]);
  }

  float2 acc[4][TN / 2];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) acc[i][j] = make_float2(0.f, 0.f);
  auto row_times = [&](float a0, float a1, float a2, float a3, const float* right) {
    float2 b[TN / 2];
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) b[j] = *reinterpret_cast<const float2*>(right + tn + 32 * j);
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) {
      acc[0][j] = fma2(make_float2(a0, a0), b[j], acc[0][j]);
      acc[1][j] = fma2(make_float2(a1, a1), b[j], acc[1][j]);
      acc[2][j] = fma2(make_float2(a2, a2), b[j], acc[2][j]);
      acc[3][j] = fma2(make_float2(a3, a3), b[j], acc[3][j]);
    }
  };
  const int slabs = (d + kRetSlab - 1) / kRetSlab;
  for (int slab = 0; slab < slabs; ++slab) {
    ret_wait<0>();
    __syncthreads();                                  // the slab is here; the other one is read
    if (slab + 1 < slabs) fetch(slab + 1);
    const float* right = s_s + (slab & 1) * kRetSlab * BS;
    const int r0 = slab * kRetSlab, rows = min(kRetSlab, dp - r0);
#pragma unroll 2
    for (int r = 0; r < rows; r += 4) {               // rows of the slab behind d are zeros, and so are q's elements there
      float4 a[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(q_s + (tm + i) * qs + r0 + r);
      row_times(a[0].x, a[1].x, a[2].x, a[3].x, right + r * BS);
      row_times(a[0].y, a[1].y, a[2].y, a[3].y, right + (r + 1) * BS);
      row_times(a[0].z, a[1].z, a[2].z, a[3].z, right + (r + 2) * BS);
      row_times(a[0].w, a[1].w, a[2].w, a[3].w, right + (r + 3) * BS);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) {
      acc[i][j].x *= pw[tm + i + 1];
      acc[i][j].y *= pw[tm + i + 1];
    }
  const int s_end = (warp + 1) * 8;                   // a warp's rows end at 8 warp + 7: no later s counts
#pragma unroll 4
  for (int s = 0; s < s_end; ++s) {
    const float4 a = *reinterpret_cast<const float4*>(a_t + s * kRetChunk + tm);
    row_times(a.x, a.y, a.z, a.w, v_s + s * BS);
  }

  // a row's columns lie with the 16 threads of its ty
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int s = tm + i;
    const size_t t = home.t0 + s;
    float inv = 1.f;
    if (!o_out) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) ss += acc[i][j].x * acc[i][j].x + acc[i][j].y * acc[i][j].y;
#pragma unroll
      for (int x = 8; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
      inv = 1.f / sqrtf(ss / (float)dv + eps);
    }
    if (s >= home.n) continue;
#pragma unroll
    for (int j = 0; j < TN / 2; ++j)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int col = c0 + tn + 32 * j + c;
        if (col >= dv) continue;
        const float v = c ? acc[i][j].y : acc[i][j].x;
        if (o_out) {
          o_out[(t * H + h) * dv + col] = v;
        } else {
          const float z = proj[t * ldp + 2 * (size_t)H * d + (size_t)H * dv + (size_t)h * dv + col];
          out[(t * H + h) * dv + col] = from_float<TO>(v * inv * (z / (1.f + expf(-z))));
        }
      }
  }
}

// A warp per (token, head): out = o / sqrt(mean(o^2) + eps) * silu(gate).
template <typename TO>
__global__ void retention_output_kernel(const float* __restrict__ o, float eps, const float* __restrict__ proj, long long ldp,
                                        int g_off, TO* __restrict__ out, long long heads_total, int H, int dv) {
  pdl_wait();
  pdl_trigger();
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= heads_total) return;
  const int lane = threadIdx.x & 31, h = (int)(w % H);
  const long long t = w / H;
  const float* src = o + w * dv;
  float ss = 0.f;
  for (int i = lane; i < dv; i += 32) ss += src[i] * src[i];
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int i = lane; i < dv; i += 32) {
    const float z = proj[t * ldp + g_off + (size_t)h * dv + i];
    out[w * dv + i] = from_float<TO>(src[i] * inv * (z / (1.f + expf(-z))));
  }
}

}  // namespace srlm

using namespace srlm;

// Whether srlm_retention_walk norms and gates itself (one tile of columns holds a head).
extern "C" int srlm_retention_walk_finishes(int dv) { return dv <= 128; }

// cos_t, sin_t float32 [T, pairs] (pairs 0: no rotation); state float32 [slots, state_stride]; out [T, H dv] when a head is
// one tile (srlm_retention_walk_finishes), else o_out float32 [T, H dv] (retention_output follows).
extern "C" int srlm_retention_walk(const float* proj, long long ldp, const float* cos_t, const float* sin_t, int pairs,
                                   const float* decay, float eps, float* state, long long state_stride, const int* cu_q,
                                   const int* slots, float* o_out, void* out, int out_dtype, int n_entries, int H, int d,
                                   int dv, int walk_max, cudaStream_t stream) {
  if (n_entries <= 0) return ST_OK;
  if (H <= 0 || d <= 0 || d > 512 || dv <= 0 || pairs < 0 || 2 * pairs > d || (pairs && (!cos_t || !sin_t)) || !(eps > 0.f) ||
      ldp < 2LL * H * d + 2LL * H * dv || state_stride < (long long)H * d * dv || n_entries > 65535 || H > 65535)
    return refuse(ST_BAD_SIZE, "retention_walk: heads=%d dim=%d (at most 512) vdim=%d pairs=%d ld=%lld", H, d, dv, pairs, ldp);
  const int vec = dv % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0 ? 4 : 1;
  const int cols = dv < 128 ? dv : 128, tiles = (dv + cols - 1) / cols;
  const bool finishes = tiles == 1;
  if (finishes ? !out : !o_out) return refuse(ST_BAD_SIZE, "retention_walk: no buffer for the result");
  const int col_threads = (cols + vec - 1) / vec;
  int row_groups = kRetThreads / col_threads;
  if (row_groups > d) row_groups = d;
  const int rpt = (d + row_groups - 1) / row_groups;
  const int threads = (col_threads * row_groups + 31) / 32 * 32;
  const size_t smem = (2 * (size_t)d + (size_t)row_groups * cols + cols) * sizeof(float);
  dim3 grid(tiles, H, n_entries);
#define SRLM_WALK(V, R)                                                                                                \
  SRLM_DISPATCH_ACT(out_dtype, TO, launch_pdl(retention_walk_kernel<V, R, TO>, grid, dim3(threads), smem, stream, proj, ldp, \
      cos_t, sin_t, pairs, decay, eps, state, state_stride, cu_q, slots, finishes ? nullptr : o_out, (TO*)out, H, d, dv, cols, \
      col_threads, row_groups, walk_max))
#define SRLM_WALK_R(V)                \
  do {                                \
    if (rpt <= 1) SRLM_WALK(V, 1);    \
    else if (rpt <= 2) SRLM_WALK(V, 2);   \
    else if (rpt <= 4) SRLM_WALK(V, 4);   \
    else if (rpt <= 8) SRLM_WALK(V, 8);   \
    else if (rpt <= 16) SRLM_WALK(V, 16); \
    else SRLM_WALK(V, 32);            \
  } while (0)
  // 16-byte columns: at most 32 rows a thread (32 column threads, 16 row groups, d <= 512); single columns: 128
  if (vec == 4) SRLM_WALK_R(4);
  else if (rpt > 32) SRLM_WALK(1, 128);
  else SRLM_WALK_R(1);
#undef SRLM_WALK_R
#undef SRLM_WALK
  return launched();
}

extern "C" int srlm_retention_output(const float* o, float eps, const float* proj, long long ldp, int g_off, void* out,
                                     int out_dtype, int T, int H, int dv, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (H <= 0 || dv <= 0 || !(eps > 0.f) || g_off < 0 || ldp < g_off + (long long)H * dv)
    return refuse(ST_BAD_SIZE, "retention_output: heads=%d vdim=%d g_off=%d ld=%lld", H, dv, g_off, ldp);
  const long long total = (long long)T * H;
  SRLM_DISPATCH_ACT(out_dtype, TO, launch_pdl(retention_output_kernel<TO>, dim3((unsigned)((total + 3) / 4)), dim3(128), 0,
                                              stream, o, eps, proj, ldp, g_off, (TO*)out, total, H, dv));
  return launched();
}

static size_t ret_read_smem(int d, int tn) {
  const size_t qs = (d + 3) / 4 * 4 + 4, bs = 16 * tn + 4;
  const size_t third = kRetChunk * kRetChunk + 2 * kRetSlab * bs;
  return (kRetChunk * qs + kRetChunk * bs + (kRetChunk * qs > third ? kRetChunk * qs : third)) * sizeof(float);
}
static int ret_rows_padded(int d, int t) { return (d + 16 * t - 1) / (16 * t) * (16 * t); }
static size_t ret_chunks_smem(int d, int t) { return (size_t)kRetChunk * (ret_rows_padded(d, t) + 4 + 16 * t + 4) * sizeof(float); }
static int ret_tile(int n) { return n <= 32 ? 2 : n <= 64 ? 4 : 8; }

// Whether entries may be taken in chunks: heads of up to 256 elements.
extern "C" int srlm_retention_chunks_take(int d, int dv) {
  const int tm = ret_tile(d), tn = ret_tile(dv);
  return d > 0 && dv > 0 && d <= 256 && ret_read_smem(d, tn) <= 220 * 1024 && ret_chunks_smem(d, tm > tn ? tm : tn) <= 220 * 1024;
}
extern "C" int srlm_retention_chunk_tokens() { return kRetChunk; }

// The entries of more than walk_max tokens, in chunks; chunks: how many chunks they have together; U float32
// [chunks, H, d, dv].  out [T, H dv] when a head's values are at most 128, else o_out (retention_output follows).
extern "C" int srlm_retention_in_chunks(const float* proj, long long ldp, const float* cos_t, const float* sin_t, int pairs,
                                        const float* decay, float eps, float* state, long long state_stride,
                                        const int* cu_q, const int* slots, float* U, float* o_out, void* out, int out_dtype,
                                        int n_entries, int H, int d, int dv, int walk_max, int chunks, cudaStream_t stream) {
  if (n_entries <= 0 || chunks <= 0) return ST_OK;
  if (H <= 0 || !srlm_retention_chunks_take(d, dv) || pairs < 0 || 2 * pairs > d || (pairs && (!cos_t || !sin_t)) || !(eps > 0.f) ||
      ldp < 2LL * H * d + 2LL * H * dv || state_stride < (long long)H * d * dv || n_entries > 65535 || H > 65535 || !U)
    return refuse(ST_BAD_SIZE, "retention_in_chunks: heads=%d dim=%d vdim=%d pairs=%d ld=%lld", H, d, dv, pairs, ldp);
  const int tm = ret_tile(d), tn = ret_tile(dv), t = tm > tn ? tm : tn;
  const bool finishes = dv <= 128;
  if (finishes ? !out : !o_out) return refuse(ST_BAD_SIZE, "retention_in_chunks: no buffer for the result");
  // 16-byte accesses: every row of the projection, of U and of the state starts on 16 bytes
  const int vec = d % 4 == 0 && dv % 4 == 0 && ldp % 4 == 0 && state_stride % 4 == 0 &&
                  (((uintptr_t)proj | (uintptr_t)U | (uintptr_t)state) & 15) == 0;
  {
    const size_t smem = ret_chunks_smem(d, t);
    const dim3 grid(chunks, H, (dv + 16 * t - 1) / (16 * t));
#define SRLM_CHUNKS(X)                                                                                                      \
  do {                                                                                                                      \
    auto kern = retention_chunks_kernel<X, X>;                                                                              \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);               \
    launch_pdl(kern, grid, dim3(256), smem, stream, proj, ldp, cos_t, sin_t, pairs, decay, cu_q, n_entries, walk_max, U, H, d, dv, \
               ret_rows_padded(d, t), vec);                                                                                 \
  } while (0)
    if (t == 2) SRLM_CHUNKS(2);
    else if (t == 4) SRLM_CHUNKS(4);
    else SRLM_CHUNKS(8);
#undef SRLM_CHUNKS
  }
  const size_t elements = (size_t)H * d * dv;
  if (vec) launch_pdl(retention_fold_kernel<4>, dim3((unsigned)((elements / 4 + 255) / 256), n_entries), dim3(256), 0, stream, U,
                      decay, state, state_stride, cu_q, slots, walk_max, H, d, dv);
  else launch_pdl(retention_fold_kernel<1>, dim3((unsigned)((elements + 255) / 256), n_entries), dim3(256), 0, stream, U, decay,
                  state, state_stride, cu_q, slots, walk_max, H, d, dv);
  const size_t smem = ret_read_smem(d, tn);
  const dim3 grid(chunks, H, (dv + 16 * tn - 1) / (16 * tn));
#define SRLM_READ(X)                                                                                                       \
  SRLM_DISPATCH_ACT(out_dtype, TO, {                                                                                       \
    auto kern = retention_read_kernel<X, TO>;                                                                              \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);              \
    launch_pdl(kern, grid, dim3(256), smem, stream, proj, ldp, cos_t, sin_t, pairs, decay, eps, cu_q, n_entries, walk_max, U, \
               finishes ? (float*)nullptr : o_out, (TO*)out, H, d, dv, (d + 3) / 4 * 4, vec);                                                    \
  })
  if (tn == 2) SRLM_READ(2);
  else if (tn == 4) SRLM_READ(4);
  else SRLM_READ(8);
#undef SRLM_READ
  return launched();
}
