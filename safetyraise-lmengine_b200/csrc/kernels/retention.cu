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
#include "common.cuh"

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

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(d)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)),
        "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&d);
}

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

// An element of a rotated head: x its projected elements, cs and sn the token's angles.
__device__ __forceinline__ float rotated(const float* __restrict__ x, int i, const float* __restrict__ cs,
                                         const float* __restrict__ sn, int pairs) {
  const float own = x[i];
  if (i >= 2 * pairs) return own;
  return i < pairs ? own * cs[i] - x[i + pairs] * sn[i] : own * cs[i - pairs] + x[i - pairs] * sn[i - pairs];
}

// U of a chunk and head: a tile of 16 TM rows (of d) x 16 TN columns (of dv) a block, TM x TN of it a thread.
template <int TM, int TN>
__global__ void __launch_bounds__(256)
retention_chunks_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ cos_t,
                        const float* __restrict__ sin_t, int pairs, const float* __restrict__ decay,
                        const int* __restrict__ cu_q, int n_entries, int walk_max, float* __restrict__ U, int H, int d, int dv) {
  pdl_wait();
  pdl_trigger();
  constexpr int BM = 16 * TM, BN = 16 * TN;
  extern __shared__ __align__(16) float ret_chunk_smem[];
  float* k_s = ret_chunk_smem;                       // [64][BM + 4]
  float* v_s = k_s + kRetChunk * (BM + 4);           // [64][BN + 4]
  __shared__ float fade[kRetChunk];
  const int h = blockIdx.y, col_tiles = (dv + BN - 1) / BN;
  const int m0 = (blockIdx.z / col_tiles) * BM, c0 = (blockIdx.z % col_tiles) * BN;
  const ChunkHome home = chunk_home(cu_q, n_entries, walk_max, blockIdx.x);
  if (home.entry < 0) return;
  const int tid = threadIdx.x;
  if (tid < home.n) fade[tid] = decay_power(decay[h], home.n - 1 - tid) / sqrtf((float)d);
  __syncthreads();
  for (int idx = tid; idx < kRetChunk * BM; idx += blockDim.x) {
    const int s = idx / BM, i = idx - s * BM, t = home.t0 + s;
    float v = 0.f;
    if (s < home.n && m0 + i < d)
      v = rotated(proj + (size_t)t * ldp + (size_t)(H + h) * d, m0 + i, cos_t + (size_t)t * pairs, sin_t + (size_t)t * pairs, pairs) * fade[s];
    k_s[s * (BM + 4) + i] = v;
  }
  for (int idx = tid; idx < kRetChunk * BN; idx += blockDim.x) {
    const int s = idx / BN, i = idx - s * BN;
    v_s[s * (BN + 4) + i] = s < home.n && c0 + i < dv ? proj[(size_t)(home.t0 + s) * ldp + 2 * (size_t)H * d + (size_t)h * dv + c0 + i] : 0.f;
  }
  __syncthreads();
  const int tm = (tid / 16) * TM, tn = (tid % 16) * 2;        // a thread's columns: tn, tn + 1 of every 32
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
    for (int i = 0; i < TM; ++i) a[i] = k_s[s * (BM + 4) + tm + i];
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) b[j] = *reinterpret_cast<const float2*>(v_s + s * (BN + 4) + tn + 32 * j);
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) acc[i][j] = fma2(make_float2(a[i], a[i]), b[j], acc[i][j]);
  }
  float* dst = U + ((size_t)blockIdx.x * H + h) * d * dv;
#pragma unroll
  for (int i = 0; i < TM; ++i) {
    const int r = m0 + tm + i;
    if (r >= d) continue;
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) {
      const int c = c0 + tn + 32 * j;
      if (c < dv) dst[(size_t)r * dv + c] = acc[i][j].x;
      if (c + 1 < dv) dst[(size_t)r * dv + c + 1] = acc[i][j].y;
    }
  }
}

// grid (elements of a state / 256, entries): S of the slot through the entry's chunks; U_c <- the state ahead of chunk c.
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
  const size_t per = (size_t)H * d * dv, i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= per) return;
  const int h = (int)(i / ((size_t)d * dv)), chunks = (len + kRetChunk - 1) / kRetChunk;
  const float whole = decay_power(decay[h], kRetChunk), rest = decay_power(decay[h], len - (chunks - 1) * kRetChunk);
  float* u = U + (size_t)base * per + i;
  float* slot = state + (size_t)slots[e] * state_stride + i;
  float S = *slot;
  constexpr int kAhead = 8;
  for (int c = 0; c < chunks; c += kAhead) {
    float next[kAhead];
#pragma unroll
    for (int x = 0; x < kAhead; ++x) next[x] = c + x < chunks ? u[(size_t)(c + x) * per] : 0.f;
#pragma unroll
    for (int x = 0; x < kAhead; ++x) {
      if (c + x < chunks) {
        u[(size_t)(c + x) * per] = S;
        S = fmaf(c + x + 1 < chunks ? whole : rest, S, next[x]);
      }
    }
  }
  *slot = S;
}

// A chunk of 64 tokens, one head, a tile of 16 TN value columns a block: thread (ty, tx) holds rows 4 ty .. 4 ty + 3 and
// the column pairs 2 tx + 32 j.  Where one tile holds the head it norms and gates; else o_out.
template <int TN, typename TO>
__global__ void __launch_bounds__(256)
retention_read_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ cos_t,
                      const float* __restrict__ sin_t, int pairs, const float* __restrict__ decay, float eps,
                      const int* __restrict__ cu_q, int n_entries, int walk_max, const float* __restrict__ U,
                      float* __restrict__ o_out, TO* __restrict__ out, int H, int d, int dv) {
  pdl_wait();
  pdl_trigger();
  constexpr int BN = 16 * TN, TR = kRetChunk + 4;
  extern __shared__ __align__(16) float ret_chunk_smem[];
  float* q_t = ret_chunk_smem;                        // [d][68]: element, token
  float* k_t = q_t + (size_t)d * TR;                  // [d][68], then slabs of S: [slab rows][BN + 4]
  float* a_t = k_t + (size_t)d * TR;                  // [64][68]: (s, t): what token t takes of v_s
  float* v_s = a_t + (size_t)kRetChunk * TR;          // [64][BN + 4]
  __shared__ float pw[kRetChunk + 1];
  const int h = blockIdx.y, c0 = blockIdx.z * BN;
  const ChunkHome home = chunk_home(cu_q, n_entries, walk_max, blockIdx.x);
  if (home.entry < 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid <= kRetChunk) pw[tid] = decay_power(decay[h], tid);
  const float k_scale = 1.f / sqrtf((float)d);
  // q and k turned and transposed: a warp stores 8 elements x 4 tokens at a time, one bank each
  const int dim_groups = (d + 7) / 8;
  for (int job = warp; job < dim_groups * (kRetChunk / 4); job += 8) {
    const int i = (job % dim_groups) * 8 + (lane & 7), s = (job / dim_groups) * 4 + (lane >> 3), t = home.t0 + s;
    if (i < d) {
      float q = 0.f, k = 0.f;
      if (s < home.n) {
        const float* x = proj + (size_t)t * ldp + (size_t)h * d;
        q = rotated(x, i, cos_t + (size_t)t * pairs, sin_t + (size_t)t * pairs, pairs);
        k = rotated(x + (size_t)H * d, i, cos_t + (size_t)t * pairs, sin_t + (size_t)t * pairs, pairs) * k_scale;
      }
      q_t[i * TR + s] = q;
      k_t[i * TR + s] = k;
    }
  }
  for (int idx = tid; idx < kRetChunk * BN; idx += blockDim.x) {
    const int s = idx / BN, i = idx - s * BN;
    v_s[s * (BN + 4) + i] = s < home.n && c0 + i < dv ? proj[(size_t)(home.t0 + s) * ldp + 2 * (size_t)H * d + (size_t)h * dv + c0 + i] : 0.f;
  }
  __syncthreads();

  const int ty = tid / 16, tx = tid % 16, tm = ty * 4, tn = tx * 2;
  {
    // a_t[s][t] = decay^(t - s) q_t . k_s: 4 tokens t x 4 tokens s a thread (s = tx + 16 j), nothing above the diagonal
    float2 dot[4][2];                                 // [s][t pair]
#pragma unroll
    for (int j = 0; j < 4; ++j) dot[j][0] = dot[j][1] = make_float2(0.f, 0.f);
    for (int i = 0; i < d; ++i) {
      const float4 a = *reinterpret_cast<const float4*>(q_t + i * TR + tm);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float b = k_t[i * TR + tx + 16 * j];
        dot[j][0] = fma2(make_float2(b, b), make_float2(a.x, a.y), dot[j][0]);
        dot[j][1] = fma2(make_float2(b, b), make_float2(a.z, a.w), dot[j][1]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = tx + 16 * j;
      float4 v;
      v.x = s <= tm ? dot[j][0].x * pw[tm - s] : 0.f;
      v.y = s <= tm + 1 ? dot[j][0].y * pw[tm + 1 - s] : 0.f;
      v.z = s <= tm + 2 ? dot[j][1].x * pw[tm + 2 - s] : 0.f;
      v.w = s <= tm + 3 ? dot[j][1].y * pw[tm + 3 - s] : 0.f;
      *reinterpret_cast<float4*>(a_t + s * TR + tm) = v;
    }
  }
  __syncthreads();                                    // a_t is written; k_t and the unscaled q_t are read

  float2 acc[4][TN / 2];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) acc[i][j] = make_float2(0.f, 0.f);
  // rows s of `left` (4 tokens of it a thread) times rows s of `right`
  auto product = [&](const float* left, const float* right, int rows) {
#pragma unroll 4
    for (int s = 0; s < rows; ++s) {
      const float4 a = *reinterpret_cast<const float4*>(left + s * TR + tm);
      float2 b[TN / 2];
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) b[j] = *reinterpret_cast<const float2*>(right + s * (BN + 4) + tn + 32 * j);
#pragma unroll
      for (int j = 0; j < TN / 2; ++j) {
        acc[0][j] = fma2(make_float2(a.x, a.x), b[j], acc[0][j]);
        acc[1][j] = fma2(make_float2(a.y, a.y), b[j], acc[1][j]);
        acc[2][j] = fma2(make_float2(a.z, a.z), b[j], acc[2][j]);
        acc[3][j] = fma2(make_float2(a.w, a.w), b[j], acc[3][j]);
      }
    }
  };
  const float* S = U + ((size_t)blockIdx.x * H + h) * d * dv;
  const int slab_rows = d * TR / (BN + 4) < d ? d * TR / (BN + 4) : d;
  for (int r0 = 0; r0 < d; r0 += slab_rows) {
    const int rows = min(slab_rows, d - r0);
    if (r0) __syncthreads();
    for (int idx = tid; idx < rows * BN; idx += blockDim.x) {
      const int r = idx / BN, i = idx - r * BN;
      k_t[r * (BN + 4) + i] = c0 + i < dv ? S[(size_t)(r0 + r) * dv + c0 + i] : 0.f;
    }
    __syncthreads();
    product(q_t + (size_t)r0 * TR, k_t, rows);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < TN / 2; ++j) {
      acc[i][j].x *= pw[tm + i + 1];
      acc[i][j].y *= pw[tm + i + 1];
    }
  product(a_t, v_s, min(kRetChunk, (warp + 1) * 8));  // a warp's rows end at 8 warp + 7: no later s counts

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
  const int tr = kRetChunk + 4;
  return (2 * (size_t)d * tr + (size_t)kRetChunk * tr + (size_t)kRetChunk * (16 * tn + 4)) * sizeof(float);
}
static int ret_tile(int n) { return n <= 32 ? 2 : n <= 64 ? 4 : 8; }

// Whether entries may be taken in chunks: heads of up to 256 elements.
extern "C" int srlm_retention_chunks_take(int d, int dv) {
  return d > 0 && dv > 0 && d * (kRetChunk + 4) >= 16 * ret_tile(dv) + 4 && ret_read_smem(d, ret_tile(dv)) <= 220 * 1024;
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
  {
    const size_t smem = (size_t)kRetChunk * (2 * (16 * t + 4)) * sizeof(float);
    const dim3 grid(chunks, H, ((d + 16 * t - 1) / (16 * t)) * ((dv + 16 * t - 1) / (16 * t)));
#define SRLM_CHUNKS(X)                                                                                                      \
  do {                                                                                                                      \
    auto kern = retention_chunks_kernel<X, X>;                                                                              \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);               \
    launch_pdl(kern, grid, dim3(256), smem, stream, proj, ldp, cos_t, sin_t, pairs, decay, cu_q, n_entries, walk_max, U, H, d, dv); \
  } while (0)
    if (t == 2) SRLM_CHUNKS(2);
    else if (t == 4) SRLM_CHUNKS(4);
    else SRLM_CHUNKS(8);
#undef SRLM_CHUNKS
  }
  launch_pdl(retention_fold_kernel, dim3((unsigned)(((size_t)H * d * dv + 255) / 256), n_entries), dim3(256), 0, stream, U, decay,
             state, state_stride, cu_q, slots, walk_max, H, d, dv);
  const size_t smem = ret_read_smem(d, tn);
  const dim3 grid(chunks, H, (dv + 16 * tn - 1) / (16 * tn));
#define SRLM_READ(X)                                                                                                       \
  SRLM_DISPATCH_ACT(out_dtype, TO, {                                                                                       \
    auto kern = retention_read_kernel<X, TO>;                                                                              \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);              \
    launch_pdl(kern, grid, dim3(256), smem, stream, proj, ldp, cos_t, sin_t, pairs, decay, eps, cu_q, n_entries, walk_max, U, \
               finishes ? (float*)nullptr : o_out, (TO*)out, H, d, dv);                                                    \
  })
  if (tn == 2) SRLM_READ(2);
  else if (tn == 4) SRLM_READ(4);
  else SRLM_READ(8);
#undef SRLM_READ
  return launched();
}
