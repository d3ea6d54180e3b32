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
#include "common.cuh"

namespace srlm {

constexpr int kRetThreads = 512;

template <int VEC, int RPT, typename TO>
__global__ void __launch_bounds__(kRetThreads)
retention_walk_kernel(const float* __restrict__ proj, long long ldp, const float* __restrict__ cos_t,
                      const float* __restrict__ sin_t, int pairs, const float* __restrict__ decay, float eps,
                      float* __restrict__ state, long long state_stride, const int* __restrict__ cu_q,
                      const int* __restrict__ slots, float* __restrict__ o_out, TO* __restrict__ out, int H, int d, int dv,
                      int cols, int col_threads, int row_groups) {
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
                                   int dv, cudaStream_t stream) {
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
      col_threads, row_groups))
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
