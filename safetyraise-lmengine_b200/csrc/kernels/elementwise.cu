// Embedding gather, residual-add + RMSNorm or layer norm, SwiGLU and casts.
//
// The residual stream is float32 in every mode; norms reduce in float32 in an
// order fixed by the row width alone, so a row's result does not depend on
// what else is in the batch.  Formulas: src/model/native.rs:213-229 (gather),
// src/model/math.rs:28-50 (RMSNorm), src/model/math.rs:11-22 (SiLU).
#include "common.cuh"

namespace srlm {

__global__ void patch_words_kernel(int* __restrict__ words, long long words_len, const int* __restrict__ pairs,
                                   const int* __restrict__ src, int src_len, int n, int* __restrict__ flag) {
  pdl_wait();
  pdl_trigger();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int to = pairs[2 * i], from = pairs[2 * i + 1];
  if (to < 0 || to >= words_len || from < 0 || from >= src_len) {
    atomicExch(flag, 1);
    return;
  }
  words[to] = src[from];
}

template <typename TW>
__global__ void embed_gather_kernel(const int* __restrict__ ids, const TW* __restrict__ table,
                                    float* __restrict__ out, int H, int vocab, int* __restrict__ bad, float scale, int add) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const int id = ids[t];
  if (id < 0 || id >= vocab) {          // the host checks too; never read outside the table
    if (threadIdx.x == 0) atomicExch(bad, 1);
    for (int i = threadIdx.x; i < H && !add; i += blockDim.x) out[(size_t)t * H + i] = 0.f;
    return;
  }
  const TW* row = table + (size_t)id * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = to_float(row[i]) * scale;
    out[(size_t)t * H + i] = add ? out[(size_t)t * H + i] + v : v;
  }
}

// x = residual[src] (+ delta_scale * delta[src]); residual[src] = x when rows == nullptr;
// out[r] = x * rsqrt(mean(x^2) + eps) * (w (+1)).  CENTER: the mean of the row is taken off x first (layer norm: the
// residual keeps it), so that the second moment is the variance.
template <typename TA, bool CENTER>
__global__ void add_norm_kernel(float* __restrict__ residual, const TA* __restrict__ delta, float delta_scale,
                                const float* __restrict__ weight, float eps, TA* __restrict__ out,
                                const int* __restrict__ rows, int H, int unit_offset) {
  __shared__ float scratch[32];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* res = residual + src * H;
  const TA* del = delta ? delta + src * H : nullptr;
  float ss = 0.f, sum = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float x = res[i];
    if (del) {
      x = fmaf(delta_scale, to_float(del[i]), x);
      if (!rows) res[i] = x;
    }
    if (CENTER) sum += x;
    else ss += x * x;
  }
  float mean = 0.f;
  if (CENTER) {
    mean = block_sum(sum, scratch) / (float)H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float x = res[i];
      if (del && rows) x = fmaf(delta_scale, to_float(del[i]), x);
      ss += (x - mean) * (x - mean);
    }
  }
  const float total = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(total / (float)H + eps);
  TA* o = out + (size_t)r * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float x = res[i];
    if (del && rows) x = fmaf(delta_scale, to_float(del[i]), x);
    const float w = weight[i] + (unit_offset ? 1.f : 0.f);
    o[i] = from_float<TA>((CENTER ? x - mean : x) * inv * w);
  }
}

// The same with rows of H = 4 * k elements read and written as 16-byte (float32) and 8-byte (bfloat16)
// pieces; a thread keeps up to CACHE pieces in registers, so a row of up to 4 * CACHE * blockDim elements
// is read once.  The sum of squares adds a thread's elements in index order, then the threads in the
// order of block_sum: fixed by the width.
template <int CACHE, bool CENTER>
__global__ void __launch_bounds__(1024)
add_norm_vec_kernel(float* __restrict__ residual, const bf16* __restrict__ delta, float delta_scale,
                    const float* __restrict__ weight, float eps, bf16* __restrict__ out, const int* __restrict__ rows, int H,
                    int unit_offset) {
  __shared__ float scratch[32];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float4* res = reinterpret_cast<float4*>(residual + src * H);
  const uint2* del = delta ? reinterpret_cast<const uint2*>(delta + src * H) : nullptr;
  const int pieces = H / 4;
  float4 x[CACHE];
  float ss = 0.f, sum = 0.f;
#pragma unroll
  for (int c = 0; c < CACHE; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < pieces) {
      float4 v = res[i];
      if (del) {
        const uint2 d = del[i];
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&d.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&d.y));
        v.x = fmaf(delta_scale, lo.x, v.x); v.y = fmaf(delta_scale, lo.y, v.y);
        v.z = fmaf(delta_scale, hi.x, v.z); v.w = fmaf(delta_scale, hi.y, v.w);
        if (!rows) res[i] = v;
      }
      if (CENTER) sum += (v.x + v.y) + (v.z + v.w);
      else { ss += v.x * v.x; ss += v.y * v.y; ss += v.z * v.z; ss += v.w * v.w; }
      x[c] = v;
    }
  }
  if (CENTER) {
    const float mean = block_sum(sum, scratch) / (float)H;
#pragma unroll
    for (int c = 0; c < CACHE; ++c) {
      if (threadIdx.x + c * blockDim.x < pieces) {
        x[c].x -= mean; x[c].y -= mean; x[c].z -= mean; x[c].w -= mean;
        ss += x[c].x * x[c].x; ss += x[c].y * x[c].y; ss += x[c].z * x[c].z; ss += x[c].w * x[c].w;
      }
    }
  }
  const float total = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(total / (float)H + eps);
  uint2* o = reinterpret_cast<uint2*>(out + (size_t)r * H);
  const float4* w4 = reinterpret_cast<const float4*>(weight);
  const float off = unit_offset ? 1.f : 0.f;
#pragma unroll
  for (int c = 0; c < CACHE; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < pieces) {
      const float4 w = w4[i];
      const __nv_bfloat162 lo = __floats2bfloat162_rn(x[c].x * inv * (w.x + off), x[c].y * inv * (w.y + off));
      const __nv_bfloat162 hi = __floats2bfloat162_rn(x[c].z * inv * (w.z + off), x[c].w * inv * (w.w + off));
      uint2 p;
      p.x = *reinterpret_cast<const uint32_t*>(&lo);
      p.y = *reinterpret_cast<const uint32_t*>(&hi);
      o[i] = p;
    }
  }
}

__device__ __forceinline__ float silu_f(float x) {
  // branch-stable logistic, src/model/math.rs:11-22
  if (x >= 0.f) return x / (1.f + expf(-x));
  const float e = expf(x);
  return x * (e / (1.f + e));
}

// in[T, 2I]: gate in columns [0, I), up in [I, 2I)  ->  out[T, I]
template <typename TA>
__global__ void swiglu_kernel(const TA* __restrict__ in, TA* __restrict__ out, int I, size_t total) {
  pdl_wait();
  pdl_trigger();
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x) {
    const size_t t = idx / I, i = idx % I;
    const float g = to_float(in[t * 2 * I + i]);
    const float u = to_float(in[t * 2 * I + I + i]);
    out[idx] = from_float<TA>(silu_f(g) * u);
  }
}

template <typename TI, typename TO>
__global__ void cast_kernel(const TI* __restrict__ in, TO* __restrict__ out, size_t n) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    out[i] = from_float<TO>(to_float(in[i]));
}

// out[t, c] = in[t * ld + c], c < width: a run of columns of a wider row-major tensor, contiguous, in another type
template <typename TO>
__global__ void cast_columns_kernel(const float* __restrict__ in, long long ld, TO* __restrict__ out, int width, size_t n) {
  pdl_wait();
  pdl_trigger();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / width, c = i - t * width;
    out[i] = from_float<TO>(in[t * ld + c]);
  }
}

// out[t] += delta[t]  (float32 residual, any activation type)
template <typename TA>
__global__ void residual_add_kernel(float* __restrict__ residual, const TA* __restrict__ delta, float scale, size_t n) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    residual[i] = fmaf(scale, to_float(delta[i]), residual[i]);
}

// The stream beside the embedding, a product's input: x = residual[t] (+ scale * delta[t]), x0 = the token's row of the
// table times table_scale (or kept[t], when given).  float32: out[t] = [x | x0].  bfloat16: out[t] = [hi | lo | x0] with
// hi = x rounded and lo = the rounded rest, so that a product whose weights repeat the columns of x sees 16 bits of it.
template <typename TA, typename TW>
__global__ void stream_beside_embedding_kernel(const float* __restrict__ residual, const TA* __restrict__ delta, float scale,
                                               const int* __restrict__ ids, const TW* __restrict__ table, float table_scale,
                                               int vocab, const float* __restrict__ kept, TA* __restrict__ out, int H) {
  pdl_wait();
  pdl_trigger();
  constexpr bool kSplit = sizeof(TA) == 2;
  const size_t t = blockIdx.x;
  const int id = ids[t];
  const bool known = id >= 0 && id < vocab;           // the gather has raised the step's fault word for any other
  TA* o = out + t * H * (kSplit ? 3 : 2);
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float x = residual[t * H + i];
    if (delta) x = fmaf(scale, to_float(delta[t * H + i]), x);
    const TA hi = from_float<TA>(x);
    o[i] = hi;
    if (kSplit) o[H + i] = from_float<TA>(x - to_float(hi));
    const float x0 = kept ? kept[t * H + i] : known ? to_float(table[(size_t)id * H + i]) * table_scale : 0.f;
    o[(size_t)H * (kSplit ? 2 : 1) + i] = from_float<TA>(x0);
  }
}

// residual[t] += row, for every t
__global__ void add_row_kernel(float* __restrict__ residual, const float* __restrict__ row, int H, size_t n) {
  pdl_wait();
  pdl_trigger();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    residual[i] += row[i % H];
}

// flag[0] = 1 if any a[i] (+ b[i], when b is given) is NaN or infinite.
template <typename TB>
__global__ void check_finite_kernel(const float* __restrict__ a, const TB* __restrict__ b, size_t n,
                                    int* __restrict__ flag) {
  pdl_wait();
  pdl_trigger();
  bool bad = false;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    float x = a[i];
    if (b) x += to_float(b[i]);
    bad |= !(fabsf(x) <= 3.402823466e+38f);
  }
  if (__syncthreads_or(bad) && threadIdx.x == 0) atomicExch(flag, 1);
}

// x <- cap * tanh(x / cap), in place
__global__ void softcap_kernel(float* __restrict__ x, float cap, size_t n) {
  pdl_wait();
  pdl_trigger();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    x[i] = cap * tanhf(x[i] / cap);
}

static inline int norm_block(int H) {
  int b = 32;
  while (b < 1024 && b * 4 < H) b <<= 1;
  return b;
}
static inline int flat_grid(size_t n, int block) {
  size_t g = (n + block - 1) / block;
  return (int)(g > 148 * 16 ? 148 * 16 : (g == 0 ? 1 : g));
}

}  // namespace srlm

using namespace srlm;

extern "C" int srlm_embed_gather(const int* ids, const void* table, int table_dtype, float* out, int T,
                                 int H, int vocab, int* bad_flag, float scale, int add, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (H <= 0 || vocab <= 0) return refuse(ST_BAD_SIZE, "embed_gather: H=%d vocab=%d", H, vocab);
  const int block = H >= 1024 ? 256 : 128;
  SRLM_DISPATCH_ACT(table_dtype, TW, launch_pdl(embed_gather_kernel<TW>, dim3(T), dim3(block), 0, stream,
      ids, (const TW*)table, out, H, vocab, bad_flag, scale, add));
  return launched();
}

// center: layer norm (the row's mean is taken off first); delta_scale: a factor on delta
extern "C" int srlm_add_norm(float* residual, const void* delta, float delta_scale, const float* weight, float eps,
                             void* out, int act_dtype, const int* rows, int R, int H, int unit_offset, int center,
                             cudaStream_t stream) {
  if (R <= 0) return ST_OK;
  if (H <= 0 || !(eps > 0.f)) return refuse(ST_BAD_SIZE, "add_norm: H=%d eps=%g", H, (double)eps);
  if (act_dtype == DT_BF16 && H % 4 == 0 && H <= 4 * 4 * 1024 &&
      (((uintptr_t)residual | (uintptr_t)weight) & 15) == 0 && (((uintptr_t)delta | (uintptr_t)out) & 7) == 0) {
    // whole rows in registers: one read of the residual, vector loads and stores
    const int pieces = H / 4;
    // a thread keeps up to 4 pieces: blocks of 256 threads for rows of up to 4096 elements (several blocks
    // share an SM and their loads overlap each other's reductions), wider blocks only for wider rows
    int block = 32;
    while (block < 1024 && block * 4 < pieces) block <<= 1;
    const int per_thread = (pieces + block - 1) / block;
#define SRLM_NORM_VEC(C)                                                                                                    \
  do {                                                                                                                      \
    if (center) launch_pdl(add_norm_vec_kernel<C, true>, dim3(R), dim3(block), 0, stream, residual, (const bf16*)delta,    \
                           delta_scale, weight, eps, (bf16*)out, rows, H, unit_offset);                                    \
    else launch_pdl(add_norm_vec_kernel<C, false>, dim3(R), dim3(block), 0, stream, residual, (const bf16*)delta,          \
                    delta_scale, weight, eps, (bf16*)out, rows, H, unit_offset);                                           \
  } while (0)
    if (per_thread <= 1) SRLM_NORM_VEC(1);
    else if (per_thread <= 2) SRLM_NORM_VEC(2);
    else SRLM_NORM_VEC(4);
#undef SRLM_NORM_VEC
    return launched();
  }
  SRLM_DISPATCH_ACT(act_dtype, TA, {
    if (center) launch_pdl(add_norm_kernel<TA, true>, dim3(R), dim3(norm_block(H)), 0, stream, residual, (const TA*)delta,
                           delta_scale, weight, eps, (TA*)out, rows, H, unit_offset);
    else launch_pdl(add_norm_kernel<TA, false>, dim3(R), dim3(norm_block(H)), 0, stream, residual, (const TA*)delta,
                    delta_scale, weight, eps, (TA*)out, rows, H, unit_offset);
  });
  return launched();
}

extern "C" int srlm_swiglu(const void* in, void* out, int act_dtype, int T, int I, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (I <= 0) return refuse(ST_BAD_SIZE, "swiglu: I=%d", I);
  const size_t total = (size_t)T * I;
  SRLM_DISPATCH_ACT(act_dtype, TA, launch_pdl(swiglu_kernel<TA>, dim3(flat_grid(total, 256)), dim3(256), 0, stream,
      (const TA*)in, (TA*)out, I, total));
  return launched();
}

extern "C" int srlm_cast(const void* in, int in_dtype, void* out, int out_dtype, long long n,
                         cudaStream_t stream) {
  if (n <= 0) return ST_OK;
  const int grid = flat_grid((size_t)n, 256);
  if (in_dtype == DT_F32 && out_dtype == DT_BF16)
    cast_kernel<float, bf16><<<grid, 256, 0, stream>>>((const float*)in, (bf16*)out, (size_t)n);
  else if (in_dtype == DT_BF16 && out_dtype == DT_F32)
    cast_kernel<bf16, float><<<grid, 256, 0, stream>>>((const bf16*)in, (float*)out, (size_t)n);
  else
    return refuse(ST_BAD_DTYPE, "cast: %d -> %d is not offered", in_dtype, out_dtype);
  return launched();
}

// in: float32, the first of the wanted columns of row 0; rows ld apart; out [T, width] contiguous in out_dtype
extern "C" int srlm_cast_columns(const float* in, long long ld, void* out, int out_dtype, int T, int width,
                                 cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (width <= 0 || ld < width) return refuse(ST_BAD_SIZE, "cast_columns: width=%d ld=%lld", width, ld);
  const size_t n = (size_t)T * width;
  SRLM_DISPATCH_ACT(out_dtype, TO, launch_pdl(cast_columns_kernel<TO>, dim3(flat_grid(n, 256)), dim3(256), 0, stream, in, ld,
                                              (TO*)out, width, n));
  return launched();
}

extern "C" int srlm_residual_add(float* residual, const void* delta, int act_dtype, float scale, long long n,
                                 cudaStream_t stream) {
  if (n <= 0) return ST_OK;
  SRLM_DISPATCH_ACT(act_dtype, TA, (residual_add_kernel<TA><<<flat_grid((size_t)n, 256), 256, 0, stream>>>(
      residual, (const TA*)delta, scale, (size_t)n)));
  return launched();
}

// delta (act_dtype) or null; table [vocab, H] (float32 or bfloat16), not read when kept (float32 [T, H]) is given; out
// [T, 2 H] in float32 or [T, 3 H] in bfloat16
extern "C" int srlm_stream_beside_embedding(const float* residual, const void* delta, float scale, const int* ids,
                                            const void* table, int table_dtype, float table_scale, int vocab,
                                            const float* kept, void* out, int act_dtype, int T, int H, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (H <= 0 || vocab <= 0) return refuse(ST_BAD_SIZE, "stream_beside_embedding: H=%d vocab=%d", H, vocab);
  SRLM_DISPATCH_ACT(act_dtype, TA, SRLM_DISPATCH_ACT(table_dtype, TW, launch_pdl(stream_beside_embedding_kernel<TA, TW>,
      dim3(T), dim3(H >= 1024 ? 256 : 128), 0, stream, residual, (const TA*)delta, scale, ids, (const TW*)table, table_scale,
      vocab, kept, (TA*)out, H)));
  return launched();
}

extern "C" int srlm_add_row(float* residual, const float* row, int T, int H, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (H <= 0) return refuse(ST_BAD_SIZE, "add_row: H=%d", H);
  const size_t n = (size_t)T * H;
  launch_pdl(add_row_kernel, dim3(flat_grid(n, 256)), dim3(256), 0, stream, residual, row, H, n);
  return launched();
}

// words[pairs[2 i]] = src[pairs[2 i + 1]] for i < n: token ids that a step takes from what the step before
// it sampled, while the host has not read them yet.  A source index outside [0, src_len) or a destination
// outside [0, words_len) is skipped and raises the flag (the host checks too).
extern "C" int srlm_patch_words(int* words, long long words_len, const int* pairs, const int* src, int src_len,
                                int n, int* flag, cudaStream_t stream) {
  if (n <= 0) return ST_OK;
  if (!words || !pairs || !src || !flag) return refuse(ST_BAD_SIZE, "patch_words: a null argument");
  launch_pdl(patch_words_kernel, dim3((n + 127) / 128), dim3(128), 0, stream, words, words_len, pairs, src, src_len,
             n, flag);
  return launched();
}

// The non-finite test of a step (src/model/native.rs:276-278, 292-294): a [n] float32, b [n] of the
// activation dtype or null; flag[0] becomes 1 if any a[i] + b[i] is NaN or infinite.
extern "C" int srlm_check_finite(const float* a, const void* b, int b_dtype, long long n, int* flag,
                                 cudaStream_t stream) {
  if (n <= 0) return ST_OK;
  if (!flag) return refuse(ST_BAD_SIZE, "check_finite: no flag");
  const int grid = flat_grid((size_t)n, 256);
  SRLM_DISPATCH_ACT(b_dtype, TB, launch_pdl(check_finite_kernel<TB>, dim3(grid), dim3(256), 0, stream,
      a, (const TB*)b, (size_t)n, flag));
  return launched();
}

// Logits bounded by a smooth cap: x <- cap * tanh(x / cap), float32 in place.
extern "C" int srlm_softcap(float* x, float cap, long long n, cudaStream_t stream) {
  if (n <= 0) return ST_OK;
  if (!(cap > 0.f)) return refuse(ST_BAD_SIZE, "softcap: cap=%g", (double)cap);
  launch_pdl(softcap_kernel, dim3(flat_grid((size_t)n, 256)), dim3(256), 0, stream, x, cap, (size_t)n);
  return launched();
}
