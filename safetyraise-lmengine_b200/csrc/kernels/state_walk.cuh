// What the walks over a matrix of recurrent state share (channel_delta.cu, state_space.cu).
//
// A head's state S [rows, columns] lies column by column in the request's slot ([column][row] floats).  Eight lanes hold
// one column in registers, lane l the rows 32 j + 4 l + {0..3}; so a vector over the rows is read from shared memory 16
// bytes a lane, and a sum over the rows is three exchanges.
#pragma once

#include "common.cuh"

namespace srlm {

constexpr int kStateLanes = 8;        // lanes that share a column of the state
constexpr int kStateGroup = 8;        // tokens that a grouped walk takes at a time: lane l finishes token l

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(d)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)),
        "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&d);
}

__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float logistic_f(float z) { return 1.f / (1.f + expf(-z)); }

__device__ __forceinline__ void state_copy_16(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src));
}
__device__ __forceinline__ void state_copy_4(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src));
}
__device__ __forceinline__ void state_copy_commit() { asm volatile("cp.async.commit_group;" ::); }
template <int N> __device__ __forceinline__ void state_copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }

// One column of S to and from a lane's registers.  vec: the columns start on 16 bytes and rows % 4 == 0.
template <int RPL>
__device__ __forceinline__ void load_column(float (&S)[RPL], const float* column, int l, int rows, bool live, bool vec) {
#pragma unroll
  for (int j = 0; j < RPL / 4; ++j) {
    const int r = 32 * j + 4 * l;
    if (vec) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && r < rows) v = *reinterpret_cast<const float4*>(column + r);
      S[4 * j] = v.x; S[4 * j + 1] = v.y; S[4 * j + 2] = v.z; S[4 * j + 3] = v.w;
    } else {
#pragma unroll
      for (int x = 0; x < 4; ++x) S[4 * j + x] = live && r + x < rows ? column[r + x] : 0.f;
    }
  }
}
template <int RPL>
__device__ __forceinline__ void store_column(const float (&S)[RPL], float* column, int l, int rows, bool live, bool vec) {
  if (!live) return;
#pragma unroll
  for (int j = 0; j < RPL / 4; ++j) {
    const int r = 32 * j + 4 * l;
    if (vec) {
      if (r < rows) *reinterpret_cast<float4*>(column + r) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
    } else {
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (r + x < rows) column[r + x] = S[4 * j + x];
    }
  }
}

// p[0..7]: a lane's share of eight sums over the 8 lanes of a column; returns sum number l to lane l.
__device__ __forceinline__ float scatter_sums_8(const float (&p)[kStateGroup], int l) {
  float a[4], b[2];
#pragma unroll
  for (int s = 0; s < 4; ++s) {
    const float keep = l & 4 ? p[s + 4] : p[s], give = l & 4 ? p[s] : p[s + 4];
    a[s] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
  }
#pragma unroll
  for (int s = 0; s < 2; ++s) {
    const float keep = l & 2 ? a[s + 2] : a[s], give = l & 2 ? a[s] : a[s + 2];
    b[s] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
  }
  const float keep = l & 1 ? b[1] : b[0], give = l & 1 ? b[0] : b[1];
  return keep + __shfl_xor_sync(0xffffffffu, give, 1);
}

// Sums 2^k values over the 32 lanes of a warp; afterwards lane's first N / 32 values are the sums numbered
// [first, first + N / 32), first = the return value.
template <int N>
__device__ __forceinline__ int scatter_sums_warp(float (&p)[N], int lane) {
  static_assert(N >= 32, "at least one sum a lane");
  int first = 0;
#pragma unroll
  for (int o = 16, half = N / 2; o > 0; o >>= 1, half >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int s = 0; s < N / 2; ++s) {
      if (s >= half) break;
      const float keep = up ? p[s + half] : p[s], give = up ? p[s] : p[s + half];
      p[s] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
    if (up) first += half;
  }
  return first;
}

// The groups of a step: every entry's tokens in groups of kStateGroup, numbered along the entries.
struct GroupHome {
  int entry, t0, n;
};
__device__ __forceinline__ GroupHome group_home(const int* __restrict__ cu_q, int n_entries, int index) {
  int base = 0;
  for (int e = 0; e < n_entries; ++e) {
    const int a = cu_q[e], len = cu_q[e + 1] - a;
    const int groups = (len + kStateGroup - 1) / kStateGroup;
    if (index < base + groups) {
      const int at = (index - base) * kStateGroup;
      return GroupHome{e, a + at, min(kStateGroup, len - at)};
    }
    base += groups;
  }
  return GroupHome{-1, 0, 0};
}
__device__ __forceinline__ int first_group(const int* __restrict__ cu_q, int entry) {
  int base = 0;
  for (int e = 0; e < entry; ++e) base += (cu_q[e + 1] - cu_q[e] + kStateGroup - 1) / kStateGroup;
  return base;
}

// The inputs of a short causal convolution over time (short_conv.cu has the layout of the carried ones).
struct ConvInput {
  const float* proj;        // [T, ld], the channels' columns start at proj
  long long ld;
  const float* in_bias;     // [C] or null: added to every input of the step (the carried ones hold it already)
  const float* state;       // [slots, state_stride]
  long long state_stride;
  int state_off;
  int taps, C;
};

// The convolution of channel c at token t, which is token `idx` of its entry's portion.
__device__ __forceinline__ float conv_at(const ConvInput& in, const float* __restrict__ w, int t, int idx, int slot, int c) {
  float acc = 0.f;
  const float bias = in.in_bias ? in.in_bias[c] : 0.f;
  for (int j = 0; j < in.taps; ++j) {
    const int back = in.taps - 1 - j;
    float u;
    if (back <= idx) u = in.proj[(size_t)(t - back) * in.ld + c] + bias;
    else u = in.state[(size_t)slot * in.state_stride + in.state_off + (size_t)(in.taps - 1 - (back - idx)) * in.C + c];
    acc = fmaf(w[(size_t)c * in.taps + j], u, acc);
  }
  return acc;
}
__device__ __forceinline__ float silu_of(float y) { return y / (1.f + expf(-y)); }

}  // namespace srlm
