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

// A warp of a grouped walk holds four columns of S: L lanes a set of L / 8 columns, lane hl of the set the rows
// 4 hl + 4 L j + {0..3}.  More lanes a column mean fewer bytes of shared memory a product (a lane's row pieces serve L / 8
// columns), fewer lanes mean fewer exchanges a sum.
//
// Lane hl finishes token hl & 7 of the set's column hl >> 3.  It keeps its columns in slots, slot c for column
// c ^ (hl >> 3), and forms a group's sums in slots of tokens, slot i for token i ^ (hl & 7): then the half of the sums
// that a lane gives away in an exchange always lies in the upper slots (permuted_sums), and no value is selected by lane.
template <int ROWS, int L>
struct StateTile {
  static constexpr int kColumns = L / kStateLanes;          // a lane's columns
  static constexpr int kPieces = ROWS / (4 * L);            // a lane's pieces of four rows
  static_assert(L >= 8 && L <= 32 && kPieces * 4 * L == ROWS, "whole pieces");
  float2 s[kColumns][2 * kPieces];

  __device__ __forceinline__ void load(const float* head, int first, int columns, int hl, int rows, bool vec) {
#pragma unroll
    for (int c = 0; c < kColumns; ++c)
#pragma unroll
      for (int j = 0; j < kPieces; ++j) {
        const int r = 4 * hl + 4 * L * j, col = first + (c ^ (hl >> 3));
        const float* at = head + (size_t)col * rows + r;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (col < columns) {
          if (vec) {
            if (r < rows) v = *reinterpret_cast<const float4*>(at);
          } else {
            if (r < rows) v.x = at[0];
            if (r + 1 < rows) v.y = at[1];
            if (r + 2 < rows) v.z = at[2];
            if (r + 3 < rows) v.w = at[3];
          }
        }
        s[c][2 * j] = make_float2(v.x, v.y);
        s[c][2 * j + 1] = make_float2(v.z, v.w);
      }
  }
  __device__ __forceinline__ void store(float* head, int first, int columns, int hl, int rows, bool vec) const {
#pragma unroll
    for (int c = 0; c < kColumns; ++c)
#pragma unroll
      for (int j = 0; j < kPieces; ++j) {
        const int r = 4 * hl + 4 * L * j, col = first + (c ^ (hl >> 3));
        float* at = head + (size_t)col * rows + r;
        if (col >= columns) continue;
        const float2 a = s[c][2 * j], b = s[c][2 * j + 1];
        if (vec) {
          if (r < rows) *reinterpret_cast<float4*>(at) = make_float4(a.x, a.y, b.x, b.y);
        } else {
          if (r < rows) at[0] = a.x;
          if (r + 1 < rows) at[1] = a.y;
          if (r + 2 < rows) at[2] = b.x;
          if (r + 3 < rows) at[3] = b.y;
        }
      }
  }
  // The lane's share of x . S[:, c] for its columns; x: where its first piece of a vector over the rows lies in shared memory.
  __device__ __forceinline__ void dot(const float* x, float (&out)[kColumns]) const {
    float2 acc[kColumns];
#pragma unroll
    for (int j = 0; j < kPieces; ++j) {
      const float4 v = *reinterpret_cast<const float4*>(x + 4 * L * j);
      const float2 lo = make_float2(v.x, v.y), hi = make_float2(v.z, v.w);
#pragma unroll
      for (int c = 0; c < kColumns; ++c) {
        acc[c] = fma2(lo, s[c][2 * j], j == 0 ? make_float2(0.f, 0.f) : acc[c]);
        acc[c] = fma2(hi, s[c][2 * j + 1], acc[c]);
      }
    }
#pragma unroll
    for (int c = 0; c < kColumns; ++c) out[c] = acc[c].x + acc[c].y;
  }
  // S[:, c] += x u[c]
  __device__ __forceinline__ void add(const float* x, const float (&u)[kColumns]) {
#pragma unroll
    for (int j = 0; j < kPieces; ++j) {
      const float4 v = *reinterpret_cast<const float4*>(x + 4 * L * j);
      const float2 lo = make_float2(v.x, v.y), hi = make_float2(v.z, v.w);
#pragma unroll
      for (int c = 0; c < kColumns; ++c) {
        const float2 uu = make_float2(u[c], u[c]);
        s[c][2 * j] = fma2(lo, uu, s[c][2 * j]);
        s[c][2 * j + 1] = fma2(hi, uu, s[c][2 * j + 1]);
      }
    }
  }

  // A number a (token, column) to all lanes of the column's set, by way of shared memory (32 kColumns floats a warp; a
  // __syncwarp between share and shared): every lane reads its columns in the order of its slots.
  static __device__ __forceinline__ void share(float* buf, int set, int hl, float u) {
#pragma unroll
    for (int x = 0; x < kColumns; ++x)
      buf[((set * kColumns + x) * kStateGroup + (hl & 7)) * kColumns + ((hl >> 3) ^ x)] = u;
  }
  static __device__ __forceinline__ void shared(const float* buf, int set, int hl, int token, float (&u)[kColumns]) {
    const float* at = buf + ((set * kColumns + (hl >> 3)) * kStateGroup + token) * kColumns;
    if (kColumns == 4) *reinterpret_cast<float4*>(u) = *reinterpret_cast<const float4*>(at);
    else if (kColumns == 2) *reinterpret_cast<float2*>(u) = *reinterpret_cast<const float2*>(at);
    else u[0] = at[0];
  }
};

// N values a lane in permuted slots (see StateTile), summed over the L lanes of its set: the first N / L values of lane hl
// are the sums of its own column and token.
template <int N, int L>
__device__ __forceinline__ void permuted_sums(float (&p)[N]) {
  static_assert(N >= L, "at least one sum a lane");
  int half = N / 2;
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1, half >>= 1) {
#pragma unroll
    for (int s = 0; s < N / 2; ++s) {
      if (s >= half) break;
      p[s] += __shfl_xor_sync(0xffffffffu, p[s + half], o);
    }
  }
}

// N values a lane, summed over the L lanes of its set (N >= L); afterwards lane hl's first N / L values are the sums
// numbered hl * (N / L) onwards.
template <int N, int L>
__device__ __forceinline__ void scatter_sums(float (&p)[N], int hl) {
  static_assert(N >= L, "at least one sum a lane");
  int half = N / 2;
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1, half >>= 1) {
    const bool up = hl & o;
#pragma unroll
    for (int s = 0; s < N / 2; ++s) {
      if (s >= half) break;
      const float keep = up ? p[s + half] : p[s], give = up ? p[s] : p[s + half];
      p[s] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
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
