// What the forms of the mixed-head attention share: the mask, the bias by distance, the gate per element.
#pragma once

#include "common.cuh"

namespace srlm {

// A query sees itself, the window - 1 keys before it and the sequence's first `keep` tokens (window 0: every earlier key).
struct MixMask {
  int window, keep;
  __device__ __forceinline__ int first_key(int pos) const { return window > 0 && pos >= window ? pos - window + 1 : 0; }
  __device__ __forceinline__ bool visible(int pos, int j) const {
    return j <= pos && (window <= 0 || pos - j < window || j < keep);
  }
};

// table float32 [heads, n]: the bias of a distance; distances from n - 1 on share the last one.  table null: none.
struct DistanceBias {
  const float* table;
  int n;
  __device__ __forceinline__ const float* of(int head, int distance) const {
    return table + (size_t)head * n + (distance < n ? distance : n - 1);
  }
  __device__ __forceinline__ float at(int head, int distance) const { return table ? *of(head, distance) : 0.f; }
};

// Element c (head * dv + d) of token t is multiplied by logistic(logits[t * ld + c]); logits null: no gate.
struct ElementGate {
  const float* logits;
  long long ld;
  __device__ __forceinline__ float at(size_t token, int c) const {
    return logits ? 1.f / (1.f + expf(-logits[token * ld + c])) : 1.f;
  }
};

}  // namespace srlm
