// What a product may do with an element of its result before it is rounded and stored (`post` of the C interface):
//   0 nothing
//   1 gelu in its exact form, x * Phi(x) = x / 2 * (1 + erf(x / sqrt 2))          (a feed-forward without a gate)
//   2 a cap, c * tanh(x / c)                                                      (capped logits)
// All in 32-bit.
#pragma once

#include "common.cuh"

namespace lb {

enum PostOp : int { POST_NONE = 0, POST_GELU = 1, POST_CAP = 2 };

__device__ __forceinline__ float gelu_erf(float x) { return 0.5f * x * (1.f + erff(x * 0.7071067811865476f)); }

__device__ __forceinline__ float post_op(int post, float c, float x) {
  if (post == POST_GELU) return gelu_erf(x);
  if (post == POST_CAP) return c * tanhf(x / c);
  return x;
}

inline bool valid_post(int post, float c) { return post == POST_NONE || post == POST_GELU || (post == POST_CAP && c > 0.f); }

}  // namespace lb
