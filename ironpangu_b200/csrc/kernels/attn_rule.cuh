// What the softmax attention kernels over pages share besides the products: which keys a query sees, and what happens to a score
// between the product and the softmax.
//
//   mask    the last `size` positions (0: all), or with `chunked` the positions of the query's own stretch of `size`, counted from
//           position 0 of the sequence
//   score   s = q k scale; with a cap s = cap tanh(s / cap); with slopes s -= slope_h (distance of the key)
#pragma once
#include "common.cuh"

namespace ifab {

struct ScoreRule {
  float cap;               // 0: none
  const float* slopes;     // [H], or null
  int chunked;
  __host__ __device__ bool plain() const { return cap == 0.f && !slopes; }
};

__host__ __device__ __forceinline__ int first_key(int pos, int size, int chunked) {
  if (size <= 0) return 0;
  if (chunked) return pos / size * size;
  return pos + 1 > size ? pos + 1 - size : 0;
}

// cap tanh(z / cap). FAST: through the hardware exponential, absolute error below 1e-6 cap
template <bool FAST = false>
__device__ __forceinline__ float soft_limit(float z, float cap) {
  return FAST ? cap - __fdividef(2.f * cap, 1.f + __expf(z * (2.f / cap))) : cap * tanhf(z / cap);
}

template <bool FAST>
__device__ __forceinline__ float ruled_score(float s, const ScoreRule& r, float slope, int distance) {
  if (r.cap > 0.f) s = soft_limit<FAST>(s, r.cap);
  return s - slope * (float)distance;
}

}  // namespace ifab
