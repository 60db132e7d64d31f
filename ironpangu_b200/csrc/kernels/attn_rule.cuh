// What the softmax attention kernels over pages share besides the products: which keys a query sees, and what happens to a score
// between the product and the softmax.
//
//   mask    the last `size` positions (0: all), or with `chunked` the positions of the query's own stretch of `size`, counted from
//           position 0 of the sequence
//   ahead   entries that a windowed query sees beside its window, in the same softmax: of the positions before the window's first the first `keep` ones,
//           or the blocks of `pool` positions (from position 0 on) that lie wholly there, one key and value each: the means of theirs.
//           A block's entry lives in the page of its last position, [pages, ceil(page_tokens / pool), G, .]
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

struct AheadRule {
  int keep, pool;          // at most one of them above 0
  const void *k, *v;       // pool: the entries' keys and values
  int per_page;            // pool: entries a page has room for
  __host__ __device__ bool any() const { return keep > 0 || pool > 0; }
  // entries that a query sees whose window starts at position `first`: 0 .. count - 1
  __host__ __device__ __forceinline__ int count(int first) const { return keep > 0 ? (first < keep ? first : keep) : pool > 0 ? first / pool : 0; }
  // position whose page holds entry i, and its row there
  __host__ __device__ __forceinline__ int position(int i) const { return pool > 0 ? i * pool + pool - 1 : i; }
  __host__ __device__ __forceinline__ int row(int i, int page_tokens) const { return pool > 0 ? i - position(i) / page_tokens * page_tokens / pool : i % page_tokens; }
  __host__ __device__ __forceinline__ int rows(int page_tokens) const { return pool > 0 ? per_page : page_tokens; }
};
__host__ __forceinline__ AheadRule ahead_rule(int keep, int pool, const void* k, const void* v, int page_tokens) {
  return {keep, pool, k, v, pool > 0 ? (page_tokens + pool - 1) / pool : 0};
}
__host__ __forceinline__ bool ahead_ok(const AheadRule& a, int window, int chunked) {
  return a.keep >= 0 && a.pool >= 0 && (!a.any() || (window > 0 && !chunked && !(a.keep && a.pool) && (!a.pool || (a.k && a.v))));
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
