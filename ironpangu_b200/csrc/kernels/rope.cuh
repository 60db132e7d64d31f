// Rotation angles in full precision for any pair layout: the angle position * frequency is formed and reduced in double (the
// frequencies come as doubles), so cos / sin are exact to float rounding at every position.
#pragma once
#include "common.cuh"

namespace ifab {

__device__ __forceinline__ void rope_angle(int pos, double freq, float* c, float* s) {
  double a = (double)pos * freq;
  a -= 6.283185307179586 * rint(a * 0.15915494309189535);
  sincosf((float)a, s, c);
}

// (cos, sin) of pair i for a row of the step: tables float2 [rows, pairs] made once per step (ifab_rope_table)
struct RopeTable {
  const float2* cs;      // [rows, rot / 2]
  int rot, interleaved;  // rotated columns of a head (0: none), pair layout
};

// columns of pair i among the first `rot` columns of a head: (i, i + rot / 2), or (2 i, 2 i + 1) when interleaved
__device__ __forceinline__ void rope_pair(int i, int rot, int interleaved, int* a, int* b) {
  *a = interleaved ? 2 * i : i;
  *b = interleaved ? 2 * i + 1 : i + rot / 2;
}

// activations and caches exist in bf16 (serving) and f32 (exact mode): loads and stores by type
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename A>
__device__ __forceinline__ A from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// rotated value of column c of a head (`head[c']` holds the plain values); columns from rt.rot on pass
template <typename A>
__device__ __forceinline__ float rotated(const RopeTable& rt, const float2* row_cs, const A* head, int c) {
  const int i = rt.interleaved ? c >> 1 : (c < rt.rot / 2 ? c : c - rt.rot / 2);
  int ia, ib;
  rope_pair(i, rt.rot, rt.interleaved, &ia, &ib);
  const float2 t = row_cs[i];
  const float a = to_f32(head[ia]), b = to_f32(head[ib]);
  return c == ia ? a * t.x - b * t.y : b * t.x + a * t.y;
}

// FAST: for results that are rounded to bf16 (the hardware exponential, ~1e-6 relative); GELU's 0.5 (1 + tanh u) is sigmoid(2 u)
template <bool FAST = false>
__device__ __forceinline__ float sigmoid_f32(float x) {
  return FAST ? __fdividef(1.f, 1.f + __expf(-x)) : 1.f / (1.f + expf(-x));      // __fdividef gives 0 for a huge divisor: the limit
}
template <bool FAST = false>
__device__ __forceinline__ float gelu_tanh_f32(float z) { return z * sigmoid_f32<FAST>(1.5957691216057308f * (z + 0.044715f * z * z * z)); }

// 0.5 z (1 + erf(z / sqrt 2)) = z - 0.5 z erfc(z / sqrt 2). FAST: erfc by formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions
// (absolute error below 1.5e-7)
template <bool FAST = false>
__device__ __forceinline__ float gelu_erf_f32(float z) {
  if (!FAST) return 0.5f * z * erfcf(-0.70710678118654752f * z);
  const float x = 0.70710678118654752f * fabsf(z), t = __fdividef(1.f, fmaf(0.3275911f, x, 1.f));
  const float c = t * (0.254829592f + t * (-0.284496736f + t * (1.421413741f + t * (-1.453152027f + t * 1.061405429f)))) * __expf(-x * x);
  return fmaxf(z, 0.f) - 0.5f * fabsf(z) * c;
}

// elementwise activations by number: 0 none, 1 SiLU, 2 sigmoid, 3 GELU (tanh form), 4 GELU (erf form)
template <bool FAST = false>
__device__ __forceinline__ float activate(float z, int act) {
  switch (act) {
    case 1: return z * sigmoid_f32<FAST>(z);
    case 2: return sigmoid_f32<FAST>(z);
    case 3: return gelu_tanh_f32<FAST>(z);
    case 4: return gelu_erf_f32<FAST>(z);
    default: return z;
  }
}

// What a gated feed-forward makes of its two projections: 0 silu(g) u, 1 relu(g) u, 2 g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit) and
// u' = u within [-limit, limit]
struct GatedUnit {
  int kind;
  float limit, alpha;
};
template <bool FAST = false>
__device__ __forceinline__ float gated_value(float g, float u, const GatedUnit& unit) {
  if (unit.kind == 1) return fmaxf(g, 0.f) * u;
  if (unit.kind == 2) {
    g = fminf(g, unit.limit);
    return g * sigmoid_f32<FAST>(unit.alpha * g) * (fminf(fmaxf(u, -unit.limit), unit.limit) + 1.f);
  }
  return g * sigmoid_f32<FAST>(g) * u;
}
// the same of projections that count as bf16 rows for SiLU units (the form of the kernels that store them)
__device__ __forceinline__ float gated_bf16(float g, float u, const GatedUnit& unit) {
  if (unit.kind) return gated_value<true>(g, u, unit);
  g = bf16_round(g);
  return g / (1.f + __expf(-g)) * bf16_round(u);
}
__host__ __forceinline__ bool gated_ok(const GatedUnit& u) { return u.kind >= 0 && u.kind <= 2 && (u.kind != 2 || u.limit > 0.f); }

// sum over the block (blockDim.x a multiple of 32, at most 1024); `red` holds 33 floats; every thread gets the sum
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < n; ++i) s += red[i];
  return s;
}

}  // namespace ifab
