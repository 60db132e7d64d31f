// Parameters shared by the linear-attention kernels (linear_attn.cu, linear_attn_tc.cu).
#pragma once
#include "rope.cuh"
#include "ifab_kernels.h"

namespace ifab {

constexpr int LA_POW = 129;      // entries of the decay table per head: decay^0 .. decay^128

struct LaParams {
  const void* proj; long ldp;
  int q_off, k_off, v_off;       // columns of the packed projection
  int H, d, e;
  RopeTable rope;                // of q and k (rot 0: none)
  int act;                       // activation of q, k (columns past the rotation) and v
  float k_scale;
  const float* powers;           // [H, LA_POW]: decay^n
  float* state;                  // [slots, H, e, d]
  const int32_t* positions; const int32_t* slots;
  int T;
};

// an activated value is a value of the activation type, whichever kernel computes it
template <typename A>
__device__ __forceinline__ float activated(const LaParams& p, A v) {
  return p.act ? to_f32(from_f32<A>(activate<sizeof(A) == 2>(to_f32(v), p.act))) : to_f32(v);
}

// states ahead of every chunk, in place of what the chunks add (linear_attn.cu)
int la_scan(float* cstate, float* state, const int32_t* chunks, int n, const int32_t* positions, const float* powers, int H, int d, int e, cudaStream_t s);

}  // namespace ifab
