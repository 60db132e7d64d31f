// Shared by the kernels of recurrences with a decay per token (gated_recurrence.cu, gated_delta.cu, gated_tiles.cu).
#pragma once
#include "rope.cuh"
#include "ifab_kernels.h"

namespace ifab {

enum { GR_SSD = 0, GR_DELTA = 1, GR_MEMORY = 2 };
constexpr int GR_CHUNK = 64;      // rows of a chunk of the f32 form
constexpr int GR_TILE = 128;      // of the tensor-core form

// Operands of a step's rows, as gr_prepare_kernel leaves them: q, k [T, G, d] and v [T, H, e] in the activation type (head h reads q / k head h / (H / G)), factors
// of the rows of q and k [T, G] (null: q_factor and 1), log_decay [T, H], weight [T, H] (a factor, null: 1; MEMORY: the log of it), m [T, H]
// (MEMORY, chunks: the running maximum, made by gr_maximum_kernel). E value columns in the state: e, and for MEMORY one more that is always 1.
struct GrRows {
  const void *q, *k, *v;
  const float *qs, *ks; float q_factor;
  const float *log_decay, *weight;
  float* m;
  int kind, H, G, d, e, E;
};

template <typename A>
__device__ __forceinline__ float gr_q(const GrRows& r, long t, int g, int c) {
  const float f = r.qs ? r.qs[t * r.G + g] : r.q_factor;
  return to_f32(reinterpret_cast<const A*>(r.q)[(t * r.G + g) * r.d + c]) * f;
}
template <typename A>
__device__ __forceinline__ float gr_k(const GrRows& r, long t, int g, int c) {
  const float v = to_f32(reinterpret_cast<const A*>(r.k)[(t * r.G + g) * r.d + c]);
  return r.ks ? v * r.ks[t * r.G + g] : v;
}
template <typename A>
__device__ __forceinline__ float gr_v(const GrRows& r, long t, int h, int c) {
  return c < r.e ? to_f32(reinterpret_cast<const A*>(r.v)[(t * r.H + h) * r.e + c]) : 1.f;
}

// State [slots, H, E, d]; MEMORY: m_state [slots, 2, H] by epoch sides
struct GrState {
  float *s, *m;
  const int32_t* epoch;
};

struct GrChunks {
  GrRows r;
  const int32_t* chunks;      // [n, 4]: first row, rows, slot, 2 * chunks of the run + 1 at the first chunk of a run
  int n;
  const int32_t* positions;
  float* cstate;              // [n, H, E, d]: what a chunk adds, then the state ahead of it
  float* cdecay;              // [n, H]
  float* o; long ldo;         // [T, H * E]
};

// The factors of a chunk's rows in shared memory. `total`: log decays summed up to and with each row (double: differences of large sums), `off`: what the
// running maximum takes off the row, start: off of the row ahead of the chunk
template <int N>
struct GrFactors {
  double total[N];
  float off[N], lw[N], w[N];
  double start;
};

// call with the whole CTA (at least N threads); ends with a barrier
template <int N>
__device__ __forceinline__ void gr_load_factors(const GrChunks& p, int c, int h, const GrState& st, GrFactors<N>& f) {
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1], slot = p.chunks[c * 4 + 2], j = threadIdx.x;
  const GrRows& r = p.r;
  if (j < N) {
    const bool live = j < L;
    const long at = (long)(row0 + (live ? j : 0)) * r.H + h;
    f.total[j] = live ? (double)r.log_decay[at] : 0.0;
    f.off[j] = live && r.kind == GR_MEMORY ? r.m[at] : 0.f;
    f.lw[j] = live && r.kind == GR_MEMORY ? r.weight[at] : 0.f;
    f.w[j] = !live ? 0.f : r.kind == GR_MEMORY || !r.weight ? 1.f : r.weight[at];
    if (j == 0) {
      float s = 0.f;
      if (r.kind == GR_MEMORY && p.positions[row0] != 0)
        s = (p.chunks[c * 4 + 3] & 1) ? st.m[((long)slot * 2 + (st.epoch[slot] & 1)) * r.H + h] : r.m[at - r.H];      // a run's later chunks start behind their own row
      f.start = (double)s;
    }
  }
  __syncthreads();
  if (j < 32) {      // running sums, some rows per lane
    constexpr int R = N / 32;
    double a[R], v = 0.0;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      v += f.total[R * j + i];
      a[i] = v;
    }
    double before = v;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double n = __shfl_up_sync(0xffffffffu, before, o);
      if (j >= o) before += n;
    }
    before -= v;
#pragma unroll
    for (int i = 0; i < R; ++i) f.total[R * j + i] = before + a[i];
  }
  __syncthreads();
}

// weight of row j's write as row i sees it (j <= i), of the state ahead of the chunk as row i sees it
template <int N>
__device__ __forceinline__ float gr_pair(const GrFactors<N>& f, int i, int j) {
  return expf((float)(f.total[i] - f.total[j] + (double)f.lw[j] - (double)f.off[i])) * f.w[j];
}
template <int N>
__device__ __forceinline__ float gr_carry(const GrFactors<N>& f, int i) { return expf((float)(f.total[i] + f.start - (double)f.off[i])); }

// gated_recurrence.cu: the running maximum of every row; the states ahead of every chunk from what the chunks add
int gr_maximum(const GrChunks& p, const GrState& st, cudaStream_t s);
int gr_scan(const GrChunks& p, const GrState& st, cudaStream_t s);
// gated_delta.cu: corrected values u_rows [T, H, e] of every row, and the states ahead of every chunk
int gr_delta_chunks(const GrChunks& p, const GrState& st, int f32, float* w_rows, float* u_rows, cudaStream_t s);

}  // namespace ifab
