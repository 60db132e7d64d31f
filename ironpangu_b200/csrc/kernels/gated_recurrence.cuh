// Shared by the kernels of recurrences with a decay per token (gated_recurrence.cu, gated_delta.cu).
#pragma once
#include "rope.cuh"
#include "ifab_kernels.h"

namespace ifab {

enum { GR_SSD = 0, GR_DELTA = 1, GR_MEMORY = 2 };
constexpr int GR_CHUNK = 64;      // rows of a chunk

// Operands of a step's rows: q, k [T, G, d] and v [T, H, E] in f32 (head h reads q / k head h / (H / G)), log_decay [T, H], weight [T, H]
// (a factor, null: 1; MEMORY: the log of it), m [T, H] (MEMORY, chunks: the running maximum, made by gr_maximum_kernel)
struct GrRows {
  const float *q, *k, *v, *log_decay, *weight;
  float* m;
  int kind, H, G, d, E;
};

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
struct GrFactors {
  double total[GR_CHUNK];
  float off[GR_CHUNK], lw[GR_CHUNK], w[GR_CHUNK];
  double start;
};

// call with the whole CTA (at least 64 threads); ends with a barrier
__device__ __forceinline__ void gr_load_factors(const GrChunks& p, int c, int h, const GrState& st, GrFactors& f) {
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1], slot = p.chunks[c * 4 + 2], j = threadIdx.x;
  const GrRows& r = p.r;
  if (j < GR_CHUNK) {
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
  if (j < 32) {      // running sums, two rows per lane
    const double a = f.total[2 * j], b = f.total[2 * j + 1];
    double v = a + b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double n = __shfl_up_sync(0xffffffffu, v, o);
      if (j >= o) v += n;
    }
    f.total[2 * j] = v - b;
    f.total[2 * j + 1] = v;
  }
  __syncthreads();
}

// weight of row j's write as row i sees it (j <= i), of the state ahead of the chunk as row i sees it, of the latter for the state behind
// the chunk's L rows, and of row j there
__device__ __forceinline__ float gr_pair(const GrFactors& f, int i, int j) { return expf((float)(f.total[i] - f.total[j] + (double)f.lw[j] - (double)f.off[i])) * f.w[j]; }
__device__ __forceinline__ float gr_carry(const GrFactors& f, int i) { return expf((float)(f.total[i] + f.start - (double)f.off[i])); }
__device__ __forceinline__ float gr_add(const GrFactors& f, int L, int j) { return gr_pair(f, L - 1, j); }

// gated_delta.cu: corrected values of every row, in place of v, and the states ahead of every chunk
int gr_delta_chunks(const GrChunks& p, const GrState& st, float* w_rows, float* u_rows, cudaStream_t s);

}  // namespace ifab
