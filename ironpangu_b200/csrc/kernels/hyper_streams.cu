// Residual streams side by side (hyper-connections with fixed mixing weights) around sublayers that read a norm and a causal convolution:
//
//   u = sum_s in[s] x_s,   h = u / rms(u) * gain,   operand = h + conv(h),   y = sublayer(operand),   x_t <- sum_s mix[s, t] x_s + out[t] y
//
//   embed_norm_kernel    rows of the embedding table divided by their rms, times one number (f32)
//   streams_rows_kernel  the end of one sublayer and the front of the next in one pass over the streams: x_out from x_in and y, then u, its
//                        norm, the convolution and the operand of the next linears. A CTA takes `block` consecutive rows and recomputes h
//                        of the few rows ahead of them that the convolution reaches (x_out must not be x_in); the last taps - 1
//                        values of h before a step come from the sequence's history
//   streams_tile_kernel  the same for steps of many rows: a warp per row up to the norm, then a thread per column group down the rows
//
// History [slots, 2, taps - 1, width] f32, newest first, two sides per slot: a step reads the side `epoch[slot]` names and writes the other
// (ifab_step_epoch turns the epochs over once per step), so rows of a step may be worked on in any order.
//
// Streams are f32 [T, streams, width] at given strides (stream stride 0: all streams are the same row, as after the embedding). With
// S = 1 and unit weights this is a plain residual.
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

constexpr int MAX_S = 16, MAX_TAPS = 16, THREADS = 256;

template <typename A>
__global__ void __launch_bounds__(THREADS) embed_norm_kernel(const int32_t* ids, const A* table, long ldt, const float* gain, float eps, float* x, long ldx, int D,
                                                             int vocab, uint32_t* status) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0 && status) atomicOr(status, IFAB_STATUS_BAD_INDEX);
    id = 0;
  }
  const A* r = table + (long)id * ldt;
  float ss = 0.f;
  for (int c = threadIdx.x; c < D; c += THREADS) {
    const float v = to_f32(r[c]);
    ss += v * v;
  }
  const float f = gain[0] / sqrtf(block_sum(ss, red) / (float)D + eps);
  for (int c = threadIdx.x; c < D; c += THREADS) x[(long)t * ldx + c] = to_f32(r[c]) * f;
}

struct StreamsParams {
  const float* x_in; long ldr_in, lds_in;      // row and stream strides
  float* x_out; long ldr_out, lds_out;         // written when y is given
  const float* y; long ldy; int parts; long part_stride;      // result of the last sublayer (parts of a sum), or null
  const float *mix, *out;                      // [S, S] (from, to), [S]
  const float* in;                             // [S], or null: all ones
  const float* gain; float eps;                // one number
  const float* taps_w; int taps;               // [taps, D], the last row is the current token's; 0: no convolution
  float* history; const int32_t* epoch;
  const int32_t *positions, *slots;
  float* sum; long ldsum;                      // u on request
  void* xa; long lda;                          // operand, or null
  int T, S, D, block;
};

template <int V>
struct Vec { float f[V]; };
template <int V>
__device__ __forceinline__ Vec<V> ld(const float* p) {
  Vec<V> v;
  if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v.f[0] = a.x; v.f[1] = a.y; v.f[2] = a.z; v.f[3] = a.w;
  } else {
    v.f[0] = *p;
  }
  return v;
}
template <int V>
__device__ __forceinline__ void st(float* p, const Vec<V>& v) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v.f[0], v.f[1], v.f[2], v.f[3]);
  else *p = v.f[0];
}
template <int V>
__device__ __forceinline__ void st(bf16* p, const Vec<V>& v) {
  if constexpr (V == 4) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.f[0], v.f[1]), b = __floats2bfloat162_rn(v.f[2], v.f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(v.f[0]);
  }
}

// SMAX: most streams; V: columns of a thread at a time. Shared memory: the last `taps` (at least 1) rows of h, columns private to their threads
template <typename A, int SMAX, int V>
__global__ void __launch_bounds__(SMAX <= 2 ? 1024 : SMAX <= 4 ? 512 : THREADS) streams_rows_kernel(StreamsParams p) {
  extern __shared__ __align__(16) float ring[];
  __shared__ float red[33], mix[SMAX * SMAX], in[SMAX], out[SMAX];
  grid_dep_launch();
  const int nthr = blockDim.x;
  for (int i = threadIdx.x; i < p.S * p.S; i += nthr) mix[i] = p.mix ? p.mix[i] : 0.f;
  if ((int)threadIdx.x < p.S) {
    in[threadIdx.x] = p.in ? p.in[threadIdx.x] : 1.f;
    out[threadIdx.x] = p.out ? p.out[threadIdx.x] : 0.f;
  }
  const float gain = p.gain ? p.gain[0] : 1.f;
  __syncthreads();
  grid_dep_wait();
  const int r0 = blockIdx.x * p.block, r1 = min(p.T, r0 + p.block), back = p.taps - 1, deep = max(p.taps, 1);
  int o = 0;                                   // rows of the same run ahead of this one in the step (as many as matter)
  while (o < back && r0 - o - 1 >= 0 && p.slots[r0 - o - 1] == p.slots[r0]) ++o;
  int run = 0;                                 // of them, rows in the ring
  for (int r = r0 - o; r < r1; ++r) {
    if (r > r0 - o) run = p.slots[r] == p.slots[r - 1] ? run + 1 : 0;
    const bool mine = r >= r0;
    float* h = ring + (long)(r % deep) * p.D;
    const float* xr = p.x_in + (long)r * p.ldr_in;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < p.D; c += nthr * V) {
      Vec<V> x[SMAX], u;
#pragma unroll
      for (int s = 0; s < SMAX; ++s)
        if (s < p.S) x[s] = ld<V>(xr + s * p.lds_in + c);
      if (p.y) {
        Vec<V> y = ld<V>(p.y + (long)r * p.ldy + c), n[SMAX];
        for (int q = 1; q < p.parts; ++q) {
          const Vec<V> a = ld<V>(p.y + q * p.part_stride + (long)r * p.ldy + c);
#pragma unroll
          for (int i = 0; i < V; ++i) y.f[i] += a.f[i];
        }
#pragma unroll
        for (int t = 0; t < SMAX; ++t) {
          if (t >= p.S) break;
#pragma unroll
          for (int i = 0; i < V; ++i) n[t].f[i] = out[t] * y.f[i];
#pragma unroll
          for (int s = 0; s < SMAX; ++s) {
            if (s >= p.S) break;
#pragma unroll
            for (int i = 0; i < V; ++i) n[t].f[i] = fmaf(mix[s * p.S + t], x[s].f[i], n[t].f[i]);
          }
          if (mine && p.x_out) st<V>(p.x_out + (long)r * p.ldr_out + t * p.lds_out + c, n[t]);
        }
#pragma unroll
        for (int t = 0; t < SMAX; ++t) x[t] = n[t];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) u.f[i] = 0.f;
#pragma unroll
      for (int s = 0; s < SMAX; ++s) {
        if (s >= p.S) break;
#pragma unroll
        for (int i = 0; i < V; ++i) u.f[i] = fmaf(in[s], x[s].f[i], u.f[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(u.f[i], u.f[i], ss);
      st<V>(h + c, u);
      if (mine && p.sum) st<V>(p.sum + (long)r * p.ldsum + c, u);
    }
    if (!p.xa) continue;
    const float f = gain / sqrtf(block_sum(ss, red) / (float)p.D + p.eps);
    const int pos = p.taps ? p.positions[r] : 0, slot = p.taps ? p.slots[r] : 0;
    const int side = p.taps > 1 ? p.epoch[slot] & 1 : 0;
    const float* old = p.history + ((long)slot * 2 + side) * back * p.D;
    const bool last = p.taps > 1 && mine && (r + 1 == p.T || p.slots[r + 1] != slot);
    float* fresh = p.history + ((long)slot * 2 + (side ^ 1)) * back * p.D;
    for (int c = threadIdx.x * V; c < p.D; c += nthr * V) {
      Vec<V> v = ld<V>(h + c);
#pragma unroll
      for (int i = 0; i < V; ++i) v.f[i] *= f;
      st<V>(h + c, v);
      if (!mine) continue;
      Vec<V> a = v;
      if (p.taps) {
        const Vec<V> w = ld<V>(p.taps_w + (long)back * p.D + c);
#pragma unroll
        for (int i = 0; i < V; ++i) a.f[i] = fmaf(w.f[i], v.f[i], a.f[i]);
        if (last) st<V>(fresh + c, v);
        for (int j = 1; j < p.taps; ++j) {     // h of position pos - j
          Vec<V> b;
          if (j > pos) {
#pragma unroll
            for (int i = 0; i < V; ++i) b.f[i] = 0.f;
          } else {
            b = j <= run ? ld<V>(ring + (long)((r - j) % deep) * p.D + c) : ld<V>(old + (long)(j - run - 1) * p.D + c);
          }
          const Vec<V> wj = ld<V>(p.taps_w + (long)(back - j) * p.D + c);
#pragma unroll
          for (int i = 0; i < V; ++i) a.f[i] = fmaf(wj.f[i], b.f[i], a.f[i]);
          if (last && j < back) st<V>(fresh + (long)j * p.D + c, b);
        }
      }
      st<V>(reinterpret_cast<A*>(p.xa) + (long)r * p.lda + c, a);
    }
  }
}

// Shared memory: h of the CTA's rows and of those recomputed ahead of them, then 1 / rms times the gain of each
constexpr int tile_threads(int smax) { return smax <= 2 ? 768 : 512; }
template <typename A, int SMAX>
__global__ void __launch_bounds__(tile_threads(SMAX)) streams_tile_kernel(StreamsParams p) {
  extern __shared__ __align__(16) float hs[];
  __shared__ float mix[SMAX * SMAX], in[SMAX], out[SMAX];
  grid_dep_launch();
  for (int i = threadIdx.x; i < p.S * p.S; i += blockDim.x) mix[i] = p.mix ? p.mix[i] : 0.f;
  if ((int)threadIdx.x < p.S) {
    in[threadIdx.x] = p.in ? p.in[threadIdx.x] : 1.f;
    out[threadIdx.x] = p.out ? p.out[threadIdx.x] : 0.f;
  }
  const float gain = p.gain ? p.gain[0] : 1.f;
  __syncthreads();
  grid_dep_wait();
  const int r0 = blockIdx.x * p.block, r1 = min(p.T, r0 + p.block), back = max(p.taps - 1, 0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int o = 0;                                   // rows of the same run ahead of this CTA's (as many as matter)
  while (o < back && r0 - o - 1 >= 0 && p.slots[r0 - o - 1] == p.slots[r0]) ++o;
  const int rows = o + r1 - r0;
  float* inv = hs + (long)(p.block + back) * p.D;
  for (int i = warp; i < rows; i += blockDim.x >> 5) {
    const int r = r0 - o + i;
    const bool mine = i >= o;
    const float* xr = p.x_in + (long)r * p.ldr_in;
    float* h = hs + (long)i * p.D;
    float ss = 0.f;
    constexpr int U = SMAX <= 1 ? 4 : 2;        // column groups whose loads are in flight together
    for (int c0 = lane * 4; c0 < p.D; c0 += 128 * U) {
      Vec<4> x[U][SMAX], y[U];
#pragma unroll
      for (int z = 0; z < U; ++z) {
        const int c = c0 + 128 * z;
        if (c >= p.D) break;
#pragma unroll
        for (int s = 0; s < SMAX; ++s)
          if (s < p.S) x[z][s] = ld<4>(xr + s * p.lds_in + c);
        if (p.y) {
          y[z] = ld<4>(p.y + (long)r * p.ldy + c);
          for (int q = 1; q < p.parts; ++q) {
            const Vec<4> a = ld<4>(p.y + q * p.part_stride + (long)r * p.ldy + c);
#pragma unroll
            for (int k = 0; k < 4; ++k) y[z].f[k] += a.f[k];
          }
        }
      }
#pragma unroll
      for (int z = 0; z < U; ++z) {
        const int c = c0 + 128 * z;
        if (c >= p.D) break;
        Vec<4> u;
#pragma unroll
        for (int k = 0; k < 4; ++k) u.f[k] = 0.f;
        if (p.y) {
#pragma unroll
          for (int t = 0; t < SMAX; ++t) {
            if (t >= p.S) break;
            Vec<4> n;
#pragma unroll
            for (int k = 0; k < 4; ++k) n.f[k] = out[t] * y[z].f[k];
#pragma unroll
            for (int s = 0; s < SMAX; ++s) {
              if (s >= p.S) break;
#pragma unroll
              for (int k = 0; k < 4; ++k) n.f[k] = fmaf(mix[s * p.S + t], x[z][s].f[k], n.f[k]);
            }
            if (mine && p.x_out) st<4>(p.x_out + (long)r * p.ldr_out + t * p.lds_out + c, n);
#pragma unroll
            for (int k = 0; k < 4; ++k) u.f[k] = fmaf(in[t], n.f[k], u.f[k]);
          }
        } else {
#pragma unroll
          for (int s = 0; s < SMAX; ++s) {
            if (s >= p.S) break;
#pragma unroll
            for (int k = 0; k < 4; ++k) u.f[k] = fmaf(in[s], x[z][s].f[k], u.f[k]);
          }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) ss = fmaf(u.f[k], u.f[k], ss);
        st<4>(h + c, u);
        if (mine && p.sum) st<4>(p.sum + (long)r * p.ldsum + c, u);
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) inv[i] = gain / sqrtf(ss / (float)p.D + p.eps);
  }
  __syncthreads();
  if (!p.xa) return;
  for (int c = threadIdx.x * 4; c < p.D; c += blockDim.x * 4) {
    int run = o;                               // rows of the run ahead of row r in the step (as many as matter)
    for (int i = o; i < rows; ++i) {
      const int r = r0 - o + i, slot = p.slots[r];
      if (i > o) run = p.slots[r - 1] == slot ? run + 1 : 0;
      Vec<4> v = ld<4>(hs + (long)i * p.D + c);
      const float f = inv[i];
#pragma unroll
      for (int k = 0; k < 4; ++k) v.f[k] *= f;
      Vec<4> a = v;
      if (p.taps) {
        const int pos = p.positions[r], side = p.taps > 1 ? p.epoch[slot] & 1 : 0;
        const float* old = p.history + ((long)slot * 2 + side) * back * p.D;
        const bool last = p.taps > 1 && (r + 1 == p.T || p.slots[r + 1] != slot);
        float* fresh = p.history + ((long)slot * 2 + (side ^ 1)) * back * p.D;
        const Vec<4> w = ld<4>(p.taps_w + (long)back * p.D + c);
#pragma unroll
        for (int k = 0; k < 4; ++k) a.f[k] = fmaf(w.f[k], v.f[k], a.f[k]);
        if (last) st<4>(fresh + c, v);
        for (int j = 1; j < p.taps; ++j) {
          Vec<4> b;
          float g = 1.f;
          if (j > pos) {
#pragma unroll
            for (int k = 0; k < 4; ++k) b.f[k] = 0.f;
          } else if (j <= run) {
            b = ld<4>(hs + (long)(i - j) * p.D + c);
            g = inv[i - j];
          } else {
            b = ld<4>(old + (long)(j - run - 1) * p.D + c);
          }
          const Vec<4> wj = ld<4>(p.taps_w + (long)(back - j) * p.D + c);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            b.f[k] *= g;
            a.f[k] = fmaf(wj.f[k], b.f[k], a.f[k]);
          }
          if (last && j < back) st<4>(fresh + (long)j * p.D + c, b);
        }
      }
      st<4>(reinterpret_cast<A*>(p.xa) + (long)r * p.lda + c, a);
    }
  }
}

// rows of a CTA: even waves of CTAs, as many as shared memory asks for; 0: the other kernel
int tile_rows(const StreamsParams& p) {
  const int back = p.taps > 1 ? p.taps - 1 : 0, room = (int)(200 * 1024 / (p.D * sizeof(float) + sizeof(float))) - back;
  if (p.T <= 256 || room < 4) return 0;
  const int want = (p.T + 147) / 148, waves = (want + room - 1) / room, rows = (want + waves - 1) / waves;
  return rows < 4 ? 4 : rows;
}
template <typename A, int SMAX>
int launch_tile(StreamsParams p, cudaStream_t s) {
  p.block = tile_rows(p);
  const int rows = p.block + (p.taps > 1 ? p.taps - 1 : 0);
  const size_t smem = (size_t)rows * (p.D + 1) * sizeof(float);
  auto k = streams_tile_kernel<A, SMAX>;
  if (int rc = opt_in_smem(k, smem)) return rc;
  return launch_chain(k, dim3((p.T + p.block - 1) / p.block), dim3(rows < 8 ? 256 : 32 * rows < tile_threads(SMAX) ? 32 * rows : tile_threads(SMAX)), smem, s, p);
}

template <typename A, int SMAX, int V>
int launch_rows(const StreamsParams& p, cudaStream_t s) {
  const size_t smem = (size_t)(p.taps > 1 ? p.taps : 1) * p.D * sizeof(float);
  auto k = streams_rows_kernel<A, SMAX, V>;
  if (smem > 200 * 1024) return -1;
  if (int rc = opt_in_smem(k, smem)) return rc;
  const int most = SMAX <= 2 ? 1024 : SMAX <= 4 ? 512 : THREADS, want = (p.D + 32 * V - 1) / (32 * V) * 32;
  return launch_chain(k, dim3((p.T + p.block - 1) / p.block), dim3(want < 64 ? 64 : want < most ? want : most), smem, s, p);
}
template <typename A>
int by_streams(const StreamsParams& p, cudaStream_t s) {
  const auto odd = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; };
  const bool four = !((p.D | p.ldr_in | p.lds_in | p.ldr_out | p.lds_out | p.ldy | p.part_stride | p.ldsum | p.lda) % 4) && !odd(p.x_in) && !odd(p.x_out) && !odd(p.y) &&
                    !odd(p.taps_w) && !odd(p.history) && !odd(p.sum) && !odd(p.xa);
  if (!four) return launch_rows<A, MAX_S, 1>(p, s);
  if (p.S <= 4 && tile_rows(p)) return p.S <= 1 ? launch_tile<A, 1>(p, s) : p.S == 2 ? launch_tile<A, 2>(p, s) : launch_tile<A, 4>(p, s);
  if (p.S == 1) return launch_rows<A, 1, 4>(p, s);
  if (p.S == 2) return launch_rows<A, 2, 4>(p, s);
  if (p.S <= 4) return launch_rows<A, 4, 4>(p, s);
  return launch_rows<A, MAX_S, 4>(p, s);
}

// one thread per row: the first row of a run turns its sequence's epoch over
__global__ void __launch_bounds__(128) step_epoch_kernel(const int32_t* slots, int32_t* epoch, int T) {
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x * 128 + threadIdx.x;
  if (t < T && (t == 0 || slots[t - 1] != slots[t])) epoch[slots[t]] ^= 1;
}

}  // namespace

extern "C" int ifab_embed_norm(const int32_t* ids, const void* table, long ldt, const float* gain, float eps, float* x, long ldx, int f32, int T, int D, int vocab,
                               uint32_t* status, void* stream) {
  if (T < 1 || D < 1 || vocab < 1 || !gain) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? launch_chain(embed_norm_kernel<float>, dim3(T), dim3(THREADS), 0, s, ids, (const float*)table, ldt, gain, eps, x, ldx, D, vocab, status)
             : launch_chain(embed_norm_kernel<bf16>, dim3(T), dim3(THREADS), 0, s, ids, (const bf16*)table, ldt, gain, eps, x, ldx, D, vocab, status);
}

// epoch [slots]: rows of a sequence are consecutive in a step
extern "C" int ifab_step_epoch(const int32_t* slots, int32_t* epoch, int T, void* stream) {
  if (T < 1) return -1;
  return launch_chain(step_epoch_kernel, dim3((T + 127) / 128), dim3(128), 0, (cudaStream_t)stream, slots, epoch, T);
}

extern "C" int ifab_streams_rows(const float* x_in, long ldr_in, long lds_in, float* x_out, long ldr_out, long lds_out, const float* y, long ldy, int parts,
                                 long part_stride, const float* mix, const float* out, const float* in, const float* gain, float eps, const float* taps_w, int taps,
                                 float* history, const int32_t* epoch, const int32_t* positions, const int32_t* slots, float* sum, long ldsum, void* xa, long lda,
                                 int f32, int T, int S, int D, int block, void* stream) {
  if (T < 1 || D < 1 || S < 1 || S > MAX_S || taps < 0 || taps > MAX_TAPS || parts < 1 || block < 1 || (y && (!mix || !out)) || (x_out && x_out == x_in)) return -1;
  if (taps && (!taps_w || !positions || !xa || (taps > 1 && (!history || !epoch)))) return -1;
  if (!slots) return -1;
  StreamsParams p{x_in, ldr_in, lds_in, x_out, ldr_out, lds_out, y, ldy, parts, part_stride, mix, out, in, gain, eps, taps_w, taps, history, epoch, positions, slots, sum, ldsum,
                  xa, lda, T, S, D, block};
  return f32 ? by_streams<float>(p, (cudaStream_t)stream) : by_streams<bf16>(p, (cudaStream_t)stream);
}
