// Decode-time launches (one or two rows) of decoders with residual streams and gated recurrences. The weight stream of the linears is the one of gemv.cuh (prefetched
// ahead of the wait on the producer); their prologues finish what lies ahead of them, so that a layer needs no row kernels between its linears:
//
//   gemv_streams_kernel  the streams behind the last sublayer, norm and convolution (hyper_streams.cu), then a linear over that operand. Every CTA computes the rows it
//                        needs; the CTAs of the first column write the streams (x_out must not be x_in) and the history's other side
//   gemv_mixed_kernel    a linear over [bf16 columns | result of a recurrence, finished: division, skip, gate, norm of equal groups, gain (gr_finish_kernel)]
//   gr_decode_kernel     gr_prepare_kernel and gr_step_kernel in one: a CTA convolves what its head and its 32 value columns need
#include "gated_recurrence.cuh"
#include "gemv.cuh"

using namespace ifab;

namespace {

struct Linear {
  const bf16* w; int N, K;
  void* z; long ldz; int out_f32, act;
  int T;
};

// the dot products of R weight rows per warp with T staged rows, and the epilogue
template <int T, int R>
__device__ __forceinline__ void finish_linear(const Linear& p, const bf16* const (&rows)[R], const bf16* xs, RowBatch<R>& pf, int n0) {
  const int lane = threadIdx.x & 31;
  if (n0 >= p.N) return;
  float acc[R][T];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int t = 0; t < T; ++t) acc[r][t] = 0.f;
  warp_rows_dot<T, R>(rows, xs, p.K, acc, pf);
  warp_reduce_acc<T, R>(acc);
  if (lane != 0) return;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (n0 + r >= p.N) continue;
#pragma unroll
    for (int t = 0; t < T; ++t) {
      if (t >= p.T) continue;
      const float v = activate<true>(acc[r][t], p.act);
      if (p.out_f32) reinterpret_cast<float*>(p.z)[(long)t * p.ldz + n0 + r] = v;
      else reinterpret_cast<bf16*>(p.z)[(long)t * p.ldz + n0 + r] = __float2bfloat16_rn(v);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// a linear behind the streams
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int MAX_S = 4;
struct StreamsIn {
  const float* x_in; long ldr_in, lds_in;
  float* x_out; long ldr_out, lds_out;
  const float* y; long ldy;
  const float *mix, *out, *in, *gain; float eps;
  const float* taps_w; int taps;               // [taps, K]
  float* history; const int32_t* epoch;
  const int32_t *positions, *slots;
  int S;
};

template <int T, int R>
__global__ void __launch_bounds__(256, 2) gemv_streams_kernel(Linear p, StreamsIn q) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  float* u = reinterpret_cast<float*>(smem_raw);           // [T][K]
  float* ahead = u + (long)T * p.K;                        // [T][K]: what the history gives to the convolution
  bf16* xs = reinterpret_cast<bf16*>(ahead + (long)T * p.K);
  __shared__ float red[T][8];
  grid_dep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = (blockIdx.x * 8 + warp) * R;
  const bf16* rows[R];
#pragma unroll
  for (int r = 0; r < R; ++r) rows[r] = (n0 + r < p.N) ? p.w + (long)(n0 + r) * p.K : nullptr;
  RowBatch<R> pf;
  prefetch_rows<R>(rows, p.K, pf);
  __shared__ float mix[MAX_S][MAX_S], in[MAX_S], out[MAX_S];
  if ((int)threadIdx.x < MAX_S * MAX_S) {
    const int s = threadIdx.x / MAX_S, t = threadIdx.x % MAX_S;
    mix[s][t] = q.y && s < q.S && t < q.S ? q.mix[s * q.S + t] : 0.f;
    if (t == 0) {
      in[s] = s < q.S ? q.in[s] : 0.f;
      out[s] = q.y && s < q.S ? q.out[s] : 0.f;
    }
  }
  const float gain = q.gain[0];
  grid_dep_wait();
  __syncthreads();
  const int K = p.K, back = q.taps - 1;
  const bool writer = blockIdx.x == 0;
  int run = 0;                                             // of the second row
  if (T == 2 && p.T == 2) run = q.slots[0] == q.slots[1];
#pragma unroll
  for (int t = 0; t < T; ++t) {
    float ss = 0.f;
    if (t < p.T) {
      const int pos = q.taps ? q.positions[t] : 0, slot = q.taps ? q.slots[t] : 0, side = q.taps > 1 ? q.epoch[slot] & 1 : 0, mine = t ? run : 0;
      const float* old = q.history + ((long)slot * 2 + side) * back * K;
      float* fresh = q.history + ((long)slot * 2 + (side ^ 1)) * back * K;
      const bool last = writer && q.taps > 1 && (t + 1 == p.T || !run);
      const float* xr = q.x_in + (long)t * q.ldr_in;
      for (int c = threadIdx.x * 4; c < K; c += 1024) {
        float4 x[MAX_S];
#pragma unroll
        for (int s = 0; s < MAX_S; ++s)
          if (s < q.S) x[s] = *reinterpret_cast<const float4*>(xr + s * q.lds_in + c);
        const float4 y = q.y ? *reinterpret_cast<const float4*>(q.y + (long)t * q.ldy + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        float4 h = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int j = 1; j < q.taps; ++j) {                 // what lies ahead of the step
          if (j <= mine) continue;
          float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
          if (j <= pos) {
            v = *reinterpret_cast<const float4*>(old + (long)(j - mine - 1) * K + c);
            const float4 w = *reinterpret_cast<const float4*>(q.taps_w + (long)(back - j) * K + c);
            h.x = fmaf(w.x, v.x, h.x);
            h.y = fmaf(w.y, v.y, h.y);
            h.z = fmaf(w.z, v.z, h.z);
            h.w = fmaf(w.w, v.w, h.w);
          }
          if (last && j < back) *reinterpret_cast<float4*>(fresh + (long)j * K + c) = v;
        }
        *reinterpret_cast<float4*>(ahead + (long)t * K + c) = h;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (q.y) {
#pragma unroll
          for (int o = 0; o < MAX_S; ++o) {
            if (o >= q.S) break;
            float4 n = make_float4(out[o] * y.x, out[o] * y.y, out[o] * y.z, out[o] * y.w);
#pragma unroll
            for (int s = 0; s < MAX_S; ++s) {
              if (s >= q.S) break;
              n.x = fmaf(mix[s][o], x[s].x, n.x);
              n.y = fmaf(mix[s][o], x[s].y, n.y);
              n.z = fmaf(mix[s][o], x[s].z, n.z);
              n.w = fmaf(mix[s][o], x[s].w, n.w);
            }
            if (writer) *reinterpret_cast<float4*>(q.x_out + (long)t * q.ldr_out + o * q.lds_out + c) = n;
            a.x = fmaf(in[o], n.x, a.x);
            a.y = fmaf(in[o], n.y, a.y);
            a.z = fmaf(in[o], n.z, a.z);
            a.w = fmaf(in[o], n.w, a.w);
          }
        } else {
#pragma unroll
          for (int s = 0; s < MAX_S; ++s) {
            if (s >= q.S) break;
            a.x = fmaf(in[s], x[s].x, a.x);
            a.y = fmaf(in[s], x[s].y, a.y);
            a.z = fmaf(in[s], x[s].z, a.z);
            a.w = fmaf(in[s], x[s].w, a.w);
          }
        }
        *reinterpret_cast<float4*>(u + (long)t * K + c) = a;
        ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[t][warp] = ss;
  }
  __syncthreads();
  float inv[T];
#pragma unroll
  for (int t = 0; t < T; ++t) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s += red[t][i];
    inv[t] = gain / sqrtf(s / (float)K + q.eps);
  }
  // columns are still the threads' own
#pragma unroll
  for (int t = 0; t < T; ++t) {
    const bool live = t < p.T;
    const int slot = live && q.taps > 1 ? q.slots[t] : 0, side = live && q.taps > 1 ? q.epoch[slot] & 1 : 0;
    float* fresh = q.history + ((long)slot * 2 + (side ^ 1)) * back * K;
    const bool last = live && writer && q.taps > 1 && (t + 1 == p.T || !run);
    for (int c = threadIdx.x * 4; c < K; c += 1024) {
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live) {
        float4 h = *reinterpret_cast<const float4*>(u + (long)t * K + c);
        h.x *= inv[t]; h.y *= inv[t]; h.z *= inv[t]; h.w *= inv[t];
        f = h;
        if (q.taps) {
          const float4 a = *reinterpret_cast<const float4*>(ahead + (long)t * K + c), w = *reinterpret_cast<const float4*>(q.taps_w + (long)back * K + c);
          f.x += fmaf(w.x, h.x, a.x);
          f.y += fmaf(w.y, h.y, a.y);
          f.z += fmaf(w.z, h.z, a.z);
          f.w += fmaf(w.w, h.w, a.w);
          if (last) *reinterpret_cast<float4*>(fresh + c) = h;
          if (T == 2 && t == 1 && run && q.taps > 1 && q.positions[1] > 0) {        // the row ahead in the step
            float4 b = *reinterpret_cast<const float4*>(u + c);
            b.x *= inv[0]; b.y *= inv[0]; b.z *= inv[0]; b.w *= inv[0];
            const float4 v = *reinterpret_cast<const float4*>(q.taps_w + (long)(back - 1) * K + c);
            f.x = fmaf(v.x, b.x, f.x);
            f.y = fmaf(v.y, b.y, f.y);
            f.z = fmaf(v.z, b.z, f.z);
            f.w = fmaf(v.w, b.w, f.w);
            if (last && back > 1) *reinterpret_cast<float4*>(fresh + K + c) = b;
          }
        }
      }
      __nv_bfloat162 a = __floats2bfloat162_rn(f.x, f.y), b = __floats2bfloat162_rn(f.z, f.w);
      *reinterpret_cast<uint2*>(xs + (long)t * K + c) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    }
  }
  __syncthreads();
  finish_linear<T, R>(p, rows, xs, pf, n0);
}

// ---------------------------------------------------------------------------------------------------------------------------
// a linear behind a recurrence
// ---------------------------------------------------------------------------------------------------------------------------
struct MixedIn {
  const bf16* x; long ldx; int K1;             // columns 0 .. K1 - 1 as they are (a multiple of 8)
  const float* o; long ldo; int H, e, E;       // then H * e of the recurrence
  const float* m;
  const bf16* v; const float* skip;
  const bf16* gate; long ldg; int act, gate_first;
  int groups; float eps; const float* gain;
};

template <int T, int R>
__global__ void __launch_bounds__(256, 2) gemv_mixed_kernel(Linear p, MixedIn q) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* xs = reinterpret_cast<bf16*>(smem_raw);                               // [T][K]
  float* val = reinterpret_cast<float*>(xs + (long)T * p.K);                  // [T][H * e]
  const int n2 = q.H * q.e, n = n2 / q.groups;
  float* inv = val + (long)T * n2;                                            // [T][groups]: sums, then factors
  grid_dep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = (blockIdx.x * 8 + warp) * R;
  const bf16* rows[R];
#pragma unroll
  for (int r = 0; r < R; ++r) rows[r] = (n0 + r < p.N) ? p.w + (long)(n0 + r) * p.K : nullptr;
  RowBatch<R> pf;
  prefetch_rows<R>(rows, p.K, pf);
  for (int i = threadIdx.x; i < T * q.groups; i += 256) inv[i] = 0.f;
  grid_dep_wait();
  __syncthreads();
#pragma unroll
  for (int t = 0; t < T; ++t) {
    const bool live = t < p.T;
    bf16* row = xs + (long)t * p.K;
    for (int c = threadIdx.x * 8; c < q.K1; c += 2048)
      *reinterpret_cast<uint4*>(row + c) = live ? *reinterpret_cast<const uint4*>(q.x + (long)t * q.ldx + c) : make_uint4(0, 0, 0, 0);
    for (int c = q.K1 + n2 + (int)threadIdx.x; c < p.K; c += 256) row[c] = __float2bfloat16_rn(0.f);
    if (!live) {
      for (int c = threadIdx.x; c < n2; c += 256) row[q.K1 + c] = __float2bfloat16_rn(0.f);
      continue;
    }
    // whole warps at a time: 32 lanes x 4 columns of one group each
    for (int c0 = warp * 128; c0 < n2; c0 += 1024) {
      const int c = c0 + lane * 4;
      float ss = 0.f;
      if (c < n2) {
        const int h = c / q.e, j = c - h * q.e;
        const float* oh = q.o + (long)t * q.ldo + (long)h * q.E;
        float4 a = make_float4(oh[j], oh[j + 1], oh[j + 2], oh[j + 3]);       // heads of a memory are not whole 16-byte chunks
        if (q.m) {
          const float f = 1.f / (fmaxf(fabsf(oh[q.e]), expf(-q.m[(long)t * q.H + h])) + 1e-6f);
          a.x *= f; a.y *= f; a.z *= f; a.w *= f;
        }
        if (q.skip) {
          const uint2 raw = *reinterpret_cast<const uint2*>(q.v + (long)t * n2 + c);
          const float2 v0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), v1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
          const float s = q.skip[h];
          a.x = fmaf(s, v0.x, a.x); a.y = fmaf(s, v0.y, a.y); a.z = fmaf(s, v1.x, a.z); a.w = fmaf(s, v1.y, a.w);
        }
        const uint2 raw = *reinterpret_cast<const uint2*>(q.gate + (long)t * q.ldg + c);
        const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        const float4 z = make_float4(activate<true>(g0.x, q.act), activate<true>(g0.y, q.act), activate<true>(g1.x, q.act), activate<true>(g1.y, q.act));
        if (q.gate_first) {
          a.x *= z.x; a.y *= z.y; a.z *= z.z; a.w *= z.w;
        }
        ss = a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
        const float4 g = *reinterpret_cast<const float4*>(q.gain + c);
        a.x *= g.x; a.y *= g.y; a.z *= g.z; a.w *= g.w;
        if (!q.gate_first) {
          a.x *= z.x; a.y *= z.y; a.z *= z.z; a.w *= z.w;
        }
        *reinterpret_cast<float4*>(val + (long)t * n2 + c) = a;
      }
      if (n % 128 == 0) {
        ss = warp_sum(ss);
        if (lane == 0) atomicAdd(&inv[t * q.groups + c0 / n], ss);
      } else if (c < n2) {
        atomicAdd(&inv[t * q.groups + c / n], ss);                            // 4 columns lie in one group (n % 4 == 0)
      }
    }
  }
  __syncthreads();
  for (int t = 0; t < min(T, p.T); ++t)
    for (int c = threadIdx.x * 4; c < n2; c += 1024) {
      const float f = 1.f / sqrtf(inv[t * q.groups + c / n] / (float)n + q.eps);
      const float4 a = *reinterpret_cast<const float4*>(val + (long)t * n2 + c);
      __nv_bfloat162 x = __floats2bfloat162_rn(a.x * f, a.y * f), y = __floats2bfloat162_rn(a.z * f, a.w * f);
      *reinterpret_cast<uint2*>(xs + (long)t * p.K + q.K1 + c) = make_uint2(*reinterpret_cast<uint32_t*>(&x), *reinterpret_cast<uint32_t*>(&y));
    }
  __syncthreads();
  finish_linear<T, R>(p, rows, xs, pf, n0);
}

template <template <int, int> class Launch, typename... Args>
int by_rows(int T, int N, Args... args) {
  // rows per warp: the widest that still gives every SM a CTA, so that the grid is one wave
  const int R = N >= 148 * 8 * 4 ? 4 : N >= 148 * 8 * 2 ? 2 : 1;
  if (T == 1) return R == 4 ? Launch<1, 4>::run(args...) : R == 2 ? Launch<1, 2>::run(args...) : Launch<1, 1>::run(args...);
  return R == 4 ? Launch<2, 4>::run(args...) : R == 2 ? Launch<2, 2>::run(args...) : Launch<2, 1>::run(args...);
}
template <int T, int R>
struct LaunchStreams {
  static int run(const Linear& p, const StreamsIn& q, cudaStream_t s) {
    const size_t smem = (size_t)T * p.K * 10;
    auto k = gemv_streams_kernel<T, R>;
    if (smem > 220 * 1024) return -1;
    if (int rc = opt_in_smem(k, smem)) return rc;
    return launch_chain(k, dim3((p.N + 8 * R - 1) / (8 * R)), dim3(256), smem, s, p, q);
  }
};
template <int T, int R>
struct LaunchMixed {
  static int run(const Linear& p, const MixedIn& q, cudaStream_t s) {
    const size_t smem = (size_t)T * (p.K * 2 + q.H * q.e * 4 + q.groups * 4);
    auto k = gemv_mixed_kernel<T, R>;
    if (smem > 220 * 1024) return -1;
    if (int rc = opt_in_smem(k, smem)) return rc;
    return launch_chain(k, dim3((p.N + 8 * R - 1) / (8 * R)), dim3(256), smem, s, p, q);
  }
};

// ---------------------------------------------------------------------------------------------------------------------------
// convolution, gates and step in one
// ---------------------------------------------------------------------------------------------------------------------------
struct DecodeParams {
  const bf16* proj; long ldp;
  int col[3], channel[3];                      // q, k, v: where they start in a projection row and among the channels (-1: no convolution)
  const float *taps_w, *bias; int taps, C;
  bf16* history;
  int decay_col, weight_col;
  const float *a_log, *decay_bias, *weight_bias; float cap;
  int unit; float q_factor;
  int kind, H, G, d, e, E;
  GrState st;
  bf16* v;                                     // [T, H * e] as convolved, for a skip
  float* o; long ldo;
  float* m_rows;
  const int32_t *positions, *slots;
  int T;
};

// grid (H, T, ceil(E / 32)), 256 threads: a CTA walks a run of rows of one slot; a warp owns 4 value columns = rows of the state, lanes their d columns (REG float4s
// each). Shared memory: q [d], k [d], v [32]
template <int REG>
__global__ void __launch_bounds__(256) gr_decode_kernel(DecodeParams p) {
  __shared__ __align__(16) float sq[128 * REG], sk[128 * REG];
  __shared__ float sv[32], red[2][8], gates[2];
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, t0 = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, z0 = blockIdx.z * 32, col0 = z0 + warp * 4, d = p.d, group = p.H / p.G, g = h / group;
  const int slot = p.slots[t0];
  if (p.positions[t0] < 0 || (t0 > 0 && p.slots[t0 - 1] == slot && p.positions[t0 - 1] >= 0)) return;      // not the head of a run
  const int side = p.st.epoch[slot] & 1, nc = max(0, min(4, p.E - col0)), back = p.taps - 1;
  float* S = p.st.s + (((long)slot * p.H + h) * p.E + col0) * d;
  const bool empty = p.positions[t0] == 0;
  float4 s[4][REG];
#pragma unroll
  for (int u = 0; u < 4; ++u)
#pragma unroll
    for (int x = 0; x < REG; ++x) {
      const int c = (lane + 32 * x) * 4;
      s[u][x] = (u < nc && c < d && !empty) ? *reinterpret_cast<const float4*>(S + (long)u * d + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  float m = p.kind == GR_MEMORY && !empty ? p.st.m[((long)slot * 2 + side) * p.H + h] : 0.f;
  const bf16* old = p.history + ((long)slot * 2 + side) * back * p.C;
  bf16* fresh = p.history + ((long)slot * 2 + (side ^ 1)) * back * p.C;
  const bool keeps = blockIdx.z == 0 && h % group == 0;      // this CTA writes the history of its q and k
  for (int t = t0; t < p.T && p.slots[t] == slot && p.positions[t] >= 0; ++t) {
    const bf16* row = p.proj + (long)t * p.ldp;
    const int pos = p.positions[t], run = t - t0;
    const bool last = p.taps > 1 && (t + 1 == p.T || p.slots[t + 1] != slot);
    float ssq = 0.f, ssk = 0.f;
    for (int i = tid; i < 2 * d + 32; i += 256) {
      const int which = i < d ? 0 : i < 2 * d ? 1 : 2, c = i - (which == 0 ? 0 : which == 1 ? d : 2 * d);
      if (which == 2 && z0 + c >= p.e) {
        sv[c] = 1.f;                           // the memory's column of ones
        continue;
      }
      const int at = which == 2 ? h * p.e + z0 + c : g * d + c;
      float x = to_f32(row[p.col[which] + at]);
      if (p.taps) {
        const int ch = p.channel[which] + at;
        const bool keep = last && (which == 2 || keeps);
        const bf16 here = row[p.col[which] + at];
        const float bias = p.bias ? p.bias[ch] : 0.f;
        float acc = x * p.taps_w[(long)back * p.C + ch];
        for (int j0 = 1; j0 < p.taps; j0 += 3) {         // three taps' loads ahead of the stores
          bf16 b[3];
          float w[3];
#pragma unroll
          for (int y = 0; y < 3; ++y) {
            const int j = j0 + y;
            b[y] = __float2bfloat16_rn(0.f);
            w[y] = j < p.taps ? p.taps_w[(long)(back - j) * p.C + ch] : 0.f;
            if (j < p.taps && j <= pos) b[y] = j <= run ? row[p.col[which] + at - (long)j * p.ldp] : old[(long)(j - run - 1) * p.C + ch];
          }
#pragma unroll
          for (int y = 0; y < 3; ++y) {
            acc = fmaf(w[y], to_f32(b[y]), acc);
            if (keep && j0 + y < back) fresh[(long)(j0 + y) * p.C + ch] = b[y];
          }
        }
        if (keep) fresh[ch] = here;
        acc += bias;
        x = bf16_round(acc * sigmoid_f32<true>(acc));
      }
      if (which == 0) {
        sq[c] = x;
        ssq = fmaf(x, x, ssq);
      } else if (which == 1) {
        sk[c] = x;
        ssk = fmaf(x, x, ssk);
      } else {
        sv[c] = x;
        if (p.v) p.v[(long)t * p.H * p.e + at] = __float2bfloat16_rn(x);
      }
    }
    if (tid == 0) {
      const float a = to_f32(row[p.decay_col + h]) + (p.decay_bias ? p.decay_bias[h] : 0.f), b = to_f32(row[p.weight_col + h]) + (p.weight_bias ? p.weight_bias[h] : 0.f);
      const auto softplus = [](float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); };
      float f, w;
      if (p.kind == GR_MEMORY) {
        f = -softplus(-p.cap * tanhf(a / p.cap));
        w = p.cap * tanhf(b / p.cap);
      } else {
        const float sp = softplus(a);
        f = -expf(p.a_log[h]) * sp;
        w = p.kind == GR_SSD ? sp : sigmoid_f32(b);
      }
      gates[0] = f;
      gates[1] = w;
    }
    if (p.unit) {
      ssq = warp_sum(ssq);
      ssk = warp_sum(ssk);
      if (lane == 0) {
        red[0][warp] = ssq;
        red[1][warp] = ssk;
      }
    }
    __syncthreads();
    float fq = p.q_factor, fk = 1.f;
    if (p.unit) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        a += red[0][i];
        b += red[1][i];
      }
      fq /= sqrtf(a + 1e-6f);
      fk = 1.f / sqrtf(b + 1e-6f);
    }
    const float ld = gates[0];
    float w = gates[1], a;
    if (p.kind == GR_MEMORY) {
      const float mn = fmaxf(ld + m, w);
      a = expf(ld + m - mn);
      w = expf(w - mn);
      m = mn;
      if (blockIdx.z == 0 && tid == 0) p.m_rows[(long)t * p.H + h] = m;
    } else {
      a = expf(ld);
    }
    float4 kr[REG], qr[REG];
#pragma unroll
    for (int x = 0; x < REG; ++x) {
      const int c = (lane + 32 * x) * 4;
      kr[x] = c < d ? *reinterpret_cast<const float4*>(sk + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      qr[x] = c < d ? *reinterpret_cast<const float4*>(sq + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      kr[x].x *= fk; kr[x].y *= fk; kr[x].z *= fk; kr[x].w *= fk;
      qr[x].x *= fq; qr[x].y *= fq; qr[x].z *= fq; qr[x].w *= fq;
    }
    float v[4], acc[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      v[u] = u < nc ? sv[warp * 4 + u] : 0.f;
      float kk = 0.f;
#pragma unroll
      for (int x = 0; x < REG; ++x) {
        s[u][x].x *= a; s[u][x].y *= a; s[u][x].z *= a; s[u][x].w *= a;
        if (p.kind == GR_DELTA) kk = fmaf(kr[x].x, s[u][x].x, fmaf(kr[x].y, s[u][x].y, fmaf(kr[x].z, s[u][x].z, fmaf(kr[x].w, s[u][x].w, kk))));
      }
      if (p.kind == GR_DELTA) v[u] -= warp_sum(kk);
      const float wv = w * v[u];
      acc[u] = 0.f;
#pragma unroll
      for (int x = 0; x < REG; ++x) {
        s[u][x].x = fmaf(kr[x].x, wv, s[u][x].x);
        s[u][x].y = fmaf(kr[x].y, wv, s[u][x].y);
        s[u][x].z = fmaf(kr[x].z, wv, s[u][x].z);
        s[u][x].w = fmaf(kr[x].w, wv, s[u][x].w);
        acc[u] = fmaf(qr[x].x, s[u][x].x, fmaf(qr[x].y, s[u][x].y, fmaf(qr[x].z, s[u][x].z, fmaf(qr[x].w, s[u][x].w, acc[u]))));
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float x = warp_sum(acc[u]);
      if (lane == 0 && u < nc) p.o[(long)t * p.ldo + (long)h * p.E + col0 + u] = x;
    }
    __syncthreads();                           // q, k, v are used up
  }
#pragma unroll
  for (int u = 0; u < 4; ++u)
#pragma unroll
    for (int x = 0; x < REG; ++x) {
      const int c = (lane + 32 * x) * 4;
      if (u < nc && c < d) *reinterpret_cast<float4*>(S + (long)u * d + c) = s[u][x];
    }
  if (p.kind == GR_MEMORY && blockIdx.z == 0 && tid == 0) p.st.m[((long)slot * 2 + (side ^ 1)) * p.H + h] = m;
}

bool odd16(const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; }

}  // namespace

// z = act(bf16(h + conv(h)) w^T) for T <= 2 rows, S <= 4 streams: see ifab_streams_rows for the streams (y: one f32 row per row). w [N, K] bf16
extern "C" int ifab_gemv_streams(const float* x_in, long ldr_in, long lds_in, float* x_out, long ldr_out, long lds_out, const float* y, long ldy, const float* mix,
                                 const float* out, const float* in, const float* gain, float eps, const float* taps_w, int taps, float* history,
                                 const int32_t* epoch, const int32_t* positions, const int32_t* slots, int S, const void* w, void* z, long ldz, int out_f32, int act,
                                 int T, int N, int K, void* stream) {
  if (T < 1 || T > 2 || N < 1 || K < 8 || K % 8 || S < 1 || S > MAX_S || !in || !gain || (y && (!x_out || !mix || !out || x_out == x_in)) || taps < 0) return -1;
  if (taps && (!taps_w || !positions || !slots || (taps > 1 && (!history || !epoch)))) return -1;
  if (!slots || ((ldr_in | lds_in | ldr_out | lds_out | ldy) % 4) || odd16(x_in) || odd16(x_out) || odd16(y) || odd16(taps_w) || odd16(history) || odd16(w)) return -1;
  const Linear p{(const bf16*)w, N, K, z, ldz, out_f32, act, T};
  const StreamsIn q{x_in, ldr_in, lds_in, x_out, ldr_out, lds_out, y, ldy, mix, out, in, gain, eps, taps_w, taps, history, epoch, positions, slots, S};
  return by_rows<LaunchStreams, const Linear&, const StreamsIn&>(T, N, p, q, (cudaStream_t)stream);
}

// z (f32) = [x's first K1 columns | finished recurrence (ifab_gr_finish), zero up to K] w^T for T <= 2 rows; e and the groups' columns multiples of 4
extern "C" int ifab_gemv_mixed(const void* x, long ldx, int K1, const float* o, long ldo, int H, int e, int E, const float* m, const void* v, const float* skip,
                               const void* gate, long ldg, int gate_act, int gate_first, int groups, float eps, const float* gain, const void* w, float* z, long ldz,
                               int T, int N, int K, void* stream) {
  if (T < 1 || T > 2 || N < 1 || K < 8 || K % 8 || K1 < 0 || K1 % 8 || H < 1 || e < 1 || K < K1 + H * e || groups < 1 || (H * e) % groups || (e % 4) || (H * e / groups) % 4) return -1;
  if (!gate || !gain || (skip && !v) || (m && E <= e) || (K1 && (!x || ldx % 8 || odd16(x))) || ldg % 4 || (reinterpret_cast<uintptr_t>(gate) & 7) || odd16(gain) || odd16(w) || odd16(v))
    return -1;
  const Linear p{(const bf16*)w, N, K, z, ldz, 1, 0, T};
  const MixedIn q{(const bf16*)x, ldx, K1, o, ldo, H, e, E, m, (const bf16*)v, skip, (const bf16*)gate, ldg, gate_act, gate_first, groups, eps, gain};
  return by_rows<LaunchMixed, const Linear&, const MixedIn&>(T, N, p, q, (cudaStream_t)stream);
}

// ifab_gr_prepare and ifab_gr_step in one launch (bf16, d a multiple of 4 up to 256). cols, channels: of q, k, v
extern "C" int ifab_gr_decode(const void* proj, long ldp, const int32_t* cols, const int32_t* channels, int unit, float q_factor, const float* taps_w, const float* bias,
                              int taps, int C, void* history, int kind, int H, int G, int d, int e, int decay_col, int weight_col, const float* a_log,
                              const float* decay_bias, const float* weight_bias, float cap, float* state, float* m_state, const int32_t* epoch, void* v, float* m_rows,
                              const int32_t* positions, const int32_t* slots, float* o, long ldo, int T, void* stream) {
  const int E = e + (kind == GR_MEMORY);
  if (T < 1 || T > 65535 || kind < GR_SSD || kind > GR_MEMORY || H < 1 || H > 65535 || G < 1 || H % G || d < 4 || d > 256 || d % 4 || e < 1 || E > 1024 || !epoch) return -1;
  if (taps < 0 || (taps && !taps_w) || (taps > 1 && !history) || (kind == GR_MEMORY ? cap <= 0.f || !m_state || !m_rows : !a_log)) return -1;
  DecodeParams p{(const bf16*)proj, ldp, {cols[0], cols[1], cols[2]}, {channels[0], channels[1], channels[2]}, taps_w, bias, taps, C, (bf16*)history, decay_col, weight_col,
                 a_log, decay_bias, weight_bias, cap, unit, q_factor, kind, H, G, d, e, E, {state, m_state, epoch}, (bf16*)v, o, ldo, m_rows, positions, slots, T};
  const dim3 grid(H, T, (E + 31) / 32);
  return d <= 128 ? launch_chain(gr_decode_kernel<1>, grid, dim3(256), 0, (cudaStream_t)stream, p) : launch_chain(gr_decode_kernel<2>, grid, dim3(256), 0, (cudaStream_t)stream, p);
}
