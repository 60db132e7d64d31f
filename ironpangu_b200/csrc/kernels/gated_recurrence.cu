// Recurrences over a matrix state per head with a decay per token, for any head sizes; states, gates and products in f32:
//
//   SSD      S = a S + w k v^T                                   o = S^T q      (state-space duality: a = exp(-exp(A) dt), w = dt)
//   DELTA    S = a S,  u = w (v - S^T k),  S += k u^T            o = S^T q      (gated delta rule: w = beta)
//   MEMORY   m' = max(f + m, i),  S = exp(f + m - m') S + exp(i - m') k v^T     (exponential gates; one more value column of ones keeps
//            the sum of the keys, so that S^T q ends with n q)
//
//   gr_prepare_kernel  packed projection rows -> q, k, v (short causal convolution + SiLU) in the activation type, the factors that make q and k
//                      unit vectors, and the gates (softplus, exponentials, soft limits). The convolution reads rows of the step and the
//                      sequence's last taps - 1 rows before it (history [slots, 2, taps - 1, C] in the activation type, two sides by epoch as in
//                      hyper_streams.cu)
//   gr_step_kernel     decode: one CTA per (head, run of rows of one slot, 32 value columns); a run walks its rows through the state.
//                      The grid depends on the row count only (graph capture)
//   prompts, by chunks of 64 consecutive rows of one sequence with f32 products (the tensor-core form: gated_tiles.cu):
//     gr_maximum_kernel  MEMORY: the running maximum of every row
//     gr_state_kernel    what a chunk adds to the state; gr_scan_kernel: the states ahead of every chunk (DELTA: gated_delta.cu)
//     gr_out_kernel      the outputs of a chunk from the state ahead of it and from its rows
//   gr_finish_kernel   o -> the operand of the output projection: the division of MEMORY, a skip D v, gate before or after a norm over
//                      equal groups of columns, a gain per column
//
// The state is [slots, H, E, d] (a row of it meets q and k), one per sequence slot; a row at position 0 starts from zero whatever the
// slot held before.
#include "gated_recurrence.cuh"

using namespace ifab;

namespace {

struct Section {
  int col, heads, n;          // where it starts in a projection row, heads and columns of a head
  int channel;                // of the convolution, -1: none
  void* dst;                  // [T, heads * n]
  float* factors; float factor;      // [T, heads]: factor / sqrt(sum of squares + 1e-6); or null
};

struct PrepareParams {
  const void* proj; long ldp;
  Section sec[3];
  const float *taps_w, *bias; int taps, C;      // [taps, C] (last: the current row's), [C] or null
  void* history; const int32_t* epoch;
  int kind, H, decay_col, weight_col;
  const float *a_log, *decay_bias, *weight_bias; float cap;
  float *log_decay, *weight;
  const int32_t *positions, *slots;
  int T, rows;                // rows of a CTA
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

template <typename A, int V>
__device__ __forceinline__ void load_v(const A* p, float* f) {
  if constexpr (V == 4 && sizeof(A) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    f[0] = to_f32(*p);
  }
}
template <typename A, int V>
__device__ __forceinline__ void store_v(A* p, const float* f) {
  if constexpr (V == 4 && sizeof(A) == 2) {
    __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  } else if constexpr (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    *p = from_f32<A>(f[0]);
  }
}

// grid (ceil(heads of all sections / 8) + 1, ceil(T / rows)), 256 threads: a warp per head, V columns per lane at a time; the last CTAs make the gates
template <typename A, int V>
__global__ void __launch_bounds__(256) gr_prepare_kernel(PrepareParams p) {
  grid_dep_launch();
  grid_dep_wait();
  const int t0 = blockIdx.y * p.rows, t1 = min(p.T, t0 + p.rows), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (blockIdx.x == gridDim.x - 1) {
    for (int i = threadIdx.x; i < (t1 - t0) * p.H; i += 256) {
      const int t = t0 + i / p.H, h = i % p.H;
      const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
      const float a = to_f32(row[p.decay_col + h]) + (p.decay_bias ? p.decay_bias[h] : 0.f), b = to_f32(row[p.weight_col + h]) + (p.weight_bias ? p.weight_bias[h] : 0.f);
      float g, w;
      if (p.kind == GR_MEMORY) {
        g = -softplus(-p.cap * tanhf(a / p.cap));
        w = p.cap * tanhf(b / p.cap);
      } else {
        const float sp = softplus(a);
        g = -expf(p.a_log[h]) * sp;
        w = p.kind == GR_SSD ? sp : sigmoid_f32(b);
      }
      p.log_decay[(long)t * p.H + h] = g;
      p.weight[(long)t * p.H + h] = w;
    }
    return;
  }
  // what the rows need to know: rows of their sequence ahead of them in the step, position, slot, whether they are its last
  __shared__ int run_of[8], pos_of[8], slot_of[8], last_of[8], side_of[8];
  const int back = p.taps - 1;
  if ((int)threadIdx.x < t1 - t0) {
    const int t = t0 + threadIdx.x, slot = p.slots[t];
    int run = 0;
    while (run < back && t - run - 1 >= 0 && p.slots[t - run - 1] == slot) ++run;
    run_of[threadIdx.x] = run;
    pos_of[threadIdx.x] = p.positions[t];
    slot_of[threadIdx.x] = slot;
    last_of[threadIdx.x] = p.taps > 1 && (t + 1 == p.T || p.slots[t + 1] != slot);
    side_of[threadIdx.x] = p.taps > 1 ? p.epoch[slot] & 1 : 0;
  }
  __syncthreads();
  const int i = blockIdx.x * 8 + warp, h0 = p.sec[0].heads, h1 = h0 + p.sec[1].heads;
  if (i >= h1 + p.sec[2].heads) return;
  const Section& s = p.sec[i < h0 ? 0 : i < h1 ? 1 : 2];
  const int h = i - (i < h0 ? 0 : i < h1 ? h0 : h1);
  float sum[8];
#pragma unroll
  for (int z = 0; z < 8; ++z) sum[z] = 0.f;
  // eight rows in the middle of a run: every input is loaded once
  if (t1 - t0 == 8 && run_of[0] == back && run_of[7] == back && slot_of[0] == slot_of[7] && pos_of[0] >= 0 && p.taps <= 4 && s.channel >= 0) {
    const A* row = reinterpret_cast<const A*>(p.proj) + (long)t0 * p.ldp + s.col + h * s.n;
    A* dst = reinterpret_cast<A*>(s.dst) + ((long)t0 * s.heads + h) * s.n;
    A* fresh = reinterpret_cast<A*>(p.history) + ((long)slot_of[0] * 2 + (side_of[0] ^ 1)) * back * p.C + s.channel + h * s.n;
    for (int c = lane * V; c < s.n; c += 32 * V) {
      float x[11][V], w[4][V], bias[V];        // x[3 + z]: of row z
#pragma unroll
      for (int z = 0; z < 11; ++z)
        if (z >= 3 - back) load_v<A, V>(row + (long)(z - 3) * p.ldp + c, x[z]);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j < p.taps) load_v<float, V>(p.taps_w + (long)(back - j) * p.C + s.channel + h * s.n + c, w[j]);
#pragma unroll
      for (int u = 0; u < V; ++u) bias[u] = 0.f;
      if (p.bias) load_v<float, V>(p.bias + s.channel + h * s.n + c, bias);
#pragma unroll
      for (int z = 0; z < 8; ++z) {
        float v[V];
#pragma unroll
        for (int u = 0; u < V; ++u) {
          float acc = bias[u];
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j < p.taps) acc = fmaf(w[j][u], x[3 + z - j][u], acc);
          v[u] = to_f32(from_f32<A>(acc * sigmoid_f32<sizeof(A) == 2>(acc)));
          sum[z] = fmaf(v[u], v[u], sum[z]);
        }
        store_v<A, V>(dst + (long)z * s.heads * s.n + c, v);
      }
      if (last_of[7])
#pragma unroll
        for (int j = 0; j < 3; ++j)
          if (j < back) store_v<A, V>(fresh + (long)j * p.C + c, x[10 - j]);
    }
  } else
  for (int c = lane * V; c < s.n; c += 32 * V) {
    float w0[V], bias[V];
    if (s.channel >= 0) {
      load_v<float, V>(p.taps_w + (long)back * p.C + s.channel + h * s.n + c, w0);
      if (p.bias) load_v<float, V>(p.bias + s.channel + h * s.n + c, bias);
    }
#pragma unroll
    for (int z = 0; z < 8; ++z) {
      const int t = t0 + z, pos = t < t1 ? pos_of[z] : -1;
      if (pos < 0) continue;
      const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp + s.col + h * s.n;
      A* dst = reinterpret_cast<A*>(s.dst) + ((long)t * s.heads + h) * s.n;
      float v[V];
      load_v<A, V>(row + c, v);
      if (s.channel >= 0) {
        const int run = run_of[z], ch = s.channel + h * s.n + c;
        const bool last = last_of[z];
        A* fresh = reinterpret_cast<A*>(p.history) + ((long)slot_of[z] * 2 + (side_of[z] ^ 1)) * back * p.C + ch;
        const A* old = reinterpret_cast<const A*>(p.history) + ((long)slot_of[z] * 2 + side_of[z]) * back * p.C + ch;
        float w[V], x[V], acc[V];
#pragma unroll
        for (int u = 0; u < V; ++u) acc[u] = v[u] * w0[u];
        if (last) store_v<A, V>(fresh, v);
        for (int j = 1; j < p.taps; ++j) {
          if (j <= pos) {
            load_v<A, V>(j <= run ? row + c - (long)j * p.ldp : old + (long)(j - run - 1) * p.C, x);
            load_v<float, V>(p.taps_w + (long)(back - j) * p.C + ch, w);
#pragma unroll
            for (int u = 0; u < V; ++u) acc[u] = fmaf(w[u], x[u], acc[u]);
          } else {
#pragma unroll
            for (int u = 0; u < V; ++u) x[u] = 0.f;
          }
          if (last && j < back) store_v<A, V>(fresh + (long)j * p.C, x);
        }
        if (p.bias) {
#pragma unroll
          for (int u = 0; u < V; ++u) acc[u] += bias[u];
        }
#pragma unroll
        for (int u = 0; u < V; ++u) v[u] = to_f32(from_f32<A>(acc[u] * sigmoid_f32<sizeof(A) == 2>(acc[u])));
      }
      store_v<A, V>(dst + c, v);
#pragma unroll
      for (int u = 0; u < V; ++u) sum[z] = fmaf(v[u], v[u], sum[z]);
    }
  }
  if (s.factors) {
#pragma unroll
    for (int z = 0; z < 8; ++z) {
      if (t0 + z >= t1 || pos_of[z] < 0) continue;
      const float ss = warp_sum(sum[z]);
      if (lane == 0) s.factors[(long)(t0 + z) * s.heads + h] = s.factor / sqrtf(ss + 1e-6f);
    }
  }
}

struct StepParams {
  GrRows r;
  GrState st;
  const int32_t *positions, *slots;
  float* o; long ldo;
  float* m_rows;              // MEMORY: [T, H]
  int T;
};

// a warp owns 4 value columns = rows of the state, lanes their d columns (float4s: REG of them per lane; 0: any d, one column at a time)
template <typename A, int REG>
__global__ void __launch_bounds__(256) gr_step_kernel(StepParams p) {
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int h = blockIdx.x, t0 = blockIdx.y, lane = threadIdx.x & 31, col0 = blockIdx.z * 32 + (threadIdx.x >> 5) * 4, d = r.d, g = h / (r.H / r.G);
  const int slot = p.slots[t0];
  if (p.positions[t0] < 0 || (t0 > 0 && p.slots[t0 - 1] == slot && p.positions[t0 - 1] >= 0)) return;      // not the head of a run
  const int nc = min(4, r.E - col0);
  if (nc <= 0) return;
  float* S = p.st.s + (((long)slot * r.H + h) * r.E + col0) * d;
  const int side = r.kind == GR_MEMORY ? p.st.epoch[slot] & 1 : 0;
  const bool empty = p.positions[t0] == 0;
  float m = r.kind == GR_MEMORY && !empty ? p.st.m[((long)slot * 2 + side) * r.H + h] : 0.f;
  constexpr int R = REG ? REG : 1;
  float4 s[4][R];
  if (REG) {
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
      for (int x = 0; x < R; ++x) {
        const int c = (lane + 32 * x) * 4;
        s[u][x] = (u < nc && c < d && !empty) ? *reinterpret_cast<const float4*>(S + (long)u * d + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
  }
  bool first = empty;
  for (int t = t0; t < p.T && p.slots[t] == slot && p.positions[t] >= 0; ++t) {
    const A *q = reinterpret_cast<const A*>(r.q) + ((long)t * r.G + g) * d, *k = reinterpret_cast<const A*>(r.k) + ((long)t * r.G + g) * d;
    const float fq = r.qs ? r.qs[(long)t * r.G + g] : r.q_factor, fk = r.ks ? r.ks[(long)t * r.G + g] : 1.f;
    const float ld = r.log_decay[(long)t * r.H + h];
    float w = r.weight[(long)t * r.H + h], a;
    if (r.kind == GR_MEMORY) {
      const float mn = fmaxf(ld + m, w);
      a = expf(ld + m - mn);
      w = expf(w - mn);
      m = mn;
      if (blockIdx.z == 0 && threadIdx.x == 0) p.m_rows[(long)t * r.H + h] = m;
    } else {
      a = expf(ld);
    }
    float v[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int u = 0; u < 4; ++u) v[u] = u < nc ? gr_v<A>(r, t, h, col0 + u) : 0.f;
    if (REG) {
      float4 kr[R], qr[R];
#pragma unroll
      for (int x = 0; x < R; ++x) {
        const int c = (lane + 32 * x) * 4;
        float a4[4] = {0.f, 0.f, 0.f, 0.f}, b4[4] = {0.f, 0.f, 0.f, 0.f};
        if (c < d) {
          load_v<A, 4>(k + c, a4);
          load_v<A, 4>(q + c, b4);
        }
        kr[x] = make_float4(a4[0] * fk, a4[1] * fk, a4[2] * fk, a4[3] * fk);
        qr[x] = make_float4(b4[0] * fq, b4[1] * fq, b4[2] * fq, b4[3] * fq);
      }
      float kk[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        kk[u] = 0.f;
#pragma unroll
        for (int x = 0; x < R; ++x) {
          s[u][x].x *= a; s[u][x].y *= a; s[u][x].z *= a; s[u][x].w *= a;
          if (r.kind == GR_DELTA) kk[u] = fmaf(kr[x].x, s[u][x].x, fmaf(kr[x].y, s[u][x].y, fmaf(kr[x].z, s[u][x].z, fmaf(kr[x].w, s[u][x].w, kk[u]))));
        }
      }
      if (r.kind == GR_DELTA) {
#pragma unroll
        for (int u = 0; u < 4; ++u) v[u] -= warp_sum(kk[u]);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float wv = w * v[u];
#pragma unroll
        for (int x = 0; x < R; ++x) {
          s[u][x].x = fmaf(kr[x].x, wv, s[u][x].x);
          s[u][x].y = fmaf(kr[x].y, wv, s[u][x].y);
          s[u][x].z = fmaf(kr[x].z, wv, s[u][x].z);
          s[u][x].w = fmaf(kr[x].w, wv, s[u][x].w);
          acc[u] = fmaf(qr[x].x, s[u][x].x, fmaf(qr[x].y, s[u][x].y, fmaf(qr[x].z, s[u][x].z, fmaf(qr[x].w, s[u][x].w, acc[u]))));
        }
      }
    } else {
      if (r.kind == GR_DELTA && !first) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          float kk = 0.f;
          for (int c = lane; c < d && u < nc; c += 32) kk = fmaf(to_f32(k[c]) * fk, S[(long)u * d + c], kk);
          v[u] = fmaf(-a, warp_sum(kk), v[u]);
        }
      }
      for (int c = lane; c < d; c += 32)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (u >= nc) break;
          const float x = fmaf(to_f32(k[c]) * fk, w * v[u], first ? 0.f : a * S[(long)u * d + c]);
          S[(long)u * d + c] = x;
          acc[u] = fmaf(to_f32(q[c]) * fq, x, acc[u]);
        }
    }
    first = false;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float x = warp_sum(acc[u]);
      if (lane == 0 && u < nc) p.o[(long)t * p.ldo + (long)h * r.E + col0 + u] = x;
    }
  }
  if (REG) {
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
      for (int x = 0; x < R; ++x) {
        const int c = (lane + 32 * x) * 4;
        if (u < nc && c < d) *reinterpret_cast<float4*>(S + (long)u * d + c) = s[u][x];
      }
  }
  if (r.kind == GR_MEMORY && blockIdx.z == 0 && threadIdx.x == 0) p.st.m[((long)slot * 2 + (side ^ 1)) * r.H + h] = m;
}

// grid (H, chunks), 256 threads: CTAs of a run's first chunk walk its rows, 2048 at a time. m_t = G_t + max(m_0, max over j <= t of (i_j - G_j)), G the sums of f
__global__ void __launch_bounds__(256) gr_maximum_kernel(GrChunks p, GrState st) {
  constexpr int R = 8;
  __shared__ double sums[8], tops[8];
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, c = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, meta = p.chunks[c * 4 + 3];
  if (!(meta & 1)) return;
  const int row0 = p.chunks[c * 4], slot = p.chunks[c * 4 + 2], count = meta >> 1, lc = c + count - 1;
  const int n = p.chunks[lc * 4] + p.chunks[lc * 4 + 1] - row0, side = st.epoch[slot] & 1;
  const GrRows& r = p.r;
  double sum = 0.0, best = p.positions[row0] == 0 ? 0.0 : (double)st.m[((long)slot * 2 + side) * r.H + h];
  for (int t0 = 0; t0 < n; t0 += 256 * R) {
    const int t = t0 + threadIdx.x * R;
    float f[R], in[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const long at = (long)(row0 + min(t + i, n - 1)) * r.H + h;
      f[i] = t + i < n ? r.log_decay[at] : 0.f;
      in[i] = t + i < n ? r.weight[at] : -INFINITY;
    }
    double G = 0.0, b = -INFINITY;      // of this thread's rows, from their start
#pragma unroll
    for (int i = 0; i < R; ++i) {
      G += (double)f[i];
      b = fmax(b, (double)in[i] - G);
    }
    // of everything up to and with this thread's rows: sums add, a later maximum is moved back by the sums ahead of it
    double GS = G, bS = b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double g = __shfl_up_sync(0xffffffffu, GS, o), x = __shfl_up_sync(0xffffffffu, bS, o);
      if (lane >= o) {
        bS = fmax(x, bS - g);
        GS += g;
      }
    }
    __syncthreads();
    if (lane == 31) {
      sums[warp] = GS;
      tops[warp] = bS;
    }
    __syncthreads();
    double ahead = sum, top = best;     // up to this thread's rows
    for (int w = 0; w < warp; ++w) {
      top = fmax(top, tops[w] - ahead);
      ahead += sums[w];
    }
    const double gl = __shfl_up_sync(0xffffffffu, GS, 1), bl = __shfl_up_sync(0xffffffffu, bS, 1);
    if (lane > 0) {
      top = fmax(top, bl - ahead);
      ahead += gl;
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      ahead += (double)f[i];
      top = fmax(top, (double)in[i] - ahead);
      if (t + i < n) r.m[(long)(row0 + t + i) * r.H + h] = (float)(ahead + top);
      if (t + i == n - 1) st.m[((long)slot * 2 + (side ^ 1)) * r.H + h] = (float)(ahead + top);
    }
    for (int w = 0; w < 8; ++w) {
      best = fmax(best, tops[w] - sum);
      sum += sums[w];
    }
  }
}

// grid (n, H, tiles of 64 x 64 of the state): sum over the chunk's rows of (weight at the chunk's end) k_j v_j^T
template <typename A>
__global__ void __launch_bounds__(256) gr_state_kernel(GrChunks p, GrState st) {
  __shared__ float ks[GR_CHUNK][68], vs[GR_CHUNK][68];
  __shared__ GrFactors<GR_CHUNK> f;
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int c = blockIdx.x, h = blockIdx.y, te = (r.E + 63) / 64, d0 = blockIdx.z / te * 64, e0 = blockIdx.z % te * 64, g = h / (r.H / r.G);
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  gr_load_factors(p, c, h, st, f);
  if (threadIdx.x < GR_CHUNK) {
    const int j = threadIdx.x;
    vs[j][64] = j < L ? gr_pair(f, L - 1, j) : 0.f;
    if (j == 0 && blockIdx.z == 0) p.cdecay[(long)c * r.H + h] = gr_carry(f, L - 1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < GR_CHUNK * 64; i += 256) {
    const int j = i >> 6, x = i & 63;
    ks[j][x] = (j < L && d0 + x < r.d) ? gr_k<A>(r, row0 + j, g, d0 + x) * vs[j][64] : 0.f;
    vs[j][x] = (j < L && e0 + x < r.E) ? gr_v<A>(r, row0 + j, h, e0 + x) : 0.f;
  }
  __syncthreads();
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int j = 0; j < L; ++j) {
    const float4 a = *reinterpret_cast<const float4*>(&vs[j][ty * 4]), b = *reinterpret_cast<const float4*>(&ks[j][tx * 4]);
    const float ar[4] = {a.x, a.y, a.z, a.w}, br[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int y = 0; y < 4; ++y)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[y][x] = fmaf(ar[y], br[x], acc[y][x]);
  }
  float* out = p.cstate + ((long)c * r.H + h) * r.d * r.E;
#pragma unroll
  for (int y = 0; y < 4; ++y) {
    const int e = e0 + ty * 4 + y, x0 = d0 + tx * 4;
    if (e >= r.E) break;
    if (r.d % 4 == 0) {
      if (x0 < r.d) *reinterpret_cast<float4*>(out + (long)e * r.d + x0) = make_float4(acc[y][0], acc[y][1], acc[y][2], acc[y][3]);
    } else {
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (x0 + x < r.d) out[(long)e * r.d + x0 + x] = acc[y][x];
    }
  }
}

// grid (ceil(H * d * E / 256), n): CTAs of a run's first chunk walk its chunks; cstate becomes the state AHEAD of the chunk
template <int V>
__global__ void __launch_bounds__(256) gr_scan_kernel(GrChunks p, float* state) {
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int first = blockIdx.y, count = p.chunks[first * 4 + 3] >> 1;
  if (!(p.chunks[first * 4 + 3] & 1)) return;
  const long sz = (long)r.d * r.E, total = (long)r.H * sz, i = ((long)blockIdx.x * 256 + threadIdx.x) * V;
  if (i >= total) return;
  const float* dec = p.cdecay + (long)first * r.H + i / sz;
  float* st = state + (long)p.chunks[first * 4 + 2] * total + i;
  float* cs = p.cstate + (long)first * total + i;
  const bool fresh = p.positions[p.chunks[first * 4]] == 0;
  __align__(16) float s[V];
#pragma unroll
  for (int x = 0; x < V; ++x) s[x] = fresh ? 0.f : st[x];
  constexpr int AHEAD = 8;
  for (int c0 = 0; c0 < count; c0 += AHEAD) {
    __align__(16) float add[AHEAD][V];
    float f[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < count) {
        if (V == 4) *reinterpret_cast<float4*>(add[u]) = *reinterpret_cast<const float4*>(cs + (long)(c0 + u) * total);
        else add[u][0] = cs[(long)(c0 + u) * total];
        f[u] = dec[(long)(c0 + u) * r.H];
      }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < count) {
        if (V == 4) *reinterpret_cast<float4*>(cs + (long)(c0 + u) * total) = *reinterpret_cast<const float4*>(s);
        else cs[(long)(c0 + u) * total] = s[0];
#pragma unroll
        for (int x = 0; x < V; ++x) s[x] = fmaf(f[u], s[x], add[u][x]);
      }
  }
#pragma unroll
  for (int x = 0; x < V; ++x) st[x] = s[x];
}

// grid (n, H, ceil(E / 64)): o_i = carry_i S^T q_i + sum over j <= i of pair(i, j) (q_i . k_j) v_j
template <typename A, typename AV>
__global__ void __launch_bounds__(256) gr_out_kernel(GrChunks p, GrState st) {
  extern __shared__ float sm[];
  __shared__ GrFactors<GR_CHUNK> f;
  float(*qs)[68] = reinterpret_cast<float(*)[68]>(sm);                 // [column of q][row], one 64-column slice
  float(*ks)[68] = reinterpret_cast<float(*)[68]>(sm + 64 * 68);       // [column of k][row]; then v rows
  float(*ss)[68] = reinterpret_cast<float(*)[68]>(sm + 2 * 64 * 68);   // a slice of the state; then the weights [j][i]
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int c = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * 64, g = h / (r.H / r.G);
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  gr_load_factors(p, c, h, st, f);
  const float* S = p.cstate + ((long)c * r.H + h) * r.d * r.E;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float w[4][4] = {}, acc[4][4] = {};
  for (int d0 = 0; d0 < r.d; d0 += 64) {
    __syncthreads();
    for (int i = threadIdx.x; i < GR_CHUNK * 64; i += 256) {
      const int j = i >> 6, x = i & 63;
      const bool ok = j < L && d0 + x < r.d;
      qs[x][j] = ok ? gr_q<A>(r, row0 + j, g, d0 + x) : 0.f;
      ks[x][j] = ok ? gr_k<A>(r, row0 + j, g, d0 + x) : 0.f;
      ss[x][j] = (d0 + x < r.d && e0 + j < r.E) ? S[(long)(e0 + j) * r.d + d0 + x] : 0.f;
    }
    __syncthreads();
    const int n = min(64, r.d - d0);
    for (int x = 0; x < n; ++x) {
      const float4 a = *reinterpret_cast<const float4*>(&qs[x][ty * 4]), b = *reinterpret_cast<const float4*>(&ks[x][tx * 4]),
                   s = *reinterpret_cast<const float4*>(&ss[x][tx * 4]);
      const float ar[4] = {a.x, a.y, a.z, a.w}, br[4] = {b.x, b.y, b.z, b.w}, sr[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
      for (int y = 0; y < 4; ++y)
#pragma unroll
        for (int z = 0; z < 4; ++z) {
          w[y][z] = fmaf(ar[y], br[z], w[y][z]);
          acc[y][z] = fmaf(ar[y], sr[z], acc[y][z]);
        }
    }
  }
  __syncthreads();
#pragma unroll
  for (int y = 0; y < 4; ++y) {
    const int i = ty * 4 + y;
    const float carry = gr_carry(f, i < L ? i : 0);
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      const int j = tx * 4 + z;
      acc[y][z] *= carry;
      ss[j][i] = (j <= i && i < L) ? w[y][z] * gr_pair(f, i, j) : 0.f;
    }
  }
  for (int i = threadIdx.x; i < GR_CHUNK * 64; i += 256) {
    const int j = i >> 6, x = i & 63;
    ks[j][x] = (j < L && e0 + x < r.E) ? gr_v<AV>(r, row0 + j, h, e0 + x) : 0.f;
  }
  __syncthreads();
  for (int j = 0; j < L; ++j) {
    const float4 a = *reinterpret_cast<const float4*>(&ss[j][ty * 4]), b = *reinterpret_cast<const float4*>(&ks[j][tx * 4]);
    const float ar[4] = {a.x, a.y, a.z, a.w}, br[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int y = 0; y < 4; ++y)
#pragma unroll
      for (int z = 0; z < 4; ++z) acc[y][z] = fmaf(ar[y], br[z], acc[y][z]);
  }
#pragma unroll
  for (int y = 0; y < 4; ++y)
#pragma unroll
    for (int z = 0; z < 4; ++z)
      if (ty * 4 + y < L && e0 + tx * 4 + z < r.E) p.o[(long)(row0 + ty * 4 + y) * p.ldo + (long)h * r.E + e0 + tx * 4 + z] = acc[y][z];
}

struct FinishParams {
  const float* o; long ldo; int H, e, E;       // heads of e columns at stride E in a row
  const float *m;                              // MEMORY: [T, H]
  const void* v; const float* skip;            // SSD: [T, H * e] and D [H], or null
  const void* gate; long ldg; int act, gate_first;
  int groups; float eps; const float* gain;    // [H * e]
  void* y; long ldy;
};

// grid (CTAs of a row's groups, T), 256 threads; WPG warps per group
template <typename A, int WPG>
__global__ void __launch_bounds__(256) gr_finish_kernel(FinishParams p) {
  __shared__ float red[33];
  extern __shared__ float den[];               // MEMORY: 1 / the denominator of every head
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.y, n = p.H * p.e / p.groups;
  const float* o = p.o + (long)t * p.ldo;
  const A* gate = reinterpret_cast<const A*>(p.gate) + (long)t * p.ldg;
  if (p.m) {
    for (int h = threadIdx.x; h < p.H; h += 256) den[h] = 1.f / (fmaxf(fabsf(o[(long)h * p.E + p.e]), expf(-p.m[(long)t * p.H + h])) + 1e-6f);
    __syncthreads();
  }
  auto value = [&](int c, float* g) {
    const int h = c / p.e, j = c - h * p.e;
    float x = o[(long)h * p.E + j];
    if (p.m) x *= den[h];
    if (p.skip) x = fmaf(p.skip[h], to_f32(reinterpret_cast<const A*>(p.v)[((long)t * p.H + h) * p.e + j]), x);
    *g = activate<sizeof(A) == 2>(to_f32(gate[c]), p.act);
    return p.gate_first ? x * *g : x;
  };
  constexpr int TPG = 32 * WPG, GPB = 8 / WPG;
  for (int g0 = blockIdx.x * GPB; g0 < p.groups; g0 += gridDim.x * GPB) {
    const int g = g0 + threadIdx.x / TPG, i0 = threadIdx.x % TPG;
    if (WPG == 1 && g >= p.groups) break;
    float ss = 0.f, z;
    for (int c = i0; c < n; c += TPG) {
      const float x = value(g * n + c, &z);
      ss = fmaf(x, x, ss);
    }
    ss = WPG == 1 ? warp_sum(ss) : block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)n + p.eps);
    for (int c = i0; c < n; c += TPG) {
      const float x = value(g * n + c, &z) * inv * p.gain[g * n + c];
      reinterpret_cast<A*>(p.y)[(long)t * p.ldy + g * n + c] = from_f32<A>(p.gate_first ? x : x * z);
    }
  }
}

// One CTA per row and group, the values in registers between the sum and the stores; whole chunks of 4 columns. ITER: chunks of a thread
template <typename A, int ITER>
__global__ void __launch_bounds__(256) gr_finish_wide_kernel(FinishParams p) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.y, n = p.H * p.e / p.groups, base = blockIdx.x * n;
  const float* o = p.o + (long)t * p.ldo;
  const A* gate = reinterpret_cast<const A*>(p.gate) + (long)t * p.ldg;
  float x[ITER][4], z[ITER][4], ss = 0.f;
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int k = (threadIdx.x + i * 256) * 4, c = base + k;
    if (k >= n) break;
    const int h = c / p.e, j = c - h * p.e;
    load_v<float, 4>(o + (long)h * p.E + j, x[i]);
    load_v<A, 4>(gate + c, z[i]);
    if (p.skip) {
      float v[4];
      load_v<A, 4>(reinterpret_cast<const A*>(p.v) + (long)t * p.H * p.e + c, v);
#pragma unroll
      for (int u = 0; u < 4; ++u) x[i][u] = fmaf(p.skip[h], v[u], x[i][u]);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      z[i][u] = activate<sizeof(A) == 2>(z[i][u], p.act);
      if (p.gate_first) x[i][u] *= z[i][u];
      ss = fmaf(x[i][u], x[i][u], ss);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)n + p.eps);
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int k = (threadIdx.x + i * 256) * 4, c = base + k;
    if (k >= n) break;
    float g[4];
    load_v<float, 4>(p.gain + c, g);
#pragma unroll
    for (int u = 0; u < 4; ++u) g[u] *= x[i][u] * inv * (p.gate_first ? 1.f : z[i][u]);
    store_v<A, 4>(reinterpret_cast<A*>(p.y) + (long)t * p.ldy + c, g);
  }
}

bool rows_ok(const GrRows& r) {
  return r.kind >= GR_SSD && r.kind <= GR_MEMORY && r.H >= 1 && r.G >= 1 && r.H % r.G == 0 && r.d >= 1 && r.e >= 1 && r.E == r.e + (r.kind == GR_MEMORY) && r.d <= 1024 &&
         r.E <= 1024 && r.H <= 65535;
}

}  // namespace

int ifab::gr_maximum(const GrChunks& p, const GrState& st, cudaStream_t s) { return launch_chain(gr_maximum_kernel, dim3(p.r.H, p.n), dim3(256), 0, s, p, st); }

int ifab::gr_scan(const GrChunks& p, const GrState& st, cudaStream_t s) {
  const long total = (long)p.r.H * p.r.d * p.r.E;
  if ((long)p.r.d * p.r.E % 4 == 0) return launch_chain(gr_scan_kernel<4>, dim3((unsigned)((total + 1023) / 1024), p.n), dim3(256), 0, s, p, st.s);
  return launch_chain(gr_scan_kernel<1>, dim3((unsigned)((total + 255) / 256), p.n), dim3(256), 0, s, p, st.s);
}

// Sections q, k, v: {column, heads, columns of a head, convolution channel or -1}. factors: of q and k [T, heads] (DELTA), or null. History in the type of proj.
extern "C" int ifab_gr_prepare(const void* proj, long ldp, int f32, const int32_t* sections, void* q, void* k, void* v, float* q_factors, float* k_factors, float q_factor,
                               const float* taps_w, const float* bias, int taps, int C, void* history, const int32_t* epoch, int kind, int H, int decay_col,
                               int weight_col, const float* a_log, const float* decay_bias, const float* weight_bias, float cap, float* log_decay, float* weight,
                               const int32_t* positions, const int32_t* slots, int T, void* stream) {
  if (T < 1 || H < 1 || taps < 0 || taps > 64 || (taps && !taps_w) || (taps > 1 && (!history || !epoch)) || kind < GR_SSD || kind > GR_MEMORY || (kind == GR_MEMORY ? cap <= 0.f : !a_log))
    return -1;
  PrepareParams p{proj, ldp, {}, taps_w, bias, taps, C, history, epoch, kind, H, decay_col, weight_col, a_log, decay_bias, weight_bias, cap, log_decay, weight,
                  positions, slots, T, T <= 256 ? 1 : 8};
  void* dst[3] = {q, k, v};
  float* factors[3] = {q_factors, k_factors, nullptr};
  const auto odd = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; };
  bool four = !((ldp | C) % 4) && !odd(proj) && !odd(history) && !odd(taps_w) && !odd(bias);
  int heads = 0;
  for (int i = 0; i < 3; ++i) {
    const int32_t* s = sections + 4 * i;
    if (s[0] < 0 || s[1] < 1 || s[2] < 1 || (s[3] >= 0 && (!taps || s[3] + s[1] * s[2] > C))) return -1;
    p.sec[i] = Section{s[0], s[1], s[2], s[3], dst[i], factors[i], i == 0 ? q_factor : 1.f};
    four = four && !((s[0] | s[2] | (s[3] < 0 ? 0 : s[3])) % 4) && !odd(dst[i]);
    heads += s[1];
  }
  const dim3 grid((heads + 7) / 8 + 1, (T + p.rows - 1) / p.rows);
  cudaStream_t s = (cudaStream_t)stream;
  if (grid.y > 65535) return -1;
  if (four) return f32 ? launch_chain(gr_prepare_kernel<float, 4>, grid, dim3(256), 0, s, p) : launch_chain(gr_prepare_kernel<bf16, 4>, grid, dim3(256), 0, s, p);
  return f32 ? launch_chain(gr_prepare_kernel<float, 1>, grid, dim3(256), 0, s, p) : launch_chain(gr_prepare_kernel<bf16, 1>, grid, dim3(256), 0, s, p);
}

// rows at negative positions are skipped
extern "C" int ifab_gr_step(const void* q, const void* k, const void* v, int f32, const float* qs, const float* ks, float q_factor, const float* log_decay,
                            const float* weight, int kind, int H, int G, int d, int e, float* state, float* m_state, const int32_t* epoch, float* m_rows,
                            const int32_t* positions, const int32_t* slots, float* o, long ldo, int T, void* stream) {
  const int E = e + (kind == GR_MEMORY);
  StepParams p{{q, k, v, qs, ks, q_factor, log_decay, weight, m_rows, kind, H, G, d, e, E}, {state, m_state, epoch}, positions, slots, o, ldo, m_rows, T};
  if (T < 1 || T > 65535 || !rows_ok(p.r) || (kind == GR_MEMORY && (!m_state || !epoch || !m_rows))) return -1;
  const dim3 grid(H, T, (E + 31) / 32);
  cudaStream_t s = (cudaStream_t)stream;
  const int reg = d % 4 || d > 256 ? 0 : d <= 128 ? 1 : 2;
  if (f32)
    return reg == 0 ? launch_chain(gr_step_kernel<float, 0>, grid, dim3(256), 0, s, p)
                    : reg == 1 ? launch_chain(gr_step_kernel<float, 1>, grid, dim3(256), 0, s, p) : launch_chain(gr_step_kernel<float, 2>, grid, dim3(256), 0, s, p);
  return reg == 0 ? launch_chain(gr_step_kernel<bf16, 0>, grid, dim3(256), 0, s, p)
                  : reg == 1 ? launch_chain(gr_step_kernel<bf16, 1>, grid, dim3(256), 0, s, p) : launch_chain(gr_step_kernel<bf16, 2>, grid, dim3(256), 0, s, p);
}

// Chunks of at most 64 rows. scratch: cstate f32 [n, H, E, d], cdecay [n, H]; DELTA: w_rows [T, H, d] and u_rows [T, H, e] (the corrected values)
extern "C" int ifab_gr_chunks(const void* q, const void* k, const void* v, int f32, const float* qs, const float* ks, float q_factor, const float* log_decay,
                              const float* weight, int kind, int H, int G, int d, int e, const int32_t* chunks, int n, const int32_t* positions, float* cstate,
                              uint64_t cstate_bytes, float* cdecay, float* w_rows, float* u_rows, float* state, float* m_state, const int32_t* epoch, float* m_rows,
                              float* o, long ldo, void* stream) {
  const int E = e + (kind == GR_MEMORY);
  GrChunks p{{q, k, v, qs, ks, q_factor, log_decay, weight, m_rows, kind, H, G, d, e, E}, chunks, n, positions, cstate, cdecay, o, ldo};
  const GrState st{state, m_state, epoch};
  if (n < 1 || n > 65535 || !rows_ok(p.r) || (kind == GR_MEMORY && (!m_state || !epoch || !m_rows)) || (kind == GR_DELTA && (!w_rows || !u_rows))) return -1;
  if ((uint64_t)n * H * d * E * sizeof(float) > cstate_bytes) return -5;
  cudaStream_t s = (cudaStream_t)stream;
  const int td = (d + 63) / 64, te = (E + 63) / 64;
  if (kind == GR_DELTA) {
    if (int rc = gr_delta_chunks(p, st, f32, w_rows, u_rows, s)) return rc;
    p.r.v = u_rows;
    p.r.kind = GR_SSD;             // the outputs: corrected values that count once
    p.r.weight = nullptr;
  } else {
    if (kind == GR_MEMORY)
      if (int rc = gr_maximum(p, st, s)) return rc;
    const dim3 grid(n, H, td * te);
    if (int rc = f32 ? launch_chain(gr_state_kernel<float>, grid, dim3(256), 0, s, p, st) : launch_chain(gr_state_kernel<bf16>, grid, dim3(256), 0, s, p, st)) return rc;
    if (int rc = gr_scan(p, st, s)) return rc;
  }
  const size_t smem = 3 * 64 * 68 * sizeof(float);
  const auto out = [&](auto kernel) {
    if (int rc = opt_in_smem(kernel, smem)) return rc;
    return launch_chain(kernel, dim3(n, H, te), dim3(256), smem, s, p, st);
  };
  return f32 ? out(gr_out_kernel<float, float>) : kind == GR_DELTA ? out(gr_out_kernel<bf16, float>) : out(gr_out_kernel<bf16, bf16>);
}

// y [T, H * e]: see the top of the file. m: MEMORY (heads of o end with n q); v, skip: a skip
extern "C" int ifab_gr_finish(const float* o, long ldo, int H, int e, int E, const float* m, const void* v, const float* skip, const void* gate, long ldg, int act,
                              int gate_first, int groups, float eps, const float* gain, void* y, long ldy, int f32, int T, void* stream) {
  if (T < 1 || T > 65535 || H < 1 || H > 2048 || e < 1 || E < e || (m && E <= e) || groups < 1 || (H * e) % groups || !gate || !gain || (skip && !v)) return -1;
  FinishParams p{o, ldo, H, e, E, m, v, skip, gate, ldg, act, gate_first, groups, eps, gain, y, ldy};
  const size_t smem = m ? (size_t)H * sizeof(float) : 0;
  cudaStream_t s = (cudaStream_t)stream;
  const int n = H * e / groups;
  const auto odd = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; };
  const auto off = [&](const void* a) { return (reinterpret_cast<uintptr_t>(a) & (f32 ? 15 : 7)) != 0; };
  if (n > 256 && n <= 8192 && !m && !((n | e | E | ldo | ldg | ldy) % 4) && !odd(o) && !odd(gain) && !off(gate) && !off(y) && !off(v)) {
    const dim3 grid(groups, T);
    if (f32) return n <= 4096 ? launch_chain(gr_finish_wide_kernel<float, 4>, grid, dim3(256), 0, s, p) : launch_chain(gr_finish_wide_kernel<float, 8>, grid, dim3(256), 0, s, p);
    return n <= 4096 ? launch_chain(gr_finish_wide_kernel<bf16, 4>, grid, dim3(256), 0, s, p) : launch_chain(gr_finish_wide_kernel<bf16, 8>, grid, dim3(256), 0, s, p);
  }
  if (n > 256) {
    const dim3 grid(groups < 8 ? groups : 8, T);
    return f32 ? launch_chain(gr_finish_kernel<float, 8>, grid, dim3(256), smem, s, p) : launch_chain(gr_finish_kernel<bf16, 8>, grid, dim3(256), smem, s, p);
  }
  const dim3 grid(T <= 256 ? (groups + 7) / 8 : 1, T);
  return f32 ? launch_chain(gr_finish_kernel<float, 1>, grid, dim3(256), smem, s, p) : launch_chain(gr_finish_kernel<bf16, 1>, grid, dim3(256), smem, s, p);
}
