// Recurrences over a matrix state per head with a decay per token, for any head sizes; everything in f32:
//
//   SSD      S = a S + w k v^T                                   o = S^T q      (state-space duality: a = exp(-exp(A) dt), w = dt)
//   DELTA    S = a S,  u = w (v - S^T k),  S += k u^T            o = S^T q      (gated delta rule: w = beta)
//   MEMORY   m' = max(f + m, i),  S = exp(f + m - m') S + exp(i - m') k v^T     (exponential gates; one more value column of ones keeps
//            the sum of the keys, so that S^T q ends with n q)
//
//   gr_prepare_kernel  packed projection rows -> q, k, v in f32 (short causal convolution + SiLU, unit vectors or a factor) and the
//                      gates (softplus, exponentials, soft limits), one CTA per row. The convolution reads rows of the step and the
//                      sequence's last taps - 1 rows before it (history [slots, 2, taps - 1, C] in the activation type, two sides by epoch as in
//                      hyper_streams.cu)
//   gr_step_kernel     decode: one CTA per (head, run of rows of one slot, 32 value columns); a run walks its rows through the state.
//                      The grid depends on the row count only (graph capture)
//   prompts, by chunks of 64 consecutive rows of one sequence:
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
  float scale; int unit;      // a factor; unit: divided by sqrt(sum of squares + 1e-6) first
  float* dst; int stride;     // f32 [T, heads * stride]; columns past n get 1
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
  int T;
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// grid T, 256 threads: a warp per head
template <typename A>
__global__ void __launch_bounds__(256) gr_prepare_kernel(PrepareParams p) {
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
  const int pos = p.positions[t], slot = p.slots[t], back = p.taps - 1;
  if (pos < 0) return;
  int run = 0;                // rows of the sequence ahead of this one in the step
  while (run < back && t - run - 1 >= 0 && p.slots[t - run - 1] == slot) ++run;
  const int side = p.taps > 1 ? p.epoch[slot] & 1 : 0;
  const A* old = reinterpret_cast<const A*>(p.history) + ((long)slot * 2 + side) * back * p.C;
  A* fresh = reinterpret_cast<A*>(p.history) + ((long)slot * 2 + (side ^ 1)) * back * p.C;
  const bool last = p.taps > 1 && (t + 1 == p.T || p.slots[t + 1] != slot);
  const int total = p.sec[0].heads + p.sec[1].heads + p.sec[2].heads;
  for (int i = warp; i < total; i += 8) {
    const int which = i < p.sec[0].heads ? 0 : i < p.sec[0].heads + p.sec[1].heads ? 1 : 2;
    const Section& s = p.sec[which];
    const int h = i - (which > 0 ? p.sec[0].heads : 0) - (which > 1 ? p.sec[1].heads : 0);
    float* dst = s.dst + ((long)t * s.heads + h) * s.stride;
    float ss = 0.f;
    for (int c = lane; c < s.n; c += 32) {
      const int col = h * s.n + c;
      float v = to_f32(row[s.col + col]);
      if (s.channel >= 0) {
        const int ch = s.channel + col;
        if (last) fresh[ch] = row[s.col + col];
        v *= p.taps_w[(long)back * p.C + ch];
        for (int j = 1; j < p.taps; ++j) {
          A b = from_f32<A>(0.f);
          if (j <= pos) b = j <= run ? row[s.col + col - (long)j * p.ldp] : old[(long)(j - run - 1) * p.C + ch];
          v = fmaf(p.taps_w[(long)(back - j) * p.C + ch], to_f32(b), v);
          if (last && j < back) fresh[(long)j * p.C + ch] = b;
        }
        if (p.bias) v += p.bias[ch];
        v *= sigmoid_f32(v);
      }
      if (s.unit) {
        dst[c] = v;
        ss = fmaf(v, v, ss);
      } else {
        dst[c] = v * s.scale;
      }
    }
    if (s.unit) {
      const float f = s.scale / sqrtf(warp_sum(ss) + 1e-6f);
      for (int c = lane; c < s.n; c += 32) dst[c] *= f;
    }
    for (int c = s.n + lane; c < s.stride; c += 32) dst[c] = 1.f;
  }
  for (int h = threadIdx.x; h < p.H; h += 256) {
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
template <int REG>
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
    const float *q = r.q + ((long)t * r.G + g) * d, *k = r.k + ((long)t * r.G + g) * d;
    const float* vr = r.v + ((long)t * r.H + h) * r.E + col0;
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
    for (int u = 0; u < 4; ++u) v[u] = u < nc ? vr[u] : 0.f;
    if (REG) {
      float4 kr[R], qr[R];
#pragma unroll
      for (int x = 0; x < R; ++x) {
        const int c = (lane + 32 * x) * 4;
        kr[x] = c < d ? *reinterpret_cast<const float4*>(k + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        qr[x] = c < d ? *reinterpret_cast<const float4*>(q + c) : make_float4(0.f, 0.f, 0.f, 0.f);
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
          for (int c = lane; c < d && u < nc; c += 32) kk = fmaf(k[c], S[(long)u * d + c], kk);
          v[u] = fmaf(-a, warp_sum(kk), v[u]);
        }
      }
      for (int c = lane; c < d; c += 32)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (u >= nc) break;
          const float x = fmaf(k[c], w * v[u], first ? 0.f : a * S[(long)u * d + c]);
          S[(long)u * d + c] = x;
          acc[u] = fmaf(q[c], x, acc[u]);
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

// grid (H, chunks), 32 threads: CTAs of a run's first chunk walk its rows, 32 at a time. m_t = G_t + max(m_0, max over j <= t of (i_j - G_j)), G the sums of f
__global__ void __launch_bounds__(32) gr_maximum_kernel(GrChunks p, GrState st) {
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, c = blockIdx.y, lane = threadIdx.x, meta = p.chunks[c * 4 + 3];
  if (!(meta & 1)) return;
  const int row0 = p.chunks[c * 4], slot = p.chunks[c * 4 + 2], count = meta >> 1, lc = c + count - 1;
  const int n = p.chunks[lc * 4] + p.chunks[lc * 4 + 1] - row0, side = st.epoch[slot] & 1;
  const GrRows& r = p.r;
  double sum = 0.0, best = p.positions[row0] == 0 ? 0.0 : (double)st.m[((long)slot * 2 + side) * r.H + h];
  for (int t0 = 0; t0 < n; t0 += 32) {
    const int t = t0 + lane;
    const bool live = t < n;
    const long at = (long)(row0 + (live ? t : 0)) * r.H + h;
    double G = live ? (double)r.log_decay[at] : 0.0;
    const double i = live ? (double)r.weight[at] : -INFINITY;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double x = __shfl_up_sync(0xffffffffu, G, o);
      if (lane >= o) G += x;
    }
    G += sum;
    double b = i - G;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double x = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) b = fmax(b, x);
    }
    b = fmax(b, best);
    if (live) r.m[at] = (float)(G + b);
    if (live && t == n - 1) st.m[((long)slot * 2 + (side ^ 1)) * r.H + h] = (float)(G + b);
    sum = __shfl_sync(0xffffffffu, G, 31);
    best = __shfl_sync(0xffffffffu, b, 31);
  }
}

// grid (n, H, tiles of 64 x 64 of the state): sum over the chunk's rows of (weight at the chunk's end) k_j v_j^T
__global__ void __launch_bounds__(256) gr_state_kernel(GrChunks p, GrState st) {
  __shared__ float ks[GR_CHUNK][68], vs[GR_CHUNK][68];
  __shared__ GrFactors f;
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int c = blockIdx.x, h = blockIdx.y, te = (r.E + 63) / 64, d0 = blockIdx.z / te * 64, e0 = blockIdx.z % te * 64, g = h / (r.H / r.G);
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  gr_load_factors(p, c, h, st, f);
  if (threadIdx.x < GR_CHUNK) {
    const int j = threadIdx.x;
    vs[j][64] = j < L ? gr_add(f, L, j) : 0.f;
    if (j == 0 && blockIdx.z == 0) p.cdecay[(long)c * r.H + h] = gr_carry(f, L - 1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < GR_CHUNK * 64; i += 256) {
    const int j = i >> 6, x = i & 63;
    ks[j][x] = (j < L && d0 + x < r.d) ? r.k[((long)(row0 + j) * r.G + g) * r.d + d0 + x] * vs[j][64] : 0.f;
    vs[j][x] = (j < L && e0 + x < r.E) ? r.v[((long)(row0 + j) * r.H + h) * r.E + e0 + x] : 0.f;
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
__global__ void __launch_bounds__(256) gr_out_kernel(GrChunks p, GrState st) {
  extern __shared__ float sm[];
  __shared__ GrFactors f;
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
      const long at = ((long)(row0 + j) * r.G + g) * r.d + d0 + x;
      qs[x][j] = ok ? r.q[at] : 0.f;
      ks[x][j] = ok ? r.k[at] : 0.f;
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
    ks[j][x] = (j < L && e0 + x < r.E) ? r.v[((long)(row0 + j) * r.H + h) * r.E + e0 + x] : 0.f;
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
  const float *v, *skip;                       // SSD: [T, H * E] and D [H], or null
  const void* gate; long ldg; int act, gate_first;
  int groups; float eps; const float* gain;    // [H * e]
  void* y; long ldy;
};

// grid T, 256 threads; WPG warps per group
template <typename A, int WPG>
__global__ void __launch_bounds__(256) gr_finish_kernel(FinishParams p) {
  __shared__ float red[33];
  extern __shared__ float den[];               // MEMORY: 1 / the denominator of every head
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, n = p.H * p.e / p.groups;
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
    if (p.skip) x = fmaf(p.skip[h], p.v[((long)t * p.H + h) * p.E + j], x);
    *g = activate<sizeof(A) == 2>(to_f32(gate[c]), p.act);
    return p.gate_first ? x * *g : x;
  };
  constexpr int TPG = 32 * WPG, GPB = 8 / WPG;
  for (int g0 = 0; g0 < p.groups; g0 += GPB) {
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

bool rows_ok(const GrRows& r) {
  return r.kind >= GR_SSD && r.kind <= GR_MEMORY && r.H >= 1 && r.G >= 1 && r.H % r.G == 0 && r.d >= 1 && r.E >= 1 && r.d <= 1024 && r.E <= 1024 && r.H <= 65535;
}

}  // namespace

// Sections q, k, v: {column, heads, columns of a head, convolution channel or -1, unit, stride}, scales apart. History in the type of proj.
extern "C" int ifab_gr_prepare(const void* proj, long ldp, int f32, const int32_t* sections, const float* scales, float* q, float* k, float* v, const float* taps_w,
                               const float* bias, int taps, int C, void* history, const int32_t* epoch, int kind, int H, int decay_col, int weight_col,
                               const float* a_log, const float* decay_bias, const float* weight_bias, float cap, float* log_decay, float* weight,
                               const int32_t* positions, const int32_t* slots, int T, void* stream) {
  if (T < 1 || H < 1 || taps < 0 || taps > 64 || (taps && !taps_w) || (taps > 1 && (!history || !epoch)) || kind < GR_SSD || kind > GR_MEMORY || (kind == GR_MEMORY ? cap <= 0.f : !a_log))
    return -1;
  PrepareParams p{proj, ldp, {}, taps_w, bias, taps, C, history, epoch, kind, H, decay_col, weight_col, a_log, decay_bias, weight_bias, cap, log_decay, weight,
                  positions, slots, T};
  float* dst[3] = {q, k, v};
  for (int i = 0; i < 3; ++i) {
    const int32_t* s = sections + 6 * i;
    if (s[0] < 0 || s[1] < 1 || s[2] < 1 || s[5] < s[2] || (s[3] >= 0 && (!taps || s[3] + s[1] * s[2] > C))) return -1;
    p.sec[i] = Section{s[0], s[1], s[2], s[3], scales[i], s[4], dst[i], s[5]};
  }
  return f32 ? launch_chain(gr_prepare_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, p)
             : launch_chain(gr_prepare_kernel<bf16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, p);
}

// rows at negative positions are skipped
extern "C" int ifab_gr_step(const float* q, const float* k, const float* v, const float* log_decay, const float* weight, int kind, int H, int G, int d, int E,
                            float* state, float* m_state, const int32_t* epoch, float* m_rows, const int32_t* positions, const int32_t* slots, float* o, long ldo,
                            int T, void* stream) {
  StepParams p{{q, k, v, log_decay, weight, m_rows, kind, H, G, d, E}, {state, m_state, epoch}, positions, slots, o, ldo, m_rows, T};
  if (T < 1 || T > 65535 || !rows_ok(p.r) || (kind == GR_MEMORY && (!m_state || !epoch || !m_rows))) return -1;
  const dim3 grid(H, T, (E + 31) / 32);
  cudaStream_t s = (cudaStream_t)stream;
  if (d % 4 || d > 256) return launch_chain(gr_step_kernel<0>, grid, dim3(256), 0, s, p);
  return d <= 128 ? launch_chain(gr_step_kernel<1>, grid, dim3(256), 0, s, p) : launch_chain(gr_step_kernel<2>, grid, dim3(256), 0, s, p);
}

// Chunks of at most 64 rows. scratch: cstate f32 [n, H, E, d], cdecay [n, H]; DELTA: w_rows [T, H, d] and u_rows [T, H, E] (the corrected values)
extern "C" int ifab_gr_chunks(const float* q, const float* k, const float* v, const float* log_decay, const float* weight, int kind, int H, int G, int d, int E,
                              const int32_t* chunks, int n, const int32_t* positions, float* cstate, uint64_t cstate_bytes, float* cdecay, float* w_rows,
                              float* u_rows, float* state, float* m_state, const int32_t* epoch, float* m_rows, float* o, long ldo, void* stream) {
  GrChunks p{{q, k, v, log_decay, weight, m_rows, kind, H, G, d, E}, chunks, n, positions, cstate, cdecay, o, ldo};
  const GrState st{state, m_state, epoch};
  if (n < 1 || n > 65535 || !rows_ok(p.r) || (kind == GR_MEMORY && (!m_state || !epoch || !m_rows)) || (kind == GR_DELTA && (!w_rows || !u_rows))) return -1;
  if ((uint64_t)n * H * d * E * sizeof(float) > cstate_bytes) return -5;
  cudaStream_t s = (cudaStream_t)stream;
  const int td = (d + 63) / 64, te = (E + 63) / 64;
  if (kind == GR_DELTA) {
    if (int rc = gr_delta_chunks(p, st, w_rows, u_rows, s)) return rc;
    p.r.v = u_rows;
    p.r.kind = GR_SSD;             // the outputs: corrected values that count once
    p.r.weight = nullptr;
  } else {
    if (kind == GR_MEMORY)
      if (int rc = launch_chain(gr_maximum_kernel, dim3(H, n), dim3(32), 0, s, p, st)) return rc;
    if (int rc = launch_chain(gr_state_kernel, dim3(n, H, td * te), dim3(256), 0, s, p, st)) return rc;
    const long total = (long)H * d * E;
    if ((long)d * E % 4 == 0) {
      if (int rc = launch_chain(gr_scan_kernel<4>, dim3((unsigned)((total + 1023) / 1024), n), dim3(256), 0, s, p, state)) return rc;
    } else {
      if (int rc = launch_chain(gr_scan_kernel<1>, dim3((unsigned)((total + 255) / 256), n), dim3(256), 0, s, p, state)) return rc;
    }
  }
  const size_t smem = 3 * 64 * 68 * sizeof(float);
  if (int rc = opt_in_smem(gr_out_kernel, smem)) return rc;
  return launch_chain(gr_out_kernel, dim3(n, H, te), dim3(256), smem, s, p, st);
}

// y [T, H * e]: see the top of the file. m: MEMORY (heads of o end with n q); v, skip: a skip
extern "C" int ifab_gr_finish(const float* o, long ldo, int H, int e, int E, const float* m, const float* v, const float* skip, const void* gate, long ldg, int act,
                              int gate_first, int groups, float eps, const float* gain, void* y, long ldy, int f32, int T, void* stream) {
  if (T < 1 || H < 1 || H > 2048 || e < 1 || E < e || (m && E <= e) || groups < 1 || (H * e) % groups || !gate || !gain || (skip && !v)) return -1;
  FinishParams p{o, ldo, H, e, E, m, v, skip, gate, ldg, act, gate_first, groups, eps, gain, y, ldy};
  const size_t smem = m ? (size_t)H * sizeof(float) : 0;
  cudaStream_t s = (cudaStream_t)stream;
  if (H * e / groups > 256)
    return f32 ? launch_chain(gr_finish_kernel<float, 8>, dim3(T), dim3(256), smem, s, p) : launch_chain(gr_finish_kernel<bf16, 8>, dim3(T), dim3(256), smem, s, p);
  return f32 ? launch_chain(gr_finish_kernel<float, 1>, dim3(T), dim3(256), smem, s, p) : launch_chain(gr_finish_kernel<bf16, 1>, dim3(T), dim3(256), smem, s, p);
}
