// Linear attention with a fixed decay per head, for any head sizes:  S_t = decay_h S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t.
//
// Query, key and value come out of one packed projection row ([.. q heads .. k heads .. v heads ..], column offsets given);
// what happens to them before the recurrence is a parameter: a rotation of q and k (any pair layout, first `rot` columns), or an
// activation of q, k and v (rounded to the activation type), and a factor on k. Everything after that is f32. The state is f32
// [slots, H, e, d] (value columns outside: a row of the state meets q and k), one per sequence slot; a row at position 0 starts
// from zero whatever the slot held before.
//
//   la_step_kernel     decode: rows in position order, one CTA per (head, run of rows of one slot, 32 value columns); a run
//                      walks its rows through the state in memory. The grid depends on the row count only (graph capture)
//   prompts, by chunks of consecutive rows of one sequence, in three launches: what each chunk adds to the state (all chunks in
//   parallel), the states ahead of every chunk (la_scan_kernel: over the chunks of a sequence, elementwise), and the outputs of
//   every chunk from that state and from the rows of the chunk (all in parallel). Two forms of the first and the last:
//     la_chunk_*       f32 products of any size, chunks of 64 rows, on q / k / v rows written by la_prepare_kernel (exact mode)
//     la_tile_*        linear_attn_tc.cu: tensor cores, chunks of 128 rows, heads up to 128 columns
//
// decay^n comes from a table [H, 129] made in double on the host. Chunk table: int32 [n, 4] = first row, rows, slot, 2 * chunks of
// the run + 1 at the first chunk of a run and 0 at the others; the position of a run's first row from `positions`.
#include "linear_attn.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

constexpr int CH = 64;          // rows of a chunk of the f32 form

// column c of a head of q or k as it enters the recurrence
template <typename A>
__device__ __forceinline__ float qk_value(const LaParams& p, const A* head, int t, int c, float scale) {
  const float v = c < p.rope.rot ? rotated(p.rope, p.rope.cs + (long)t * (p.rope.rot / 2), head, c) : activated(p, head[c]);
  return v * scale;
}

// grid (H, T, ceil(e / 32)), 256 threads: a warp owns 4 value columns = rows of the state, lanes their q / k columns
template <typename A>
__global__ void __launch_bounds__(256) la_step_kernel(LaParams p, float* o, long ldo) {
  extern __shared__ float sm[];        // q [d], k [d]
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, t0 = blockIdx.y, lane = threadIdx.x & 31, col0 = blockIdx.z * 32 + (threadIdx.x >> 5) * 4, d = p.d;
  const int slot = p.slots[t0];
  if (p.positions[t0] < 0 || (t0 > 0 && p.slots[t0 - 1] == slot && p.positions[t0 - 1] >= 0)) return;      // not the head of a run
  float* S = p.state + (((long)slot * p.H + h) * p.e + col0) * d;
  const float decay = p.powers[(long)h * LA_POW + 1];
  const int nc = min(4, p.e - col0);
  for (int t = t0; t < p.T && p.slots[t] == slot && p.positions[t] >= 0; ++t) {
    const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
    const bool fresh = p.positions[t] == 0;
    __syncthreads();
    for (int c = threadIdx.x; c < 2 * d; c += blockDim.x) {
      const bool is_k = c >= d;
      sm[c] = qk_value(p, row + (is_k ? p.k_off : p.q_off) + (long)h * d, t, is_k ? c - d : c, is_k ? p.k_scale : 1.f);
    }
    __syncthreads();
    if (nc <= 0) continue;
    float v[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int u = 0; u < 4; ++u) v[u] = u < nc ? activated(p, row[p.v_off + (long)h * p.e + col0 + u]) : 0.f;
    if (d % 4 == 0) {
      for (int c = lane * 4; c < d; c += 128) {
        const float4 q = *reinterpret_cast<const float4*>(sm + c), k = *reinterpret_cast<const float4*>(sm + d + c);
        float4 s[4];
#pragma unroll
        for (int u = 0; u < 4; ++u)
          s[u] = (fresh || u >= nc) ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + (long)u * d + c);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (u >= nc) break;
          s[u].x = fmaf(k.x, v[u], decay * s[u].x);
          s[u].y = fmaf(k.y, v[u], decay * s[u].y);
          s[u].z = fmaf(k.z, v[u], decay * s[u].z);
          s[u].w = fmaf(k.w, v[u], decay * s[u].w);
          *reinterpret_cast<float4*>(S + (long)u * d + c) = s[u];
          acc[u] = fmaf(q.x, s[u].x, fmaf(q.y, s[u].y, fmaf(q.z, s[u].z, fmaf(q.w, s[u].w, acc[u]))));
        }
      }
    } else {
      for (int c = lane; c < d; c += 32)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (u >= nc) break;
          const float s = fmaf(sm[d + c], v[u], fresh ? 0.f : decay * S[(long)u * d + c]);
          S[(long)u * d + c] = s;
          acc[u] = fmaf(sm[c], s, acc[u]);
        }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float r = warp_sum(acc[u]);
      if (lane == 0 && u < nc) o[(long)t * ldo + (long)h * p.e + col0 + u] = r;
    }
  }
}

// grid (H, T), 128 threads
template <typename A>
__global__ void __launch_bounds__(128) la_prepare_kernel(LaParams p, float* q, float* k, float* v) {
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, t = blockIdx.y;
  const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
  const long qk = ((long)t * p.H + h) * p.d;
  const A *qh = row + p.q_off + (long)h * p.d, *kh = row + p.k_off + (long)h * p.d;
  for (int c = threadIdx.x; c < p.d; c += blockDim.x) {
    q[qk + c] = qk_value(p, qh, t, c, 1.f);
    k[qk + c] = qk_value(p, kh, t, c, p.k_scale);
  }
  const A* vh = row + p.v_off + (long)h * p.e;
  for (int c = threadIdx.x; c < p.e; c += blockDim.x) v[((long)t * p.H + h) * p.e + c] = activated(p, vh[c]);
}

struct ChunkParams {
  const float *q, *k, *v;
  const int32_t* chunks;         // [n, 4]
  int H, d, e;
  const float* powers;
  float* cstate;                 // [n, H, e, d]
  float* o; long ldo;
};

// grid (n, H, tiles of 64 x 64 of the state): sum over the chunk's rows of decay^(L - 1 - j) k_j v_j^T
__global__ void __launch_bounds__(256) la_chunk_state_kernel(ChunkParams p) {
  __shared__ float ks[CH][68], vs[CH][68];
  grid_dep_launch();
  grid_dep_wait();
  const int c = blockIdx.x, h = blockIdx.y, te = (p.e + 63) / 64, d0 = blockIdx.z / te * 64, e0 = blockIdx.z % te * 64;
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  const float* pw = p.powers + (long)h * LA_POW;
  for (int i = threadIdx.x; i < CH * 64; i += 256) {
    const int j = i >> 6, x = i & 63;
    ks[j][x] = (j < L && d0 + x < p.d) ? p.k[((long)(row0 + j) * p.H + h) * p.d + d0 + x] * pw[L - 1 - j] : 0.f;
    vs[j][x] = (j < L && e0 + x < p.e) ? p.v[((long)(row0 + j) * p.H + h) * p.e + e0 + x] : 0.f;
  }
  __syncthreads();
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int j = 0; j < L; ++j) {
    const float4 a = *reinterpret_cast<const float4*>(&ks[j][ty * 4]), b = *reinterpret_cast<const float4*>(&vs[j][tx * 4]);
    const float ar[4] = {a.x, a.y, a.z, a.w}, br[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int y = 0; y < 4; ++y)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[y][x] = fmaf(ar[y], br[x], acc[y][x]);
  }
  float* out = p.cstate + ((long)c * p.H + h) * p.d * p.e;
#pragma unroll
  for (int y = 0; y < 4; ++y)
#pragma unroll
    for (int x = 0; x < 4; ++x)
      if (d0 + ty * 4 + y < p.d && e0 + tx * 4 + x < p.e) out[(long)(e0 + tx * 4 + x) * p.d + d0 + ty * 4 + y] = acc[y][x];
}

// grid (ceil(H * d * e / (256 V)), n): CTAs of a run's first chunk walk its chunks; cstate becomes the state AHEAD of the chunk. The chunks
// of a run are whole (the rows of the first) up to the last one. V values per thread, eight chunks' loads in flight
template <int V>
__global__ void __launch_bounds__(256) la_scan_kernel(float* cstate, float* state, const int32_t* chunks, const int32_t* positions, const float* powers,
                                                      int H, int d, int e) {
  grid_dep_launch();
  grid_dep_wait();
  const int first = blockIdx.y, count = chunks[first * 4 + 3] >> 1;
  if (!(chunks[first * 4 + 3] & 1)) return;
  const long sz = (long)d * e, total = (long)H * sz, i = ((long)blockIdx.x * 256 + threadIdx.x) * V;
  if (i >= total) return;
  const float* pw = powers + (i / sz) * LA_POW;
  const float whole = pw[chunks[first * 4 + 1]], ragged = pw[chunks[(first + count - 1) * 4 + 1]];
  float* st = state + (long)chunks[first * 4 + 2] * total + i;
  __align__(16) float s[V];
  const bool fresh = positions[chunks[first * 4]] == 0;
#pragma unroll
  for (int x = 0; x < V; ++x) s[x] = fresh ? 0.f : st[x];
  float* cs = cstate + (long)first * total + i;
  constexpr int AHEAD = 8;
  for (int c0 = 0; c0 < count; c0 += AHEAD) {
    __align__(16) float add[AHEAD][V];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < count) {
        if (V == 4) *reinterpret_cast<float4*>(add[u]) = *reinterpret_cast<const float4*>(cs + (long)(c0 + u) * total);
        else add[u][0] = cs[(long)(c0 + u) * total];
      }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < count) {
        if (V == 4) *reinterpret_cast<float4*>(cs + (long)(c0 + u) * total) = *reinterpret_cast<const float4*>(s);
        else cs[(long)(c0 + u) * total] = s[0];
        const float f = c0 + u + 1 < count ? whole : ragged;
#pragma unroll
        for (int x = 0; x < V; ++x) s[x] = fmaf(f, s[x], add[u][x]);
      }
  }
#pragma unroll
  for (int x = 0; x < V; ++x) st[x] = s[x];
}

// grid (n, H, ceil(e / 64)): o_i = decay^(i + 1) q_i S + sum_{j <= i} decay^(i - j) (q_i . k_j) v_j
__global__ void __launch_bounds__(256) la_chunk_out_kernel(ChunkParams p) {
  extern __shared__ float sm[];
  float(*qs)[68] = reinterpret_cast<float(*)[68]>(sm);                 // [column of q][row], one 64-column slice
  float(*ks)[68] = reinterpret_cast<float(*)[68]>(sm + 64 * 68);       // [column of k][row]; then v rows
  float(*ss)[68] = reinterpret_cast<float(*)[68]>(sm + 2 * 64 * 68);   // a slice of the state; then the weights [j][i]
  grid_dep_launch();
  grid_dep_wait();
  const int c = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * 64;
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  const float* pw = p.powers + (long)h * LA_POW;
  const float* S = p.cstate + ((long)c * p.H + h) * p.d * p.e;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float w[4][4] = {}, acc[4][4] = {};
  for (int d0 = 0; d0 < p.d; d0 += 64) {
    __syncthreads();
    for (int i = threadIdx.x; i < CH * 64; i += 256) {
      const int j = i >> 6, x = i & 63;
      const bool ok = j < L && d0 + x < p.d;
      const long at = ((long)(row0 + j) * p.H + h) * p.d + d0 + x;
      qs[x][j] = ok ? p.q[at] : 0.f;
      ks[x][j] = ok ? p.k[at] : 0.f;
      ss[x][j] = (d0 + x < p.d && e0 + j < p.e) ? S[(long)(e0 + j) * p.d + d0 + x] : 0.f;
    }
    __syncthreads();
    const int n = min(64, p.d - d0);
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
  for (int y = 0; y < 4; ++y)
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      const int i = ty * 4 + y, j = tx * 4 + z;
      acc[y][z] *= pw[i + 1];
      ss[j][i] = (j <= i && i < L) ? w[y][z] * pw[i - j] : 0.f;
    }
  for (int i = threadIdx.x; i < CH * 64; i += 256) {
    const int j = i >> 6, x = i & 63;
    ks[j][x] = (j < L && e0 + x < p.e) ? p.v[((long)(row0 + j) * p.H + h) * p.e + e0 + x] : 0.f;
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
      if (ty * 4 + y < L && e0 + tx * 4 + z < p.e) p.o[(long)(row0 + ty * 4 + y) * p.ldo + (long)h * p.e + e0 + tx * 4 + z] = acc[y][z];
}

}  // namespace

static bool la_ok(int T, int H, int d, int e, int rot, const void* rope) {
  return T >= 1 && T <= 65535 && H >= 1 && d >= 1 && d <= 1024 && e >= 1 && e <= 1024 && rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || rope);
}

extern "C" int ifab_la_step(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved,
                            const void* rope, int act, float k_scale, const float* powers, float* state, const int32_t* positions, const int32_t* slots,
                            float* o, long ldo, int T, void* stream) {
  if (!la_ok(T, H, d, e, rot, rope)) return -1;
  LaParams p{proj, ldp, q_off, k_off, v_off, H, d, e, {(const float2*)rope, rot, interleaved}, act, k_scale, powers, state, positions, slots, T};
  const dim3 grid(H, T, (e + 31) / 32);
  const size_t smem = (size_t)2 * d * sizeof(float);
  return f32 ? launch_chain(la_step_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, p, o, ldo)
             : launch_chain(la_step_kernel<bf16>, grid, dim3(256), smem, (cudaStream_t)stream, p, o, ldo);
}

extern "C" int ifab_la_prepare(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved,
                               const void* rope, int act, float k_scale, float* q, float* k, float* v, int T, void* stream) {
  if (!la_ok(T, H, d, e, rot, rope)) return -1;
  LaParams p{proj, ldp, q_off, k_off, v_off, H, d, e, {(const float2*)rope, rot, interleaved}, act, k_scale, nullptr, nullptr, nullptr, nullptr, T};
  return f32 ? launch_chain(la_prepare_kernel<float>, dim3(H, T), dim3(128), 0, (cudaStream_t)stream, p, q, k, v)
             : launch_chain(la_prepare_kernel<bf16>, dim3(H, T), dim3(128), 0, (cudaStream_t)stream, p, q, k, v);
}

int ifab::la_scan(float* cstate, float* state, const int32_t* chunks, int n, const int32_t* positions, const float* powers, int H, int d, int e,
                  cudaStream_t s) {
  const long total = (long)H * d * e;
  if ((long)d * e % 4 == 0)
    return launch_chain(la_scan_kernel<4>, dim3((unsigned)((total + 1023) / 1024), n), dim3(256), 0, s, cstate, state, chunks, positions, powers, H, d, e);
  return launch_chain(la_scan_kernel<1>, dim3((unsigned)((total + 255) / 256), n), dim3(256), 0, s, cstate, state, chunks, positions, powers, H, d, e);
}

extern "C" int ifab_la_chunks(const float* q, const float* k, const float* v, const int32_t* chunks, int n, const int32_t* positions, int H, int d, int e,
                              const float* powers, float* cstate, uint64_t cstate_bytes, float* state, float* o, long ldo, void* stream) {
  if (!la_ok(n, H, d, e, 0, nullptr)) return -1;
  if ((uint64_t)n * H * d * e * sizeof(float) > cstate_bytes) return -5;
  ChunkParams p{q, k, v, chunks, H, d, e, powers, cstate, o, ldo};
  cudaStream_t s = (cudaStream_t)stream;
  const int td = (d + 63) / 64, te = (e + 63) / 64;
  if (int rc = launch_chain(la_chunk_state_kernel, dim3(n, H, td * te), dim3(256), 0, s, p)) return rc;
  if (int rc = la_scan(cstate, state, chunks, n, positions, powers, H, d, e, s)) return rc;
  const size_t smem = 3 * 64 * 68 * sizeof(float);
  if (int rc = opt_in_smem(la_chunk_out_kernel, smem)) return rc;
  return launch_chain(la_chunk_out_kernel, dim3(n, H, te), dim3(256), smem, s, p);
}
