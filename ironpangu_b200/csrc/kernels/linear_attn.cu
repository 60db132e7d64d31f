// Linear attention with a fixed decay per head, for any head sizes:  S_t = decay_h S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t.
//
// Query, key and value come out of one packed projection row ([.. q heads .. k heads .. v heads ..], column offsets given);
// what happens to them before the recurrence is a parameter: a rotation of q and k (any pair layout, first `rot` columns, angles
// in double), or an activation of q, k and v, and a factor on k. The state is f32 [slots, H, d, e], one per sequence slot; a
// row at position 0 starts from zero whatever the slot held before. Everything after the projection is f32.
//
//   la_step_kernel     decode: rows in position order, one CTA per (head, run of rows of one slot, 32 value columns); a run
//                      walks its rows through the state in memory. The grid depends on the row count only (graph capture)
//   la_prepare_kernel  prompts: q, k (rotated / activated / scaled) and v as f32 rows [T, H, d], [T, H, d], [T, H, e]
//   la_chunk_state_kernel / la_scan_kernel / la_chunk_out_kernel
//                      prompts by chunks of at most 64 rows of one sequence: what each chunk adds to the state (all chunks in
//                      parallel), the states ahead of every chunk (a scan over the chunks of a sequence, elementwise), and the
//                      outputs of every chunk from that state and from the rows of the chunk (all in parallel)
//
// decay^n comes from a table [H, 65] made in double on the host. Chunk table: int32 [n, 4] = first row, rows, slot, flags (bit 0:
// first chunk of its segment, bit 1: last); position of a segment's first row from `positions`.
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

constexpr int CH = 64;          // rows of a chunk
constexpr int POW = CH + 1;     // entries of the decay table per head

struct LaParams {
  const void* proj; long ldp;
  int q_off, k_off, v_off;       // columns of the packed projection
  int H, d, e;
  int rot, interleaved;          // rotated columns of q and k (0: none)
  const double* freq;            // [rot / 2]
  int act;                       // activation of q, k, v
  float k_scale;
  const float* powers;           // [H, POW]: decay^n
  float* state;                  // [slots, H, d, e]
  const int32_t* positions; const int32_t* slots;
  int T;
};

template <typename A>
__device__ __forceinline__ float qk_value(const LaParams& p, const A* head, int c, int pos, float scale) {
  float v;
  if (c < p.rot) {
    const int i = p.interleaved ? c >> 1 : (c < p.rot / 2 ? c : c - p.rot / 2);
    int ia, ib;
    rope_pair(i, p.rot, p.interleaved, &ia, &ib);
    float cs, sn;
    rope_angle(pos, p.freq[i], &cs, &sn);
    const float a = to_f32(head[ia]), b = to_f32(head[ib]);
    v = c == ia ? a * cs - b * sn : b * cs + a * sn;
  } else {
    v = activate(to_f32(head[c]), p.act);
  }
  return v * scale;
}

// grid (H, T, ceil(e / 32)), 256 threads: 32 value columns x 8 rows of the state in flight
template <typename A>
__global__ void __launch_bounds__(256) la_step_kernel(LaParams p, float* o, long ldo) {
  extern __shared__ float sm[];        // q [d], k [d], then 8 x 32 partial outputs
  float* qs = sm;
  float* ks = sm + p.d;
  float* part = sm + 2 * p.d;
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, t0 = blockIdx.y, tx = threadIdx.x & 31, ty = threadIdx.x >> 5, col = blockIdx.z * 32 + tx;
  const int slot = p.slots[t0];
  if (p.positions[t0] < 0 || (t0 > 0 && p.slots[t0 - 1] == slot && p.positions[t0 - 1] >= 0)) return;      // not the head of a run
  float* S = p.state + ((long)slot * p.H + h) * p.d * p.e;
  const float decay = p.powers[(long)h * POW + 1];
  for (int t = t0; t < p.T && p.slots[t] == slot && p.positions[t] >= 0; ++t) {
    const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
    const int pos = p.positions[t];
    __syncthreads();
    for (int c = threadIdx.x; c < 2 * p.d; c += blockDim.x) {
      const bool is_k = c >= p.d;
      const int cc = is_k ? c - p.d : c;
      sm[c] = qk_value(p, row + (is_k ? p.k_off : p.q_off) + (long)h * p.d, cc, pos, is_k ? p.k_scale : 1.f);
    }
    __syncthreads();
    float acc = 0.f;
    if (col < p.e) {
      const float v = activate(to_f32(row[p.v_off + (long)h * p.e + col]), p.act);
      const bool fresh = pos == 0;
      int i = ty;
      for (; i + 56 < p.d; i += 64) {
        float s[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) s[u] = fresh ? 0.f : S[(long)(i + 8 * u) * p.e + col];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          s[u] = fmaf(ks[i + 8 * u], v, decay * s[u]);
          S[(long)(i + 8 * u) * p.e + col] = s[u];
          acc = fmaf(qs[i + 8 * u], s[u], acc);
        }
      }
      for (; i < p.d; i += 8) {
        const float s = fmaf(ks[i], v, fresh ? 0.f : decay * S[(long)i * p.e + col]);
        S[(long)i * p.e + col] = s;
        acc = fmaf(qs[i], s, acc);
      }
    }
    part[ty * 32 + tx] = acc;
    __syncthreads();
    if (ty == 0 && col < p.e) {
      float r = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) r += part[k * 32 + tx];
      o[(long)t * ldo + (long)h * p.e + col] = r;
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
  const int pos = p.positions[t];
  const long qk = ((long)t * p.H + h) * p.d;
  const A *qh = row + p.q_off + (long)h * p.d, *kh = row + p.k_off + (long)h * p.d;
  for (int i = threadIdx.x; i < p.rot / 2; i += blockDim.x) {
    int ia, ib;
    rope_pair(i, p.rot, p.interleaved, &ia, &ib);
    float cs, sn;
    rope_angle(pos, p.freq[i], &cs, &sn);
    const float a = to_f32(qh[ia]), b = to_f32(qh[ib]), c = to_f32(kh[ia]), d = to_f32(kh[ib]);
    q[qk + ia] = a * cs - b * sn;
    q[qk + ib] = b * cs + a * sn;
    k[qk + ia] = (c * cs - d * sn) * p.k_scale;
    k[qk + ib] = (d * cs + c * sn) * p.k_scale;
  }
  for (int c = p.rot + threadIdx.x; c < p.d; c += blockDim.x) {
    q[qk + c] = activate(to_f32(qh[c]), p.act);
    k[qk + c] = activate(to_f32(kh[c]), p.act) * p.k_scale;
  }
  const A* vh = row + p.v_off + (long)h * p.e;
  for (int c = threadIdx.x; c < p.e; c += blockDim.x) v[((long)t * p.H + h) * p.e + c] = activate(to_f32(vh[c]), p.act);
}

struct ChunkParams {
  const float *q, *k, *v;
  const int32_t* chunks;         // [n, 4]
  const int32_t* positions;
  int n, H, d, e;
  const float* powers;
  float* cstate;                 // [n, H, d, e]
  float* state;                  // [slots, H, d, e]
  float* o; long ldo;
};

// grid (n, H, tiles of 64 x 64 of the state): sum over the chunk's rows of decay^(L - 1 - j) k_j v_j^T
__global__ void __launch_bounds__(256) la_chunk_state_kernel(ChunkParams p) {
  __shared__ float ks[CH][68], vs[CH][68];
  grid_dep_launch();
  grid_dep_wait();
  const int c = blockIdx.x, h = blockIdx.y, te = (p.e + 63) / 64, d0 = blockIdx.z / te * 64, e0 = blockIdx.z % te * 64;
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  const float* pw = p.powers + (long)h * POW;
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
      if (d0 + ty * 4 + y < p.d && e0 + tx * 4 + x < p.e) out[(long)(d0 + ty * 4 + y) * p.e + e0 + tx * 4 + x] = acc[y][x];
}

// grid (ceil(H * d * e / 256), n): CTAs of a segment's first chunk walk its chunks; cstate becomes the state AHEAD of the chunk
__global__ void __launch_bounds__(256) la_scan_kernel(ChunkParams p) {
  grid_dep_launch();
  grid_dep_wait();
  int c = blockIdx.y;
  if (!(p.chunks[c * 4 + 3] & 1)) return;
  const long sz = (long)p.d * p.e, total = (long)p.H * sz, i = (long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const float* pw = p.powers + (i / sz) * POW;
  float* st = p.state + (long)p.chunks[c * 4 + 2] * total + i;
  float s = p.positions[p.chunks[c * 4]] == 0 ? 0.f : *st;
  for (;; ++c) {
    float* cs = p.cstate + (long)c * total + i;
    const float add = *cs;
    *cs = s;
    s = fmaf(pw[p.chunks[c * 4 + 1]], s, add);
    if (p.chunks[c * 4 + 3] & 2) break;
  }
  *st = s;
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
  const float* pw = p.powers + (long)h * POW;
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
      ss[j][x] = (d0 + j < p.d && e0 + x < p.e) ? S[(long)(d0 + j) * p.e + e0 + x] : 0.f;
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

static bool la_ok(int T, int H, int d, int e, int rot) { return T >= 1 && H >= 1 && d >= 1 && d <= 1024 && e >= 1 && e <= 1024 && rot >= 0 && rot % 2 == 0 && rot <= d; }

extern "C" int ifab_la_step(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved,
                            const double* freq, int act, float k_scale, const float* powers, float* state, const int32_t* positions, const int32_t* slots,
                            float* o, long ldo, int T, void* stream) {
  if (!la_ok(T, H, d, e, rot) || T > 65535 || (rot && !freq)) return -1;
  LaParams p{proj, ldp, q_off, k_off, v_off, H, d, e, rot, interleaved, freq, act, k_scale, powers, state, positions, slots, T};
  const dim3 grid(H, T, (e + 31) / 32);
  const size_t smem = (size_t)(2 * d + 256) * sizeof(float);
  return f32 ? launch_chain(la_step_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, p, o, ldo)
             : launch_chain(la_step_kernel<bf16>, grid, dim3(256), smem, (cudaStream_t)stream, p, o, ldo);
}

extern "C" int ifab_la_prepare(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved,
                               const double* freq, int act, float k_scale, const int32_t* positions, float* q, float* k, float* v, int T, void* stream) {
  if (!la_ok(T, H, d, e, rot) || T > 65535 || (rot && !freq)) return -1;
  LaParams p{proj, ldp, q_off, k_off, v_off, H, d, e, rot, interleaved, freq, act, k_scale, nullptr, nullptr, positions, nullptr, T};
  return f32 ? launch_chain(la_prepare_kernel<float>, dim3(H, T), dim3(128), 0, (cudaStream_t)stream, p, q, k, v)
             : launch_chain(la_prepare_kernel<bf16>, dim3(H, T), dim3(128), 0, (cudaStream_t)stream, p, q, k, v);
}

extern "C" int ifab_la_chunks(const float* q, const float* k, const float* v, const int32_t* chunks, int n, const int32_t* positions, int H, int d, int e,
                              const float* powers, float* cstate, uint64_t cstate_bytes, float* state, float* o, long ldo, void* stream) {
  if (!la_ok(1, H, d, e, 0) || n < 1 || n > 65535) return -1;
  if ((uint64_t)n * H * d * e * sizeof(float) > cstate_bytes) return -5;
  ChunkParams p{q, k, v, chunks, positions, n, H, d, e, powers, cstate, state, o, ldo};
  cudaStream_t s = (cudaStream_t)stream;
  const int td = (d + 63) / 64, te = (e + 63) / 64;
  if (int rc = launch_chain(la_chunk_state_kernel, dim3(n, H, td * te), dim3(256), 0, s, p)) return rc;
  if (int rc = launch_chain(la_scan_kernel, dim3((unsigned)(((long)H * d * e + 255) / 256), n), dim3(256), 0, s, p)) return rc;
  const size_t smem = 3 * 64 * 68 * sizeof(float);
  if (int rc = opt_in_smem(la_chunk_out_kernel, smem)) return rc;
  return launch_chain(la_chunk_out_kernel, dim3(n, H, te), dim3(256), smem, s, p);
}
