// Chunks of the gated delta rule (gated_recurrence.cu). With g_i the decay from ahead of the chunk up to row i, the corrected values of a chunk's
// rows solve a unit lower triangular system,
//
//   u_i + sum over j < i of A_ij u_j = b_i (v_i - g_i S^T k_i),   A_ij = b_i (g_i / g_j) (k_i . k_j)
//
// so with T = (1 + A)^-1:  u = T (b v) - T (b g k) S  and the state behind the chunk is g_L S + sum_j (g_L / g_j) k_j u_j^T.
//
//   gr_delta_local_kernel  T (by blocks of 16, 32, 64 rows), T (b v) and T (b g k) of every chunk, all chunks in parallel
//   gr_delta_scan_kernel   over the chunks of a sequence: u in place of T (b v), the state ahead of every chunk. One CTA per (head, 16 value
//                          columns), its slice of the state in shared memory
#include "gated_recurrence.cuh"

using namespace ifab;

namespace {

constexpr int C = GR_CHUNK, EB = 16;

struct LocalSmem {
  float a[C][C + 1], t[C][C + 1], tmp[C / 2][C / 2 + 1];
  float x[C][68];
  GrFactors<GR_CHUNK> f;
};

// grid (n, H), 256 threads
template <typename A>
__global__ void __launch_bounds__(256) gr_delta_local_kernel(GrChunks p, GrState st, float* w_rows, float* u_rows) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  LocalSmem& S = *reinterpret_cast<LocalSmem*>(smem_raw);
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int c = blockIdx.x, h = blockIdx.y, g = h / (r.H / r.G), tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  gr_load_factors(p, c, h, st, S.f);
  float acc[4][4] = {};
  for (int d0 = 0; d0 < r.d; d0 += 64) {
    __syncthreads();
    for (int i = tid; i < C * 64; i += 256) {
      const int j = i >> 6, x = i & 63;
      S.x[x][j] = (j < L && d0 + x < r.d) ? gr_k<A>(r, row0 + j, g, d0 + x) : 0.f;
    }
    __syncthreads();
    const int n = min(64, r.d - d0);
    for (int x = 0; x < n; ++x) {
      const float4 a = *reinterpret_cast<const float4*>(&S.x[x][ty * 4]), b = *reinterpret_cast<const float4*>(&S.x[x][tx * 4]);
      const float ar[4] = {a.x, a.y, a.z, a.w}, br[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int y = 0; y < 4; ++y)
#pragma unroll
        for (int z = 0; z < 4; ++z) acc[y][z] = fmaf(ar[y], br[z], acc[y][z]);
    }
  }
#pragma unroll
  for (int y = 0; y < 4; ++y)
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      const int i = ty * 4 + y, j = tx * 4 + z;
      S.a[i][j] = (j < i && i < L) ? acc[y][z] * S.f.w[i] * expf((float)(S.f.total[i] - S.f.total[j])) : 0.f;
      S.t[i][j] = 0.f;
    }
  __syncthreads();
  if (tid < C) {      // the diagonal blocks of 16 rows: a column of the inverse per thread
    const int b0 = tid & ~15, col = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float v = i == col ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) v = fmaf(-S.a[b0 + i][b0 + j], x[j], v);
      x[i] = v;
      S.t[b0 + i][b0 + col] = v;
    }
  }
#pragma unroll
  for (int s = 16; s < C; s *= 2) {      // two inverted blocks of s rows and what lies below the first: -T22 (A21 T11)
    const int pairs = C / (2 * s);
    __syncthreads();
    for (int i = tid; i < pairs * s * s; i += 256) {
      const int b = i / (s * s), y = i / s % s, x = i % s, r0 = 2 * s * b;
      float v = 0.f;
      for (int k = x; k < s; ++k) v = fmaf(S.a[r0 + s + y][r0 + k], S.t[r0 + k][r0 + x], v);
      S.tmp[(s == 16 ? 16 * b : 0) + y][x] = v;
    }
    __syncthreads();
    for (int i = tid; i < pairs * s * s; i += 256) {
      const int b = i / (s * s), y = i / s % s, x = i % s, r0 = 2 * s * b;
      float v = 0.f;
      for (int k = 0; k <= y; ++k) v = fmaf(S.t[r0 + s + y][r0 + s + k], S.tmp[(s == 16 ? 16 * b : 0) + k][x], v);
      S.t[r0 + s + y][r0 + x] = -v;
    }
  }
  // T times the scaled values, then the scaled keys, 64 columns at a time
  const int te = (r.E + 63) / 64, td = (r.d + 63) / 64;
  for (int tile = 0; tile < te + td; ++tile) {
    const bool val = tile < te;
    const int c0 = (val ? tile : tile - te) * 64, n = val ? r.E : r.d;
    __syncthreads();
    for (int i = tid; i < C * 64; i += 256) {
      const int j = i >> 6, x = i & 63;
      float v = 0.f;
      if (j < L && c0 + x < n) {
        v = val ? gr_v<A>(r, row0 + j, h, c0 + x) : gr_k<A>(r, row0 + j, g, c0 + x);
        v *= val ? S.f.w[j] : S.f.w[j] * expf((float)S.f.total[j]);
      }
      S.x[j][x] = v;
    }
    __syncthreads();
    float o[4][4] = {};
    for (int j = 0; j < min(L, ty * 4 + 4); ++j) {
      const float4 b = *reinterpret_cast<const float4*>(&S.x[j][tx * 4]);
      const float br[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int y = 0; y < 4; ++y) {
        const float a = S.t[ty * 4 + y][j];
#pragma unroll
        for (int z = 0; z < 4; ++z) o[y][z] = fmaf(a, br[z], o[y][z]);
      }
    }
    float* out = val ? u_rows : w_rows;
#pragma unroll
    for (int y = 0; y < 4; ++y)
#pragma unroll
      for (int z = 0; z < 4; ++z)
        if (ty * 4 + y < L && c0 + tx * 4 + z < n) out[((long)(row0 + ty * 4 + y) * r.H + h) * n + c0 + tx * 4 + z] = o[y][z];
  }
}

struct ScanSmem {
  float x[C][68];            // 64 columns of T (b g k), or of the decayed keys, [row][column]
  float u[C][EB + 4];
  GrFactors<GR_CHUNK> f;
};

// grid (ceil(E / EB), H, n): CTAs of a run's first chunk walk its chunks. Dynamic shared memory: ScanSmem, then the state slice [d][EB]
template <typename A>
__global__ void __launch_bounds__(256) gr_delta_scan_kernel(GrChunks p, GrState st, const float* w_rows, float* u_rows) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  ScanSmem& S = *reinterpret_cast<ScanSmem*>(smem_raw);
  float* s = reinterpret_cast<float*>(smem_raw + (sizeof(ScanSmem) + 15) / 16 * 16);
  grid_dep_launch();
  grid_dep_wait();
  const GrRows& r = p.r;
  const int first = blockIdx.z, h = blockIdx.y, e0 = blockIdx.x * EB, g = h / (r.H / r.G), tid = threadIdx.x;
  if (!(p.chunks[first * 4 + 3] & 1)) return;
  const int count = p.chunks[first * 4 + 3] >> 1, slot = p.chunks[first * 4 + 2], ne = min(EB, r.E - e0);
  const bool fresh = p.positions[p.chunks[first * 4]] == 0;
  float* state = st.s + (((long)slot * r.H + h) * r.E + e0) * r.d;
  for (int i = tid; i < r.d * EB; i += 256) {
    const int e = i / r.d, x = i - e * r.d;
    s[x * EB + e] = (e < ne && !fresh) ? state[(long)e * r.d + x] : 0.f;
  }
  const int ur = (tid >> 3) * 2, uc = (tid & 7) * 2;      // 2 x 2 values of u
  const int sx = (tid >> 2) & 63, se = (tid & 3) * 4;     // 1 x 4 values of a 64-column slice of the state
  for (int c = first; c < first + count; ++c) {
    const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
    gr_load_factors(p, c, h, st, S.f);
    float* ahead = p.cstate + (((long)c * r.H + h) * r.E + e0) * r.d;
    for (int i = tid; i < r.d * ne; i += 256) {
      const int e = i / r.d, x = i - e * r.d;
      ahead[i] = s[x * EB + e];
    }
    float acc[2][2];
#pragma unroll
    for (int y = 0; y < 2; ++y)
#pragma unroll
      for (int z = 0; z < 2; ++z) acc[y][z] = (ur + y < L && uc + z < ne) ? u_rows[((long)(row0 + ur + y) * r.H + h) * r.E + e0 + uc + z] : 0.f;
    for (int d0 = 0; d0 < r.d; d0 += 64) {
      const int n = min(64, r.d - d0);
      __syncthreads();
      for (int i = tid; i < C * 64; i += 256) {
        const int j = i >> 6, x = i & 63;
        S.x[j][x] = (j < L && x < n) ? w_rows[((long)(row0 + j) * r.H + h) * r.d + d0 + x] : 0.f;
      }
      __syncthreads();
#pragma unroll 8
      for (int x = 0; x < n; ++x) {
        const float2 b = *reinterpret_cast<const float2*>(s + (d0 + x) * EB + uc);
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const float a = S.x[ur + y][x];
          acc[y][0] = fmaf(-a, b.x, acc[y][0]);
          acc[y][1] = fmaf(-a, b.y, acc[y][1]);
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int y = 0; y < 2; ++y)
#pragma unroll
      for (int z = 0; z < 2; ++z) {
        const bool ok = ur + y < L && uc + z < ne;
        if (ok) u_rows[((long)(row0 + ur + y) * r.H + h) * r.E + e0 + uc + z] = acc[y][z];
        S.u[ur + y][uc + z] = ok ? acc[y][z] * expf((float)(S.f.total[L - 1] - S.f.total[ur + y])) : 0.f;
      }
    const float carry = expf((float)S.f.total[L - 1]);
    for (int d0 = 0; d0 < r.d; d0 += 64) {
      const int n = min(64, r.d - d0);
      __syncthreads();
      for (int i = tid; i < C * 64; i += 256) {
        const int j = i >> 6, x = i & 63;
        S.x[j][x] = (j < L && x < n) ? gr_k<A>(r, row0 + j, g, d0 + x) : 0.f;
      }
      __syncthreads();
      if (sx < n) {
        float4* at = reinterpret_cast<float4*>(s + (d0 + sx) * EB + se);
        float4 v = *at;
        v.x *= carry; v.y *= carry; v.z *= carry; v.w *= carry;
#pragma unroll 8
        for (int j = 0; j < L; ++j) {
          const float a = S.x[j][sx];
          const float4 b = *reinterpret_cast<const float4*>(&S.u[j][se]);
          v.x = fmaf(a, b.x, v.x);
          v.y = fmaf(a, b.y, v.y);
          v.z = fmaf(a, b.z, v.z);
          v.w = fmaf(a, b.w, v.w);
        }
        *at = v;
      }
    }
    __syncthreads();
  }
  for (int i = tid; i < r.d * ne; i += 256) {
    const int e = i / r.d, x = i - e * r.d;
    state[i] = s[x * EB + e];
  }
}

}  // namespace

template <typename A>
static int chunks(const GrChunks& p, const GrState& st, float* w_rows, float* u_rows, cudaStream_t s) {
  if (int rc = opt_in_smem(gr_delta_local_kernel<A>, sizeof(LocalSmem))) return rc;
  if (int rc = launch_chain(gr_delta_local_kernel<A>, dim3(p.n, p.r.H), dim3(256), sizeof(LocalSmem), s, p, st, w_rows, u_rows)) return rc;
  const size_t smem = (sizeof(ScanSmem) + 15) / 16 * 16 + (size_t)p.r.d * EB * sizeof(float);
  if (int rc = opt_in_smem(gr_delta_scan_kernel<A>, smem)) return rc;
  return launch_chain(gr_delta_scan_kernel<A>, dim3((p.r.E + EB - 1) / EB, p.r.H, p.n), dim3(256), smem, s, p, st, (const float*)w_rows, u_rows);
}

int ifab::gr_delta_chunks(const GrChunks& p, const GrState& st, int f32, float* w_rows, float* u_rows, cudaStream_t s) {
  return f32 ? chunks<float>(p, st, w_rows, u_rows, s) : chunks<bf16>(p, st, w_rows, u_rows, s);
}
