// C[M,N] = act(A[M,K] * B[N,K]^T) in true f32 (FMA, no reduced-precision matrix mode): the linear of the exact 32-bit mode.
// 64 x 64 output tile per CTA, 256 threads with a 4 x 4 register tile each, K in steps of 16 through shared memory. Three forms share the
// tile loop: one product; a batch of products at fixed strides (heads side by side in a row); and products grouped by a device tile
// table (experts), whose rows may be gathered and whose A may be a gate | up pair taken as a gated unit (rope.cuh). The one product may
// add a bias and limit its result softly (cap tanh(result / cap)).
#include "attn_rule.cuh"
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

// rows m0 .. of C from rows m0 .. of A (through `index` when given); PAIR: A holds gate columns [0, K) and up columns [K, 2 K)
template <bool PAIR>
__device__ __forceinline__ void tile_f32(const float* a, long lda, const int32_t* index, const float* b, long ldb, float* c, long ldc, int m0, int M, int n0, int N,
                                         int K, int act, const GatedUnit& unit, const float* bias = nullptr, float cap = 0.f) {
  __shared__ float as[16][68], bs[16][68];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (threadIdx.x >> 4) + 16 * i, k = threadIdx.x & 15;
      float v = 0.f;
      if (m0 + r < M && k0 + k < K) {
        const float* ar = a + (long)(index ? index[m0 + r] : m0 + r) * lda + k0 + k;
        v = PAIR ? gated_value(ar[0], ar[K], unit) : ar[0];
      }
      as[k][r] = v;
      bs[k][r] = (n0 + r < N && k0 + k < K) ? b[(long)(n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&as[k][ty * 4]), bv = *reinterpret_cast<const float4*>(&bs[k][tx * 4]);
      const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], br[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= M || n >= N) continue;
      const float v = activate(bias ? acc[i][j] + bias[n] : acc[i][j], act);
      c[(long)m * ldc + n] = cap > 0.f ? soft_limit(v, cap) : v;
    }
}

__global__ void __launch_bounds__(256) linear_f32_kernel(const float* a, long lda, const float* b, long ldb, float* c, long ldc, int M, int N, int K, int act,
                                                         long sa, long sb, long sc, const float* bias, float cap) {
  grid_dep_launch();
  grid_dep_wait();
  const long z = blockIdx.z;
  tile_f32<false>(a + z * sa, lda, nullptr, b + z * sb, ldb, c + z * sc, ldc, blockIdx.y * 64, M, blockIdx.x * 64, N, K, act, GatedUnit{}, bias, cap);
}

// tiles: {group, first row, valid rows <= 128, 0}; grid (ceil(N / 64), 2 * max_tiles)
template <bool PAIR>
__global__ void __launch_bounds__(256) grouped_f32_kernel(const float* a, long lda, const int32_t* index, const float* b, float* c, long ldc, int N, int K,
                                                          const int4* tiles, const int32_t* num_tiles, int rows, GatedUnit unit) {
  grid_dep_launch();
  grid_dep_wait();
  if ((int)(blockIdx.y >> 1) >= *num_tiles) return;
  const int4 t = tiles[blockIdx.y >> 1];
  const int m0 = t.y + (blockIdx.y & 1) * 64;
  const int end = min(t.y + t.z, rows);
  if (m0 >= end) return;
  tile_f32<PAIR>(a, lda, index, b + (long)t.x * N * K, K, c, ldc, m0, end, blockIdx.x * 64, N, K, 0, unit);
}

}  // namespace

// bias [N] or null; cap > 0: cap tanh(result / cap)
extern "C" int ifab_linear_f32(const float* a, long lda, const float* b, long ldb, float* c, long ldc, const float* bias, float cap, int M, int N, int K, int act,
                               void* stream) {
  if (M < 1 || N < 1 || K < 1 || cap < 0.f) return -1;
  return launch_chain(linear_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, (cudaStream_t)stream, a, lda, b, ldb, c, ldc, M, N, K, act, 0L, 0L, 0L,
                      bias, cap);
}

// n products at strides sa, sb, sc (elements)
extern "C" int ifab_linear_f32_batched(const float* a, long lda, long sa, const float* b, long ldb, long sb, float* c, long ldc, long sc, int n, int M, int N, int K,
                                       void* stream) {
  if (n < 1 || n > 65535 || M < 1 || N < 1 || K < 1) return -1;
  return launch_chain(linear_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64, n), dim3(256), 0, (cudaStream_t)stream, a, lda, b, ldb, c, ldc, M, N, K, 0, sa, sb, sc,
                      (const float*)nullptr, 0.f);
}

// C[r] = A[index ? index[r] : r] * B[group(r)]^T for r < rows over the tiles of ifab_moe_dispatch; pair: A is [gate | up] ([rows, 2 K]), taken as the gated
// unit of that number (0 SiLU, 1 ReLU, 2 limited)
extern "C" int ifab_grouped_linear_f32(const float* a, long lda, const int32_t* index, int pair, int unit, float limit, float alpha, const float* b, int N, int K,
                                       const int32_t* tiles, const int32_t* num_tiles, int max_tiles, int rows, float* c, long ldc, void* stream) {
  const GatedUnit gu{unit, limit, alpha};
  if (N < 1 || K < 1 || rows < 1 || max_tiles < 1 || max_tiles > 32767 || !gated_ok(gu)) return -1;
  const dim3 grid((N + 63) / 64, 2 * max_tiles);
  return pair ? launch_chain(grouped_f32_kernel<true>, grid, dim3(256), 0, (cudaStream_t)stream, a, lda, index, b, c, ldc, N, K, (const int4*)tiles, num_tiles, rows, gu)
              : launch_chain(grouped_f32_kernel<false>, grid, dim3(256), 0, (cudaStream_t)stream, a, lda, index, b, c, ldc, N, K, (const int4*)tiles, num_tiles, rows, gu);
}
