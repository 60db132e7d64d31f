// C[M,N] = act(A[M,K] * B[N,K]^T) in true f32 (FMA, no reduced-precision matrix mode): the linear of the exact 32-bit mode.
// 64 x 64 output tile per CTA, 256 threads with a 4 x 4 register tile each, K in steps of 16 through shared memory.
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

__global__ void __launch_bounds__(256) linear_f32_kernel(const float* a, long lda, const float* b, long ldb, float* c, long ldc, int M, int N, int K,
                                                         int act) {
  __shared__ float as[16][68], bs[16][68];
  grid_dep_launch();
  grid_dep_wait();
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (threadIdx.x >> 4) + 16 * i, k = threadIdx.x & 15;
      as[k][r] = (m0 + r < M && k0 + k < K) ? a[(long)(m0 + r) * lda + k0 + k] : 0.f;
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
    for (int j = 0; j < 4; ++j)
      if (m0 + ty * 4 + i < M && n0 + tx * 4 + j < N) c[(long)(m0 + ty * 4 + i) * ldc + n0 + tx * 4 + j] = activate(acc[i][j], act);
}

}  // namespace

extern "C" int ifab_linear_f32(const float* a, long lda, const float* b, long ldb, float* c, long ldc, int M, int N, int K, int act, void* stream) {
  if (M < 1 || N < 1 || K < 1) return -1;
  return launch_chain(linear_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, (cudaStream_t)stream, a, lda, b, ldb, c, ldc, M, N, K, act);
}
