// One small product per head on tcgen05: C[t, h * c_stride + n] = sum_k A[t, h * a_stride + k] * B[h, n, k], heads side by side in the rows of
// A and C. The absorbed projections of latent attention for many rows: query part -> latent (B = W_uk transposed) and latent -> value
// (B = W_uv). One launch for all heads; columns of A past K belong to other parts of the row and meet the zero fill of B.
#include "tc_gemm_core.cuh"
#include "ifab_kernels.h"

using namespace ifab;
using namespace ifab::tc;

namespace {

struct HeadsParams {
  void* c; long ldc; int c_stride, out_f32;
  int a_stride, M, N, K, a_rows;
  uint32_t* status;
  uint32_t spin_limit;
};

// grid (ceil(N / BN), ceil(M / 128), heads)
template <int BN, int ST>
__global__ void __launch_bounds__(192) tc_heads_kernel(const __grid_constant__ CUtensorMap tmap_a, const __grid_constant__ CUtensorMap tmap_b, HeadsParams p) {
  extern __shared__ unsigned char smem_raw[];
  Pipe<BN, ST> pipe;
  pipe.setup(smem_raw, &tmap_a, &tmap_b);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.z;
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN, num_kb = (p.K + BK - 1) / BK;
  grid_dep_launch();
  grid_dep_wait();
  if (warp == 0 && lane == 0) {
    pipe.produce(&tmap_a, &tmap_b, num_kb, m0, n0, h, p.spin_limit, p.status, -1, p.a_rows, h * p.a_stride);
  } else if (warp == 1 && lane == 0) {
    pipe.mma(num_kb, p.spin_limit, p.status);
  } else if (warp >= 2 && pipe.wait_accumulator(p.spin_limit, p.status)) {
    const int q = warp & 3, row = m0 + q * 32 + lane;
#pragma unroll 1
    for (int c0 = 0; c0 < BN; c0 += 32) {
      float v[32];
      tmem_ld_32x32(pipe.tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)c0, v);
      tmem_ld_wait();
      if (row < p.M && n0 + c0 < p.N) {
        const int n = min(32, p.N - n0 - c0);
        const long at = (long)row * p.ldc + (long)h * p.c_stride + n0 + c0;
        if (p.out_f32) {
          float* out = reinterpret_cast<float*>(p.c) + at;
          if (n == 32 && (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
  #pragma unroll
            for (int i = 0; i < 8; ++i) reinterpret_cast<float4*>(out)[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
          } else {
  #pragma unroll
            for (int i = 0; i < 32; ++i)
              if (i < n) out[i] = v[i];
          }
        } else {
          bf16* out = reinterpret_cast<bf16*>(p.c) + at;
          if (n == 32 && (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
  #pragma unroll
            for (int i = 0; i < 4; ++i) reinterpret_cast<uint4*>(out)[i] = pack8(v + 8 * i);
          } else {
  #pragma unroll
            for (int i = 0; i < 32; ++i)
              if (i < n) out[i] = __float2bfloat16_rn(v[i]);
          }
        }
      }
    }
  }
  pipe.teardown();
}

template <int BN, int ST>
int launch_heads(const CUtensorMap& ta, const CUtensorMap& tb, const HeadsParams& p, int heads, cudaStream_t s) {
  auto k = tc_heads_kernel<BN, ST>;
  if (int rc = opt_in_smem(k, Cfg<BN, ST>::SMEM)) return rc;
  return launch_chain(k, dim3((p.N + BN - 1) / BN, (p.M + BM - 1) / BM, heads), dim3(192), (size_t)Cfg<BN, ST>::SMEM, s, ta, tb, p);
}

}  // namespace

// a: bf16 [M, lda], head h at columns h * a_stride + [0, K); b: bf16 [heads, N, ldb] (K columns valid); strides and leading dimensions of a and b
// multiples of 8
extern "C" int ifab_gemm_heads_bf16(const void* a, long lda, int a_stride, const void* b, long ldb, void* c, long ldc, int c_stride, int out_f32, int heads, int M,
                                    int N, int K, uint32_t* status, void* stream) {
  if (heads < 1 || heads > 65535 || M < 1 || N < 1 || K < 1 || lda % 8 || a_stride % 8 || ldb % 8 || (heads - 1L) * a_stride + K > lda) return -1;
  // enough CTAs to fill the SMs: narrow tiles when there are few rows
  const int rows = (M + BM - 1) / BM;
  int BN = 32;
  while (BN < 128 && (long)rows * heads * ((N + BN - 1) / BN) > 296) BN *= 2;
  const int a_rows = M <= BM ? (M + 7) / 8 * 8 : BM;
  CUtensorMap ta, tb;
  if (int rc = make_tmap_bf16_2d(&ta, a, (uint64_t)M, (uint64_t)((heads - 1L) * a_stride + K), (uint64_t)lda, (uint32_t)a_rows)) return rc;
  if (int rc = make_tmap_bf16_3d(&tb, b, (uint64_t)heads, (uint64_t)N, (uint64_t)K, (uint64_t)ldb, (uint64_t)N * ldb, (uint32_t)BN)) return rc;
  HeadsParams p{c, ldc, c_stride, out_f32, a_stride, M, N, K, a_rows, status, 4000000u};
  cudaStream_t s = (cudaStream_t)stream;
  return BN == 128 ? launch_heads<128, 4>(ta, tb, p, heads, s) : BN == 64 ? launch_heads<64, 4>(ta, tb, p, heads, s) : launch_heads<32, 5>(ta, tb, p, heads, s);
}
