// Routed experts of decoders with an f32 residual stream, for any number of rows, around the dispatch of moe_prefill.cu and the grouped
// GEMMs (tc_grouped.cu in bf16, linear_f32.cu in the exact mode):
//
//   moe_route_kernel         f32 router logits (+ bias) -> ids and weights of the chosen experts (moe_select.cuh), and the shared
//                            expert's weight sigmoid(logits[:, E]) when the logits carry that column
//   moe_combine_norm_kernel  y = sum of the chosen experts' rows by weight + shared weight * shared row (f32, slot order); then the
//                            residual update x += rms(y) * w and the next operand xa = rms(x) * w2 (or x). Without w, y is added
//                            as it is, together with f32 rows `base` (what ran beside the experts, perhaps in parts of a
//                            sum) and `extra`
#include "moe_select.cuh"
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

struct RouteParams {
  const float* logits; long ld; const float* bias;
  int M, E, topk, scoring, renorm; float scale;
  int32_t* ids; float* wts; float* shared_w;
  int groups, keep;
};

// one warp per row
__global__ void __launch_bounds__(128) moe_route_kernel(RouteParams p) {
  grid_dep_launch();
  grid_dep_wait();
  const int m = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= p.M) return;
  const float* z = p.logits + (long)m * p.ld;
  select_topk_row(z, p.bias, p.E, p.topk, p.scoring, p.renorm, p.scale, p.ids + (long)m * p.topk, p.wts + (long)m * p.topk, p.groups, p.keep);
  if (p.shared_w && lane == 0) p.shared_w[m] = sigmoid_f32(z[p.E]);
}

__device__ __forceinline__ void load4(const bf16* p, float* f) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void load4(const float* p, float* f) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void store4(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
__device__ __forceinline__ void store4(bf16* p, const float* f) {
  __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

struct CombineNormParams {
  const void* y; long ldy;               // expert outputs by permuted row
  const int32_t* route_row; const float* wts; int topk;
  const void* shared; long lds; const float* shared_w;      // shared expert's rows (or null) and their weights (null: 1)
  const float *w, *w2; float eps;
  float* x; long ldx; void* xa; long lda;
  const float *base, *extra; long ldb, lde;      // rows of the residual update (without w), or null
  int parts; long part_stride;           // of base
  int D, Dp;                             // Dp: D padded to 4 columns; the padding of every operand is zero
};

// one CTA per row; a thread keeps NV quads of the row in registers
template <typename A, int NV>
__global__ void __launch_bounds__(256) moe_combine_norm_kernel(CombineNormParams p) {
  __shared__ float red[33];
  __shared__ int s_row[MAX_TOPK];
  __shared__ float s_w[MAX_TOPK];
  grid_dep_launch();
  grid_dep_wait();
  const int m = blockIdx.x;
  if ((int)threadIdx.x < p.topk) {
    s_row[threadIdx.x] = p.route_row[(long)m * p.topk + threadIdx.x];
    s_w[threadIdx.x] = p.wts[(long)m * p.topk + threadIdx.x];
  }
  const float sw = p.shared && p.shared_w ? p.shared_w[m] : 1.f;
  __syncthreads();
  float v[NV][4];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) v[i][j] = 0.f;
    if (c < p.Dp) {
#pragma unroll 4
      for (int k = 0; k < p.topk; ++k) {
        const int r = s_row[k];
        if (r < 0) continue;
        float f[4];
        load4(reinterpret_cast<const A*>(p.y) + (long)r * p.ldy + c, f);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i][j] = fmaf(s_w[k], f[j], v[i][j]);
      }
      if (p.shared) {
        float f[4];
        load4(reinterpret_cast<const A*>(p.shared) + (long)m * p.lds + c, f);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i][j] = fmaf(sw, f[j], v[i][j]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += v[i][j] * v[i][j];
    }
  }
  const float inv = p.w ? 1.f / sqrtf(block_sum(ss, red) / (float)p.D + p.eps) : 1.f;
  float* xr = p.x + (long)m * p.ldx;
  A* ar = reinterpret_cast<A*>(p.xa) + (long)m * p.lda;
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 4;
    if (c < p.Dp) {
      float r[4];
      load4(xr + c, r);
      if (p.base) {
        float b[4];
        load4(p.base + (long)m * p.ldb + c, b);
        for (int q = 1; q < p.parts; ++q) {
          float f[4];
          load4(p.base + q * p.part_stride + (long)m * p.ldb + c, f);
#pragma unroll
          for (int j = 0; j < 4; ++j) b[j] += f[j];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i][j] += b[j];
      }
      if (p.extra) {
        float f[4];
        load4(p.extra + (long)m * p.lde + c, f);
#pragma unroll
        for (int j = 0; j < 4; ++j) r[j] += f[j];
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        v[i][j] = c + j < p.D ? r[j] + (p.w ? v[i][j] * inv * p.w[c + j] : v[i][j]) : 0.f;
        ss += v[i][j] * v[i][j];
      }
      store4(xr + c, v[i]);
    }
  }
  const float inv2 = p.w2 ? 1.f / sqrtf(block_sum(ss, red) / (float)p.D + p.eps) : 1.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 4;
    if (c < p.Dp) {
      if (p.w2)
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i][j] = c + j < p.D ? v[i][j] * inv2 * p.w2[c + j] : 0.f;
      store4(ar + c, v[i]);
    }
  }
}

template <typename A>
int combine(const CombineNormParams& p, int M, cudaStream_t s) {
  if (p.Dp <= 1024) return launch_chain(moe_combine_norm_kernel<A, 1>, dim3(M), dim3(256), 0, s, p);
  if (p.Dp <= 2048) return launch_chain(moe_combine_norm_kernel<A, 2>, dim3(M), dim3(256), 0, s, p);
  if (p.Dp <= 4096) return launch_chain(moe_combine_norm_kernel<A, 4>, dim3(M), dim3(256), 0, s, p);
  if (p.Dp <= 8192) return launch_chain(moe_combine_norm_kernel<A, 8>, dim3(M), dim3(256), 0, s, p);
  return -2;
}

}  // namespace

extern "C" int ifab_moe_route(const float* logits, long ld, const float* bias, int M, int E, int topk, int scoring, int renorm, float scale, int groups, int keep,
                              int32_t* ids, float* wts, float* shared_w, void* stream) {
  if (M < 1 || !select_ok(E, topk, scoring, groups, keep)) return -1;
  RouteParams p{logits, ld, bias, M, E, topk, scoring, renorm, scale, ids, wts, shared_w, groups, keep};
  return launch_chain(moe_route_kernel, dim3((M + 3) / 4), dim3(128), 0, (cudaStream_t)stream, p);
}

extern "C" int ifab_moe_combine_norm(const void* y, long ldy, const int32_t* route_row, const float* wts, int topk, const void* shared, long lds,
                                     const float* shared_w, const float* w, const float* w2, float eps, const float* base, long ldb, int parts, long part_stride, const float* extra, long lde,
                                     float* x, long ldx, void* xa, long lda, int f32, int M, int D, void* stream) {
  const int Dp = (D + 3) / 4 * 4;
  if (M < 1 || D < 1 || topk < 1 || topk > MAX_TOPK || ldy % 4 || ldx % 4 || lda % 4 || (shared && lds % 4) || ldy < Dp || ldx < Dp || lda < Dp || (shared && lds < Dp))
    return -1;
  if ((w && base) || (base && (ldb % 4 || ldb < Dp || parts < 1 || part_stride % 4)) || (extra && (lde % 4 || lde < Dp))) return -1;
  CombineNormParams p{y, ldy, route_row, wts, topk, shared, lds, shared_w, w, w2, eps, x, ldx, xa, lda, base, extra, ldb, lde, parts, part_stride, D, Dp};
  return f32 ? combine<float>(p, M, (cudaStream_t)stream) : combine<bf16>(p, M, (cudaStream_t)stream);
}
