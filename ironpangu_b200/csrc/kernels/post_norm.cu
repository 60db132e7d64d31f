// Row operators of decoders that keep an f32 residual stream and normalise a sublayer's OUTPUT before adding it:
//
//   embed_rows_kernel      x = table[id] * scale (f32) and its copy in the activation type (the operand of the next linears), of rms(x) * w
//                          when a gain is given (the norm ahead of the first sublayer); a second f32 copy on request
//   post_norm_add_kernel   x += rms(y) * w; copy in the activation type (of rms(x) * w2 when a second gain is given: the norm ahead
//                          of the output matrix). y is the f32 output of the sublayer's last linear; without w
//                          it is added as it is, without y nothing is; rows of `extra` join the update. y may
//                          come in parts of a sum
//   rms_rows_kernel        rms(x[row]) * w of selected rows, in the activation type (the norm ahead of the output matrix)
//   group_norm_gate_kernel (o / rms of each group of columns [* w]) * act(gate): the normalised, gated heads of a recurrent
//                          mixer. group = one head without a gain, or all heads together with one
//   gate_rows_kernel       o * act(gate), reading heads at a padded stride
//   gated_rows_kernel      [gate | up] rows -> the gated unit's value (rope.cuh)
//
// Every kernel exists for bf16 activations and for f32 ones; norms and the residual are f32 in both.
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

__device__ __forceinline__ void store4(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
__device__ __forceinline__ void store4(bf16* p, const float* f) {
  __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

template <typename A>
__global__ void __launch_bounds__(256) embed_rows_kernel(const int32_t* ids, const A* table, long ldt, float scale, const float* w, float eps, float* x, long ldx,
                                                         float* copy, A* xa, long lda, int D, int vocab, uint32_t* status) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0 && status) atomicOr(status, IFAB_STATUS_BAD_INDEX);
    id = 0;
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    const float v = to_f32(table[(long)id * ldt + c]) * scale;
    x[(long)t * ldx + c] = v;
    if (copy) copy[(long)t * ldx + c] = v;
    if (!w) xa[(long)t * lda + c] = from_f32<A>(v);
    ss += v * v;
  }
  if (!w) return;
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
  for (int c = threadIdx.x; c < D; c += blockDim.x) xa[(long)t * lda + c] = from_f32<A>(to_f32(table[(long)id * ldt + c]) * scale * inv * w[c]);
}

// one CTA per row
template <typename A>
__global__ void __launch_bounds__(256) post_norm_add_kernel(const float* y, long ldy, int parts, long part_stride, const float* w, const float* w2, float eps, float* x, long ldx,
                                                            const float* extra, long lde, A* xa, long lda, int D) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x;
  const float* yr = y ? y + (long)t * ldy : nullptr;
  const float* er = extra ? extra + (long)t * lde : nullptr;
  float* xr = x + (long)t * ldx;
  A* ar = xa + (long)t * lda;
  if (D % 4 == 0 && ldy % 4 == 0 && ldx % 4 == 0 && lda % 4 == 0 && lde % 4 == 0 && part_stride % 4 == 0 && D <= 256 * 16) {     // the row stays in registers between the passes
    float4 v[4], r[4], g[4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      r[i] = v[i];
      g[i] = make_float4(1.f, 1.f, 1.f, 1.f);
      if (c < D) {
        if (yr) v[i] = *reinterpret_cast<const float4*>(yr + c);
        for (int q = 1; q < parts; ++q) {
          const float4 a = *reinterpret_cast<const float4*>(yr + q * part_stride + c);
          v[i].x += a.x;
          v[i].y += a.y;
          v[i].z += a.z;
          v[i].w += a.w;
        }
        r[i] = *reinterpret_cast<const float4*>(xr + c);
        if (w) g[i] = *reinterpret_cast<const float4*>(w + c);
        if (er) {
          const float4 e = *reinterpret_cast<const float4*>(er + c);
          r[i].x += e.x;
          r[i].y += e.y;
          r[i].z += e.z;
          r[i].w += e.w;
        }
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = w ? 1.f / sqrtf(block_sum(ss, red) / (float)D + eps) : 1.f;
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      r[i].x += v[i].x * inv * g[i].x;
      r[i].y += v[i].y * inv * g[i].y;
      r[i].z += v[i].z * inv * g[i].z;
      r[i].w += v[i].w * inv * g[i].w;
      if (c < D) *reinterpret_cast<float4*>(xr + c) = r[i];
      ss += r[i].x * r[i].x + r[i].y * r[i].y + r[i].z * r[i].z + r[i].w * r[i].w;
    }
    const float inv2 = w2 ? 1.f / sqrtf(block_sum(ss, red) / (float)D + eps) : 1.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= D) break;
      float f[4] = {r[i].x, r[i].y, r[i].z, r[i].w};
      if (w2) {
        const float4 h = *reinterpret_cast<const float4*>(w2 + c);
        f[0] *= inv2 * h.x;
        f[1] *= inv2 * h.y;
        f[2] *= inv2 * h.z;
        f[3] *= inv2 * h.w;
      }
      store4(ar + c, f);
    }
    return;
  }
  float ss = 0.f;
  auto value = [&](int c) {
    float v = yr[c];
    for (int q = 1; q < parts; ++q) v += yr[q * part_stride + c];
    return v;
  };
  if (yr && w)
    for (int c = threadIdx.x; c < D; c += blockDim.x) {
      const float v = value(c);
      ss += v * v;
    }
  const float inv = yr && w ? 1.f / sqrtf(block_sum(ss, red) / (float)D + eps) : 1.f;
  ss = 0.f;
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    float v = xr[c] + (er ? er[c] : 0.f);
    if (yr) v += value(c) * inv * (w ? w[c] : 1.f);
    xr[c] = v;
    ss += v * v;
    if (!w2) ar[c] = from_f32<A>(v);
  }
  if (!w2) return;
  const float inv2 = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
  for (int c = threadIdx.x; c < D; c += blockDim.x) ar[c] = from_f32<A>(xr[c] * inv2 * w2[c]);
}

template <typename A>
__global__ void __launch_bounds__(256) rms_rows_kernel(const float* x, long ldx, const int32_t* rows, const float* w, float eps, A* y, long ldy, int D) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x;
  const float* xr = x + (long)(rows ? rows[t] : t) * ldx;
  float ss = 0.f;
  for (int c = threadIdx.x; c < D; c += blockDim.x) ss += xr[c] * xr[c];
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
  for (int c = threadIdx.x; c < D; c += blockDim.x) y[(long)t * ldy + c] = from_f32<A>(xr[c] * inv * w[c]);
}

// one warp per (row, group) for narrow groups, one CTA per row for a single wide one: grid (ceil(groups / WPB), rows)
template <typename A, int WARPS_PER_GROUP>
__global__ void __launch_bounds__(256) group_norm_gate_kernel(const float* o, long ldo, const float* w, float eps, const A* gate, long ldg, int act,
                                                              A* y, long ldy, int groups, int n) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.y;
  constexpr int GPB = 8 / WARPS_PER_GROUP, TPG = 32 * WARPS_PER_GROUP;
  const int g = blockIdx.x * GPB + threadIdx.x / TPG, i0 = threadIdx.x % TPG;
  if (WARPS_PER_GROUP == 1 && g >= groups) return;
  const float* r = o + (long)t * ldo + (long)g * n;
  float ss = 0.f;
  for (int c = i0; c < n; c += TPG) ss += r[c] * r[c];
  ss = WARPS_PER_GROUP == 1 ? warp_sum(ss) : block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)n + eps);
  for (int c = i0; c < n; c += TPG) {
    float v = r[c] * inv;
    if (w) v *= w[(long)g * n + c];
    y[(long)t * ldy + (long)g * n + c] = from_f32<A>(v * activate<sizeof(A) == 2>(to_f32(gate[(long)t * ldg + (long)g * n + c]), act));
  }
}

template <typename A>
__global__ void __launch_bounds__(256) gate_rows_kernel(const A* o, long ldo, int head_stride, const A* gate, long ldg, int act, A* y, long ldy, int H,
                                                        int n) {
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x;
  for (int c = threadIdx.x; c < H * n; c += blockDim.x) {
    const int h = c / n, j = c - h * n;
    y[(long)t * ldy + c] = from_f32<A>(to_f32(o[(long)t * ldo + (long)h * head_stride + j]) * activate<sizeof(A) == 2>(to_f32(gate[(long)t * ldg + c]), act));
  }
}

template <typename A>
__global__ void __launch_bounds__(256) gated_rows_kernel(const A* gu, long ld, int up, GatedUnit unit, A* y, long ldy, int F) {
  grid_dep_launch();
  grid_dep_wait();
  const A* r = gu + (long)blockIdx.x * ld;
  for (int c = threadIdx.x; c < F; c += blockDim.x) y[(long)blockIdx.x * ldy + c] = from_f32<A>(gated_value<sizeof(A) == 2>(to_f32(r[c]), to_f32(r[up + c]), unit));
}

template <typename A>
int embed(const int32_t* ids, const void* table, long ldt, float scale, const float* w, float eps, float* x, long ldx, float* copy, void* xa, long lda, int T, int D,
          int vocab, uint32_t* status, cudaStream_t s) {
  return launch_chain(embed_rows_kernel<A>, dim3(T), dim3(256), 0, s, ids, (const A*)table, ldt, scale, w, eps, x, ldx, copy, (A*)xa, lda, D, vocab, status);
}
template <typename A>
int group_norm(const float* o, long ldo, const float* w, float eps, const void* gate, long ldg, int act, void* y, long ldy, int T, int groups, int n,
               cudaStream_t s) {
  if (n > 512)
    return launch_chain(group_norm_gate_kernel<A, 8>, dim3(groups, T), dim3(256), 0, s, o, ldo, w, eps, (const A*)gate, ldg, act, (A*)y, ldy, groups, n);
  return launch_chain(group_norm_gate_kernel<A, 1>, dim3((groups + 7) / 8, T), dim3(256), 0, s, o, ldo, w, eps, (const A*)gate, ldg, act, (A*)y, ldy,
                      groups, n);
}

}  // namespace

// copy: a second f32 copy of x (row stride ldx), or null
extern "C" int ifab_embed_rows(const int32_t* ids, const void* table, long ldt, float scale, const float* w, float eps, float* x, long ldx, float* copy, void* xa,
                               long lda, int f32, int T, int D, int vocab, uint32_t* status, void* stream) {
  if (T < 1 || D < 1 || vocab < 1) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? embed<float>(ids, table, ldt, scale, w, eps, x, ldx, copy, xa, lda, T, D, vocab, status, s)
             : embed<bf16>(ids, table, ldt, scale, w, eps, x, ldx, copy, xa, lda, T, D, vocab, status, s);
}

// y: the sum of `parts` rows, part_stride elements apart
extern "C" int ifab_post_norm_add(const float* y, long ldy, int parts, long part_stride, const float* w, const float* w2, float eps, float* x, long ldx, const float* extra, long lde, void* xa,
                                  long lda, int f32, int T, int D, void* stream) {
  if (T < 1 || D < 1 || parts < 1) return -1;
  if (!y) parts = 1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? launch_chain(post_norm_add_kernel<float>, dim3(T), dim3(256), 0, s, y, ldy, parts, part_stride, w, w2, eps, x, ldx, extra, lde, (float*)xa, lda, D)
             : launch_chain(post_norm_add_kernel<bf16>, dim3(T), dim3(256), 0, s, y, ldy, parts, part_stride, w, w2, eps, x, ldx, extra, lde, (bf16*)xa, lda, D);
}

// y [T, F] = unit(gu[:, c], gu[:, up + c])
extern "C" int ifab_gated_rows(const void* gu, long ld, int up, int unit, float limit, float alpha, void* y, long ldy, int f32, int T, int F, void* stream) {
  const GatedUnit u{unit, limit, alpha};
  if (T < 1 || F < 1 || up < F || !gated_ok(u)) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? launch_chain(gated_rows_kernel<float>, dim3(T), dim3(256), 0, s, (const float*)gu, ld, up, u, (float*)y, ldy, F)
             : launch_chain(gated_rows_kernel<bf16>, dim3(T), dim3(256), 0, s, (const bf16*)gu, ld, up, u, (bf16*)y, ldy, F);
}

extern "C" int ifab_rms_rows(const float* x, long ldx, const int32_t* rows, const float* w, float eps, void* y, long ldy, int f32, int T, int D,
                             void* stream) {
  if (T < 1 || D < 1) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? launch_chain(rms_rows_kernel<float>, dim3(T), dim3(256), 0, s, x, ldx, rows, w, eps, (float*)y, ldy, D)
             : launch_chain(rms_rows_kernel<bf16>, dim3(T), dim3(256), 0, s, x, ldx, rows, w, eps, (bf16*)y, ldy, D);
}

extern "C" int ifab_group_norm_gate(const float* o, long ldo, const float* w, float eps, const void* gate, long ldg, int act, void* y, long ldy, int f32,
                                    int T, int groups, int n, void* stream) {
  if (T < 1 || groups < 1 || n < 1 || T > 65535) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? group_norm<float>(o, ldo, w, eps, gate, ldg, act, y, ldy, T, groups, n, s) : group_norm<bf16>(o, ldo, w, eps, gate, ldg, act, y, ldy, T, groups, n, s);
}

extern "C" int ifab_gate_rows(const void* o, long ldo, int head_stride, const void* gate, long ldg, int act, void* y, long ldy, int f32, int T, int H, int n,
                              void* stream) {
  if (T < 1 || H < 1 || n < 1) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? launch_chain(gate_rows_kernel<float>, dim3(T), dim3(256), 0, s, (const float*)o, ldo, head_stride, (const float*)gate, ldg, act, (float*)y, ldy,
                            H, n)
             : launch_chain(gate_rows_kernel<bf16>, dim3(T), dim3(256), 0, s, (const bf16*)o, ldo, head_stride, (const bf16*)gate, ldg, act, (bf16*)y, ldy, H, n);
}
