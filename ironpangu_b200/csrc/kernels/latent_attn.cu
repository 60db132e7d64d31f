// Latent attention over a paged cache of one row per token, for any sizes: [latent (normed), padded to Lp | rotated key part shared by
// all heads, padded to Rp], both paddings zero, 16-byte aligned. bf16 (serving) or f32 (exact mode) activations and caches; norms,
// angles, scores, weights and sums are f32 in both.
//
//   latent_prepare_kernel   one packed projection row -> normed query latent (operand of the query up-projection), and into the page of
//                           the row's sequence: normed latent, rotated key part
//   latent_query_kernel     the same for a few rows (decode) in one launch with the query up-projection: the first CTAs stream W_uq and norm the
//                           query latent while they stage it, the last T write the pages
//   rotate_heads_kernel     rotation of the rotated columns of every query head, in place (half layout)
//   latent_absorb_kernel    q_lat[h] = q_unrotated[h] W_uk[h] for a few rows (decode), rotation of the rest included
//   latent_split_kernel     split-KV attention over the pages with an optional sliding window: every warp scores four keys for HG heads
//                           at once; the HG x 4 sums are reduced through a transposing butterfly, so each lane ends with ONE
//                           (key, head) score, takes one exponential and the weights are broadcast back
//   latent_batch_kernel     the same for many rows: the warps of a CTA split the HEADS first (four each) and the keys only with what is left of them; the
//                           keys of a split pass through a ring of shared-memory stages (cp.async) once for all heads
//   latent_merge_kernel     log-sum-exp merge of the splits, head gate -> o_lat rows (operand of the value up-projection)
//   latent_merge_vup_kernel merge, gate and value up-projection for a few rows (decode)
//   latent_gather_kernel    the rows a run of queries can see, out of the pages into dense operands of the tensor-core form
#include "gemv.cuh"
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

struct Pages {
  const int32_t *positions, *slots, *page_table;
  int max_pages, page_tokens, num_pages;
  uint32_t* status;
};

__device__ __forceinline__ long page_row(const Pages& p, int slot, int pos) {
  const int lp = pos / p.page_tokens;
  const int page = lp < p.max_pages ? p.page_table[(long)slot * p.max_pages + lp] : -1;
  return page >= 0 && page < p.num_pages ? (long)page * p.page_tokens + pos % p.page_tokens : -1;
}

__device__ __forceinline__ void load8(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
// raw registers of eight / two elements, to have many rows in flight before any is used
template <typename A>
struct Raw8;
template <>
struct Raw8<bf16> {
  uint4 v;
  __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void zero() { v = make_uint4(0, 0, 0, 0); }
  __device__ __forceinline__ void get(float* f) const { unpack8(v, f); }
};
template <>
struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = *reinterpret_cast<const float4*>(p);
    b = *reinterpret_cast<const float4*>(p + 4);
  }
  __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float* f) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
};
template <typename A>
struct Raw2;
template <>
struct Raw2<bf16> {
  __nv_bfloat162 v;
  __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const __nv_bfloat162*>(p); }
  __device__ __forceinline__ void zero() { v = __floats2bfloat162_rn(0.f, 0.f); }
  __device__ __forceinline__ float2 get() const { return __bfloat1622float2(v); }
};
template <>
struct Raw2<float> {
  float2 v;
  __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float2*>(p); }
  __device__ __forceinline__ void zero() { v = make_float2(0.f, 0.f); }
  __device__ __forceinline__ float2 get() const { return v; }
};

template <bool FAST>
__device__ __forceinline__ float exp_f32(float x) { return FAST ? __expf(x) : expf(x); }

// ------------------------------------------------------------------------------------------------
struct PrepareParams {
  const void* proj; long ldp; int q_off, q_rank, kv_off, kv_rank, rot_dim;
  const float *q_gain, *kv_gain; float eps;
  const float2* cs; int rot;                 // (cos, sin) [T, rot / 2]
  Pages pg;
  void* cq; long ldc;                        // null: the query latent is normed elsewhere
  void* cache; int Lp, Rp;
};

template <typename A>
__device__ __forceinline__ void prepare_row(const PrepareParams& p, int t, float* red) {
  const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
  if (p.cq) {
    const A* src = row + p.q_off;
    float ss = 0.f;
    for (int c = threadIdx.x; c < p.q_rank; c += blockDim.x) {
      const float v = to_f32(src[c]);
      ss += v * v;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.q_rank + p.eps);
    A* dst = reinterpret_cast<A*>(p.cq) + (long)t * p.ldc;
    for (int c = threadIdx.x; c < p.q_rank; c += blockDim.x) dst[c] = from_f32<A>(to_f32(src[c]) * inv * p.q_gain[c]);
  }
  const int pos = p.pg.positions[t];
  if (pos < 0) return;
  const long r = page_row(p.pg, p.pg.slots[t], pos);
  if (r < 0) {
    if (threadIdx.x == 0 && p.pg.status) atomicOr(p.pg.status, IFAB_STATUS_BAD_INDEX);
    return;
  }
  const A* src = row + p.kv_off;
  A* dst = reinterpret_cast<A*>(p.cache) + r * (p.Lp + p.Rp);
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.kv_rank; c += blockDim.x) {
    const float v = to_f32(src[c]);
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.kv_rank + p.eps);
  for (int c = threadIdx.x; c < p.kv_rank; c += blockDim.x) dst[c] = from_f32<A>(to_f32(src[c]) * inv * p.kv_gain[c]);
  const A* kr = src + p.kv_rank;
  A* dr = dst + p.Lp;
  const RopeTable rt{nullptr, p.rot, 0};
  const float2* cs = p.cs + (long)t * (p.rot / 2);
  for (int c = threadIdx.x; c < p.rot_dim; c += blockDim.x) dr[c] = from_f32<A>(c < p.rot ? rotated(rt, cs, kr, c) : to_f32(kr[c]));
}

template <typename A>
__global__ void __launch_bounds__(256) latent_prepare_kernel(PrepareParams p) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  prepare_row<A>(p, blockIdx.x, red);
}

template <int T, int R>
__global__ void __launch_bounds__(256) latent_query_kernel(PrepareParams p, const bf16* w_uq, const bf16* q_gain, int N, int ctas, bf16* q, long ldq, int rows) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* xs = reinterpret_cast<bf16*>(smem_raw);
  __shared__ float red[T * 33];
  grid_dep_launch();
  if ((int)blockIdx.x >= ctas) {
    grid_dep_wait();
    prepare_row<bf16>(p, blockIdx.x - ctas, red);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = (blockIdx.x * 8 + warp) * R;
  const bf16* w[R];
#pragma unroll
  for (int r = 0; r < R; ++r) w[r] = n0 + r < N ? w_uq + (long)(n0 + r) * p.q_rank : nullptr;
  RowBatch<R> pf;
  prefetch_rows<R>(w, p.q_rank, pf);
  grid_dep_wait();
  stage_x<T>(xs, reinterpret_cast<const bf16*>(p.proj) + p.q_off, p.ldp, 0, rows, p.q_rank, q_gain, p.eps, false, red);
  if (n0 >= N) return;
  float acc[R][T];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int t = 0; t < T; ++t) acc[r][t] = 0.f;
  warp_rows_dot<T, R>(w, xs, p.q_rank, acc, pf);
  warp_reduce_acc<T, R>(acc);
  if (lane == 0) {
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int t = 0; t < T; ++t)
        if (n0 + r < N && t < rows) q[(long)t * ldq + n0 + r] = __float2bfloat16_rn(acc[r][t]);
  }
}

template <int T, int R>
int launch_query(const PrepareParams& p, const bf16* w_uq, const bf16* q_gain, int N, bf16* q, long ldq, int rows, cudaStream_t s) {
  const size_t smem = (size_t)T * p.q_rank * sizeof(bf16);
  auto k = latent_query_kernel<T, R>;
  if (int rc = opt_in_smem(k, smem)) return rc;
  const int ctas = (N + 8 * R - 1) / (8 * R);
  return launch_chain(k, dim3(ctas + rows), dim3(256), smem, s, p, w_uq, q_gain, N, ctas, q, ldq, rows);
}
template <int T>
int query_rows(const PrepareParams& p, const bf16* w_uq, const bf16* q_gain, int N, bf16* q, long ldq, int rows, cudaStream_t s) {
  if (N >= 148 * 8 * 4) return launch_query<T, 4>(p, w_uq, q_gain, N, q, ldq, rows, s);
  if (N >= 148 * 8 * 2) return launch_query<T, 2>(p, w_uq, q_gain, N, q, ldq, rows, s);
  return launch_query<T, 1>(p, w_uq, q_gain, N, q, ldq, rows, s);
}

template <typename A>
__global__ void __launch_bounds__(256) rotate_heads_kernel(A* q, long ldq, int head_stride, int off, int H, int rot, const float2* cs) {
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, half = rot / 2;
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, j = i - h * half;
    A* r = q + (long)t * ldq + (long)h * head_stride + off;
    const float2 a = cs[(long)t * half + j];
    const float u = to_f32(r[j]), v = to_f32(r[j + half]);
    r[j] = from_f32<A>(u * a.x - v * a.y);
    r[j + half] = from_f32<A>(v * a.x + u * a.y);
  }
}

// ------------------------------------------------------------------------------------------------
// grid (H, T, ceil(Lp / 128)), 256 threads: thread (ds, cg) owns 8 columns and 8 query elements at a time; weights requested before the
// wait. CTA z == 0 rotates the head's rotated columns in place.
__global__ void __launch_bounds__(256) latent_absorb_kernel(bf16* q, long ldq, int head_stride, int rot_off, const bf16* w_uk, const float2* cs, int rot,
                                                            float* q_lat, int H, int d, int Lp) {
  __shared__ float qs[128];
  __shared__ float part[16][129];
  grid_dep_launch();
  const int h = blockIdx.x, t = blockIdx.y, cg = threadIdx.x & 15, ds = threadIdx.x >> 4, col = blockIdx.z * 128 + cg * 8;
  const bf16* W = w_uk + (long)h * d * Lp + col;
  uint4 wv[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) wv[j] = (ds * 8 + j < d && col < Lp) ? ld_stream16(W + (long)(ds * 8 + j) * Lp) : make_uint4(0, 0, 0, 0);
  grid_dep_wait();
  bf16* qrow = q + (long)t * ldq + (long)h * head_stride;
  float acc[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  for (int d0 = 0; d0 < d; d0 += 128) {
    __syncthreads();
    for (int i = threadIdx.x; i < 128; i += blockDim.x) qs[i] = d0 + i < d ? __bfloat162float(qrow[d0 + i]) : 0.f;
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int dd = d0 + ds * 8 + j;
      if (dd >= d || col >= Lp) break;
      float wf[8];
      unpack8(d0 == 0 ? wv[j] : ld_stream16(W + (long)dd * Lp), wf);
      const float qd = qs[ds * 8 + j];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] = fmaf(qd, wf[i], acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) part[ds][cg * 8 + i] = acc[i];
  __syncthreads();
  const int c = blockIdx.z * 128 + threadIdx.x;
  if (threadIdx.x < 128 && c < Lp) {
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < 16; ++k) v += part[k][threadIdx.x];
    q_lat[((long)t * H + h) * Lp + c] = v;
  }
  if (blockIdx.z == 0 && threadIdx.x >= 128) {
    const int half = rot / 2;
    bf16* r = qrow + rot_off;
    for (int j = threadIdx.x - 128; j < half; j += 128) {
      const float2 a = cs[(long)t * half + j];
      const float u = __bfloat162float(r[j]), v = __bfloat162float(r[j + half]);
      r[j] = __float2bfloat16_rn(u * a.x - v * a.y);
      r[j + half] = __float2bfloat16_rn(v * a.x + u * a.y);
    }
  }
}

// ------------------------------------------------------------------------------------------------
struct SplitParams {
  const float* q_lat;                               // [T, H, Lp]
  const void* q_rot; long ldq; int head_stride;     // rotated columns of head h of row t at t * ldq + h * head_stride
  const void* cache; int Lp, Rp;
  Pages pg;
  int window; float scale;
  int T, H, kps, splits;
  float* scratch;                                   // [T, H, splits, Lp + 2]
};

__device__ __forceinline__ void visible(int pos, int window, int* first, int* count) {
  *count = window > 0 ? min(pos + 1, window) : pos + 1;
  *first = pos + 1 - *count;
}

// sum of V values per lane over the warp; afterwards lane l holds the total of value l / (32 / V)
template <int V>
__device__ __forceinline__ float transpose_sum(float (&s)[V]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int n = V, off = 16; n > 1; n >>= 1, off >>= 1) {
    const bool up = lane & off;
#pragma unroll
    for (int i = 0; i < n / 2; ++i) {
      const float give = up ? s[i] : s[i + n / 2], keep = up ? s[i + n / 2] : s[i];
      s[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
    }
  }
  float v = s[0];
#pragma unroll
  for (int off = 16 / V; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
  return v;
}

constexpr int KB = 4, WARPS = 8;

// A: cache type; NL: 256-column pieces of the latent, NR: 64-column pieces of the rotated part, HG: heads of a CTA
template <typename A, int NL, int NR, int HG>
__global__ void __launch_bounds__(256) latent_split_kernel(SplitParams p) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  float* sm_acc = reinterpret_cast<float*>(smem_raw);            // [8][HG][NL * 256]
  float* sm_m = sm_acc + WARPS * HG * NL * 256;
  float* sm_l = sm_m + WARPS * HG;
  constexpr bool FAST = sizeof(A) == 2;
  constexpr int V = KB * HG, GRP = 32 / V;
  grid_dep_launch();
  grid_dep_wait();
  const int split = blockIdx.x, hg = blockIdx.y, t = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.pg.positions[t];
  if (pos < 0) return;
  int first, count;
  visible(pos, p.window, &first, &count);
  const int k_begin = split * p.kps;
  if (k_begin >= count) return;
  const int k_end = split == p.splits - 1 ? count : min(count, k_begin + p.kps);      // the last split takes what is left
  const int slot = p.pg.slots[t];
  float ql[HG][NL * 8], qr[HG][NR * 2], acc[HG][NL * 8];
#pragma unroll
  for (int g = 0; g < HG; ++g) {
    const float* a = p.q_lat + ((long)t * p.H + hg * HG + g) * p.Lp;
    const A* b = reinterpret_cast<const A*>(p.q_rot) + (long)t * p.ldq + (long)(hg * HG + g) * p.head_stride;
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      const int c = i * 256 + lane * 8;
      if (c < p.Lp) load8(a + c, &ql[g][i * 8]);
      else
#pragma unroll
        for (int j = 0; j < 8; ++j) ql[g][i * 8 + j] = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        ql[g][i * 8 + j] *= p.scale;
        acc[g][i * 8 + j] = 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = i * 64 + lane * 2;
      qr[g][2 * i] = c < p.Rp ? to_f32(b[c]) * p.scale : 0.f;
      qr[g][2 * i + 1] = c < p.Rp ? to_f32(b[c + 1]) * p.scale : 0.f;
    }
  }
  const int my_key = (lane / GRP) / HG;            // which (key, head) of a batch this lane ends up with
  float m = -INFINITY, l = 0.f;                    // of this lane's head; l: this lane's keys only
  for (int kb = k_begin + warp; kb < k_end; kb += WARPS * KB) {
    Raw8<A> rl[KB][NL];
    Raw2<A> rr[KB][NR];
    bool ok[KB];
#pragma unroll
    for (int j = 0; j < KB; ++j) {
      const int k = kb + WARPS * j;
      ok[j] = k < k_end;
      long r = -1;
      if (ok[j]) {
        r = page_row(p.pg, slot, first + k);
        if (r < 0) {
          if (lane == 0 && p.pg.status) atomicOr(p.pg.status, IFAB_STATUS_BAD_INDEX);
          ok[j] = false;
        }
      }
      const A* row = reinterpret_cast<const A*>(p.cache) + (ok[j] ? r : 0) * (p.Lp + p.Rp);
#pragma unroll
      for (int i = 0; i < NL; ++i) {
        if (ok[j] && i * 256 + lane * 8 < p.Lp) rl[j][i].load(row + i * 256 + lane * 8);
        else rl[j][i].zero();
      }
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        if (ok[j] && i * 64 + lane * 2 < p.Rp) rr[j][i].load(row + p.Lp + i * 64 + lane * 2);
        else rr[j][i].zero();
      }
    }
    float s[V];
#pragma unroll
    for (int j = 0; j < KB; ++j) {
      float kf[NL * 8];
#pragma unroll
      for (int i = 0; i < NL; ++i) rl[j][i].get(kf + i * 8);
#pragma unroll
      for (int g = 0; g < HG; ++g) {
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const float2 x = rr[j][i].get();
          v = fmaf(qr[g][2 * i], x.x, fmaf(qr[g][2 * i + 1], x.y, v));
        }
#pragma unroll
        for (int i = 0; i < NL * 8; ++i) v = fmaf(ql[g][i], kf[i], v);
        s[j * HG + g] = v;
      }
    }
    float sc = transpose_sum<V>(s);
    bool mine = false;
#pragma unroll
    for (int j = 0; j < KB; ++j)
      if (j == my_key) mine = ok[j];
    if (!mine) sc = -INFINITY;
    float mx = fmaxf(sc, __shfl_xor_sync(0xffffffffu, sc, 16));      // the keys of a batch lie along the two top bits of the lane
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
    const float mn = fmaxf(m, mx);
    const float w = mine ? exp_f32<FAST>(sc - mn) : 0.f;
    const bool moved = mn > m;
    const float corr = moved ? (m == -INFINITY ? 0.f : exp_f32<FAST>(m - mn)) : 1.f;
    m = mn;
    l = l * corr + w;
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int g = 0; g < HG; ++g) {
        const float cg = __shfl_sync(0xffffffffu, corr, g * GRP);
#pragma unroll
        for (int i = 0; i < NL * 8; ++i) acc[g][i] *= cg;
      }
    }
#pragma unroll
    for (int j = 0; j < KB; ++j) {
      float kf[NL * 8];
#pragma unroll
      for (int i = 0; i < NL; ++i) rl[j][i].get(kf + i * 8);
#pragma unroll
      for (int g = 0; g < HG; ++g) {
        const float wj = __shfl_sync(0xffffffffu, w, (j * HG + g) * GRP);
#pragma unroll
        for (int i = 0; i < NL * 8; ++i) acc[g][i] = fmaf(wj, kf[i], acc[g][i]);
      }
    }
  }
  l += __shfl_xor_sync(0xffffffffu, l, 16);
  l += __shfl_xor_sync(0xffffffffu, l, 8);
#pragma unroll
  for (int g = 0; g < HG; ++g) {
    if (lane == g * GRP) {
      sm_m[warp * HG + g] = m;
      sm_l[warp * HG + g] = l;
    }
    float* dst = sm_acc + ((long)warp * HG + g) * (NL * 256);
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      *reinterpret_cast<float4*>(dst + i * 256 + lane * 8) = make_float4(acc[g][i * 8], acc[g][i * 8 + 1], acc[g][i * 8 + 2], acc[g][i * 8 + 3]);
      *reinterpret_cast<float4*>(dst + i * 256 + lane * 8 + 4) = make_float4(acc[g][i * 8 + 4], acc[g][i * 8 + 5], acc[g][i * 8 + 6], acc[g][i * 8 + 7]);
    }
  }
  __syncthreads();
  for (int g = 0; g < HG; ++g) {
    float M = -INFINITY, wgt[WARPS], L = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) M = fmaxf(M, sm_m[w * HG + g]);
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      wgt[w] = sm_m[w * HG + g] == -INFINITY ? 0.f : exp_f32<FAST>(sm_m[w * HG + g] - M);
      L += wgt[w] * sm_l[w * HG + g];
    }
    float* out = p.scratch + (((long)t * p.H + hg * HG + g) * p.splits + split) * (p.Lp + 2);
    for (int c = threadIdx.x; c < p.Lp; c += blockDim.x) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) v = fmaf(wgt[w], sm_acc[((long)w * HG + g) * (NL * 256) + c], v);
      out[c] = v;
    }
    if (threadIdx.x == 0) {
      out[p.Lp] = M;
      out[p.Lp + 1] = L;
    }
  }
}

// ------------------------------------------------------------------------------------------------
constexpr int TILE_KEYS = 32, STAGES = 3;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool live) {
  const uint32_t dst = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gmem), "r"(live ? 16 : 0) : "memory");      // 0 bytes read: zero fill
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// bf16; grid (splits, ceil(H / 32), T). `sub` of the eight warps share four heads, each takes every sub-th batch of keys and writes partials of its
// own: split s leaves partials s * sub .. s * sub + sub - 1
template <int NL>
__global__ void __launch_bounds__(256) latent_batch_kernel(SplitParams p, int sub) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* ring = reinterpret_cast<bf16*>(smem_raw);                // [STAGES][TILE_KEYS][Lp + Rp]
  constexpr int HG = 4, V = KB * HG, GRP = 32 / V;
  grid_dep_launch();
  grid_dep_wait();
  const int split = blockIdx.x, t = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups = WARPS / sub, part = warp / groups, h0 = (blockIdx.y * WARPS + warp % groups) * HG;
  const int pos = p.pg.positions[t];
  if (pos < 0) return;
  int first, count;
  visible(pos, p.window, &first, &count);
  const int k_begin = split * p.kps;
  if (k_begin >= count) return;
  const int k_end = split == p.splits - 1 ? count : min(count, k_begin + p.kps);
  const int slot = p.pg.slots[t], row = p.Lp + p.Rp, chunks = row / 8, tiles = (k_end - k_begin + TILE_KEYS - 1) / TILE_KEYS;
  // copies: eight threads per key, each finds its key's page one tile ahead of the copy
  const int my_row = threadIdx.x >> 3, lane8 = threadIdx.x & 7;
  auto find = [&](int tile) -> long {
    const int k = k_begin + tile * TILE_KEYS + my_row;
    if (k >= k_end) return -1;
    const long r = page_row(p.pg, slot, first + k);
    if (r < 0 && lane8 == 0 && p.pg.status) atomicOr(p.pg.status, IFAB_STATUS_BAD_INDEX);
    return r;
  };
  auto copy = [&](int tile, long r) {
    bf16* dst = ring + ((long)(tile % STAGES) * TILE_KEYS + my_row) * row;
    const bf16* src = reinterpret_cast<const bf16*>(p.cache) + (r < 0 ? 0 : r) * row;
    for (int c = lane8; c < chunks; c += 8) cp_async16(dst + c * 8, src + c * 8, r >= 0);
  };
  long next = find(0);
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) {
    if (i < tiles) copy(i, next);
    cp_async_commit();
    next = find(i + 1);
  }
  float ql[HG][NL * 8], qr[HG][2], acc[HG][NL * 8];
#pragma unroll
  for (int g = 0; g < HG; ++g) {
    const bool live = h0 + g < p.H;
    const float* a = p.q_lat + ((long)t * p.H + h0 + g) * p.Lp;
    const bf16* b = reinterpret_cast<const bf16*>(p.q_rot) + (long)t * p.ldq + (long)(h0 + g) * p.head_stride;
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      const int c = i * 256 + lane * 8;
      float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (live && c < p.Lp) load8(a + c, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        ql[g][i * 8 + j] = f[j] * p.scale;
        acc[g][i * 8 + j] = 0.f;
      }
    }
    const int c = lane * 2;
    qr[g][0] = live && c < p.Rp ? __bfloat162float(b[c]) * p.scale : 0.f;
    qr[g][1] = live && c < p.Rp ? __bfloat162float(b[c + 1]) * p.scale : 0.f;
  }
  const int my_key = (lane / GRP) / HG;
  float m = -INFINITY, l = 0.f;
  for (int tile = 0; tile < tiles; ++tile) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();                             // the tile has landed for every thread, and nobody still reads the stage refilled below
    if (tile + STAGES - 1 < tiles) copy(tile + STAGES - 1, next);
    cp_async_commit();
    next = find(tile + STAGES);
    const bf16* keys = ring + (long)(tile % STAGES) * TILE_KEYS * row;
    const int live_keys = min(TILE_KEYS, k_end - k_begin - tile * TILE_KEYS);
    for (int k0 = part * KB; k0 < live_keys; k0 += KB * sub) {
      Raw8<bf16> rl[KB][NL];
      float s[V];
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        const bf16* kr = keys + (long)(k0 + j) * row;
        float2 x = make_float2(0.f, 0.f);
        if (lane * 2 < p.Rp) x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(kr + p.Lp + lane * 2));
        float kf[NL * 8];
#pragma unroll
        for (int i = 0; i < NL; ++i) {
          if (i * 256 + lane * 8 < p.Lp) rl[j][i].load(kr + i * 256 + lane * 8);
          else rl[j][i].zero();
          rl[j][i].get(kf + i * 8);
        }
#pragma unroll
        for (int g = 0; g < HG; ++g) {
          float v0 = qr[g][0] * x.x, v1 = qr[g][1] * x.y;
#pragma unroll
          for (int i = 0; i < NL * 8; i += 2) {
            v0 = fmaf(ql[g][i], kf[i], v0);
            v1 = fmaf(ql[g][i + 1], kf[i + 1], v1);
          }
          s[j * HG + g] = v0 + v1;
        }
      }
      float sc = transpose_sum<V>(s);
      if (k0 + my_key >= live_keys) sc = -INFINITY;
      float mx = fmaxf(sc, __shfl_xor_sync(0xffffffffu, sc, 16));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
      const bool moved = mx > m;
      const float mn = moved ? mx : m;
      const float w = sc == -INFINITY ? 0.f : __expf(sc - mn), corr = moved ? (m == -INFINITY ? 0.f : __expf(m - mn)) : 1.f;
      m = mn;
      l = l * corr + w;
      if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
        for (int g = 0; g < HG; ++g) {
          const float cg = __shfl_sync(0xffffffffu, corr, g * GRP);
#pragma unroll
          for (int i = 0; i < NL * 8; ++i) acc[g][i] *= cg;
        }
      }
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        float kf[NL * 8];
#pragma unroll
        for (int i = 0; i < NL; ++i) rl[j][i].get(kf + i * 8);
#pragma unroll
        for (int g = 0; g < HG; ++g) {
          const float wj = __shfl_sync(0xffffffffu, w, (j * HG + g) * GRP);
#pragma unroll
          for (int i = 0; i < NL * 8; ++i) acc[g][i] = fmaf(wj, kf[i], acc[g][i]);
        }
      }
    }
  }
  cp_async_wait<0>();
  l += __shfl_xor_sync(0xffffffffu, l, 16);
  l += __shfl_xor_sync(0xffffffffu, l, 8);
#pragma unroll
  for (int g = 0; g < HG; ++g) {
    const float mg = __shfl_sync(0xffffffffu, m, g * GRP), lg = __shfl_sync(0xffffffffu, l, g * GRP);
    if (h0 + g >= p.H) continue;
    float* out = p.scratch + ((((long)t * p.H + h0 + g) * p.splits + split) * sub + part) * (p.Lp + 2);
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      const int c = i * 256 + lane * 8;
      if (c < p.Lp) {
#pragma unroll
        for (int j = 0; j < 8; j += 2) *reinterpret_cast<float2*>(out + c + j) = make_float2(acc[g][i * 8 + j], acc[g][i * 8 + j + 1]);      // rows of Lp + 2 floats
      }
    }
    if (lane == 0) {
      out[p.Lp] = mg;
      out[p.Lp + 1] = lg;
    }
  }
}

// ------------------------------------------------------------------------------------------------
struct MergeParams {
  const float* scratch; const int32_t* positions;
  int window, kps, splits, sub, H, Lp;       // sub: partials per split
  const void* gate; long ldg;                // [T, H]: head h of row t is multiplied by sigmoid(gate); or null
};

// weights of the splits of (row t, head h) into wgt[0 .. n); returns n. All threads; ends with a barrier
template <bool FAST>
__device__ __forceinline__ int merge_weights(const MergeParams& p, int t, int h, int pos, float gate, float* wgt, const float** base) {
  int first, count;
  visible(pos, p.window, &first, &count);
  const int n = min(p.splits, (count + p.kps - 1) / p.kps) * p.sub;
  *base = p.scratch + ((long)t * p.H + h) * p.splits * p.sub * (p.Lp + 2);
  if (threadIdx.x < 32) {                    // at most 64 partials: two per lane
    const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
    const float m0 = s0 < n ? (*base)[(long)s0 * (p.Lp + 2) + p.Lp] : -INFINITY, m1 = s1 < n ? (*base)[(long)s1 * (p.Lp + 2) + p.Lp] : -INFINITY;
    const float l0 = s0 < n ? (*base)[(long)s0 * (p.Lp + 2) + p.Lp + 1] : 0.f, l1 = s1 < n ? (*base)[(long)s1 * (p.Lp + 2) + p.Lp + 1] : 0.f;
    const float M = warp_max(fmaxf(m0, m1));
    const float w0 = m0 == -INFINITY ? 0.f : exp_f32<FAST>(m0 - M), w1 = m1 == -INFINITY ? 0.f : exp_f32<FAST>(m1 - M);
    const float L = warp_sum(w0 * l0 + w1 * l1);
    const float f = L > 0.f ? gate / L : 0.f;
    wgt[s0] = w0 * f;
    wgt[s1] = w1 * f;
  }
  __syncthreads();
  return n;
}

template <typename A>
__device__ __forceinline__ float head_gate(const MergeParams& p, int t, int h) {
  return p.gate ? sigmoid_f32<sizeof(A) == 2>(to_f32(reinterpret_cast<const A*>(p.gate)[(long)t * p.ldg + h])) : 1.f;
}

template <typename A>
__global__ void __launch_bounds__(128) latent_merge_kernel(MergeParams p, A* o_lat, long ldo) {
  __shared__ float wgt[64];
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, t = blockIdx.y, pos = p.positions[t];
  A* dst = o_lat + (long)t * ldo + (long)h * p.Lp;
  if (pos < 0) {
    for (int c = threadIdx.x; c < p.Lp; c += blockDim.x) dst[c] = from_f32<A>(0.f);
    return;
  }
  const float* base;
  const int n = merge_weights<sizeof(A) == 2>(p, t, h, pos, head_gate<A>(p, t, h), wgt, &base);
  for (int c = threadIdx.x; c < p.Lp; c += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < n; ++s) v = fmaf(wgt[s], base[(long)s * (p.Lp + 2) + c], v);
    dst[c] = from_f32<A>(v);
  }
}

// grid (H, T, ceil(vdim / 64)): every CTA merges the head's splits and takes 64 value rows (8 per warp)
__global__ void __launch_bounds__(256) latent_merge_vup_kernel(MergeParams p, const bf16* w_uv, int vdim, bf16* out, long ldo) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* os = reinterpret_cast<bf16*>(smem_raw);
  __shared__ float wgt[64];
  grid_dep_launch();
  const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, j0 = blockIdx.z * 64 + warp * 8;
  const bf16* rows[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) rows[r] = j0 + r < vdim ? w_uv + ((long)h * vdim + j0 + r) * p.Lp : nullptr;
  RowBatch<8> pf;
  prefetch_rows<8>(rows, p.Lp, pf);
  grid_dep_wait();
  const int pos = p.positions[t];
  if (pos < 0) return;
  const float* base;
  const int n = merge_weights<true>(p, t, h, pos, head_gate<bf16>(p, t, h), wgt, &base);
  for (int c = threadIdx.x; c < p.Lp; c += blockDim.x) {
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < n; ++s) v = fmaf(wgt[s], base[(long)s * (p.Lp + 2) + c], v);
    os[c] = __float2bfloat16_rn(v);
  }
  __syncthreads();
  float acc[8][1];
#pragma unroll
  for (int r = 0; r < 8; ++r) acc[r][0] = 0.f;
  warp_rows_dot<1, 8>(rows, os, p.Lp, acc, pf);
  warp_reduce_acc<1, 8>(acc);
  if (lane == 0) {
#pragma unroll
    for (int r = 0; r < 8; ++r)
      if (j0 + r < vdim) out[(long)t * ldo + (long)h * vdim + j0 + r] = __float2bfloat16_rn(acc[r][0]);
  }
}

// rows first .. first + n - 1 of one sequence: lat [rows, Lp] and rot [rows, tile] (columns from Rp on zero); rows from n on zero. One warp
// per row, 16 bytes per lane and step
__global__ void __launch_bounds__(256) latent_gather_kernel(const bf16* cache, Pages pg, int slot, int first, int n, int rows, int Lp, int Rp, int tile,
                                                            bf16* lat, bf16* rot) {
  grid_dep_launch();
  grid_dep_wait();
  const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= rows) return;
  long r = -1;
  if (i < n) {
    r = page_row(pg, slot, first + i);
    if (r < 0 && lane == 0 && pg.status) atomicOr(pg.status, IFAB_STATUS_BAD_INDEX);
  }
  const bf16* src = cache + (r < 0 ? 0 : r) * (Lp + Rp);
  for (int c = lane * 8; c < Lp + tile; c += 256) {
    const bool is_rot = c >= Lp;
    const uint4 v = r >= 0 && c < Lp + Rp ? *reinterpret_cast<const uint4*>(src + c) : make_uint4(0, 0, 0, 0);
    if (is_rot) *reinterpret_cast<uint4*>(rot + (long)i * tile + c - Lp) = v;
    else *reinterpret_cast<uint4*>(lat + (long)i * Lp + c) = v;
  }
}

template <typename A, int NL, int NR, int HG>
int launch_split(const SplitParams& p, cudaStream_t s) {
  const size_t smem = (size_t)(WARPS * HG * NL * 256 + 2 * WARPS * HG) * sizeof(float);
  auto k = latent_split_kernel<A, NL, NR, HG>;
  if (int rc = opt_in_smem(k, smem)) return rc;
  return launch_chain(k, dim3(p.splits, p.H / HG, p.T), dim3(256), smem, s, p);
}
template <typename A, int NL, int NR>
int split_heads(const SplitParams& p, cudaStream_t s) {
  constexpr int MOST = sizeof(A) == 2 ? (NL * NR <= 2 ? 4 : NL <= 2 ? 2 : 1) : (NL == 1 ? 2 : 1);
  if (MOST >= 4 && p.H % 4 == 0) return launch_split<A, NL, NR, MOST>(p, s);
  if (MOST >= 2 && p.H % 2 == 0) return launch_split<A, NL, NR, MOST >= 2 ? 2 : 1>(p, s);
  return launch_split<A, NL, NR, 1>(p, s);
}
template <typename A>
int split_sizes(const SplitParams& p, cudaStream_t s) {
  const bool wide = p.Rp > 64;               // one or four 64-column pieces of the rotated part
  if (p.Lp <= 256) return wide ? split_heads<A, 1, 4>(p, s) : split_heads<A, 1, 1>(p, s);
  if (p.Lp <= 512) return wide ? split_heads<A, 2, 4>(p, s) : split_heads<A, 2, 1>(p, s);
  return wide ? split_heads<A, 4, 4>(p, s) : split_heads<A, 4, 1>(p, s);
}

template <int NL>
int launch_batch(const SplitParams& p, int sub, cudaStream_t s) {
  const size_t smem = (size_t)STAGES * TILE_KEYS * (p.Lp + p.Rp) * sizeof(bf16);
  auto k = latent_batch_kernel<NL>;
  if (int rc = opt_in_smem(k, smem)) return rc;
  return launch_chain(k, dim3(p.splits, (p.H + 31) / 32, p.T), dim3(256), smem, s, p, sub);
}

bool bad_geometry(int Lp, int Rp) { return Lp < 8 || Lp > 1024 || Lp % 8 || Rp < 0 || Rp > 256 || Rp % 8; }

}  // namespace

extern "C" int ifab_latent_prepare(const void* proj, long ldp, int f32, int q_off, int q_rank, int kv_off, int kv_rank, int rot_dim, const float* q_gain,
                                   const float* kv_gain, float eps, const void* rope, int rot, const int32_t* positions, const int32_t* slots,
                                   const int32_t* page_table, int max_pages, int page_tokens, int num_pages, void* cq, long ldc, void* cache, int Lp, int Rp,
                                   int T, uint32_t* status, void* stream) {
  if (T < 1 || kv_rank < 1 || kv_rank > Lp || rot_dim < 0 || rot_dim > Rp || rot < 0 || rot % 2 || rot > rot_dim || (rot && !rope) || bad_geometry(Lp, Rp) ||
      (cq && q_rank < 1))
    return -1;
  PrepareParams p{proj, ldp, q_off, q_rank, kv_off, kv_rank, rot_dim, q_gain, kv_gain, eps, (const float2*)rope, rot,
                  {positions, slots, page_table, max_pages, page_tokens, num_pages, status}, cq, ldc, cache, Lp, Rp};
  return f32 ? launch_chain(latent_prepare_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, p)
             : launch_chain(latent_prepare_kernel<bf16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, p);
}

// decode rows (T <= 8), bf16: q [T, N] = rms(query latent) w_uq^T and the pages of the rows; w_uq [N, q_rank], q_rank % 8 == 0, bf16 gain
extern "C" int ifab_latent_query(const void* proj, long ldp, int q_off, int q_rank, int kv_off, int kv_rank, int rot_dim, const void* q_gain, const float* kv_gain,
                                 float eps, const void* rope, int rot, const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                                 int page_tokens, int num_pages, void* cache, int Lp, int Rp, const void* w_uq, int N, void* q, long ldq, int T, uint32_t* status,
                                 void* stream) {
  if (T < 1 || T > 8 || N < 1 || q_rank < 8 || q_rank % 8 || q_off % 8 || ldp % 8 || kv_rank < 1 || kv_rank > Lp || rot_dim < 0 || rot_dim > Rp || rot < 0 ||
      rot % 2 || rot > rot_dim || (rot && !rope) || bad_geometry(Lp, Rp))
    return -1;
  PrepareParams p{proj, ldp, q_off, q_rank, kv_off, kv_rank, rot_dim, nullptr, kv_gain, eps, (const float2*)rope, rot,
                  {positions, slots, page_table, max_pages, page_tokens, num_pages, status}, nullptr, 0, cache, Lp, Rp};
  cudaStream_t s = (cudaStream_t)stream;
  const bf16 *w = (const bf16*)w_uq, *g = (const bf16*)q_gain;
  if (T <= 1) return query_rows<1>(p, w, g, N, (bf16*)q, ldq, T, s);
  if (T <= 2) return query_rows<2>(p, w, g, N, (bf16*)q, ldq, T, s);
  if (T <= 4) return query_rows<4>(p, w, g, N, (bf16*)q, ldq, T, s);
  return query_rows<8>(p, w, g, N, (bf16*)q, ldq, T, s);
}

extern "C" int ifab_rotate_heads(void* q, long ldq, int f32, int head_stride, int off, int H, int rot, const void* rope, int T, void* stream) {
  if (T < 1 || H < 1 || rot < 2 || rot % 2 || off + rot > head_stride || !rope) return -1;
  return f32 ? launch_chain(rotate_heads_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, (float*)q, ldq, head_stride, off, H, rot, (const float2*)rope)
             : launch_chain(rotate_heads_kernel<bf16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, (bf16*)q, ldq, head_stride, off, H, rot, (const float2*)rope);
}

extern "C" int ifab_latent_absorb(void* q, long ldq, int head_stride, int rot_off, const void* w_uk, const void* rope, int rot, float* q_lat, int T, int H, int d,
                                  int Lp, void* stream) {
  if (T < 1 || T > 65535 || H < 1 || d < 1 || rot < 0 || rot % 2 || (rot && !rope) || bad_geometry(Lp, 0)) return -1;
  return launch_chain(latent_absorb_kernel, dim3(H, T, (Lp + 127) / 128), dim3(256), 0, (cudaStream_t)stream, (bf16*)q, ldq, head_stride, rot_off, (const bf16*)w_uk,
                      (const float2*)rope, rot, q_lat, H, d, Lp);
}

extern "C" int ifab_latent_split(const float* q_lat, const void* q_rot, long ldq, int head_stride, const void* cache, int f32, int Lp, int Rp,
                                 const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, int num_pages,
                                 int window, float scale, int T, int H, int kps, int splits, float* scratch, uint64_t scratch_bytes, uint32_t* status,
                                 void* stream) {
  if (T < 1 || T > 65535 || H < 1 || window < 0 || kps < 1 || splits < 1 || splits > 64 || bad_geometry(Lp, Rp)) return -1;
  if ((uint64_t)T * H * splits * (Lp + 2) * sizeof(float) > scratch_bytes) return -5;
  SplitParams p{q_lat, q_rot, ldq, head_stride, cache, Lp, Rp, {positions, slots, page_table, max_pages, page_tokens, num_pages, status}, window, scale, T, H,
                kps, splits, scratch};
  return f32 ? split_sizes<float>(p, (cudaStream_t)stream) : split_sizes<bf16>(p, (cudaStream_t)stream);
}

// the same with bf16 pages, Lp <= 512, Rp <= 64, for launches of many rows: `sub` (1, 2, 4 or 8, 32 heads / sub or fewer in all when above 1) warps per
// four heads, splits * sub partials
extern "C" int ifab_latent_batch(const float* q_lat, const void* q_rot, long ldq, int head_stride, const void* cache, int Lp, int Rp, const int32_t* positions,
                                 const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, int num_pages, int window, float scale, int T,
                                 int H, int kps, int splits, int sub, float* scratch, uint64_t scratch_bytes, uint32_t* status, void* stream) {
  if (T < 1 || T > 65535 || H < 1 || window < 0 || kps < 1 || splits < 1 || bad_geometry(Lp, Rp) || Lp > 512 || Rp > 64) return -1;
  if ((sub != 1 && sub != 2 && sub != 4 && sub != 8) || (sub > 1 && H * sub > 32) || splits * sub > 64) return -1;
  if ((uint64_t)T * H * splits * sub * (Lp + 2) * sizeof(float) > scratch_bytes) return -5;
  SplitParams p{q_lat, q_rot, ldq, head_stride, cache, Lp, Rp, {positions, slots, page_table, max_pages, page_tokens, num_pages, status}, window, scale, T, H,
                kps, splits, scratch};
  return Lp <= 256 ? launch_batch<1>(p, sub, (cudaStream_t)stream) : launch_batch<2>(p, sub, (cudaStream_t)stream);
}

extern "C" int ifab_latent_merge(const float* scratch, const int32_t* positions, int window, int kps, int splits, int sub, const void* gate, long ldg, int f32, int T,
                                 int H, int Lp, void* o_lat, long ldo, void* stream) {
  if (T < 1 || T > 65535 || H < 1 || window < 0 || kps < 1 || splits < 1 || sub < 1 || splits * sub > 64 || bad_geometry(Lp, 0)) return -1;
  MergeParams p{scratch, positions, window, kps, splits, sub, H, Lp, gate, ldg};
  return f32 ? launch_chain(latent_merge_kernel<float>, dim3(H, T), dim3(128), 0, (cudaStream_t)stream, p, (float*)o_lat, ldo)
             : launch_chain(latent_merge_kernel<bf16>, dim3(H, T), dim3(128), 0, (cudaStream_t)stream, p, (bf16*)o_lat, ldo);
}

extern "C" int ifab_latent_merge_vup(const float* scratch, const int32_t* positions, int window, int kps, int splits, const void* gate, long ldg, int T, int H,
                                     int Lp, const void* w_uv, int vdim, void* out, long ldo, void* stream) {
  if (T < 1 || T > 65535 || H < 1 || window < 0 || kps < 1 || splits < 1 || splits > 64 || vdim < 1 || bad_geometry(Lp, 0)) return -1;
  MergeParams p{scratch, positions, window, kps, splits, 1, H, Lp, gate, ldg};
  return launch_chain(latent_merge_vup_kernel, dim3(H, T, (vdim + 63) / 64), dim3(256), (size_t)Lp * sizeof(bf16), (cudaStream_t)stream, p, (const bf16*)w_uv, vdim,
                      (bf16*)out, ldo);
}

extern "C" int ifab_latent_gather(const void* cache, const int32_t* page_table, int slot, int max_pages, int page_tokens, int num_pages, int first, int n,
                                  int rows, int Lp, int Rp, int tile, void* lat, void* rot, uint32_t* status, void* stream) {
  if (n < 1 || rows < n || slot < 0 || first < 0 || tile < Rp || tile % 8 || bad_geometry(Lp, Rp)) return -1;
  Pages pg{nullptr, nullptr, page_table, max_pages, page_tokens, num_pages, status};
  return launch_chain(latent_gather_kernel, dim3((rows + 7) / 8), dim3(256), 0, (cudaStream_t)stream, (const bf16*)cache, pg, slot, first, n, rows, Lp, Rp, tile,
                      (bf16*)lat, (bf16*)rot);
}
