// Decode-time linears (1..8 rows per tile) of decoders with an f32 residual stream and norms on sublayer outputs. The weight stream
// is the one of gemv.cuh (prefetched ahead of the wait on the producer); the prologue finishes the previous sublayer, so a layer
// needs no row kernels of its own between its linears:
//
//   post norm    x_out = x_in + rms(y) * w, operand bf16(x_out). Every CTA computes the rows it needs (a few KB from L2); the CTAs
//                of the first column write x_out, which must not be x_in (other CTAs still read that). With a second gain (a norm
//                ahead of the next sublayer as well) the operand is bf16(rms(x_out) * w2), also stored to xn on request. Without the
//                first gain y is added as it is; rows of `extra` join the update
//   group norm   operand bf16((o / rms of each group of columns [* gain]) * act(gate)): normalised, gated heads of a recurrent mixer
//   plain        bf16 rows
//
// parallel_in_kernel is the front of a layer whose sublayers read one norm: the mixer's projection (with bias), the gated unit of a
// feed-forward every row takes, and a router with its selection, as one launch behind one prologue.
//
// Epilogue: optional bias, f32 rows added to the result, activation, bf16 or f32 result. A router's linear goes on to the selection: the last CTA to finish turns the f32
// logits into expert ids and weights (moe_select.cuh) and the extra column, when there is one, into the shared expert's weight.
#include "gemv.cuh"
#include "moe_select.cuh"
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

enum { PLAIN = 0, POST = 1, GROUP = 2 };

struct Params {
  const bf16* x; long ldx;                                           // PLAIN
  const float *y, *norm_w, *x_in; float* x_out; long ldy, ldr;       // POST (ldr: x_in and x_out)
  const float *o, *gain; const bf16* gate; long ldo, ldg; int groups, gate_act;      // GROUP
  float eps;
  const bf16* w;
  void* z; long ldz; int out_f32, act;
  int T, N, K;
  const float* norm2_w; bf16* xn; long ldn;                          // POST: second norm
  uint32_t* ticket; const float* bias; int E, topk, scoring, renorm; float scale; int32_t* ids; float *wts, *shared_w;      // router: ticket set
  const float* extra; long lde;                                      // POST: rows added to x as well, or null
  const float *out_bias, *addend; long ldadd;                        // [N] and rows added to the result (addend may be the f32 result itself)
  int groups_of_experts, keep;                                       // router
};

// stage T rows of the operand; ends with __syncthreads(). `inv`: T * max(groups, 1) floats
template <int T, int PRO>
__device__ __forceinline__ void stage_operand(const Params& p, bf16* xs, float* inv, float* red, float* xf, int t0) {
  const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, nwarp = nthr >> 5, K = p.K;
  if (PRO == PLAIN) {
    for (int t = 0; t < T; ++t) {
      const bool live = t0 + t < p.T;
      for (int c = tid * 8; c < K; c += nthr * 8)
        *reinterpret_cast<uint4*>(xs + t * K + c) = live ? *reinterpret_cast<const uint4*>(p.x + (long)(t0 + t) * p.ldx + c) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    return;
  }
  const int groups = PRO == GROUP ? p.groups : 1, n = K / groups;
  const float* src = PRO == GROUP ? p.o : p.y;
  const long lds = PRO == GROUP ? p.ldo : p.ldy;
  if (PRO == POST && !p.norm_w) {
    // nothing to divide by
  } else if (groups == 1) {
    for (int t = 0; t < T; ++t) {
      float ss = 0.f;
      if (t0 + t < p.T)
        for (int c = tid * 4; c < K; c += nthr * 4) {
          const float4 v = *reinterpret_cast<const float4*>(src + (long)(t0 + t) * lds + c);
          ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
      ss = warp_sum(ss);
      if (lane == 0) red[t * 8 + warp] = ss;
    }
    __syncthreads();
    if (tid < T) {
      float s = 0.f;
      for (int i = 0; i < nwarp; ++i) s += red[tid * 8 + i];
      inv[tid] = 1.f / sqrtf(s / (float)K + p.eps);
    }
  } else {
    for (int i = warp; i < T * groups; i += nwarp) {
      const int t = i / groups, g = i - t * groups;
      float ss = 0.f;
      if (t0 + t < p.T)
        for (int c = lane; c < n; c += 32) {
          const float v = src[(long)(t0 + t) * lds + (long)g * n + c];
          ss += v * v;
        }
      ss = warp_sum(ss);
      if (lane == 0) inv[i] = 1.f / sqrtf(ss / (float)n + p.eps);
    }
  }
  __syncthreads();
  const bool twice = PRO == POST && p.norm2_w;
  for (int t = 0; t < T; ++t) {
    const long r = t0 + t;
    const bool live = r < p.T;
    float ss = 0.f;
    for (int c = tid * 4; c < K; c += nthr * 4) {
      float f[4] = {0.f, 0.f, 0.f, 0.f};
      if (live) {
        const float4 v = PRO == POST && !src ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(src + r * lds + c);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
        if (PRO == POST) {
          const float4 x = *reinterpret_cast<const float4*>(p.x_in + r * p.ldr + c);
          if (p.norm_w) {
            const float iv = inv[t];
            const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c);
            f[0] = x.x + f[0] * iv * w.x;
            f[1] = x.y + f[1] * iv * w.y;
            f[2] = x.z + f[2] * iv * w.z;
            f[3] = x.w + f[3] * iv * w.w;
          } else {
            f[0] += x.x;
            f[1] += x.y;
            f[2] += x.z;
            f[3] += x.w;
          }
          if (p.extra) {
            const float4 e = *reinterpret_cast<const float4*>(p.extra + r * p.lde + c);
            f[0] += e.x;
            f[1] += e.y;
            f[2] += e.z;
            f[3] += e.w;
          }
          if (blockIdx.x == 0) *reinterpret_cast<float4*>(p.x_out + r * p.ldr + c) = make_float4(f[0], f[1], f[2], f[3]);
          ss += f[0] * f[0] + f[1] * f[1] + f[2] * f[2] + f[3] * f[3];
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            f[i] *= inv[t * groups + (c + i) / n];
            if (p.gain) f[i] *= p.gain[c + i];
            f[i] *= activate<true>(__bfloat162float(p.gate[r * p.ldg + c + i]), p.gate_act);
          }
        }
      }
      if (twice) {
        *reinterpret_cast<float4*>(xf + t * K + c) = make_float4(f[0], f[1], f[2], f[3]);
        continue;
      }
      __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
      *reinterpret_cast<uint2*>(xs + t * K + c) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    }
    if (twice) {
      ss = warp_sum(ss);
      if (lane == 0) red[t * 8 + warp] = ss;
    }
  }
  __syncthreads();
  if (!twice) return;
  for (int t = 0; t < T; ++t) {
    float s = 0.f;
    for (int i = 0; i < nwarp; ++i) s += red[t * 8 + i];
    const float iv = 1.f / sqrtf(s / (float)K + p.eps);
    for (int c = tid * 4; c < K; c += nthr * 4) {
      const float4 v = *reinterpret_cast<const float4*>(xf + t * K + c), w = *reinterpret_cast<const float4*>(p.norm2_w + c);
      __nv_bfloat162 a = __floats2bfloat162_rn(v.x * iv * w.x, v.y * iv * w.y), b = __floats2bfloat162_rn(v.z * iv * w.z, v.w * iv * w.w);
      const uint2 u = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
      *reinterpret_cast<uint2*>(xs + t * K + c) = u;
      if (p.xn && blockIdx.x == 0 && t0 + t < p.T) *reinterpret_cast<uint2*>(p.xn + (long)(t0 + t) * p.ldn + c) = u;
    }
  }
  __syncthreads();
}

template <int T, int R, int PRO>
__global__ void __launch_bounds__(256) gemv_operand_kernel(Params p) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* xs = reinterpret_cast<bf16*>(smem_raw);
  float* inv = reinterpret_cast<float*>(xs + (long)T * p.K);
  float* xf = inv + 8;                          // POST with a second norm: the updated rows (T <= 8 and K % 8 keep it 16-byte aligned)
  __shared__ float red[T * 8];
  grid_dep_launch();
  const int t0 = blockIdx.y * T, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = (blockIdx.x * 8 + warp) * R;
  const bf16* rows[R];
#pragma unroll
  for (int r = 0; r < R; ++r) rows[r] = (n0 + r < p.N) ? p.w + (long)(n0 + r) * p.K : nullptr;
  RowBatch<R> pf;
  prefetch_rows<R>(rows, p.K, pf);
  grid_dep_wait();
  stage_operand<T, PRO>(p, xs, inv, red, xf, t0);
  const bool router = PRO == POST && p.ticket;
  if (n0 >= p.N && !router) return;
  float acc[R][T];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int t = 0; t < T; ++t) acc[r][t] = 0.f;
  warp_rows_dot<T, R>(rows, xs, p.K, acc, pf);
  warp_reduce_acc<T, R>(acc);
  if (lane == 0) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (n0 + r >= p.N) continue;
#pragma unroll
      for (int t = 0; t < T; ++t) {
        if (t0 + t >= p.T) continue;
        float v = acc[r][t];
        if (p.out_bias) v += p.out_bias[n0 + r];
        if (p.addend) v += p.addend[(long)(t0 + t) * p.ldadd + n0 + r];
        v = activate<true>(v, p.act);
        if (p.out_f32) reinterpret_cast<float*>(p.z)[(long)(t0 + t) * p.ldz + n0 + r] = v;
        else reinterpret_cast<bf16*>(p.z)[(long)(t0 + t) * p.ldz + n0 + r] = __float2bfloat16_rn(v);
      }
    }
  }
  if (!router) return;
  __shared__ int is_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    is_last = atomicAdd(p.ticket, 1u) == gridDim.x - 1;
    if (is_last) *p.ticket = 0;
  }
  __syncthreads();
  if (!is_last || warp >= p.T) return;          // one row tile: warp t selects for row t
  __threadfence();
  const float* logits = reinterpret_cast<const float*>(p.z) + (long)warp * p.ldz;
  select_topk_row(logits, p.bias, p.E, p.topk, p.scoring, p.renorm, p.scale, p.ids + (long)warp * p.topk, p.wts + (long)warp * p.topk, p.groups_of_experts, p.keep);
  if (p.shared_w && lane == 0) p.shared_w[warp] = sigmoid_f32(__ldcg(logits + p.E));
}

// The front of a layer with parallel sublayers. CTAs 0 .. router_ctas - 1 hold the router's rows (f32 logits; the last of them selects), the
// others warps of R weight rows: the projection (`w`, N rows, bf16 result with out_bias), then R / 2 pairs of the gated unit (gate rows
// [0, F), up rows [F, 2 F) of w_gu).
struct ParallelParams {
  Params p;
  const bf16* w_gu; int F; GatedUnit unit; bf16* unit_out; long ldu;
  const bf16* w_router; float* logits; long ldl;
  int router_ctas;
};

template <int T, int R>
__global__ void __launch_bounds__(256) parallel_in_kernel(ParallelParams q) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const Params& p = q.p;
  bf16* xs = reinterpret_cast<bf16*>(smem_raw);
  float* inv = reinterpret_cast<float*>(xs + (long)T * p.K);
  float* xf = inv + 8;
  __shared__ float red[T * 8];
  grid_dep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool router = (int)blockIdx.x < q.router_ctas;
  const int task = router ? blockIdx.x * 8 + warp : ((int)blockIdx.x - q.router_ctas) * 8 + warp;
  const int n_proj = (p.N + R - 1) / R;
  const bool pairs = !router && task >= n_proj;
  const int n0 = pairs ? (task - n_proj) * (R / 2) : task * R;
  const int live = router ? p.E - n0 : pairs ? q.F - n0 : p.N - n0;      // rows (units) from n0 on
  const bf16* rows[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = pairs ? r % (R / 2) : r;
    const bf16* base = router ? q.w_router : pairs ? q.w_gu + (r < R / 2 ? 0L : (long)q.F * p.K) : p.w;
    rows[r] = i < live ? base + (long)(n0 + i) * p.K : nullptr;
  }
  RowBatch<R> pf;
  prefetch_rows<R>(rows, p.K, pf);
  grid_dep_wait();
  stage_operand<T, POST>(p, xs, inv, red, xf, 0);
  if (live > 0) {
    float acc[R][T];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int t = 0; t < T; ++t) acc[r][t] = 0.f;
    warp_rows_dot<T, R>(rows, xs, p.K, acc, pf);
    warp_reduce_acc<T, R>(acc);
    if (lane == 0) {
#pragma unroll
      for (int t = 0; t < T; ++t) {
        if (t >= p.T) continue;
        if (pairs) {
#pragma unroll
          for (int r = 0; r < R / 2; ++r)
            if (r < live) q.unit_out[(long)t * q.ldu + n0 + r] = __float2bfloat16_rn(gated_bf16(acc[r][t], acc[R / 2 + r][t], q.unit));
        } else {
#pragma unroll
          for (int r = 0; r < R; ++r) {
            if (r >= live) continue;
            if (router) q.logits[(long)t * q.ldl + n0 + r] = acc[r][t];
            else reinterpret_cast<bf16*>(p.z)[(long)t * p.ldz + n0 + r] = __float2bfloat16_rn(acc[r][t] + (p.out_bias ? p.out_bias[n0 + r] : 0.f));
          }
        }
      }
    }
  }
  if (!router) return;
  __shared__ int is_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    is_last = atomicAdd(p.ticket, 1u) == (uint32_t)q.router_ctas - 1;
    if (is_last) *p.ticket = 0;
  }
  __syncthreads();
  if (!is_last || warp >= p.T) return;
  __threadfence();
  select_topk_row(q.logits + (long)warp * q.ldl, p.bias, p.E, p.topk, p.scoring, p.renorm, p.scale, p.ids + (long)warp * p.topk, p.wts + (long)warp * p.topk,
                  p.groups_of_experts, p.keep);
}

template <int T, int R>
int launch_parallel(ParallelParams q, cudaStream_t s) {
  const size_t smem = (size_t)T * q.p.K * (sizeof(bf16) + sizeof(float)) + 8 * sizeof(float);
  auto k = parallel_in_kernel<T, R>;
  if (int rc = opt_in_smem(k, smem)) return rc;
  q.router_ctas = q.w_router ? (q.p.E + 8 * R - 1) / (8 * R) : 0;
  const int tasks = (q.p.N + R - 1) / R + (q.F + R / 2 - 1) / (R / 2);
  return launch_chain(k, dim3(q.router_ctas + (tasks + 7) / 8), dim3(256), smem, s, q);
}
template <int T>
int parallel_rows(const ParallelParams& q, cudaStream_t s) {
  return q.p.N + 2 * q.F >= 148 * 8 * 4 ? launch_parallel<T, 4>(q, s) : launch_parallel<T, 2>(q, s);
}

template <int T, int R, int PRO>
int launch_one(const Params& p, cudaStream_t s) {
  const size_t smem = (size_t)T * p.K * sizeof(bf16) + (PRO == GROUP ? (size_t)T * p.groups : 8) * sizeof(float) +
                      (PRO == POST && p.norm2_w ? (size_t)T * p.K * sizeof(float) : 0);
  auto k = gemv_operand_kernel<T, R, PRO>;
  if (int rc = opt_in_smem(k, smem)) return rc;
  return launch_chain(k, dim3((p.N + 8 * R - 1) / (8 * R), (p.T + T - 1) / T), dim3(256), smem, s, p);
}
template <int T, int PRO>
int by_rows(const Params& p, cudaStream_t s) {
  // rows per warp: the widest that still gives every SM a CTA (two are resident), so that the grid is one wave
  if (p.N >= 148 * 8 * 4) return launch_one<T, 4, PRO>(p, s);
  if (p.N >= 148 * 8 * 2) return launch_one<T, 2, PRO>(p, s);
  return launch_one<T, 1, PRO>(p, s);
}
template <int PRO>
int dispatch(const Params& p, cudaStream_t s) {
  if (p.T < 1 || p.N < 1 || p.K < 8 || p.K % 8) return -1;
  if (p.T <= 1) return by_rows<1, PRO>(p, s);
  if (p.T <= 2) return by_rows<2, PRO>(p, s);
  if (p.T <= 4) return by_rows<4, PRO>(p, s);
  return by_rows<8, PRO>(p, s);
}

}  // namespace

extern "C" int ifab_gemv_post_norm(const float* y, long ldy, const float* norm_w, const float* norm2_w, float eps, const float* x_in, float* x_out, long ldx,
                                   const void* w, void* z, long ldz, int out_f32, int act, int T, int N, int K, void* stream) {
  if (ldy % 4 || ldx % 4 || x_in == x_out) return -1;
  Params p{};
  p.norm2_w = norm2_w;
  p.y = y; p.ldy = ldy; p.norm_w = norm_w; p.eps = eps; p.x_in = x_in; p.x_out = x_out; p.ldr = ldx;
  p.w = (const bf16*)w; p.z = z; p.ldz = ldz; p.out_f32 = out_f32; p.act = act; p.T = T; p.N = N; p.K = K;
  return dispatch<POST>(p, (cudaStream_t)stream);
}
// The router of a sublayer pair: x_out as above, xn = bf16(rms(x_out) * norm2_w), f32 logits [T, N] = xn w^T (T <= 8), then ids / wts of the chosen
// of the first E columns and, when N = E + 1, shared_w = sigmoid(logits[:, E]). ticket: one zeroed word (left zero again)
extern "C" int ifab_router_post_norm(const float* y, long ldy, const float* norm_w, const float* norm2_w, float eps, const float* x_in, float* x_out, long ldx,
                                     void* xn, long ldn, const void* w, float* logits, long ldz, const float* bias, int E, int topk, int scoring, int renorm,
                                     float scale, int32_t* ids, float* wts, float* shared_w, uint32_t* ticket, int T, int N, int K, void* stream) {
  if (ldy % 4 || ldx % 4 || ldn % 4 || x_in == x_out || T > 8 || !ticket || !norm2_w || !select_ok(E, topk, scoring, 1, 1) || N < E || N > E + 1 ||
      (shared_w && N != E + 1))
    return -1;
  Params p{};
  p.groups_of_experts = p.keep = 1;
  p.y = y; p.ldy = ldy; p.norm_w = norm_w; p.norm2_w = norm2_w; p.eps = eps; p.x_in = x_in; p.x_out = x_out; p.ldr = ldx;
  p.xn = (bf16*)xn; p.ldn = ldn; p.ticket = ticket; p.bias = bias; p.E = E; p.topk = topk; p.scoring = scoring; p.renorm = renorm; p.scale = scale;
  p.ids = ids; p.wts = wts; p.shared_w = shared_w;
  p.w = (const bf16*)w; p.z = logits; p.ldz = ldz; p.out_f32 = 1; p.act = 0; p.T = T; p.N = N; p.K = K;
  return dispatch<POST>(p, (cudaStream_t)stream);
}
extern "C" int ifab_gemv_group_norm(const float* o, long ldo, const float* gain, float eps, int groups, const void* gate, long ldg, int gate_act,
                                    const void* w, void* z, long ldz, int out_f32, int act, int T, int N, int K, void* stream) {
  if (ldo % 4 || groups < 1 || groups > 1024 || K % groups) return -1;
  Params p{};
  p.o = o; p.ldo = ldo; p.gain = gain; p.eps = eps; p.groups = groups; p.gate = (const bf16*)gate; p.ldg = ldg; p.gate_act = gate_act;
  p.w = (const bf16*)w; p.z = z; p.ldz = ldz; p.out_f32 = out_f32; p.act = act; p.T = T; p.N = N; p.K = K;
  return dispatch<GROUP>(p, (cudaStream_t)stream);
}
// z = act(x w^T + bias + addend); bias [N] and addend (f32 rows, which may be z) or null
extern "C" int ifab_gemv_act(const void* x, long ldx, const void* w, const float* bias, const float* addend, long ldadd, void* z, long ldz, int out_f32, int act, int T,
                             int N, int K, void* stream) {
  if (ldx % 8) return -1;
  Params p{};
  p.out_bias = bias; p.addend = addend; p.ldadd = ldadd;
  p.x = (const bf16*)x; p.ldx = ldx;
  p.w = (const bf16*)w; p.z = z; p.ldz = ldz; p.out_f32 = out_f32; p.act = act; p.T = T; p.N = N; p.K = K;
  return dispatch<PLAIN>(p, (cudaStream_t)stream);
}

// The front of a layer with parallel sublayers for T <= 2 rows: x_out = x_in (+ y) (+ extra); h = bf16(rms(x_out) * norm_w), also stored to xn when given;
// z (bf16) = h w^T + bias; unit_out (bf16) = unit(h gate^T, h up^T) for w_gu = [gate | up] ([2 F, K]; F 0: none); with w_router, ids / wts of the experts
// that f32 logits h w_router^T choose (moe_select.cuh; ticket: one zeroed word, left zero again).
extern "C" int ifab_parallel_in_decode(const float* y, long ldy, const float* extra, long lde, const float* norm_w, float eps, const float* x_in, float* x_out,
                                       long ldx, void* xn, long ldn, const void* w, const float* bias, void* z, long ldz, int N, const void* w_gu, int F, int unit,
                                       float limit, float alpha, void* unit_out, long ldu, const void* w_router, float* logits, long ldl, const float* correction,
                                       int E, int topk, int scoring, int renorm, float scale, int groups, int keep, int32_t* ids, float* wts, uint32_t* ticket,
                                       int T, int K, void* stream) {
  ParallelParams q{};
  q.unit = {unit, limit, alpha};
  if (T < 1 || T > 2 || K < 8 || K % 8 || N < 1 || F < 0 || !norm_w || ldx % 4 || (y && ldy % 4) || (extra && lde % 4) || (xn && ldn % 4) || x_in == x_out ||
      (F && (!w_gu || !gated_ok(q.unit))) || (w_router && (!ticket || !select_ok(E, topk, scoring, groups, keep))))
    return -1;
  Params& p = q.p;
  p.y = y; p.ldy = ldy; p.extra = extra; p.lde = lde; p.norm2_w = norm_w; p.eps = eps; p.x_in = x_in; p.x_out = x_out; p.ldr = ldx;
  p.xn = (bf16*)xn; p.ldn = ldn;
  p.w = (const bf16*)w; p.out_bias = bias; p.z = z; p.ldz = ldz; p.N = N; p.T = T; p.K = K;
  q.w_gu = (const bf16*)w_gu; q.F = F; q.unit_out = (bf16*)unit_out; q.ldu = ldu;
  q.w_router = (const bf16*)w_router; q.logits = logits; q.ldl = ldl;
  p.bias = correction; p.E = w_router ? E : 0; p.topk = topk; p.scoring = scoring; p.renorm = renorm; p.scale = scale; p.groups_of_experts = groups; p.keep = keep;
  p.ids = ids; p.wts = wts; p.ticket = ticket;
  return T == 1 ? parallel_rows<1>(q, (cudaStream_t)stream) : parallel_rows<2>(q, (cudaStream_t)stream);
}
