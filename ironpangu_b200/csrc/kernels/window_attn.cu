// Softmax attention over a window or a chunk of paged keys / values with sinks, score caps, distance biases and output gates
// (attn_rule.cuh), for any head sizes (query / key size and value size independent), bf16 or f32 activations and caches.
//
//   qk_norm_rope_write_kernel  RMS norm per head of q and k with a shared gain, rotation of the first `rot` columns (either pair
//                              layout), q to its own rows, k and v into the pages of their sequence
//   qk_rows_norm_write_kernel  the same with the norm over all heads of q (and all of k) together, a gain per column
//   qk_chunks_write_kernel     that, or no norm at all, for bf16 heads of whole 16-byte chunks
//   window_attn_kernel         one CTA per (row, query head): scores, weights and sums in f32; the denominator also holds
//                              exp(sink_h). Optional output gate, a value per column or per head, and a factor on the result
//   pool_write_kernel          means of the keys and values of the blocks that end with a row of the step, out of the pages into the
//                              entries of AheadRule
//
// v may be the columns of k (v_off == k_off): the values are then the keys as projected.
//
// Positions, slots and page tables as in the other paged kernels; pages that fell out of every window may be gone (-1).
#include "attn_rule.cuh"
#include "rope.cuh"
#include "ifab_kernels.h"

using namespace ifab;

namespace {

// cs [T, pairs]: cos and sin of position * freq[i]
__global__ void __launch_bounds__(128) rope_table_kernel(const int32_t* positions, const double* freq, float2* cs, int T, int pairs) {
  grid_dep_launch();
  grid_dep_wait();
  const long i = (long)blockIdx.x * 128 + threadIdx.x;
  if (i >= (long)T * pairs) return;
  float2 v;
  rope_angle(positions[i / pairs], freq[i % pairs], &v.x, &v.y);
  cs[i] = v;
}

struct QkParams {
  const void* proj; long ldp; int q_off, k_off, v_off;
  const float *q_gain, *k_gain; float eps;           // gains may be null: no norm
  int H, G, d, e;
  RopeTable rope;
  const int32_t *positions, *slots, *page_table;
  int max_pages, page_tokens, num_pages;
  void* q_out; long ldq; int q_stride;      // columns from one query head to the next (>= d)
  void *k_cache, *v_cache;
  int T;
  uint32_t* status;
};

// grid (ceil((H + 2 G) / 4), T), 128 threads: one warp per head of a row
template <typename A>
__global__ void __launch_bounds__(128) qk_norm_rope_write_kernel(QkParams p) {
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.y, h = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H + 2 * p.G) return;
  const int pos = p.positions[t];
  if (pos < 0) return;
  const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
  long dst_row = -1;
  if (h >= p.H) {
    const int lp = pos / p.page_tokens;
    const int page = lp < p.max_pages ? p.page_table[(long)p.slots[t] * p.max_pages + lp] : -1;
    if (page < 0 || page >= p.num_pages) {
      if (lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_BAD_INDEX);
      return;
    }
    dst_row = (long)page * p.page_tokens + pos % p.page_tokens;
  }
  if (h >= p.H + p.G) {
    const int g = h - p.H - p.G;
    const A* src = row + p.v_off + (long)g * p.e;
    A* dst = reinterpret_cast<A*>(p.v_cache) + (dst_row * p.G + g) * p.e;
    for (int c = lane; c < p.e; c += 32) dst[c] = src[c];
    return;
  }
  const bool is_q = h < p.H;
  const A* src = is_q ? row + p.q_off + (long)h * p.d : row + p.k_off + (long)(h - p.H) * p.d;
  A* dst = is_q ? reinterpret_cast<A*>(p.q_out) + (long)t * p.ldq + (long)h * p.q_stride : reinterpret_cast<A*>(p.k_cache) + (dst_row * p.G + h - p.H) * p.d;
  const float* gain = is_q ? p.q_gain : p.k_gain;
  float inv = 1.f;
  if (gain) {
    float ss = 0.f;
    for (int c = lane; c < p.d; c += 32) {
      const float v = to_f32(src[c]);
      ss += v * v;
    }
    inv = 1.f / sqrtf(warp_sum(ss) / (float)p.d + p.eps);
  }
  const float2* cs = p.rope.cs + (long)t * (p.rope.rot / 2);
  for (int i = lane; i < p.rope.rot / 2; i += 32) {
    int ia, ib;
    rope_pair(i, p.rope.rot, p.rope.interleaved, &ia, &ib);
    const float2 r = cs[i];
    const float a = to_f32(src[ia]) * inv * (gain ? gain[ia] : 1.f), b = to_f32(src[ib]) * inv * (gain ? gain[ib] : 1.f);
    dst[ia] = from_f32<A>(a * r.x - b * r.y);
    dst[ib] = from_f32<A>(b * r.x + a * r.y);
  }
  for (int c = p.rope.rot + lane; c < p.d; c += 32) dst[c] = from_f32<A>(to_f32(src[c]) * inv * (gain ? gain[c] : 1.f));
}

// grid T, 256 threads: the two row sums first, then pairs of neighbouring columns
template <typename A>
__global__ void __launch_bounds__(256) qk_rows_norm_write_kernel(QkParams p) {
  __shared__ float red[2][8];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[t];
  if (pos < 0) return;
  const A* row = reinterpret_cast<const A*>(p.proj) + (long)t * p.ldp;
  const int lp = pos / p.page_tokens;
  const int page = lp < p.max_pages ? p.page_table[(long)p.slots[t] * p.max_pages + lp] : -1;
  if (page < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, IFAB_STATUS_BAD_INDEX);
    return;
  }
  const long dst_row = (long)page * p.page_tokens + pos % p.page_tokens;
  const int nq = p.H * p.d, nk = p.G * p.d, nv = p.G * p.e;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x; c < nq; c += 256) {
    const float v = to_f32(row[p.q_off + c]);
    sq += v * v;
  }
  for (int c = threadIdx.x; c < nk; c += 256) {
    const float v = to_f32(row[p.k_off + c]);
    sk += v * v;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) {
    red[0][warp] = sq;
    red[1][warp] = sk;
  }
  A* vd = reinterpret_cast<A*>(p.v_cache) + dst_row * nv;
  for (int c = threadIdx.x; c < nv; c += 256) vd[c] = row[p.v_off + c];
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    sq += red[0][i];
    sk += red[1][i];
  }
  const float iq = 1.f / sqrtf(sq / (float)nq + p.eps), ik = 1.f / sqrtf(sk / (float)nk + p.eps);
  const float2* cs = p.rope.cs + (long)t * (p.rope.rot / 2);
  const int half = p.rope.rot / 2, units = half + p.d - p.rope.rot;      // of a head: pairs, then single columns
  A* qd = reinterpret_cast<A*>(p.q_out) + (long)t * p.ldq;
  A* kd = reinterpret_cast<A*>(p.k_cache) + dst_row * nk;
  for (int i = threadIdx.x; i < (p.H + p.G) * units; i += 256) {
    const int h = i / units, u = i - h * units;
    const bool is_q = h < p.H;
    const int c0 = (is_q ? h : h - p.H) * p.d;                           // of the head among its projection's columns
    const A* src = row + (is_q ? p.q_off : p.k_off) + c0;
    const float* gain = (is_q ? p.q_gain : p.k_gain) + c0;
    A* dst = is_q ? qd + (long)h * p.q_stride : kd + c0;
    const float inv = is_q ? iq : ik;
    if (u < half) {
      int ia, ib;
      rope_pair(u, p.rope.rot, p.rope.interleaved, &ia, &ib);
      const float2 r = cs[u];
      const float a = to_f32(src[ia]) * inv * gain[ia], b = to_f32(src[ib]) * inv * gain[ib];
      dst[ia] = from_f32<A>(a * r.x - b * r.y);
      dst[ib] = from_f32<A>(b * r.x + a * r.y);
    } else {
      const int c = p.rope.rot + u - half;
      dst[c] = from_f32<A>(to_f32(src[c]) * inv * gain[c]);
    }
  }
}

// grid T, 256 threads: a thread keeps up to NV chunks of 8 columns (q, then k, then v) in registers between the row sums and the stores.
// NORM: gains of all columns of q and k
template <int NV, bool NORM>
__global__ void __launch_bounds__(256) qk_chunks_write_kernel(QkParams p) {
  __shared__ float red[2][8];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[t];
  if (pos < 0) return;
  const bf16* row = reinterpret_cast<const bf16*>(p.proj) + (long)t * p.ldp;
  const int lp = pos / p.page_tokens;
  const int page = lp < p.max_pages ? p.page_table[(long)p.slots[t] * p.max_pages + lp] : -1;
  if (page < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, IFAB_STATUS_BAD_INDEX);
    return;
  }
  const long dst_row = (long)page * p.page_tokens + pos % p.page_tokens;
  const int nq = p.H * p.d, nk = p.G * p.d, nv = p.G * p.e;
  const bool same = p.v_off == p.k_off;            // the values are the keys
  const int total = nq + nk + (same ? 0 : nv);
  uint4 raw[NV];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 8;
    raw[i] = make_uint4(0, 0, 0, 0);
    if (c < total) raw[i] = *reinterpret_cast<const uint4*>(row + (c < nq ? p.q_off + c : c < nq + nk ? p.k_off + c - nq : p.v_off + c - nq - nk));
    if (NORM && c < nq + nk) {
      float f[8], ss = 0.f;
      unpack8(raw[i], f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
      if (c < nq) sq += ss;
      else sk += ss;
    }
  }
  float iq = 1.f, ik = 1.f;
  if (NORM) {
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      red[0][warp] = sq;
      red[1][warp] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      sq += red[0][i];
      sk += red[1][i];
    }
    iq = 1.f / sqrtf(sq / (float)nq + p.eps);
    ik = 1.f / sqrtf(sk / (float)nk + p.eps);
  }
  const float2* cs = p.rope.cs + (long)t * (p.rope.rot / 2);
  bf16* vd = reinterpret_cast<bf16*>(p.v_cache) + dst_row * nv;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 8;
    if (c >= total) break;
    if (c >= nq + nk) {
      *reinterpret_cast<uint4*>(vd + c - nq - nk) = raw[i];
      continue;
    }
    const bool is_q = c < nq;
    const int k = is_q ? c : c - nq, h = k / p.d, col = k - h * p.d;
    if (!is_q && same) *reinterpret_cast<uint4*>(vd + k) = raw[i];
    float f[8];
    unpack8(raw[i], f);
    if (NORM) {
      const float4 g0 = *reinterpret_cast<const float4*>((is_q ? p.q_gain : p.k_gain) + k), g1 = *reinterpret_cast<const float4*>((is_q ? p.q_gain : p.k_gain) + k + 4);
      const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w}, inv = is_q ? iq : ik;
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = f[j] * inv * g[j];
    }
    if (col < p.rope.rot) {                          // whole chunks: rot is a multiple of 8
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 r = cs[col / 2 + j];
        const float a = f[2 * j], b = f[2 * j + 1];
        f[2 * j] = a * r.x - b * r.y;
        f[2 * j + 1] = b * r.x + a * r.y;
      }
    }
    bf16* dst = is_q ? reinterpret_cast<bf16*>(p.q_out) + (long)t * p.ldq + (long)h * p.q_stride + col : reinterpret_cast<bf16*>(p.k_cache) + dst_row * nk + k;
    *reinterpret_cast<uint4*>(dst) = pack8(f);
  }
}

template <bool NORM>
int write_chunks(const QkParams& p, cudaStream_t s) {
  const int chunks = (p.H * p.d + p.G * p.d + (p.v_off == p.k_off ? 0 : p.G * p.e) + 2047) / 2048;
  if (chunks <= 2) return launch_chain(qk_chunks_write_kernel<2, NORM>, dim3(p.T), dim3(256), 0, s, p);
  return launch_chain(qk_chunks_write_kernel<4, NORM>, dim3(p.T), dim3(256), 0, s, p);
}

struct WinParams {
  const void* q; long ldq;
  const void *k_cache, *v_cache;
  const int32_t *positions, *slots, *page_table;
  int max_pages, page_tokens, num_pages;
  int H, G, d, e, window;
  float scale;
  const float* sink;             // [H] or null
  const void* gate; long ldg; int gate_act;
  void* out; long ldo;
  int q_stride;
  uint32_t* status;
  ScoreRule rule;
  int gate_head;                 // the gate has one value per head: [T, H]
  AheadRule ahead;
  float factor;                  // of the result
};

// The first n_ahead entries ahead of a window (rows 0 .. ahead_rows - 1, zero-filled), then keys and values first .. first + n - 1 of one sequence out of its pages: k [rows, G * dp] (columns d .. dp - 1 of a head zero) and
// transposed values vt [G * 128, ld] (rows e .. 127 of a head zero), rows / columns from n on zero - the operands of the tensor-core
// attention. grid (ceil(rows / 32), G): one CTA per 32 keys of a head, values turned through shared memory.
__global__ void __launch_bounds__(256) ctx_gather_pad_kernel(const bf16* k_cache, const bf16* v_cache, const int32_t* page_table, int slot, int max_pages,
                                                             int page_tokens, int num_pages, int first, int n, AheadRule ahead, int n_ahead, int ahead_rows,
                                                             int G, int d, int dp, int e, bf16* k, bf16* vt, long ldvt, uint32_t* status) {
  __shared__ bf16 tile[32][128 + 2];
  __shared__ long src_row[32];
  grid_dep_launch();
  grid_dep_wait();
  const int j0 = blockIdx.x * 32, g = blockIdx.y, t = threadIdx.x;
  const bool front = j0 < ahead_rows, pooled = front && ahead.pool > 0;
  if (pooled) {
    k_cache = reinterpret_cast<const bf16*>(ahead.k);
    v_cache = reinterpret_cast<const bf16*>(ahead.v);
  }
  if (t < 32) {
    long row = -1;
    const int i = front ? j0 + t : j0 + t - ahead_rows;
    if (i < (front ? n_ahead : n)) {
      const int pos = front ? ahead.position(i) : first + i, lp = pos / page_tokens;
      const int page = lp < max_pages ? page_table[(long)slot * max_pages + lp] : -1;
      if (page >= 0 && page < num_pages) row = pooled ? (long)page * ahead.per_page + ahead.row(i, page_tokens) : (long)page * page_tokens + pos % page_tokens;
      else if (status) atomicOr(status, IFAB_STATUS_BAD_INDEX);
    }
    src_row[t] = row;
  }
  __syncthreads();
  if ((d | e) % 8 == 0) {
    // 16-byte chunks: keys straight through, values by columns of 8 keys
    for (int i = t; i < 32 * (dp / 8); i += 256) {
      const int kk = i / (dp / 8), c = (i - kk * (dp / 8)) * 8;
      const long row = src_row[kk];
      *reinterpret_cast<uint4*>(k + (long)(j0 + kk) * G * dp + (long)g * dp + c) =
          (row >= 0 && c < d) ? *reinterpret_cast<const uint4*>(k_cache + (row * G + g) * d + c) : make_uint4(0, 0, 0, 0);
    }
    for (int i = t; i < 32 * 16; i += 256) {
      const int kk = i >> 4, c = (i & 15) * 8;
      const long row = src_row[kk];
      const uint4 v = (row >= 0 && c < e) ? *reinterpret_cast<const uint4*>(v_cache + (row * G + g) * e + c) : make_uint4(0, 0, 0, 0);
      uint32_t* w = reinterpret_cast<uint32_t*>(&tile[kk][c]);
      w[0] = v.x;
      w[1] = v.y;
      w[2] = v.z;
      w[3] = v.w;
    }
    __syncthreads();
    for (int i = t; i < 128 * 4; i += 256) {
      const int c = i >> 2, k0 = (i & 3) * 8;
      union { bf16 h[8]; uint4 u; } o;
#pragma unroll
      for (int j = 0; j < 8; ++j) o.h[j] = tile[k0 + j][c];
      *reinterpret_cast<uint4*>(vt + ((long)g * 128 + c) * ldvt + j0 + k0) = o.u;
    }
    return;
  }
  const bf16 zero = __float2bfloat16_rn(0.f);
  for (int i = t; i < 32 * dp; i += 256) {
    const int kk = i / dp, c = i - kk * dp;
    const long row = src_row[kk];
    k[(long)(j0 + kk) * G * dp + (long)g * dp + c] = (row >= 0 && c < d) ? k_cache[(row * G + g) * d + c] : zero;
  }
  for (int i = t; i < 32 * 128; i += 256) {
    const int kk = i >> 7, c = i & 127;
    const long row = src_row[kk];
    tile[kk][c] = (row >= 0 && c < e) ? v_cache[(row * G + g) * e + c] : zero;
  }
  __syncthreads();
  for (int c = t >> 5; c < 128; c += 8) vt[((long)g * 128 + c) * ldvt + j0 + (t & 31)] = tile[t & 31][c];
}

constexpr int WARPS = 8, KB = 4, EPL = 8;      // lanes own columns lane, lane + 32, ...: up to 256

template <typename A>
__global__ void __launch_bounds__(256) window_attn_kernel(WinParams p) {
  __shared__ float sm_acc[WARPS][256], sm_m[WARPS], sm_l[WARPS];
  grid_dep_launch();
  grid_dep_wait();
  const int h = blockIdx.x, t = blockIdx.y, g = h / (p.H / p.G), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[t];
  if (pos < 0) return;
  const int32_t* table = p.page_table + (long)p.slots[t] * p.max_pages;
  const int first = first_key(pos, p.window, p.rule.chunked);
  const float slope = p.rule.slopes ? p.rule.slopes[h] : 0.f;
  float q[EPL], acc[EPL];
  const A* qr = reinterpret_cast<const A*>(p.q) + (long)t * p.ldq + (long)h * p.q_stride;
#pragma unroll
  for (int u = 0; u < EPL; ++u) {
    const int c = lane + 32 * u;
    q[u] = c < p.d ? to_f32(qr[c]) : 0.f;
    acc[u] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int ahead = p.ahead.count(first), n = ahead + pos + 1 - first;      // what the query sees: entries ahead of the window, then its positions
  for (int k0 = warp; k0 < n; k0 += WARPS * KB) {
    float s[KB];
    long r[KB];
    const A* vr[KB];
#pragma unroll
    for (int b = 0; b < KB; ++b) {
      const int i = k0 + b * WARPS;
      r[b] = -1;
      s[b] = 0.f;
      if (i < n) {
        const bool pooled = i < ahead && p.ahead.pool > 0;
        const int key = i < ahead ? p.ahead.position(i) : first + i - ahead, lp = key / p.page_tokens;
        const int page = lp < p.max_pages ? table[lp] : -1;
        if (page < 0 || page >= p.num_pages) {
          if (lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_BAD_INDEX);
        } else {
          r[b] = ((pooled ? (long)page * p.ahead.per_page + p.ahead.row(i, p.page_tokens) : (long)page * p.page_tokens + key % p.page_tokens)) * p.G + g;
          const A* kr = reinterpret_cast<const A*>(pooled ? p.ahead.k : p.k_cache) + r[b] * p.d;
          vr[b] = reinterpret_cast<const A*>(pooled ? p.ahead.v : p.v_cache) + r[b] * p.e;
#pragma unroll
          for (int u = 0; u < EPL; ++u)
            if (32 * u < p.d && lane + 32 * u < p.d) s[b] = fmaf(q[u], to_f32(kr[lane + 32 * u]), s[b]);
        }
      }
    }
#pragma unroll
    for (int b = 0; b < KB; ++b) s[b] = r[b] >= 0 ? warp_sum(s[b]) * p.scale : -INFINITY;
    if (!p.rule.plain()) {
#pragma unroll
      for (int b = 0; b < KB; ++b)
        if (r[b] >= 0) s[b] = ruled_score<sizeof(A) == 2>(s[b], p.rule, slope, n - 1 - k0 - b * WARPS);
    }
    float mn = m;
#pragma unroll
    for (int b = 0; b < KB; ++b) mn = fmaxf(mn, s[b]);
    if (mn == -INFINITY) continue;
    const float corr = expf(m - mn);
    l *= corr;
#pragma unroll
    for (int u = 0; u < EPL; ++u) acc[u] *= corr;
#pragma unroll
    for (int b = 0; b < KB; ++b) {
      if (r[b] < 0) continue;
      const float w = expf(s[b] - mn);
      l += w;
#pragma unroll
      for (int u = 0; u < EPL; ++u)
        if (32 * u < p.e && lane + 32 * u < p.e) acc[u] = fmaf(w, to_f32(vr[b][lane + 32 * u]), acc[u]);
    }
    m = mn;
  }
  if (lane == 0) {
    sm_m[warp] = m;
    sm_l[warp] = l;
  }
#pragma unroll
  for (int u = 0; u < EPL; ++u) sm_acc[warp][lane + 32 * u] = acc[u];
  __syncthreads();
  float M = p.sink ? p.sink[h] : -INFINITY;
#pragma unroll
  for (int w = 0; w < WARPS; ++w) M = fmaxf(M, sm_m[w]);
  float den = p.sink ? expf(p.sink[h] - M) : 0.f, wgt[WARPS];
#pragma unroll
  for (int w = 0; w < WARPS; ++w) {
    wgt[w] = sm_m[w] == -INFINITY ? 0.f : expf(sm_m[w] - M);
    den += wgt[w] * sm_l[w];
  }
  const float inv = den > 0.f ? p.factor / den : 0.f;
  for (int c = threadIdx.x; c < p.e; c += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) v = fmaf(wgt[w], sm_acc[w][c], v);
    v *= inv;
    if (p.gate) v *= activate<sizeof(A) == 2>(to_f32(reinterpret_cast<const A*>(p.gate)[(long)t * p.ldg + (p.gate_head ? h : (long)h * p.e + c)]), p.gate_act);
    reinterpret_cast<A*>(p.out)[(long)t * p.ldo + (long)h * p.e + c] = from_f32<A>(v);
  }
}

// grid T, 128 threads: the block that ends at a row's position, if one does. All heads of a position are one row, keys and values; V columns per thread at a time
template <typename A, int V>
__global__ void __launch_bounds__(128) pool_write_kernel(const A* k_cache, const A* v_cache, const int32_t* positions, const int32_t* slots, const int32_t* page_table,
                                                         int max_pages, int page_tokens, int num_pages, int nk, int nv, AheadRule rule, uint32_t* status) {
  constexpr int B = 32;                     // positions looked up together
  __shared__ long rows[B];
  __shared__ int bad;
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, pos = positions[t], P = rule.pool;
  if (pos < 0 || (pos + 1) % P) return;
  const int32_t* table = page_table + (long)slots[t] * max_pages;
  const auto find = [&](int j) {
    const int lp = j / page_tokens, page = lp < max_pages ? table[lp] : -1;
    return page >= 0 && page < num_pages ? page : -1;
  };
  const int last = find(pos);
  if (threadIdx.x == 0) bad = last < 0;
  const long entry = (long)last * rule.per_page + rule.row(pos / P, page_tokens);
  for (int c0 = 0; c0 < nk + nv; c0 += 128 * V) {             // every thread takes every round: the barriers are the CTA's
    const int c = c0 + threadIdx.x * V;
    float acc[V];
#pragma unroll
    for (int u = 0; u < V; ++u) acc[u] = 0.f;
    for (int j0 = pos - P + 1; j0 <= pos; j0 += B) {
      __syncthreads();
      if (threadIdx.x < B) {
        const int j = min(j0 + (int)threadIdx.x, pos), page = find(j);
        if (page < 0) bad = 1;
        rows[threadIdx.x] = (long)max(page, 0) * page_tokens + j % page_tokens;
      }
      __syncthreads();
      if (bad || c >= nk + nv) continue;
      const int n = min(B, pos - j0 + 1), ld = c < nk ? nk : nv;
      const A* src = c < nk ? k_cache + c : v_cache + c - nk;
#pragma unroll 8
      for (int b = 0; b < n; ++b) {
        const A* p = src + rows[b] * ld;
        if constexpr (V == 8) {
          float f[8];
          unpack8(*reinterpret_cast<const uint4*>(p), f);
#pragma unroll
          for (int u = 0; u < 8; ++u) acc[u] += f[u];
        } else {
          acc[0] += to_f32(*p);
        }
      }
    }
    if (bad || c >= nk + nv) continue;
    A* dst = c < nk ? reinterpret_cast<A*>(const_cast<void*>(rule.k)) + entry * nk + c : reinterpret_cast<A*>(const_cast<void*>(rule.v)) + entry * nv + c - nk;
#pragma unroll
    for (int u = 0; u < V; ++u) acc[u] /= (float)P;
    if constexpr (V == 8) *reinterpret_cast<uint4*>(dst) = pack8(acc);
    else *dst = from_f32<A>(acc[0]);
  }
  __syncthreads();
  if (bad && threadIdx.x == 0 && status) atomicOr(status, IFAB_STATUS_BAD_INDEX);
}

}  // namespace

extern "C" int ifab_pool_write(const void* k_cache, const void* v_cache, int f32, const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                               int page_tokens, int num_pages, int G, int d, int e, int pool, void* pool_k, void* pool_v, int T, uint32_t* status, void* stream) {
  if (T < 1 || G < 1 || G > 65535 || d < 1 || d > 256 || e < 1 || e > 256 || pool < 1 || !pool_k || !pool_v) return -1;
  const AheadRule rule = ahead_rule(0, pool, pool_k, pool_v, page_tokens);
  const int nk = G * d, nv = G * e;
  const auto odd = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; };
  cudaStream_t s = (cudaStream_t)stream;
  if (f32)
    return launch_chain(pool_write_kernel<float, 1>, dim3(T), dim3(128), 0, s, (const float*)k_cache, (const float*)v_cache, positions, slots, page_table, max_pages,
                        page_tokens, num_pages, nk, nv, rule, status);
  if (!((nk | nv) % 8) && !odd(k_cache) && !odd(v_cache) && !odd(pool_k) && !odd(pool_v))
    return launch_chain(pool_write_kernel<bf16, 8>, dim3(T), dim3(128), 0, s, (const bf16*)k_cache, (const bf16*)v_cache, positions, slots, page_table, max_pages,
                        page_tokens, num_pages, nk, nv, rule, status);
  return launch_chain(pool_write_kernel<bf16, 1>, dim3(T), dim3(128), 0, s, (const bf16*)k_cache, (const bf16*)v_cache, positions, slots, page_table, max_pages,
                      page_tokens, num_pages, nk, nv, rule, status);
}

extern "C" int ifab_qk_norm_rope_write(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, const float* q_gain, const float* k_gain,
                                       float eps, int H, int G, int d, int e, int rot, int interleaved, const void* rope, const int32_t* positions,
                                       const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, int num_pages, void* q_out,
                                       long ldq, int q_stride, void* k_cache, void* v_cache, int whole, int T, uint32_t* status, void* stream) {
  if (T < 1 || T > 65535 || H < 1 || G < 1 || d < 1 || e < 1 || rot < 0 || rot % 2 || rot > d || (rot && !rope) || q_stride < d) return -1;
  QkParams p{proj, ldp, q_off, k_off, v_off, q_gain, k_gain, eps, H, G, d, e, {(const float2*)rope, rot, interleaved}, positions, slots, page_table, max_pages, page_tokens,
             num_pages, q_out, ldq, q_stride, k_cache, v_cache, T, status};
  const auto odd = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; };
  if (!f32 && (whole || (!q_gain && !k_gain)) && !((d | e | rot | q_off | k_off | v_off | q_stride) % 8) && !((ldp | ldq) % 8) && (interleaved || !rot) &&
      (long)H * d + (long)G * d + (v_off == k_off ? 0 : G * e) <= 8192 && !odd(proj) && !odd(q_out) && !odd(k_cache) && !odd(v_cache) && (!whole || (!odd(q_gain) && !odd(k_gain))))
    return whole ? write_chunks<true>(p, (cudaStream_t)stream) : write_chunks<false>(p, (cudaStream_t)stream);
  if (whole) {
    if (!q_gain || !k_gain) return -1;
    return f32 ? launch_chain(qk_rows_norm_write_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, p)
               : launch_chain(qk_rows_norm_write_kernel<bf16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, p);
  }
  const dim3 grid((H + 2 * G + 3) / 4, T);
  return f32 ? launch_chain(qk_norm_rope_write_kernel<float>, grid, dim3(128), 0, (cudaStream_t)stream, p)
             : launch_chain(qk_norm_rope_write_kernel<bf16>, grid, dim3(128), 0, (cudaStream_t)stream, p);
}

extern "C" int ifab_window_attn(const void* q, long ldq, int q_stride, const void* k_cache, const void* v_cache, int f32, const int32_t* positions, const int32_t* slots,
                                const int32_t* page_table, int max_pages, int page_tokens, int num_pages, int H, int G, int d, int e, int window,
                                float scale, float cap, const float* slopes, int chunked, const float* sink, const void* gate, long ldg, int gate_act,
                                int gate_per_head, int keep, int pool, const void* pool_k, const void* pool_v, float factor, void* out, long ldo, int T,
                                uint32_t* status, void* stream) {
  const AheadRule ahead = ahead_rule(keep, pool, pool_k, pool_v, page_tokens);
  if (!ahead_ok(ahead, window, chunked) || (ahead.any() && (cap > 0.f || slopes))) return -1;
  if (cap < 0.f || T < 1 || T > 65535 || H < 1 || G < 1 || H % G || d < 1 || d > 256 || e < 1 || e > 256 || window < 0) return -1;
  WinParams p{q, ldq, k_cache, v_cache, positions, slots, page_table, max_pages, page_tokens, num_pages, H, G, d, e, window, scale, sink, gate, ldg, gate_act,
              out, ldo, q_stride, status, {cap, slopes, chunked}, gate_per_head, ahead, factor};
  const dim3 grid(H, T);
  return f32 ? launch_chain(window_attn_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, p)
             : launch_chain(window_attn_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, p);
}

extern "C" int ifab_ctx_gather_pad(const void* k_cache, const void* v_cache, const int32_t* page_table, int slot, int max_pages, int page_tokens,
                                   int num_pages, int first, int n, int rows, int keep, int pool, const void* pool_k, const void* pool_v, int n_ahead, int ahead_rows,
                                   int G, int d, int dp, int e, void* k, void* vt, long ldvt, uint32_t* status, void* stream) {
  const AheadRule ahead = ahead_rule(keep, pool, pool_k, pool_v, page_tokens);
  if (!ahead_ok(ahead, 1, 0) || n_ahead < 0 || ahead_rows < n_ahead || ahead_rows % 32 || (n_ahead && !ahead.any())) return -1;
  if (n < 1 || rows < n || rows % 32 || slot < 0 || first < 0 || G < 1 || d < 1 || dp < d || e < 1 || e > 128 || ldvt < rows + ahead_rows || dp % 8 || ldvt % 8) return -1;
  if (((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(vt)) & 15)) return -1;
  return launch_chain(ctx_gather_pad_kernel, dim3((rows + ahead_rows) / 32, G), dim3(256), 0, (cudaStream_t)stream, (const bf16*)k_cache, (const bf16*)v_cache,
                      page_table, slot, max_pages, page_tokens, num_pages, first, n, ahead, n_ahead, ahead_rows, G, d, dp, e, (bf16*)k, (bf16*)vt, ldvt, status);
}

extern "C" int ifab_rope_table(const int32_t* positions, const double* freq, void* cs, int T, int pairs, void* stream) {
  if (T < 1 || pairs < 1) return -1;
  return launch_chain(rope_table_kernel, dim3((unsigned)(((long)T * pairs + 127) / 128)), dim3(128), 0, (cudaStream_t)stream, positions, freq, (float2*)cs, T,
                      pairs);
}
