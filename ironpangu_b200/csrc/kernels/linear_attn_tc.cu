// Linear attention of prompts on the tensor cores: chunks of up to 128 consecutive rows of one sequence, heads of up to 128 columns
// (see linear_attn.cu for the recurrence and the chunk scheme). One CTA per (chunk, head):
//
//   la_tile_state_kernel   what the chunk adds to the state: D[e, d] = sum_j v_j[e] * (decay^(L - 1 - j) k_j[d])
//   la_tile_out_kernel     W = Q K^T; P_ij = decay^(i - j) W_ij for j <= i; o_i = decay^(i + 1) S q_i + sum_j P_ij v_j
//
// All threads first build the operands in shared memory (rotation / activation / decay on the way, heads zero-padded to 64 or
// 128 columns, 128-byte-swizzled K-major panels), then one thread issues tcgen05.mma into tensor memory, then the row threads
// read it back. The recurrence is a 32-bit computation: an operand that is not a bf16 value by nature (rotated q and k, the
// decayed k, the state, P) enters as two bf16 terms, rounded value + remainder, and the products keep all but the smallest
// cross term (~16 bits of every factor, f32 accumulation).
// Waits are bounded: one that runs out sets the status word; nothing asynchronous but the MMAs themselves is ever in flight.
#include "linear_attn.cuh"
#include "tc_common.cuh"

using namespace ifab;
using namespace ifab::tc;

namespace {

constexpr int CT = 128;                          // rows of a chunk
constexpr int PANEL = 128 * 128;                 // 128 rows x 64 bf16
constexpr int THREADS = 512, WARPS = THREADS / 32;

struct TileParams {
  LaParams a;
  const int32_t* chunks;
  float* cstate;                                 // [n, H, e, d]
  float* o; long ldo;                            // f32 heads, or
  const bf16* gate; long ldg; int gate_act;      // (y given) heads divided by their rms and gated, in bf16
  bf16* y; long ldy; float eps;
  uint32_t* status; uint32_t spin_limit;
};

struct Bars {
  uint64_t done[3];
  uint32_t tmem_slot;
};

// byte offset of element (r, c) of an operand whose 64-column panels hold `rows` rows
__device__ __forceinline__ uint32_t at(int r, int c, int rows) {
  return (uint32_t)((c >> 6) * rows * 128 + (r >> 3) * 1024 + (r & 7) * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4) + (c & 7) * 2);
}

// 8 columns c0 .. c0 + 7 of a head of q, k (rotated or activated, times `scale`) or v (rot = 0); columns from n on are zero
__device__ __forceinline__ void load8(const LaParams& p, const bf16* head, const float2* cs, int rot, int c0, int n, bool aligned, float scale, float* f) {
  if (aligned && c0 + 8 <= n) {
    unpack8(*reinterpret_cast<const uint4*>(head + c0), f);
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = c0 + i < n ? to_f32(head[c0 + i]) : 0.f;
  }
  if (c0 < rot) {
    const int half = rot / 2;
    if (!p.rope.interleaved && aligned && half % 8 == 0) {             // the partners are one chunk too
      const bool low = c0 < half;
      float g[8];
      unpack8(*reinterpret_cast<const uint4*>(head + (low ? c0 + half : c0 - half)), g);
      const float2* t = cs + (low ? c0 : c0 - half);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = low ? f[i] * t[i].x - g[i] * t[i].y : f[i] * t[i].x + g[i] * t[i].y;
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (c0 + i < rot) f[i] = rotated(p.rope, cs, head, c0 + i);
        else if (c0 + i < n) f[i] = activated(p, __float2bfloat16_rn(f[i]));
    }
  } else if (p.act) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (c0 + i < n) f[i] = activated(p, __float2bfloat16_rn(f[i]));
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) f[i] *= scale;
}

// load8 in two halves, so that a thread can have several pieces in flight: what the vector path reads ...
struct Raw8 {
  uint4 own, other;
  float4 t[4];
};
__device__ __forceinline__ bool vector8(const LaParams& p, int rot, int c0, int n, bool aligned) {
  return aligned && c0 + 8 <= n && (c0 >= rot || (!p.rope.interleaved && (rot / 2) % 8 == 0));
}
__device__ __forceinline__ void fetch8(const LaParams& p, const bf16* head, const float2* cs, int rot, int c0, int n, bool aligned, Raw8& r) {
  if (!vector8(p, rot, c0, n, aligned)) return;
  r.own = *reinterpret_cast<const uint4*>(head + c0);
  if (c0 < rot) {
    const int half = rot / 2, low = c0 < half ? c0 : c0 - half;
    r.other = *reinterpret_cast<const uint4*>(head + (c0 < half ? c0 + half : c0 - half));
    const float4* t = reinterpret_cast<const float4*>(cs + low);
#pragma unroll
    for (int i = 0; i < 4; ++i) r.t[i] = t[i];
  }
}
// ... and what becomes of it
__device__ __forceinline__ void finish8(const LaParams& p, const bf16* head, const float2* cs, int rot, int c0, int n, bool aligned, float scale,
                                        const Raw8& r, float* f) {
  if (!vector8(p, rot, c0, n, aligned)) {
    load8(p, head, cs, rot, c0, n, aligned, scale, f);
    return;
  }
  unpack8(r.own, f);
  if (c0 < rot) {
    float g[8];
    unpack8(r.other, g);
    const float sign = c0 < rot / 2 ? -1.f : 1.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = f[2 * i] * r.t[i].x + sign * g[2 * i] * r.t[i].y;
      f[2 * i + 1] = f[2 * i + 1] * r.t[i].z + sign * g[2 * i + 1] * r.t[i].w;
    }
  } else if (p.act) {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = activated(p, __float2bfloat16_rn(f[i]));
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) f[i] *= scale;
}

// value -> rounded bf16 terms
__device__ __forceinline__ void split8(const float* f, uint4* hi, uint4* lo) {
  *hi = pack8(f);
  float r[8];
  unpack8(*hi, r);
#pragma unroll
  for (int i = 0; i < 8; ++i) r[i] = f[i] - r[i];
  *lo = pack8(r);
}

__device__ __forceinline__ bool head_aligned(const LaParams& p, int off, int w) { return ((off | w | (int)(p.ldp & 7)) & 7) == 0; }

// A transposed operand: rows = columns 0 .. width - 1 of a head (zero from n on), columns = rows of the chunk, optionally in two terms and
// times scale[L - 1 - row]. width a multiple of 64
template <bool LO>
__device__ __forceinline__ void build_t(const LaParams& p, unsigned char* dst, unsigned char* dst_lo, int width, int row0, int L, int off, int h, int n, int rot,
                                        const float* scale, float factor) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tasks = 4 * (width / 16);
  const bool al = head_aligned(p, off, n);
  for (int task = warp; task < tasks; task += WARPS) {
    const int j = (task & 3) * 32 + lane, c0 = (task >> 2) * 16;
    const bool live = j < L && c0 < n;
    const int row = row0 + (live ? j : 0);
    const bf16* head = reinterpret_cast<const bf16*>(p.proj) + (long)row * p.ldp + off + (long)h * n;
    const float2* cs = rot ? p.rope.cs + (long)row * (rot / 2) : nullptr;
    float f[16];
    if (live) {
      Raw8 r[2];
      fetch8(p, head, cs, rot, c0, n, al, r[0]);
      fetch8(p, head, cs, rot, c0 + 8, n, al, r[1]);
      const float s = factor * (scale ? scale[L - 1 - j] : 1.f);
      finish8(p, head, cs, rot, c0, n, al, s, r[0], f);
      finish8(p, head, cs, rot, c0 + 8, n, al, s, r[1], f + 8);
    } else {
#pragma unroll
      for (int i = 0; i < 16; ++i) f[i] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const bf16 hi = __float2bfloat16_rn(f[i]);
      *reinterpret_cast<bf16*>(dst + at(c0 + i, j, width)) = hi;
      if (LO) *reinterpret_cast<bf16*>(dst_lo + at(c0 + i, j, width)) = __float2bfloat16_rn(f[i] - __bfloat162float(hi));
    }
  }
}

// ends with a CTA barrier: operands written by all threads are visible to the tensor core
__device__ __forceinline__ void operands_ready() {
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
}

// D (+)= A B^T over `panels` 64-column panels of both operands
__device__ __forceinline__ void mma_panels(uint32_t d, uint32_t a, uint32_t b, int a_panel, int b_panel, int panels, uint32_t idesc, bool* acc) {
  for (int pp = 0; pp < panels; ++pp) {
    const uint64_t da = umma_desc_sw128(a + pp * a_panel), db = umma_desc_sw128(b + pp * b_panel);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      umma_bf16(d, da + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, *acc);
      *acc = true;
    }
  }
}

// NP: 64-column panels of a head of q / k
template <int NP>
__global__ void __launch_bounds__(THREADS) la_tile_state_kernel(TileParams p) {
  constexpr int DP = 64 * NP;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  unsigned char *vt = smem, *kt = smem + 2 * PANEL, *ktl = kt + 2 * DP * 128;
  Bars* B = reinterpret_cast<Bars*>(ktl + 2 * DP * 128);
  const LaParams& a = p.a;
  const int c = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&B->done[0], 1);
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc(&B->tmem_slot, DP);
  __syncthreads();               // tensor memory is taken before a dependent kernel may start beside this one
  grid_dep_launch();
  grid_dep_wait();
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  const float* pw = a.powers + (long)h * LA_POW;
  // a lane owns a row of the chunk: its 2-byte stores run along an operand's rows, so a warp's store covers 32 consecutive columns
  build_t<true>(a, kt, ktl, DP, row0, L, a.k_off, h, a.d, a.rope.rot, pw, a.k_scale);
  build_t<false>(a, vt, nullptr, 128, row0, L, a.v_off, h, a.e, 0, nullptr, 1.f);
  operands_ready();
  const uint32_t tmem = B->tmem_slot;
  if (threadIdx.x == 0) {
    constexpr uint32_t idesc = umma_idesc_bf16(128, DP);
    bool acc = false;
    mma_panels(tmem, smem_u32(vt), smem_u32(kt), PANEL, DP * 128, 2, idesc, &acc);
    mma_panels(tmem, smem_u32(vt), smem_u32(ktl), PANEL, DP * 128, 2, idesc, &acc);
    umma_commit(&B->done[0]);
  }
  const bool ok = __all_sync(0xffffffffu, mbar_wait(&B->done[0], 0, p.spin_limit));
  tc_fence_after();
  if (!ok) {
    if (lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_MBAR_TIMEOUT);
  } else {
    // four threads per value column (TMEM lane), each a quarter of the d columns (with 64 columns two of them have work)
    const int e = (warp & 3) * 32 + lane, part = warp >> 2;
    float* out = p.cstate + (((long)c * a.H + h) * a.e + e) * a.d;
#pragma unroll 1
    for (int c0 = part * 32; c0 < DP; c0 += 128) {
      float v[32];
      tmem_ld_32x32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)c0, v);
      tmem_ld_wait();
      if (e < a.e && a.d % 4 == 0) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (c0 + 4 * i < a.d) *reinterpret_cast<float4*>(out + c0 + 4 * i) = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
      } else if (e < a.e) {
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (c0 + i < a.d) out[c0 + i] = v[i];
      }
      __syncwarp();              // the next read of tensor memory is warp-wide
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, DP);
  }
}

// LO: q and k have a second term (they were rotated or scaled)
template <int NP, bool LO>
struct OutLayout {
  static constexpr int T = LO ? 2 : 1;
  static constexpr int Q = 0, K = Q + T * NP * PANEL, S = K + (T * NP > 4 ? T * NP : 4) * PANEL, V = S + 2 * NP * PANEL, POW = V + 2 * PANEL,
                       BAR = POW + 640, SMEM = BAR + 256 + 1024;
  static constexpr int P = K;                    // the weights take the place of k once W is complete
};

template <int NP, bool LO>
__global__ void __launch_bounds__(THREADS, 1) la_tile_out_kernel(TileParams p) {
  using Y = OutLayout<NP, LO>;
  constexpr int DP = 64 * NP, TERM = NP * PANEL;
  constexpr uint32_t W_COL = 0, S_COL = 128, O_COL = 256;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  float* pw = reinterpret_cast<float*>(smem + Y::POW);
  Bars* B = reinterpret_cast<Bars*>(smem + Y::BAR);
  const LaParams& a = p.a;
  const int c = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&B->done[i], 1);
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc(&B->tmem_slot, 512);
  if (threadIdx.x < LA_POW) pw[threadIdx.x] = a.powers[(long)h * LA_POW + threadIdx.x];
  __syncthreads();               // tensor memory is taken before a dependent kernel may start beside this one
  grid_dep_launch();
  grid_dep_wait();
  const int row0 = p.chunks[c * 4], L = p.chunks[c * 4 + 1];
  // q and k: eight lanes per row and panel (one 128-byte line); two positions' loads in flight per thread
  const bool alq = head_aligned(a, a.q_off, a.d), alk = head_aligned(a, a.k_off, a.d);
  for (int i0 = threadIdx.x; i0 < CT * (DP / 8); i0 += 2 * THREADS) {
    Raw8 rq[2], rk[2];
    const bf16 *qh[2], *kh[2];
    const float2* cs[2];
    bool live[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * THREADS, r = i / (DP / 8), c0 = i % (DP / 8) * 8;
      live[u] = r < L && c0 < a.d;
      const int row = row0 + (live[u] ? r : 0);
      qh[u] = reinterpret_cast<const bf16*>(a.proj) + (long)row * a.ldp + a.q_off + (long)h * a.d;
      kh[u] = reinterpret_cast<const bf16*>(a.proj) + (long)row * a.ldp + a.k_off + (long)h * a.d;
      cs[u] = a.rope.rot ? a.rope.cs + (long)row * (a.rope.rot / 2) : nullptr;
      if (live[u]) {
        fetch8(a, qh[u], cs[u], a.rope.rot, c0, a.d, alq, rq[u]);
        fetch8(a, kh[u], cs[u], a.rope.rot, c0, a.d, alk, rk[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * THREADS, r = i / (DP / 8), c0 = i % (DP / 8) * 8;
#pragma unroll
      for (int which = 0; which < 2; ++which) {
        float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (live[u])
          finish8(a, which ? kh[u] : qh[u], cs[u], a.rope.rot, c0, a.d, which ? alk : alq, which ? a.k_scale : 1.f, which ? rk[u] : rq[u], f);
        unsigned char* dst = smem + (which ? Y::K : Y::Q) + at(r, c0, 128);
        uint4 hi, lo;
        split8(f, &hi, &lo);
        *reinterpret_cast<uint4*>(dst) = hi;
        if (LO) *reinterpret_cast<uint4*>(dst + TERM) = lo;
      }
    }
  }
  operands_ready();
  const uint32_t tmem = B->tmem_slot;
  constexpr uint32_t idesc = umma_idesc_bf16(128, 128);
  if (threadIdx.x == 0) {
    const uint32_t q = smem_u32(smem + Y::Q), k = smem_u32(smem + Y::K);
    bool acc = false;
    mma_panels(tmem + W_COL, q, k, PANEL, PANEL, NP, idesc, &acc);
    if (LO) {
      mma_panels(tmem + W_COL, q, k + TERM, PANEL, PANEL, NP, idesc, &acc);
      mma_panels(tmem + W_COL, q + TERM, k, PANEL, PANEL, NP, idesc, &acc);
    }
    umma_commit(&B->done[0]);
  }
  __syncwarp();
  // the state ahead of the chunk (rows = value columns) and v^T, while W is computed
  const float* S = p.cstate + ((long)c * a.H + h) * a.e * a.d;
#pragma unroll
  for (int u = 0; u < 128 * (DP / 8) / THREADS; ++u) {
    const int i = threadIdx.x + u * THREADS, chunk = i % (DP / 8), r = i / (DP / 8), c0 = chunk * 8;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (r < a.e) {
      if (a.d % 4 == 0 && c0 + 8 <= a.d) {
        const float4 u = *reinterpret_cast<const float4*>(S + (long)r * a.d + c0), v = *reinterpret_cast<const float4*>(S + (long)r * a.d + c0 + 4);
        f[0] = u.x; f[1] = u.y; f[2] = u.z; f[3] = u.w;
        f[4] = v.x; f[5] = v.y; f[6] = v.z; f[7] = v.w;
      } else {
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (c0 + k < a.d) f[k] = S[(long)r * a.d + c0 + k];
      }
    }
    uint4 hi, lo;
    split8(f, &hi, &lo);
    unsigned char* dst = smem + Y::S + at(r, c0, 128);
    *reinterpret_cast<uint4*>(dst) = hi;
    *reinterpret_cast<uint4*>(dst + TERM) = lo;
  }
  build_t<false>(a, smem + Y::V, nullptr, 128, row0, L, a.v_off, h, a.e, 0, nullptr, 1.f);
  operands_ready();
  if (threadIdx.x == 0) {
    const uint32_t q = smem_u32(smem + Y::Q), s = smem_u32(smem + Y::S);
    bool acc = false;
    mma_panels(tmem + S_COL, q, s, PANEL, PANEL, NP, idesc, &acc);
    mma_panels(tmem + S_COL, q, s + TERM, PANEL, PANEL, NP, idesc, &acc);
    if (LO) mma_panels(tmem + S_COL, q + TERM, s, PANEL, PANEL, NP, idesc, &acc);
    umma_commit(&B->done[1]);
  }
  __syncwarp();
  // P: four threads per row, 32 columns each
  const int i = (warp & 3) * 32 + lane, part = warp >> 2, c0 = part * 32;
  const uint32_t row_addr = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  bool ok = __all_sync(0xffffffffu, mbar_wait(&B->done[0], 0, p.spin_limit));
  tc_fence_after();
  if (ok) {
    float v[32];
    tmem_ld_32x32(row_addr + W_COL + (uint32_t)c0, v);
    tmem_ld_wait();
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      float f[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int j = c0 + 8 * g + k;
        f[k] = j <= i ? v[8 * g + k] * pw[j <= i ? i - j : 0] : 0.f;
      }
      uint4 hi, lo;
      split8(f, &hi, &lo);
      unsigned char* dst = smem + Y::P + at(i, c0 + 8 * g, 128);
      *reinterpret_cast<uint4*>(dst) = hi;
      *reinterpret_cast<uint4*>(dst + 2 * PANEL) = lo;
    }
  }
  operands_ready();
  if (threadIdx.x == 0) {
    const uint32_t w = smem_u32(smem + Y::P), v = smem_u32(smem + Y::V);
    bool acc = false;
    mma_panels(tmem + O_COL, w, v, PANEL, PANEL, 2, idesc, &acc);
    mma_panels(tmem + O_COL, w + 2 * PANEL, v, PANEL, PANEL, 2, idesc, &acc);
    umma_commit(&B->done[2]);
  }
  __syncwarp();
  ok = __all_sync(0xffffffffu, mbar_wait(&B->done[1], 0, p.spin_limit) && mbar_wait(&B->done[2], 0, p.spin_limit)) && ok;
  tc_fence_after();
  if (!ok && lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_MBAR_TIMEOUT);
  // o_i = decay^(i + 1) S q_i + P v: this thread's 32 columns
  float o[32], u[32];
  const float dec = pw[i + 1];
  float ss = 0.f;
  tmem_ld_32x32(row_addr + S_COL + (uint32_t)c0, u);
  tmem_ld_32x32(row_addr + O_COL + (uint32_t)c0, o);
  tmem_ld_wait();
#pragma unroll
  for (int k = 0; k < 32; ++k) {
    o[k] = fmaf(dec, u[k], o[k]);
    if (c0 + k < a.e) ss += o[k] * o[k];
  }
  const bool live = i < L && ok;
  if (p.y) {
    // the head's rms: the four threads of a row add their sums
    float* red = reinterpret_cast<float*>(smem + Y::P);
    __syncthreads();
    red[part * 128 + i] = ss;
    __syncthreads();
    const float inv = 1.f / sqrtf(((red[i] + red[128 + i]) + (red[256 + i] + red[384 + i])) / (float)a.e + p.eps);
    if (live) {
      bf16* dst = p.y + (long)(row0 + i) * p.ldy + (long)h * a.e + c0;
      const bf16* gr = p.gate + (long)(row0 + i) * p.ldg + (long)h * a.e + c0;
      const bool wide = ((a.e | (int)(p.ldy & 7) | (int)(p.ldg & 7)) & 7) == 0 && (reinterpret_cast<uintptr_t>(p.gate) & 15) == 0;
#pragma unroll
      for (int x = 0; x < 32; x += 8) {
        if (c0 + x >= a.e) break;
        float f[8], g[8];
        if (wide) unpack8(*reinterpret_cast<const uint4*>(gr + x), g);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (!wide) g[k] = c0 + x + k < a.e ? to_f32(gr[x + k]) : 0.f;
          f[k] = o[x + k] * inv * activate<true>(g[k], p.gate_act);
        }
        if (wide) {
          *reinterpret_cast<uint4*>(dst + x) = pack8(f);
        } else {
#pragma unroll
          for (int k = 0; k < 8; ++k)
            if (c0 + x + k < a.e) dst[x + k] = __float2bfloat16_rn(f[k]);
        }
      }
    }
  } else if (live) {
    float* dst = p.o + (long)(row0 + i) * p.ldo + (long)h * a.e + c0;
    if (a.e % 4 == 0 && p.ldo % 4 == 0) {
#pragma unroll
      for (int x = 0; x < 32; x += 4)
        if (c0 + x < a.e) *reinterpret_cast<float4*>(dst + x) = make_float4(o[x], o[x + 1], o[x + 2], o[x + 3]);
    } else {
#pragma unroll
      for (int x = 0; x < 64; ++x)
        if (c0 + x < a.e) dst[x] = o[x];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int NP>
int launch_state(const TileParams& p, int n, cudaStream_t s) {
  const size_t smem = 2 * PANEL + 4 * 64 * NP * 128 + 256 + 1024;
  if (int rc = opt_in_smem(la_tile_state_kernel<NP>, smem)) return rc;
  return launch_chain(la_tile_state_kernel<NP>, dim3(n, p.a.H), dim3(THREADS), smem, s, p);
}
template <int NP, bool LO>
int launch_out(const TileParams& p, int n, cudaStream_t s) {
  static_assert(OutLayout<NP, LO>::SMEM <= 227 * 1024, "shared memory of the chunk output kernel");
  if (int rc = opt_in_smem(la_tile_out_kernel<NP, LO>, OutLayout<NP, LO>::SMEM)) return rc;
  return launch_chain(la_tile_out_kernel<NP, LO>, dim3(n, p.a.H), dim3(THREADS), (size_t)OutLayout<NP, LO>::SMEM, s, p);
}

}  // namespace

// proj bf16; d, e <= 128; chunks of at most 128 rows. Heads as f32 rows o [T, H * e], or - y given - divided by their rms (no gain),
// multiplied by act(gate) and stored as bf16 rows y [T, H * e].
extern "C" int ifab_la_tiles(const void* proj, long ldp, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved, const void* rope,
                             int act, float k_scale, const float* powers, const int32_t* chunks, int n, const int32_t* positions, float* cstate,
                             uint64_t cstate_bytes, float* state, float* o, long ldo, const void* gate, long ldg, int gate_act, void* y, long ldy, float eps,
                             uint32_t* status, void* stream) {
  if (n < 1 || n > 65535 || H < 1 || H > 65535 || d < 1 || d > 128 || e < 1 || e > 128 || rot < 0 || rot % 2 || rot > d || (rot && !rope)) return -1;
  if ((!y && !o) || (y && !gate)) return -1;
  if ((uint64_t)n * H * d * e * sizeof(float) > cstate_bytes) return -5;
  TileParams p{};
  p.a = LaParams{proj, ldp, q_off, k_off, v_off, H, d, e, {(const float2*)rope, rot, interleaved}, act, k_scale, powers, state, positions, nullptr, 0};
  p.chunks = chunks; p.cstate = cstate; p.o = o; p.ldo = ldo; p.gate = (const bf16*)gate; p.ldg = ldg; p.gate_act = gate_act;
  p.y = (bf16*)y; p.ldy = ldy; p.eps = eps; p.status = status; p.spin_limit = 4000000u;
  cudaStream_t s = (cudaStream_t)stream;
  const bool lo = rot > 0 || k_scale != 1.f;
  if (int rc = d <= 64 ? launch_state<1>(p, n, s) : launch_state<2>(p, n, s)) return rc;
  if (int rc = la_scan(cstate, state, chunks, n, positions, powers, H, d, e, s)) return rc;
  if (d <= 64) return lo ? launch_out<1, true>(p, n, s) : launch_out<1, false>(p, n, s);
  return lo ? launch_out<2, true>(p, n, s) : launch_out<2, false>(p, n, s);
}
