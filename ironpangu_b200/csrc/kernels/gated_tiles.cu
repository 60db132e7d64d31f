// Recurrences with a decay per token (gated_recurrence.cu) over prompts on the tensor cores: chunks of up to 128 consecutive rows of one sequence, heads of up to
// 128 columns, bf16 rows. One CTA per (chunk, head) unless said otherwise:
//
//   gr_tile_state_kernel   SSD, MEMORY: what the chunk adds to the state, D[e, d] = sum_j v_j[e] * (c_j k_j[d]), c_j the weight of row j's write at the chunk's
//                          end; MEMORY: the sum of the weighted keys beside it. The states ahead of every chunk: gr_scan_kernel
//   gr_tile_delta_kernel   DELTA: A_ij = b_i (g_i / g_j) (k_i . k_j) below the diagonal, T = (1 + A)^-1 by blocks of 16, 32, 64, 128 rows, and T (b v) and
//                          T (b g k) (see gated_delta.cu)
//   gr_tile_scan_kernel    DELTA, over the chunks of a sequence, one CTA per (head, 32 value columns): u = T (b v) - T (b g k) S, S = g_L S + sum_j (g_L / g_j)
//                          k_j u_j^T. The state stays in tensor memory; the operands of the next chunk arrive by bulk copies meanwhile
//   gr_tile_out_kernel     W = Q K^T; P_ij = weight of row j as row i sees it * W_ij for j <= i; o_i = carry_i S q_i + sum_j P_ij v_j; MEMORY and DELTA go on to
//                          the normed, gated operand of the output projection
//
// Operands lie in shared memory as 128-byte-swizzled K-major panels of 64 columns, built by all threads; one thread issues tcgen05.mma into tensor memory.
// Rows of q, k and v are bf16 values, their factors are 32-bit: whatever carries a factor - c_j k_j, T, P, the state, u - enters as two bf16 terms, rounded
// value + remainder, and the products keep all but the smallest cross term (~16 bits of every factor, f32 accumulation).
// Waits are bounded: one that runs out sets the status word; nothing asynchronous but the MMAs and the bulk copies of the scan is ever in flight, and
// those are waited for before a CTA returns.
#include "gated_recurrence.cuh"
#include "tc_common.cuh"

using namespace ifab;
using namespace ifab::tc;

namespace {

constexpr int CT = GR_TILE;
constexpr int PANEL = 128 * 128;                 // 128 rows x 64 bf16
constexpr int THREADS = 512, WARPS = THREADS / 32;

struct TileParams {
  GrChunks c;
  GrState st;
  const bf16* gate; long ldg; int gate_act; const float* gain; float eps;      // y given: o over its denominator and rms, times gain [H * e] and act(gate), in bf16
  bf16* y; long ldy;
  float* u;                                      // DELTA: [T, H, e], T (b v), then the corrected values
  unsigned char* images;                         // DELTA: per (chunk, head) T (b g k) in two terms, then k transposed: operands as they lie in shared memory
  uint32_t* status; uint32_t spin_limit;
};

// byte offset of element (r, c) of an operand whose 64-column panels hold `rows` rows
__device__ __forceinline__ uint32_t at(int r, int c, int rows) {
  return (uint32_t)((c >> 6) * rows * 128 + (r >> 3) * 1024 + (r & 7) * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4) + (c & 7) * 2);
}
__device__ __forceinline__ void put(unsigned char* p, uint32_t off, float v) { *reinterpret_cast<bf16*>(p + off) = __float2bfloat16_rn(v); }
// value -> rounded value in `p`, remainder in `lo`
__device__ __forceinline__ void put2(unsigned char* p, unsigned char* lo, uint32_t off, float v) {
  const bf16 hi = __float2bfloat16_rn(v);
  *reinterpret_cast<bf16*>(p + off) = hi;
  *reinterpret_cast<bf16*>(lo + off) = __float2bfloat16_rn(v - __bfloat162float(hi));
}
__device__ __forceinline__ void split8(const float* f, uint4* hi, uint4* lo) {
  *hi = pack8(f);
  float r[8];
  unpack8(*hi, r);
#pragma unroll
  for (int i = 0; i < 8; ++i) r[i] = f[i] - r[i];
  *lo = pack8(r);
}

// 8 columns from c0 on of a row of n bf16 values (zero past n)
__device__ __forceinline__ uint4 row8(const bf16* row, int c0, int n, bool aligned) {
  if (aligned && c0 + 8 <= n) return *reinterpret_cast<const uint4*>(row + c0);
  union { bf16 h[8]; uint4 u; } o;
#pragma unroll
  for (int i = 0; i < 8; ++i) o.h[i] = c0 + i < n ? row[c0 + i] : __float2bfloat16_rn(0.f);
  return o.u;
}

// An operand [128 rows of the chunk, 64 NP columns] from rows of n columns `ld` apart; rows from L on zero
template <int NP>
__device__ __forceinline__ void build_rows(unsigned char* dst, const bf16* src, long ld, int n, int L) {
  const bool al = ((n | (int)(ld & 7)) & 7) == 0;
#pragma unroll 4
  for (int i = threadIdx.x; i < CT * 8 * NP; i += THREADS) {
    const int r = i / (8 * NP), c0 = i % (8 * NP) * 8;
    *reinterpret_cast<uint4*>(dst + at(r, c0, 128)) = r < L && c0 < n ? row8(src + (long)r * ld, c0, n, al) : make_uint4(0, 0, 0, 0);
  }
}
// The transposed operand [width columns, 128 rows of the chunk]; LO: times scale[row], in two terms. width a multiple of 64
template <bool LO>
__device__ __forceinline__ void build_t(unsigned char* dst, unsigned char* dst_lo, int width, const bf16* src, long ld, int n, int L, const float* scale) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tasks = 4 * (width / 16);
  const bool al = ((n | (int)(ld & 7)) & 7) == 0;
  for (int task = warp; task < tasks; task += WARPS) {
    const int j = (task & 3) * 32 + lane, c0 = (task >> 2) * 16;
    const bool live = j < L && c0 < n;
    uint4 raw[2] = {make_uint4(0, 0, 0, 0), make_uint4(0, 0, 0, 0)};
    if (live) {
      const bf16* row = src + (long)j * ld;
      raw[0] = row8(row, c0, n, al);
      if (c0 + 8 < n) raw[1] = row8(row, c0 + 8, n, al);
    }
    float f[16];
    unpack8(raw[0], f);
    unpack8(raw[1], f + 8);
    const float s = LO ? scale[j] : 1.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      if (LO) put2(dst, dst_lo, at(c0 + i, j, width), f[i] * s);
      else put(dst, at(c0 + i, j, width), f[i]);
    }
  }
}
// The transposed operand of f32 rows in two terms
__device__ __forceinline__ void build_t_f32(unsigned char* dst, unsigned char* dst_lo, int width, const float* src, long ld, int n, int L) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tasks = 4 * (width / 8);
  const bool al = ((n | (int)(ld & 3)) & 3) == 0;
  for (int task = warp; task < tasks; task += WARPS) {
    const int j = (task & 3) * 32 + lane, c0 = (task >> 2) * 8;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (j < L && c0 < n) {
      const float* row = src + (long)j * ld;
      if (al && c0 + 8 <= n) {
        const float4 a = *reinterpret_cast<const float4*>(row + c0), b = *reinterpret_cast<const float4*>(row + c0 + 4);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
        f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (c0 + i < n) f[i] = row[c0 + i];
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) put2(dst, dst_lo, at(c0 + i, j, width), f[i]);
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

__device__ __forceinline__ unsigned char* aligned_smem(unsigned char* raw) {
  return reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~(uintptr_t)1023);
}

struct Bars {
  uint64_t done[4];
  uint32_t tmem_slot;
};

// ---------------------------------------------------------------------------------------------------------------------------
// SSD, MEMORY: what a chunk adds to the state. NP: 64-column panels of a head of k
// ---------------------------------------------------------------------------------------------------------------------------
template <int NP>
__global__ void __launch_bounds__(THREADS) gr_tile_state_kernel(TileParams p) {
  constexpr int DP = 64 * NP;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = aligned_smem(smem_raw);
  unsigned char *vt = smem, *kt = smem + 2 * PANEL, *ktl = kt + 2 * DP * 128;
  Bars* B = reinterpret_cast<Bars*>(ktl + 2 * DP * 128);
  GrFactors<CT>& f = *reinterpret_cast<GrFactors<CT>*>(ktl + 2 * DP * 128 + 128);
  __shared__ float cj[CT], nsum[4][128];
  const GrRows& r = p.c.r;
  const int c = blockIdx.x, h = blockIdx.y, g = h / (r.H / r.G), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&B->done[0], 1);
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc(&B->tmem_slot, DP);
  __syncthreads();               // tensor memory is taken before a dependent kernel may start beside this one
  grid_dep_launch();
  grid_dep_wait();
  const int row0 = p.c.chunks[c * 4], L = p.c.chunks[c * 4 + 1];
  gr_load_factors(p.c, c, h, p.st, f);
  if (threadIdx.x < CT) cj[threadIdx.x] = (int)threadIdx.x < L ? gr_pair(f, L - 1, threadIdx.x) : 0.f;
  if (threadIdx.x == 0) p.c.cdecay[(long)c * r.H + h] = gr_carry(f, L - 1);
  __syncthreads();
  const bf16* k = reinterpret_cast<const bf16*>(r.k) + ((long)row0 * r.G + g) * r.d;
  const bf16* v = reinterpret_cast<const bf16*>(r.v) + ((long)row0 * r.H + h) * r.e;
  build_t<true>(kt, ktl, DP, k, (long)r.G * r.d, r.d, L, cj);
  build_t<false>(vt, nullptr, 128, v, (long)r.H * r.e, r.e, L, nullptr);
  operands_ready();
  const uint32_t tmem = B->tmem_slot;
  if (threadIdx.x == 0) {
    constexpr uint32_t idesc = umma_idesc_bf16(128, DP);
    bool acc = false;
    mma_panels(tmem, smem_u32(vt), smem_u32(kt), PANEL, DP * 128, 2, idesc, &acc);
    mma_panels(tmem, smem_u32(vt), smem_u32(ktl), PANEL, DP * 128, 2, idesc, &acc);
    umma_commit(&B->done[0]);
  }
  __syncwarp();
  float* out = p.c.cstate + ((long)c * r.H + h) * r.E * r.d;
  if (r.kind == GR_MEMORY) {     // the sum of the weighted keys, a quarter of the rows per thread
    const int x = threadIdx.x & 127, part = threadIdx.x >> 7;
    float s = 0.f;
    if (x < r.d)
      for (int j = part * 32; j < min(L, part * 32 + 32); ++j) s = fmaf(cj[j], __bfloat162float(k[(long)j * r.G * r.d + x]), s);
    nsum[part][x] = s;
    __syncthreads();
    if (part == 0 && x < r.d) out[(long)r.e * r.d + x] = (nsum[0][x] + nsum[1][x]) + (nsum[2][x] + nsum[3][x]);
  }
  const bool ok = __all_sync(0xffffffffu, mbar_wait(&B->done[0], 0, p.spin_limit));
  tc_fence_after();
  if (!ok) {
    if (lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_MBAR_TIMEOUT);
  } else {
    // four threads per value column (TMEM lane), each a quarter of the d columns (with 64 columns two of them have work)
    const int e = (warp & 3) * 32 + lane, part = warp >> 2;
    float* row = out + (long)e * r.d;
#pragma unroll 1
    for (int c0 = part * 32; c0 < DP; c0 += 128) {
      float a[32];
      tmem_ld_32x32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)c0, a);
      tmem_ld_wait();
      if (e < r.e && r.d % 4 == 0) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (c0 + 4 * i < r.d) *reinterpret_cast<float4*>(row + c0 + 4 * i) = make_float4(a[4 * i], a[4 * i + 1], a[4 * i + 2], a[4 * i + 3]);
      } else if (e < r.e) {
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (c0 + i < r.d) row[c0 + i] = a[i];
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

// ---------------------------------------------------------------------------------------------------------------------------
// outputs. VLO: the values are f32 rows (u), two terms. Shared memory: q, k | the weights (two terms) in their place, the state (two terms), the values
// ---------------------------------------------------------------------------------------------------------------------------
struct OutLayout {
  static constexpr int QK = 0, S = QK + 4 * PANEL, V = S + 4 * PANEL;
};
struct OutSmall {
  GrFactors<CT> f;
  float qn[CT], kn[CT], carry[CT], nrow[128], red[2][4 * CT];
  Bars bars;
};
template <bool VLO>
constexpr int out_smem() { return OutLayout::V + (VLO ? 4 : 2) * PANEL + (int)sizeof(OutSmall) + 1024; }

template <int NP, bool VLO>
__global__ void __launch_bounds__(THREADS, 1) gr_tile_out_kernel(TileParams p) {
  using Y = OutLayout;
  constexpr int DP = 64 * NP;
  constexpr uint32_t W_COL = 0, S_COL = 128, O_COL = 256;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = aligned_smem(smem_raw);
  OutSmall& X = *reinterpret_cast<OutSmall*>(smem + Y::V + (VLO ? 4 : 2) * PANEL);
  Bars* B = &X.bars;
  const GrRows& r = p.c.r;
  const int c = blockIdx.x, h = blockIdx.y, g = h / (r.H / r.G), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&B->done[i], 1);
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc(&B->tmem_slot, 512);
  __syncthreads();               // tensor memory is taken before a dependent kernel may start beside this one
  grid_dep_launch();
  grid_dep_wait();
  const int row0 = p.c.chunks[c * 4], L = p.c.chunks[c * 4 + 1];
  const bf16* q = reinterpret_cast<const bf16*>(r.q) + ((long)row0 * r.G + g) * r.d;
  const bf16* k = reinterpret_cast<const bf16*>(r.k) + ((long)row0 * r.G + g) * r.d;
  unsigned char *Q = smem + Y::QK, *K = Q + 2 * PANEL, *Sm = smem + Y::S, *V = smem + Y::V;
  build_rows<NP>(Q, q, (long)r.G * r.d, r.d, L);
  build_rows<NP>(K, k, (long)r.G * r.d, r.d, L);
  gr_load_factors(p.c, c, h, p.st, X.f);
  operands_ready();
  const uint32_t tmem = B->tmem_slot;
  constexpr uint32_t idesc = umma_idesc_bf16(128, 128);
  if (threadIdx.x == 0) {
    bool acc = false;
    mma_panels(tmem + W_COL, smem_u32(Q), smem_u32(K), PANEL, PANEL, NP, idesc, &acc);
    umma_commit(&B->done[0]);
  }
  __syncwarp();
  // the state ahead of the chunk (rows = value columns), the values, the factors of the rows, while W is computed
  const float* S = p.c.cstate + ((long)c * r.H + h) * r.E * r.d;
#pragma unroll
  for (int u = 0; u < 128 * (DP / 8) / THREADS; ++u) {
    const int i = threadIdx.x + u * THREADS, a = i / (DP / 8), c0 = i % (DP / 8) * 8;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (a < r.e) {
      const float* row = S + (long)a * r.d;
      if (r.d % 4 == 0 && c0 + 8 <= r.d) {
        const float4 x = *reinterpret_cast<const float4*>(row + c0), y = *reinterpret_cast<const float4*>(row + c0 + 4);
        f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
        f[4] = y.x; f[5] = y.y; f[6] = y.z; f[7] = y.w;
      } else {
#pragma unroll
        for (int z = 0; z < 8; ++z)
          if (c0 + z < r.d) f[z] = row[c0 + z];
      }
    }
    uint4 hi, lo;
    split8(f, &hi, &lo);
    *reinterpret_cast<uint4*>(Sm + at(a, c0, 128)) = hi;
    *reinterpret_cast<uint4*>(Sm + 2 * PANEL + at(a, c0, 128)) = lo;
  }
  if (VLO) build_t_f32(V, V + 2 * PANEL, 128, p.u + ((long)row0 * r.H + h) * r.e, (long)r.H * r.e, r.e, L);
  else build_t<false>(V, nullptr, 128, reinterpret_cast<const bf16*>(r.v) + ((long)row0 * r.H + h) * r.e, (long)r.H * r.e, r.e, L, nullptr);
  if (threadIdx.x < CT) {
    const int i = threadIdx.x;
    const long t = row0 + min(i, L - 1);
    X.qn[i] = r.qs ? r.qs[t * r.G + g] : r.q_factor;
    X.kn[i] = r.ks ? r.ks[t * r.G + g] : 1.f;
    X.carry[i] = gr_carry(X.f, min(i, L - 1)) * X.qn[i];
    X.nrow[i] = r.kind == GR_MEMORY && i < r.d ? S[(long)r.e * r.d + i] : 0.f;
  }
  operands_ready();
  if (threadIdx.x == 0) {
    bool acc = false;
    mma_panels(tmem + S_COL, smem_u32(Q), smem_u32(Sm), PANEL, PANEL, NP, idesc, &acc);
    mma_panels(tmem + S_COL, smem_u32(Q), smem_u32(Sm) + 2 * PANEL, PANEL, PANEL, NP, idesc, &acc);
    umma_commit(&B->done[1]);
  }
  __syncwarp();
  // P: four threads per row, 32 columns each
  const int i = (warp & 3) * 32 + lane, part = warp >> 2, c0 = part * 32;
  const uint32_t row_addr = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  // MEMORY: n q = carry (n ahead of the chunk) q + the sum of the row's weights
  float nq = 0.f;
  if (r.kind == GR_MEMORY && c0 < DP) {
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      float f[8];
      unpack8(*reinterpret_cast<const uint4*>(Q + at(i, c0 + 8 * z, 128)), f);
#pragma unroll
      for (int y = 0; y < 8; ++y) nq = fmaf(f[y], X.nrow[c0 + 8 * z + y], nq);
    }
    nq *= X.carry[i];
  }
  bool ok = __all_sync(0xffffffffu, mbar_wait(&B->done[0], 0, p.spin_limit) && mbar_wait(&B->done[1], 0, p.spin_limit));
  __syncthreads();               // q and k are free: both products that read them are complete, and n q was formed
  tc_fence_after();
  if (ok) {
    float a[32];
    tmem_ld_32x32(row_addr + W_COL + (uint32_t)c0, a);
    tmem_ld_wait();
    const double base = X.f.total[i] - (double)X.f.off[i];
    const float qf = X.qn[i];
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      float f[8];
#pragma unroll
      for (int y = 0; y < 8; ++y) {
        const int j = c0 + 8 * z + y;
        f[y] = j <= i && i < L ? a[8 * z + y] * qf * X.kn[j] * X.f.w[j] * __expf((float)(base - X.f.total[j] + (double)X.f.lw[j])) : 0.f;
        nq += f[y];
      }
      uint4 hi, lo;
      split8(f, &hi, &lo);
      *reinterpret_cast<uint4*>(Q + at(i, c0 + 8 * z, 128)) = hi;
      *reinterpret_cast<uint4*>(Q + 2 * PANEL + at(i, c0 + 8 * z, 128)) = lo;
    }
  }
  X.red[0][part * CT + i] = nq;
  operands_ready();
  if (threadIdx.x == 0) {
    const uint32_t w = smem_u32(Q), v = smem_u32(V);
    bool acc = false;
    mma_panels(tmem + O_COL, w, v, PANEL, PANEL, 2, idesc, &acc);
    mma_panels(tmem + O_COL, w + 2 * PANEL, v, PANEL, PANEL, 2, idesc, &acc);
    if (VLO) mma_panels(tmem + O_COL, w, v + 2 * PANEL, PANEL, PANEL, 2, idesc, &acc);
    umma_commit(&B->done[2]);
  }
  __syncwarp();
  nq = (X.red[0][i] + X.red[0][CT + i]) + (X.red[0][2 * CT + i] + X.red[0][3 * CT + i]);
  ok = __all_sync(0xffffffffu, mbar_wait(&B->done[2], 0, p.spin_limit)) && ok;
  tc_fence_after();
  if (!ok && lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_MBAR_TIMEOUT);
  float o[32], u[32];
  tmem_ld_32x32(row_addr + S_COL + (uint32_t)c0, u);
  tmem_ld_32x32(row_addr + O_COL + (uint32_t)c0, o);
  tmem_ld_wait();
  const float carry = X.carry[i];
  float den = 1.f;
  if (r.kind == GR_MEMORY) den = 1.f / (fmaxf(fabsf(nq), expf(-X.f.off[i])) + 1e-6f);
  float ss = 0.f;
#pragma unroll
  for (int z = 0; z < 32; ++z) {
    o[z] = fmaf(carry, u[z], o[z]);
    if (p.y) o[z] *= den;
    if (c0 + z < r.e) ss = fmaf(o[z], o[z], ss);
  }
  const bool live = i < L && ok;
  const long t = row0 + i;
  if (p.y) {
    // the head's rms: the four threads of a row add their sums
    X.red[1][part * CT + i] = ss;
    __syncthreads();
    const float inv = 1.f / sqrtf(((X.red[1][i] + X.red[1][CT + i]) + (X.red[1][2 * CT + i] + X.red[1][3 * CT + i])) / (float)r.e + p.eps);
    if (live) {
      bf16* dst = p.y + t * p.ldy + (long)h * r.e + c0;
      const bf16* gr = p.gate + t * p.ldg + (long)h * r.e + c0;
      const float* gain = p.gain + (long)h * r.e + c0;
      const bool wide = ((r.e | (int)(p.ldy & 7) | (int)(p.ldg & 7)) & 7) == 0 && ((reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.y)) & 15) == 0;
#pragma unroll
      for (int x = 0; x < 32; x += 8) {
        if (c0 + x >= r.e) break;
        float f[8], gt[8];
        if (wide) unpack8(*reinterpret_cast<const uint4*>(gr + x), gt);
#pragma unroll
        for (int z = 0; z < 8; ++z) {
          const bool in = c0 + x + z < r.e;
          if (!wide) gt[z] = in ? to_f32(gr[x + z]) : 0.f;
          f[z] = in ? o[x + z] * inv * gain[x + z] * activate<true>(gt[z], p.gate_act) : 0.f;
        }
        if (wide) {
          *reinterpret_cast<uint4*>(dst + x) = pack8(f);
        } else {
#pragma unroll
          for (int z = 0; z < 8; ++z)
            if (c0 + x + z < r.e) dst[x + z] = __float2bfloat16_rn(f[z]);
        }
      }
    }
  } else if (live) {
    float* dst = p.c.o + t * p.c.ldo + (long)h * r.E + c0;
    if (r.e % 4 == 0 && r.E % 4 == 0 && p.c.ldo % 4 == 0) {
#pragma unroll
      for (int x = 0; x < 32; x += 4)
        if (c0 + x < r.e) *reinterpret_cast<float4*>(dst + x) = make_float4(o[x], o[x + 1], o[x + 2], o[x + 3]);
    } else {
#pragma unroll
      for (int x = 0; x < 32; ++x)
        if (c0 + x < r.e) dst[x] = o[x];
    }
    if (r.kind == GR_MEMORY && part == 0) dst[r.e] = nq;
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// DELTA: the triangular system of a chunk
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int LDA = CT + 1;
struct DeltaSmall {
  GrFactors<CT> f;
  float kn[CT], sv[CT], sk[CT];      // factor of k, of row j's value, of row j's key
  Bars bars;
};
// k rows (then v^T) | T in two terms (the blocks' products meanwhile) | k^T | A, then T, in f32
struct DeltaLayout {
  static constexpr int K = 0, T = K + 2 * PANEL, KT = T + 4 * PANEL, A = KT + 2 * PANEL, SMALL = A + (CT * LDA * 4 + 15) / 16 * 16;
  static constexpr int SMEM = SMALL + (int)sizeof(DeltaSmall) + 1024;
};
static_assert(DeltaLayout::SMEM <= 227 * 1024, "shared memory of the triangular system");
__host__ __device__ constexpr int image_bytes(int np) { return 2 * np * PANEL + 2 * PANEL; }      // two terms of T (b g k), k^T

template <int NP>
__global__ void __launch_bounds__(THREADS, 1) gr_tile_delta_kernel(TileParams p) {
  using Y = DeltaLayout;
  constexpr int DP = 64 * NP;
  constexpr uint32_t G_COL = 0, U_COL = 128, W_COL = 256;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = aligned_smem(smem_raw);
  unsigned char *K = smem + Y::K, *T = smem + Y::T, *KT = smem + Y::KT;
  float* a = reinterpret_cast<float*>(smem + Y::A);
  float* tmp = reinterpret_cast<float*>(T);
  DeltaSmall& X = *reinterpret_cast<DeltaSmall*>(smem + Y::SMALL);
  Bars* B = &X.bars;
  const GrRows& r = p.c.r;
  const int c = blockIdx.x, h = blockIdx.y, g = h / (r.H / r.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&B->done[i], 1);
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc(&B->tmem_slot, 512);
  __syncthreads();               // tensor memory is taken before a dependent kernel may start beside this one
  grid_dep_launch();
  grid_dep_wait();
  const int row0 = p.c.chunks[c * 4], L = p.c.chunks[c * 4 + 1];
  const bf16* k = reinterpret_cast<const bf16*>(r.k) + ((long)row0 * r.G + g) * r.d;
  build_rows<NP>(K, k, (long)r.G * r.d, r.d, L);
  gr_load_factors(p.c, c, h, p.st, X.f);
  operands_ready();
  const uint32_t tmem = B->tmem_slot;
  constexpr uint32_t idesc = umma_idesc_bf16(128, 128);
  if (tid == 0) {
    bool acc = false;
    mma_panels(tmem + G_COL, smem_u32(K), smem_u32(K), PANEL, PANEL, NP, idesc, &acc);
    umma_commit(&B->done[0]);
  }
  __syncwarp();
  if (tid < CT) {
    const float kn = r.ks ? r.ks[(long)(row0 + min(tid, L - 1)) * r.G + g] : 1.f;
    X.kn[tid] = kn;
    X.sv[tid] = X.f.w[tid];
    X.sk[tid] = X.f.w[tid] * kn * expf((float)X.f.total[tid]);
  }
  build_t<false>(KT, nullptr, 128, k, (long)r.G * r.d, r.d, L, nullptr);
  const int i = (warp & 3) * 32 + lane, part = warp >> 2, c0 = part * 32;
  const uint32_t row_addr = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  bool ok = __all_sync(0xffffffffu, mbar_wait(&B->done[0], 0, p.spin_limit));
  __syncthreads();
  tc_fence_after();
  if (ok) {
    float v[32];
    tmem_ld_32x32(row_addr + G_COL + (uint32_t)c0, v);
    tmem_ld_wait();
    const double total = X.f.total[i];
    const float wi = X.f.w[i] * X.kn[i];
#pragma unroll
    for (int z = 0; z < 32; ++z) {
      const int j = c0 + z;
      a[i * LDA + j] = j < i && i < L ? v[z] * wi * X.kn[j] * __expf((float)(total - X.f.total[j])) : 0.f;
    }
  }
  __syncthreads();
  {   // the diagonal blocks of 16 rows: a column of the inverse per thread, in place
    float x[16];
    const int b0 = tid & ~15, col = tid & 15;
    if (tid < CT) {
#pragma unroll
      for (int y = 0; y < 16; ++y) {
        float v = y == col ? 1.f : 0.f;
#pragma unroll
        for (int j = 0; j < y; ++j) v = fmaf(-a[(b0 + y) * LDA + b0 + j], x[j], v);
        x[y] = v;
      }
    }
    __syncthreads();
    if (tid < CT) {
#pragma unroll
      for (int y = 0; y < 16; ++y) a[(b0 + y) * LDA + b0 + col] = x[y];
    }
  }
#pragma unroll
  for (int s = 16; s < CT; s *= 2) {      // two inverted blocks of s rows and what lies below the first: -T22 (A21 T11); 2 x 2 values per thread
    const int pairs = CT / (2 * s), per = s / 2;
    __syncthreads();
    for (int n = tid; n < pairs * per * per; n += THREADS) {
      const int b = n / (per * per), y = n / per % per * 2, x = n % per * 2, r0 = 2 * s * b;
      float v[2][2] = {};
      for (int z = x; z < s; ++z) {
        const float a0 = a[(r0 + s + y) * LDA + r0 + z], a1 = a[(r0 + s + y + 1) * LDA + r0 + z], b0 = a[(r0 + z) * LDA + r0 + x], b1 = a[(r0 + z) * LDA + r0 + x + 1];
        v[0][0] = fmaf(a0, b0, v[0][0]);
        v[0][1] = fmaf(a0, b1, v[0][1]);
        v[1][0] = fmaf(a1, b0, v[1][0]);
        v[1][1] = fmaf(a1, b1, v[1][1]);
      }
      float* d = tmp + (long)b * s * (s + 1);
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int o = 0; o < 2; ++o) d[(y + m) * (s + 1) + x + o] = v[m][o];
    }
    __syncthreads();
    for (int n = tid; n < pairs * per * per; n += THREADS) {
      const int b = n / (per * per), y = n / per % per * 2, x = n % per * 2, r0 = 2 * s * b;
      const float* d = tmp + (long)b * s * (s + 1);
      float v[2][2] = {};
      for (int z = 0; z <= y + 1; ++z) {
        const float a0 = z <= y ? a[(r0 + s + y) * LDA + r0 + s + z] : 0.f, a1 = a[(r0 + s + y + 1) * LDA + r0 + s + z], b0 = d[z * (s + 1) + x], b1 = d[z * (s + 1) + x + 1];
        v[0][0] = fmaf(a0, b0, v[0][0]);
        v[0][1] = fmaf(a0, b1, v[0][1]);
        v[1][0] = fmaf(a1, b0, v[1][0]);
        v[1][1] = fmaf(a1, b1, v[1][1]);
      }
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int o = 0; o < 2; ++o) a[(r0 + s + y + m) * LDA + r0 + x + o] = -v[m][o];
    }
  }
  __syncthreads();
  // T times the scaled values, then the scaled keys: the factors go into the columns of T
  unsigned char* VT = K;
  build_t<false>(VT, nullptr, 128, reinterpret_cast<const bf16*>(r.v) + ((long)row0 * r.H + h) * r.e, (long)r.H * r.e, r.e, L, nullptr);
  for (int round = 0; round < 2; ++round) {
    const float* scale = round ? X.sk : X.sv;
    if (round) {
      ok = __all_sync(0xffffffffu, mbar_wait(&B->done[1], 0, p.spin_limit)) && ok;
      __syncthreads();           // the first product has read T
    }
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      float f[8];
#pragma unroll
      for (int y = 0; y < 8; ++y) {
        const int j = c0 + 8 * z + y;
        f[y] = j <= i && j < L ? a[i * LDA + j] * scale[j] : 0.f;
      }
      uint4 hi, lo;
      split8(f, &hi, &lo);
      *reinterpret_cast<uint4*>(T + at(i, c0 + 8 * z, 128)) = hi;
      *reinterpret_cast<uint4*>(T + 2 * PANEL + at(i, c0 + 8 * z, 128)) = lo;
    }
    operands_ready();
    if (tid == 0) {
      const uint32_t x = smem_u32(T), b = smem_u32(round ? KT : VT), d = tmem + (round ? W_COL : U_COL);
      bool acc = false;
      mma_panels(d, x, b, PANEL, PANEL, 2, idesc, &acc);
      mma_panels(d, x + 2 * PANEL, b, PANEL, PANEL, 2, idesc, &acc);
      umma_commit(&B->done[1 + round]);
    }
    __syncwarp();
  }
  unsigned char* image = p.images + ((long)c * r.H + h) * image_bytes(NP);
  // k^T as it lies here
  for (int n = tid; n < 2 * PANEL / 16; n += THREADS) reinterpret_cast<uint4*>(image + 2 * NP * PANEL)[n] = reinterpret_cast<const uint4*>(KT)[n];
  ok = __all_sync(0xffffffffu, mbar_wait(&B->done[2], 0, p.spin_limit)) && ok;
  tc_fence_after();
  if (!ok && lane == 0 && p.status) atomicOr(p.status, IFAB_STATUS_MBAR_TIMEOUT);
  float v[32];
  tmem_ld_32x32(row_addr + U_COL + (uint32_t)c0, v);
  tmem_ld_wait();
  if (i < L && ok) {
    float* dst = p.u + ((long)(row0 + i) * r.H + h) * r.e + c0;
    if (r.e % 4 == 0) {
#pragma unroll
      for (int x = 0; x < 32; x += 4)
        if (c0 + x < r.e) *reinterpret_cast<float4*>(dst + x) = make_float4(v[x], v[x + 1], v[x + 2], v[x + 3]);
    } else {
#pragma unroll
      for (int x = 0; x < 32; ++x)
        if (c0 + x < r.e) dst[x] = v[x];
    }
  }
  __syncwarp();
  if (c0 < DP) {
    tmem_ld_32x32(row_addr + W_COL + (uint32_t)c0, v);
    tmem_ld_wait();
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      float f[8];
#pragma unroll
      for (int y = 0; y < 8; ++y) f[y] = ok && c0 + 8 * z + y < r.d ? v[8 * z + y] : 0.f;
      uint4 hi, lo;
      split8(f, &hi, &lo);
      *reinterpret_cast<uint4*>(image + at(i, c0 + 8 * z, 128)) = hi;
      *reinterpret_cast<uint4*>(image + NP * PANEL + at(i, c0 + 8 * z, 128)) = lo;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// DELTA: over the chunks of a sequence. 256 threads: two per TMEM lane (a row of the chunk, then a key column of the state), half of the value columns each
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int EN = 32, EH = EN / 2;              // value columns of a CTA, of a thread
struct ScanSmall {
  double last[8];                                // scratch of the running sums
  uint64_t full[2], done[2];
  uint32_t tmem_slot;
};
template <int NP>
struct ScanLayout {
  static constexpr int IMG = 0, S = IMG + 2 * image_bytes(NP), U = S + 2 * NP * EN * 128, SMALL = U + 2 * 2 * EN * 128, SMEM = SMALL + (int)sizeof(ScanSmall) + 1024;
};
static_assert(ScanLayout<2>::SMEM <= 227 * 1024, "shared memory of the scan");

// a copy of `bytes` (a multiple of 16) from global memory into this CTA's shared memory
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
// 16 consecutive f32 columns of a thread's TMEM lane (tc_common.cuh has the form of 32)
__device__ __forceinline__ void tmem_ld_32x16(uint32_t taddr, float* v) {
  uint32_t* r = reinterpret_cast<uint32_t*>(v);
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]),
                 "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
               : "r"(taddr)
               : "memory");
}
__device__ __forceinline__ void tmem_st_32x16(uint32_t taddr, const float* v) {
  const uint32_t* r = reinterpret_cast<const uint32_t*>(v);
  asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr), "r"(r[0]), "r"(r[1]),
               "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
               : "memory");
}

// grid (ceil(e / EN), H, n): CTAs of a run's first chunk walk its chunks
template <int NP>
__global__ void __launch_bounds__(256, 1) gr_tile_scan_kernel(TileParams p) {
  using Y = ScanLayout<NP>;
  constexpr uint32_t U_COL = 0, S_COL = 32;
  constexpr int IMAGE = image_bytes(NP);
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = aligned_smem(smem_raw);
  unsigned char *Ss = smem + Y::S, *Us = smem + Y::U;
  ScanSmall& X = *reinterpret_cast<ScanSmall*>(smem + Y::SMALL);
  const GrRows& r = p.c.r;
  const int first = blockIdx.z, h = blockIdx.y, g = h / (r.H / r.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int quarter = warp & 3, half = warp >> 2, row = quarter * 32 + lane, e0 = blockIdx.x * EN + half * EH, ne = min(EH, max(r.e - e0, 0));
  grid_dep_wait();
  const int meta = p.c.chunks[first * 4 + 3], count = meta >> 1, slot = p.c.chunks[first * 4 + 2];
  if (!(meta & 1)) return;
  if (tid == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&X.full[i], 1);
      mbar_init(&X.done[i], 1);
    }
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc(&X.tmem_slot, 64);
  __syncthreads();               // tensor memory is taken before a dependent kernel may start beside this one
  grid_dep_launch();
  const uint32_t tmem = X.tmem_slot, mine = tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(half * EH);
  const bool fresh = p.c.positions[p.c.chunks[first * 4]] == 0;
  float* state = p.st.s + (((long)slot * r.H + h) * r.E + e0) * r.d;
  auto load = [&](int c) {
    const int b = (c - first) & 1;
    mbar_expect_tx(&X.full[b], IMAGE);
    bulk_load(smem + Y::IMG + b * IMAGE, p.images + ((long)c * r.H + h) * IMAGE, IMAGE, &X.full[b]);
  };
  int issued = min(count, 2);
  bool ok = true;
  if (tid == 0) {
    load(first);
    if (count > 1) load(first + 1);
  }
  // what this thread's row of a chunk brings: its part of T (b v), its log decay, the factor of its key
  struct Row {
    float u[EH], log_decay, kn;
    float* at;
    bool live;
  };
  auto fetch = [&](int c, Row& x) {
    const int row0 = p.c.chunks[c * 4], L = p.c.chunks[c * 4 + 1];
    x.live = row < L;
    const long t = row0 + (x.live ? row : 0);
    x.at = p.u + (t * r.H + h) * r.e + e0;
    x.log_decay = x.live ? r.log_decay[t * r.H + h] : 0.f;
    x.kn = x.live && r.ks ? r.ks[t * r.G + g] : 1.f;
    if (r.e % 4 == 0) {
#pragma unroll
      for (int i = 0; i < EH; i += 4) {
        const float4 v = x.live && i < ne ? *reinterpret_cast<const float4*>(x.at + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        x.u[i] = v.x; x.u[i + 1] = v.y; x.u[i + 2] = v.z; x.u[i + 3] = v.w;
      }
    } else {
#pragma unroll
      for (int i = 0; i < EH; ++i) x.u[i] = x.live && i < ne ? x.at[i] : 0.f;
    }
  };
  float s[EH];
#pragma unroll
  for (int i = 0; i < EH; ++i) s[i] = (i < ne && row < r.d && !fresh) ? state[(long)i * r.d + row] : 0.f;
  Row next;
  fetch(first, next);
  constexpr uint32_t idesc = umma_idesc_bf16(128, EN);
  for (int n = 0; n < count && ok; ++n) {
    const int c = first + n, b = n & 1;
    Row x = next;
    // running sums of the log decays
    double total = (double)x.log_decay;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double y = __shfl_up_sync(0xffffffffu, total, o);
      if (lane >= o) total += y;
    }
    if (lane == 31) X.last[warp] = total;
    // this thread's key column of the state ahead of the chunk, in two terms
    if (row < 64 * NP) {
#pragma unroll
      for (int i = 0; i < EH; ++i) put2(Ss, Ss + NP * EN * 128, at(half * EH + i, row, EN), s[i]);
    }
    operands_ready();
    unsigned char* img = smem + Y::IMG + b * IMAGE;
    if (tid == 0 && mbar_wait(&X.full[b], (n >> 1) & 1, p.spin_limit)) {
      tc_fence_after();
      const uint32_t w = smem_u32(img), sb = smem_u32(Ss);
      bool acc = false;
      mma_panels(tmem + U_COL, w, sb, PANEL, EN * 128, NP, idesc, &acc);
      mma_panels(tmem + U_COL, w, sb + NP * EN * 128, PANEL, EN * 128, NP, idesc, &acc);
      mma_panels(tmem + U_COL, w + NP * PANEL, sb, PANEL, EN * 128, NP, idesc, &acc);
      umma_commit(&X.done[0]);
    }
    __syncwarp();
    if (n + 1 < count) fetch(c + 1, next);
    // the state ahead of the chunk for the outputs; as it enters the sum: decayed
    float* ahead = p.c.cstate + (((long)c * r.H + h) * r.E + e0) * r.d;
    double all = 0.0;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const double y = X.last[half * 4 + w];
      if (w < quarter) total += y;
      all += y;
    }
    const float carry = expf((float)all), tail = x.live ? expf((float)(all - total)) * x.kn : 0.f;
#pragma unroll
    for (int i = 0; i < EH; ++i) {
      if (i < ne && row < r.d) ahead[(long)i * r.d + row] = s[i];
      s[i] *= carry;
    }
    tmem_st_32x16(mine + S_COL, s);
    tmem_st_wait();
    ok = __all_sync(0xffffffffu, mbar_wait(&X.done[0], n & 1, p.spin_limit));
    tc_fence_after();
    float wv[EH];
    tmem_ld_32x16(mine + U_COL, wv);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < EH; ++i) {
      x.u[i] -= wv[i];
      put2(Us, Us + 2 * EN * 128, at(half * EH + i, row, EN), x.u[i] * tail);
    }
    ok = __syncthreads_and(ok);      // all warps leave the loop together
    if (!ok) break;
    operands_ready();
    if (tid == 0) {
      const uint32_t kt = smem_u32(img + 2 * NP * PANEL), ub = smem_u32(Us);
      bool acc = true;
      mma_panels(tmem + S_COL, kt, ub, PANEL, EN * 128, 2, idesc, &acc);
      mma_panels(tmem + S_COL, kt, ub + 2 * EN * 128, PANEL, EN * 128, 2, idesc, &acc);
      umma_commit(&X.done[1]);
    }
    __syncwarp();
    if (x.live) {
      if (r.e % 4 == 0) {
#pragma unroll
        for (int i = 0; i < EH; i += 4)
          if (i < ne) *reinterpret_cast<float4*>(x.at + i) = make_float4(x.u[i], x.u[i + 1], x.u[i + 2], x.u[i + 3]);
      } else {
#pragma unroll
        for (int i = 0; i < EH; ++i)
          if (i < ne) x.at[i] = x.u[i];
      }
    }
    ok = __all_sync(0xffffffffu, mbar_wait(&X.done[1], n & 1, p.spin_limit));
    tc_fence_after();
    tmem_ld_32x16(mine + S_COL, s);
    tmem_ld_wait();
    ok = __syncthreads_and(ok);      // the products have read this chunk's image
    if (ok && n + 2 < count) {
      if (tid == 0) load(c + 2);
      ++issued;
    }
  }
  if (!ok) {
    if (tid == 0) {
      if (p.status) atomicOr(p.status, IFAB_STATUS_MBAR_TIMEOUT);
      for (int i = max(0, issued - 2); i < issued; ++i) mbar_wait(&X.full[i & 1], (i >> 1) & 1, p.spin_limit);      // copies must land before the CTA may exit
    }
  } else {
#pragma unroll
    for (int i = 0; i < EH; ++i)
      if (i < ne && row < r.d) state[(long)i * r.d + row] = s[i];
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 64);
  }
}

template <typename K>
int run(K kernel, dim3 grid, int threads, size_t smem, cudaStream_t s, const TileParams& p) {
  if (int rc = opt_in_smem(kernel, smem)) return rc;
  return launch_chain(kernel, grid, dim3(threads), smem, s, p);
}

template <int NP>
int tiles(const TileParams& p, cudaStream_t s) {
  const GrRows& r = p.c.r;
  const int n = p.c.n;
  if (r.kind == GR_DELTA) {
    if (int rc = run(gr_tile_delta_kernel<NP>, dim3(n, r.H), THREADS, DeltaLayout::SMEM, s, p)) return rc;
    if (int rc = run(gr_tile_scan_kernel<NP>, dim3((r.e + EN - 1) / EN, r.H, n), 256, ScanLayout<NP>::SMEM, s, p)) return rc;
    TileParams o = p;
    o.c.r.weight = nullptr;      // corrected values count once
    return run(gr_tile_out_kernel<NP, true>, dim3(n, r.H), THREADS, out_smem<true>(), s, o);
  }
  if (r.kind == GR_MEMORY)
    if (int rc = gr_maximum(p.c, p.st, s)) return rc;
  const size_t smem = 2 * PANEL + 4 * 64 * NP * 128 + 128 + sizeof(GrFactors<CT>) + 1024;
  if (int rc = run(gr_tile_state_kernel<NP>, dim3(n, r.H), THREADS, smem, s, p)) return rc;
  if (int rc = gr_scan(p.c, p.st, s)) return rc;
  return run(gr_tile_out_kernel<NP, false>, dim3(n, r.H), THREADS, out_smem<false>(), s, p);
}

static_assert(out_smem<true>() <= 227 * 1024, "shared memory of the outputs");

}  // namespace

// bf16 rows; d, e <= 128; chunks of at most 128 rows. Heads as f32 rows o [T, H * E], or - y given, not for SSD - as the normed, gated operand y [T, H * e]. DELTA: u
// f32 [T, H, e] and images, 65536 (d <= 64) or 98304 bytes per chunk and head
extern "C" int ifab_gr_tiles(const void* q, const void* k, const void* v, const float* qs, const float* ks, float q_factor, const float* log_decay, const float* weight,
                             int kind, int H, int G, int d, int e, const int32_t* chunks, int n, const int32_t* positions, float* cstate, uint64_t cstate_bytes,
                             float* cdecay, float* u, void* images, uint64_t image_bytes_given, float* state, float* m_state, const int32_t* epoch, float* m_rows,
                             float* o, long ldo, const void* gate, long ldg, int gate_act, const float* gain, float eps, void* y, long ldy, uint32_t* status,
                             void* stream) {
  const int E = e + (kind == GR_MEMORY);
  if (n < 1 || n > 65535 || kind < GR_SSD || kind > GR_MEMORY || H < 1 || H > 65535 || G < 1 || H % G || d < 1 || d > 128 || e < 1 || e > 128) return -1;
  if ((!y && !o) || (y && (!gate || !gain || kind == GR_SSD)) || (kind == GR_MEMORY && (!m_state || !epoch || !m_rows)) || (kind == GR_DELTA && (!u || !images))) return -1;
  if ((uint64_t)n * H * d * E * sizeof(float) > cstate_bytes || (kind == GR_DELTA && (uint64_t)n * H * image_bytes(d <= 64 ? 1 : 2) > image_bytes_given)) return -5;
  if (kind == GR_DELTA && (reinterpret_cast<uintptr_t>(images) & 15)) return -1;
  TileParams p{};
  p.c = GrChunks{{q, k, v, qs, ks, q_factor, log_decay, weight, m_rows, kind, H, G, d, e, E}, chunks, n, positions, cstate, cdecay, o, ldo};
  p.st = GrState{state, m_state, epoch};
  p.gate = (const bf16*)gate; p.ldg = ldg; p.gate_act = gate_act; p.gain = gain; p.eps = eps; p.y = (bf16*)y; p.ldy = ldy;
  p.u = u; p.images = (unsigned char*)images; p.status = status; p.spin_limit = 4000000u;
  return d <= 64 ? tiles<1>(p, (cudaStream_t)stream) : tiles<2>(p, (cudaStream_t)stream);
}
