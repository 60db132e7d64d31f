/* C ABI of the sm_100a kernel library (libifab_kernels.so).
 *
 * Every entry point takes raw device pointers plus a CUDA stream handle and returns 0 on success,
 * a negative value for a rejected argument, or a positive cudaError_t from the launch. Nothing here
 * allocates device memory except the functions in the "fabric" group, which own the symmetric heap.
 * All matrices are row-major; weights are [out_features, in_features] with in_features contiguous.
 */
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define IFAB_MAX_RANKS 8

/* Symmetric-heap descriptor of one rank (host struct, passed by pointer). data[r]/flags[r] are rank
 * r's staging area and flag words as mapped into this process; entries >= world are ignored. */
typedef struct IfabFabric {
  void* data[IFAB_MAX_RANKS];
  uint64_t* flags[IFAB_MAX_RANKS];
  uint64_t* seq;      /* local: number of fused-collective launches completed */
  uint32_t* done;     /* local: CTA ticket counter of the running launch */
  uint32_t* status;   /* local: IFAB_STATUS_* bits, sticky until the host clears them */
  int32_t rank;
  int32_t world;
  uint32_t spin_limit;
  uint32_t data_half_bytes;
  uint32_t flag_half_words;
  uint32_t ll_half_bytes;  /* one parity half of the tagged-store area (8 bytes per exchanged f32) */
  uint64_t ll_offset;      /* byte offset of that area from data[r]; it is used by nothing else, because a
                              reader takes any 8-byte word whose high half equals the call number as valid */
  void* mc;                /* NVLink multicast address of the same block (a store to it lands in every rank's copy, a
                              multimem.ld_reduce returns the sum over the ranks), or NULL: plain peer loads / stores */
} IfabFabric;

/* ---- fabric: symmetric heap over CUDA IPC (one process per GPU) ---- */
int ifab_device_alloc(void** out, uint64_t bytes);           /* cudaMalloc + zero fill */
int ifab_device_free(void* p);
int ifab_ipc_export(void* p, unsigned char handle[64]);      /* cudaIpcGetMemHandle */
int ifab_ipc_import(const unsigned char handle[64], void** out);
int ifab_ipc_close(void* p);
int ifab_set_device(int device);
int ifab_peek(void* dst_host, const void* src_device, uint64_t bytes);   /* synchronous small copies of */
int ifab_poke(void* dst_device, const void* src_host, uint64_t bytes);   /* control words               */
const char* ifab_error_string(int code);

/* ---- elementwise / layout ---- */
int ifab_embedding_bf16(const int32_t* ids, const void* table, void* out, int T, int D, int vocab, uint32_t* status,
                        void* stream);
int ifab_rmsnorm_bf16(const void* x, long ldx, const void* w, void* y, long ldy, int T, int D, float eps,
                      int zero_centered, void* stream);

/* ---- decode linears (T <= 8 per tile; larger T loops over tiles) ---- */
int ifab_gemv_bf16(const void* x, long ldx, const void* w, const void* norm_w, float eps, int zero_centered,
                   const void* residual, long ldr, void* y, long ldy, int out_f32, int T, int N, int K, int mode,
                   void* stream);
int ifab_gemv_allreduce_bf16(const void* x, long ldx, const void* w, const void* residual, long ldr, void* y, long ldy,
                             void* y_f32, int T, int N, int K, const IfabFabric* fab, void* stream);

/* ---- block-scaled fp8 (e4m3, one f32 scale per 1 x 128 block of a row) expert weights (decode_moe_fp8.cu) ---- */
/* w: bf16 [rows, K] (row stride ldw) -> q: u8 [rows, K], scales: f32 [rows, ceil(K / 128)] */
int ifab_quantize_fp8_block(const void* w, long ldw, long rows, int K, void* q, float* scales, void* stream);
/* the inverse, rounded to bf16 -> out: bf16 [rows, K] contiguous; K % 16 == 0 (the prompt path widens one layer's experts at a time) */
int ifab_dequantize_fp8_block(const void* q, const float* scales, long rows, int K, void* out, void* stream);
int ifab_moe_gate_up_decode_fp8(const void* x, long ldx, const void* norm_w, float eps, const int32_t* ids, int T, int D, int F, int topk, int e0,
                                int e_local, const void* w_gu, const float* s_gu, const void* w_shared_gu, const float* s_shared_gu, int Fs, void* act,
                                void* stream);
int ifab_moe_down_allreduce_decode_fp8(const void* act, const int32_t* ids, const float* wts, int T, int D, int F, int topk, int e0, int e_local,
                                       const void* w_down, const float* s_down, const void* w_shared_down, const float* s_shared_down, int Fs,
                                       const void* residual, long ldr, void* y, long ldy, const IfabFabric* fab, void* stream);

/* ---- tensor-core GEMM (tcgen05 + TMEM + TMA): C[M,N] = A[M,K] * B[N,K]^T (+ residual) ---- */
int ifab_gemm_bf16(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual,
                   long ldr, int M, int N, int K, uint32_t* status, void* stream);
/* the same with an activation of the result in the epilogue: 0 none, 1 SiLU, 2 sigmoid, 3 GELU (tanh form) */
int ifab_gemm_act_bf16(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual, long ldr, int act,
                       int M, int N, int K, uint32_t* status, void* stream);
int ifab_gemm_act_bf16_2sm(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual, long ldr, int act,
                           int persistent, int M, int N, int K, uint32_t* status, void* stream);
/* the same with a bias [N] (f32, or null) and, for cap > 0, a soft limit cap tanh(result / cap) after the activation */
int ifab_gemm_epilogue_bf16(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual, long ldr, const float* bias,
                            int act, float cap, int M, int N, int K, uint32_t* status, void* stream);
int ifab_gemm_epilogue_bf16_2sm(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual, long ldr,
                                const float* bias, int act, float cap, int persistent, int M, int N, int K, uint32_t* status, void* stream);
/* f32 parts of A * B^T + bias along K for M <= 128 rows, part_stride apart; their sum is the product */
int ifab_gemm_split_bf16(const void* a, long lda, const void* b, long ldb, float* c, long ldc, long part_stride, int parts, const float* bias, int M, int N, int K,
                         uint32_t* status, void* stream);
/* first half of a gated feed-forward, any number of rows: b = [gate rows | up rows] ([2F, K]), c[M, F] = unit(a gate^T, a up^T). Units: 0 silu(g) u,
 * 1 relu(g) u, 2 g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit), u' = u within [-limit, limit] */
int ifab_gemm_gated_bf16(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int unit, float limit, float alpha, int M, int F, int K,
                         uint32_t* status, void* stream);
int ifab_gemm_gated_bf16_2sm(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int unit, float limit, float alpha, int M, int F, int K,
                             uint32_t* status, void* stream);
/* C = act(A * B^T + bias) in true f32, softly limited for cap > 0 */
int ifab_linear_f32(const float* a, long lda, const float* b, long ldb, float* c, long ldc, const float* bias, float cap, int M, int N, int K, int act, void* stream);
/* n products at strides sa, sb, sc; and products grouped by the tile table of ifab_moe_dispatch (rows of A through `index` when given; pair: A is
 * [gate | up], taken as the gated unit of that number) */
int ifab_linear_f32_batched(const float* a, long lda, long sa, const float* b, long ldb, long sb, float* c, long ldc, long sc, int n, int M, int N, int K,
                            void* stream);
int ifab_grouped_linear_f32(const float* a, long lda, const int32_t* index, int pair, int unit, float limit, float alpha, const float* b, int N,
                            int K, const int32_t* tiles, const int32_t* num_tiles, int max_tiles, int rows, float* c, long ldc, void* stream);
/* one product per head, heads side by side in the rows of A and C: C[t, h * c_stride + n] = sum_k A[t, h * a_stride + k] B[h, n, k] (tcgen05) */
int ifab_gemm_heads_bf16(const void* a, long lda, int a_stride, const void* b, long ldb, void* c, long ldc, int c_stride, int out_f32, int heads, int M, int N,
                         int K, uint32_t* status, void* stream);

/* the same on CTA pairs (tcgen05.mma cta_group::2, 256 x 256 tiles, each CTA loads half of A and half of B); N % 32 == 0 */
int ifab_gemm_bf16_2sm(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual,
                       long ldr, int M, int N, int K, uint32_t* status, void* stream);

/* CTA pairs, persistent grid (one pair per SM pair), two accumulators in tensor memory: the epilogue of a tile runs under the next tile's MMAs */
int ifab_gemm_bf16_2sm_persistent(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int out_f32, const void* residual,
                                  long ldr, int M, int N, int K, uint32_t* status, void* stream);

/* packed gate / up projection of a SwiGLU block on CTA pairs: b = [gate rows | up rows] ([2F, K]), c[M, F] = silu(a gate^T) * (a up^T) */
int ifab_gemm_swiglu_bf16_2sm(const void* a, long lda, const void* b, long ldb, void* c, long ldc, int M, int F, int K, uint32_t* status,
                              void* stream);

int ifab_gemm_allreduce_bf16(const void* a, long lda, const void* b, long ldb, void* const* out_peers, long ldc, const void* residual,
                             long ldr, int M, int N, int K, const IfabFabric* fab, void* stream);

/* column-parallel GEMM fused with the all-gather of its row-sharded activations: C[world*rows_local, N] = gather(A_r) * B^T.
 * a_peers[r] = rank r's [rows_local, K] shard in symmetric memory as mapped here (remote tiles are copied once with peer
 * loads into `staged` [M, K] and then read by TMA; no multicast); flag_peers[r] = rank r's u64[8] flag row; tile_count =
 * local u64 [M / 128], zeroed once; `epoch` starts at 1 and grows by one per call; alternate two A buffers. */
int ifab_allgather_gemm_bf16(void* const* a_peers, long lda, const void* b, long ldb, void* c, long ldc, int rows_local, int N,
                             int K, int world, int rank, void* const* flag_peers, void* staged, long lds, void* tile_count,
                             uint64_t epoch, uint32_t* status, void* stream);

/* ---- prefill path: grouped expert GEMM (tcgen05) and its routing plumbing; all sizes are device-side counts ---- */
/* mode 0: C[rows, N] = A . B[e]^T; mode 1: N = 2F (gate rows then up rows), C[rows, F] = silu(gate) * up.
 * tiles: max_tiles x int4 {expert, first row, valid rows, 0}; *num_tiles of them are valid (written by ifab_moe_dispatch). */
int ifab_grouped_gemm_bf16(const void* a, long lda, int rows_max, const void* b, int experts, int N, int K,
                           const int32_t* tiles, const int32_t* num_tiles, int max_tiles, void* c, long ldc, int mode,
                           uint32_t* status, void* stream);
int ifab_grouped_gemm_gated_bf16(const void* a, long lda, int rows_max, const void* b, int experts, int N, int K, const int32_t* tiles, const int32_t* num_tiles,
                                 int max_tiles, void* c, long ldc, int mode, int unit, float limit, float alpha, uint32_t* status, void* stream);
/* router for any number of rows (blocks of 8 per CTA); xn (optional) receives the RMS-normalised rows */
int ifab_router_block(const void* x, long ldx, const void* norm_w, float eps, const float* w_router, const float* bias,
                      float* logits, int32_t* ids, float* wts, void* xn, long ldxn, int M, int D, int E, int topk,
                      int scoring, int renorm, float scale, void* stream);
int ifab_moe_dispatch(const int32_t* ids, int M, int topk, int e0, int e_local, int32_t* counts, int32_t* route_row,
                      int32_t* perm_token, int32_t* tiles, int32_t* num_tiles, int32_t* total_rows, int max_tiles,
                      void* stream);
int ifab_moe_gather(const void* xn, long ldxn, const int32_t* perm_token, const int32_t* total_rows, void* xp, long ldxp,
                    int D, int rows_max, void* stream);
int ifab_moe_combine(const void* y, long ldy, const int32_t* route_row, const float* wts, int M, int topk, int D,
                     const void* shared, long lds, const void* residual, long ldr, float* out_f32, void* out, long ldo,
                     void* stream);
int ifab_mla_q_rope(const void* q, long ldq, const int32_t* positions, void* q_lat, int T, int H, int nope, int rope,
                    float theta, void* stream);
int ifab_mla_merge(const float* scratch, const int32_t* positions, int n_sinks, int window, int keys_per_split,
                   int max_splits, int T, int H, void* o_lat, void* stream);
/* one-shot pull all-reduce of f32 [rows, D] partials held in symmetric memory (parts[r] = rank r's buffer as mapped here),
 * + residual, bf16 out. The caller alternates two sets of partial buffers between consecutive calls. */
/* ---- prompt attention on the tensor cores (tcgen05): one sequence, consecutive positions, causal (+ sliding window) ----
 * q: [m, ...] head h at columns h * q_head_stride + [0, d1 + d2); k: [ctx, ...] key head g = h / kv_group at columns
 * g * k_head_stride + [0, d1); k2: [ctx, d2] key columns shared by all heads (NULL when d2 = 0); vt: transposed values, key head g
 * at rows g * vt_head_stride + vt_row0 + [0, 128), one column per key (ldvt >= ctx); out: [m, H * 128].
 * d1 in {64, 128}, d2 in {0, 64}; rows of q are positions pos0 .. pos0 + m - 1 and pos0 + m <= ctx. */
int ifab_fa_prefill_bf16(const void* q, long ldq, int q_head_stride, const void* k, long ldk, int k_head_stride, const void* k2, long ldk2,
                         const void* vt, long ldvt, int vt_head_stride, int vt_row0, int vt_rows, void* out, long ldo, int m, int ctx, int H,
                         int kv_group, int d1, int d2, int pos0, int window, float scale, uint32_t* status, void* stream);
int ifab_mla_q_rope_inplace(void* q, long ldq, const int32_t* positions, int T, int H, int nope, int rope, float theta, void* stream);
int ifab_mla_ctx_gather(const void* cache, const int32_t* page_table, int slot, int max_pages, int page_tokens, int num_pages, int ctx,
                        int rows, void* lat, void* pe, uint32_t* status, void* stream);
int ifab_allreduce_rows(const void* const* parts, const void* residual, long ldr, void* out, long ldo, long rows, int D,
                        const IfabFabric* fab, void* stream);
/* NVLS (NVLink multicast) form: two-shot - each rank reduces 1/world of the buffer with multimem.ld_reduce and writes the
 * sums back to every copy with multimem.st; the buffer holds this rank's partial on entry and the sums on exit. */
int ifab_allreduce_rows_nvls(void* part_local, void* part_mc, const void* residual, long ldr, void* out, long ldo, long rows, int D,
                             uint32_t* arrive, const IfabFabric* fab, void* stream);

/* ---- expert parallelism with sharded tokens: dispatch / combine all-to-all over peer memory (ep_a2a.cu) ----
 * `*_peers` arrays hold `world` pointers into the symmetric buffers of every rank as mapped here: recv / ret bf16 [W*cap, D],
 * meta int32 [W*cap, 2], ctl = 2 x 8 u64 flags + 8 i32 counts. `epoch` grows by one per exchange, identically on all ranks. */
int ifab_ep_dispatch(const void* xn, long ldxn, const int32_t* ids, int M, int topk, int D, int e_local, int world, int rank, int cap,
                     int32_t* send_idx, void* const* recv_peers, void* const* meta_peers, void* const* ctl_peers, uint32_t* ticket,
                     int32_t* dst_count, uint64_t epoch, uint32_t* status, void* stream);
int ifab_ep_plan(const void* meta, void* ctl, int world, int cap, int e_local, int32_t* perm, int32_t* tiles, int32_t* num_tiles,
                 int32_t* total_rows, int max_tiles, uint64_t epoch, uint32_t spin_limit, uint32_t* status, void* stream);
int ifab_ep_gather(const void* recv, const int32_t* perm, const int32_t* total_rows, void* xp, long ldxp, int D, int rows_max, void* stream);
int ifab_ep_return(const void* y, long ldy, const int32_t* perm, const int32_t* total_rows, int D, int cap, int world, int rank, int rows_max,
                   void* const* ret_peers, void* const* ctl_peers, uint32_t* ticket, uint64_t epoch, void* stream);
int ifab_ep_combine(const void* ret, void* ctl, const int32_t* ids, const int32_t* send_idx, const float* wts, int M, int topk, int D,
                    int e_local, int world, int cap, const void* shared, long lds, const void* residual, long ldr, void* out, long ldo,
                    uint64_t epoch, uint32_t spin_limit, uint32_t* status, void* stream);

/* ---- MoE decode path (owner-local expert parallelism) ---- */
int ifab_router_topk(const void* x, long ldx, const void* norm_w, float eps, const float* w_router, const float* bias,
                     float* logits, int32_t* ids, float* wts, int T, int D, int E, int topk, int scoring, int renorm,
                     float scale, uint32_t* ticket, void* xn, long ldxn, void* stream);
int ifab_moe_gate_up_decode(const void* x, long ldx, const void* norm_w, float eps, const int32_t* ids, int T, int D,
                            int F, int topk, int e0, int e_local, const void* w_gu, const void* w_shared_gu, int Fs,
                            void* act, int ldact, void* stream);
int ifab_moe_gate_up_unit_decode(const void* x, long ldx, const void* norm_w, float eps, const int32_t* ids, int T, int D, int F, int topk, int e0, int e_local,
                                 const void* w_gu, const void* w_shared_gu, int Fs, void* act, int ldact, int unit, float limit, float alpha, void* stream);
/* one rank: y f32 [T, ldy] = the same sum before rounding, the shared expert's row weighted by shared_w [T] (null: 1). In both, `act` slots are
 * ldact columns apart (slot topk is the shared expert's, which may be wider or narrower than F) */
int ifab_moe_down_f32_decode(const void* act, int ldact, const int32_t* ids, const float* wts, const float* shared_w, int T, int D, int F, int topk,
                             int experts, const void* w_down, const void* w_shared_down, int Fs, float* y, long ldy, void* stream);
/* routed experts of decoders with an f32 residual (moe_rows.cu): logits f32 [M, ld] (column E: the shared expert's gate, used when shared_w is given) ->
 * ids, wts [M, topk]; scoring 0 softmax, 1 sigmoid, 2 logit + bias selected, softmax over the chosen, 3 sigmoid + bias selected, sigmoid (over the sum with
 * renorm); of `groups` groups of neighbours only the `keep` best are open (moe_select.cuh). combine_norm: y = weighted sum of the permuted rows
 * (+ shared_w * shared), x += rms(y) * w (without w: y + base, a sum of parts) (+ extra), xa = rms(x) * w2 (x without w2) */
int ifab_moe_route(const float* logits, long ld, const float* bias, int M, int E, int topk, int scoring, int renorm, float scale, int groups, int keep, int32_t* ids,
                   float* wts, float* shared_w, void* stream);
int ifab_moe_combine_norm(const void* y, long ldy, const int32_t* route_row, const float* wts, int topk, const void* shared, long lds, const float* shared_w,
                          const float* w, const float* w2, float eps, const float* base, long ldb, int parts, long part_stride, const float* extra, long lde, float* x, long ldx, void* xa,
                          long lda, int f32, int M, int D, void* stream);
int ifab_moe_down_allreduce_decode(const void* act, const int32_t* ids, const float* wts, int T, int D, int F, int topk,
                                   int e0, int e_local, const void* w_down, const void* w_shared_down, int Fs,
                                   const void* residual, long ldr, void* y, long ldy, const IfabFabric* fab,
                                   void* stream);

/* Router + shared and routed gate/up + down + all-reduce of one decode layer as ONE launch (T = 1 or 2 rows, F <= 1536).
 * The grid is sized to be resident at once; two in-grid signals (bounded waits) stand where the three kernels above
 * have kernel boundaries. Results are bit-identical to ifab_router_topk -> ifab_moe_gate_up_decode ->
 * ifab_moe_down_allreduce_decode. sync_words: 16 + 8 * T * E zero-initialised bytes (8-byte aligned) owned by the caller,
 * one set per stream;
 * y = x + reduced expert output, y may alias x. logits / ids / wts receive the router's outputs. */
int ifab_moe_block_decode(const void* x, long ldx, const void* norm_w, float eps, const float* w_router, const float* bias,
                          int E, int topk, int scoring, int renorm, float route_scale, const void* w_gu,
                          const void* w_shared_gu, const void* w_down, const void* w_shared_down, int T, int D, int F,
                          int Fs, int e0, int e_local, float* logits, int32_t* ids, float* wts, void* act, void* y,
                          long ldy, uint32_t* sync_words, const IfabFabric* fab, void* stream);

/* ---- lm_head + vocab-sharded greedy sampling ---- */
int ifab_lm_head_argmax(const void* x, long ldx, const void* norm_w, float eps, const void* w, float* logits,
                        int T, int V_local, int K, int vocab_offset, void* partial /* >= grid*T*8 bytes */,
                        uint64_t partial_bytes, int32_t* out_ids, float* out_vals, const IfabFabric* fab,
                        void* stream);
/* the same for logits cap tanh(logit / cap) (0: none) */
int ifab_lm_head_capped_argmax(const void* x, long ldx, const void* norm_w, float eps, const void* w, float* logits, float cap, int T, int V_local, int K,
                               int vocab_offset, void* partial, uint64_t partial_bytes, int32_t* out_ids, float* out_vals, const IfabFabric* fab, void* stream);

/* ---- sampling on vocabulary-sharded logits: temperature, penalties, top-k <= 64, min-p, top-p, counter-based draw ---- */
int ifab_sample_topk(const float* logits, long ld, int T, int V_local, int vocab_offset, int top_k,
                     const int32_t* top_k_rows /* optional [T]: per-row k <= top_k */,
                     const float* inv_temperature, const float* top_p, const float* min_p, const int16_t* counts, long ldc,
                     const float* penalties, const uint64_t* seeds, uint64_t* counters, void* scratch, uint64_t scratch_bytes,
                     int32_t* out_ids, float* out_probs, const IfabFabric* fab, void* stream);

/* ---- MLA (multi-head latent attention) decode path ---- */
int ifab_mla_kv_write(const void* kv, long ldkv, const void* norm_w, float eps, float theta, const int32_t* positions,
                      const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, void* cache,
                      int num_pages, int T, int latent, int rope, uint32_t* status, void* stream);
/* the same with the rotary columns in rows of their own (latent_rows [T, >= latent], rope_rows [T, >= rope]) */
int ifab_mla_kv_write_split(const void* latent_rows, long ldl, const void* rope_rows, long ldr, const void* norm_w, float eps, float theta,
                            const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens,
                            void* cache, int num_pages, int T, int latent, int rope, uint32_t* status, void* stream);
int ifab_mla_q_absorb(const void* q, long ldq, const void* w_kvb, float theta, const int32_t* positions, void* q_lat,
                      int T, int H, int nope, int rope, int latent, int vdim, void* stream);
int ifab_mla_decode_attention(const void* q_lat, const void* cache, const int32_t* positions, const int32_t* slots,
                              const int32_t* page_table, int max_pages, int page_tokens, int num_pages,
                              const void* sinks, int n_sinks, int window, float scale, int T, int H, int latent,
                              int rope, int keys_per_split, int max_splits, float* scratch, uint64_t scratch_bytes,
                              const void* w_kvb, int nope, int vdim, void* out, long ldo, uint32_t* status,
                              void* stream);

/* The attention half of an MLA decode layer as one launch (a cluster of 8 CTAs per head): cache write, q_b, absorb, attention
 * over the paged latent cache and value up-projection. qkv: [T, q_lora + 576] (output of the qkv_a linear); w_qb: [H * (nope + 64),
 * q_lora]; w_kvb: [H, nope + vdim, 512]; out: [T, H * vdim]. T <= 8, bf16 cache. */
int ifab_mla_head_decode(const void* qkv, long ldqkv, const void* q_norm, const void* kv_norm, float eps, float theta,
                         const void* w_qb, const void* w_kvb, void* cache, const int32_t* positions, const int32_t* slots,
                         const int32_t* page_table, int max_pages, int page_tokens, int num_pages, const void* sinks,
                         int n_sinks, int window, float scale, int T, int H, int q_lora, int nope, int vdim, void* out,
                         long ldo, uint32_t* status, void* stream);

/* The same, and while it runs its CTAs request up to three byte ranges (weights of the layer's later kernels) into L2. */
int ifab_mla_head_decode_pf(const void* qkv, long ldqkv, const void* q_norm, const void* kv_norm, float eps, float theta,
                            const void* w_qb, const void* w_kvb, void* cache, const int32_t* positions, const int32_t* slots,
                            const int32_t* page_table, int max_pages, int page_tokens, int num_pages, const void* sinks,
                            int n_sinks, int window, float scale, int T, int H, int q_lora, int nope, int vdim, void* out,
                            long ldo, uint32_t* status, const void* pf0, uint64_t pf0_bytes, const void* pf1, uint64_t pf1_bytes,
                            const void* pf2, uint64_t pf2_bytes, void* stream);

/* ---- row operators shared by compiled programs (hybrid_ops.cu) ---- */
/* Half-rotation RoPE over the first rotary_dim columns of every head of a row; the other columns are copied. */
int ifab_rope_prefix(const void* x, long ldx, const int32_t* positions, void* y, long ldy, int T, int heads, int head_dim, int rotary_dim,
                     float theta, void* stream);
/* y = a + b over [rows, n] bf16 (f32 sum, one rounding). */
int ifab_add_rows(const void* a, long lda, const void* b, long ldb, void* y, long ldy, int rows, int n, void* stream);
/* y = silu(gate) * up over [rows, n] bf16. */
int ifab_swiglu_pair(const void* gate, long ldg, const void* up, long ldu, void* y, long ldy, int rows, int n, void* stream);

/* ---- hyper-connection / hybrid-model operators (hc_ops.cu); all mixing arithmetic in f32 ---- */
/* causal depthwise conv with residual; w f32 [C_total, taps] (this rank's channels start at c_offset); state bf16 [slots, taps-1, C] */
int ifab_mome(const void* x, long ldx, const float* w, void* state, const int32_t* positions, const int32_t* slots, void* y,
              long ldy, int T, int C, int taps, int c_offset, void* stream);
/* X bf16 [T, S, W]; phi f32 [S*S+2S, S*W]; gamma [S*W]; alpha [3]; beta [S*S+2S] -> y bf16 [T, W], post f32 [T, S], comb f32 [T, S, S] */
int ifab_mhc_pre(const void* X, const float* phi, const float* gamma, const float* alpha, const float* beta, void* y, float* post,
                 float* comb, int T, int S, int W, int sinkhorn_iters, float eps, void* stream);
/* the same in ONE launch: `tickets` = T zeroed 32-bit words (left zero again); the CTA that finishes a token's sums last runs its tail */
int ifab_mhc_pre_ticketed(const void* X, const float* phi, const float* gamma, const float* alpha, const float* beta, void* y, float* post,
                          float* comb, int T, int S, int W, int sinkhorn_iters, float eps, uint32_t* tickets, void* stream);
int ifab_mhc_post(const void* X, const void* branch, long ldb, const float* post, const float* comb, void* Y, int T, int S, int W,
                  void* stream);
/* the same with the branch RMS-normalised first (gain norm_w bf16 [W], result rounded to bf16 like a stand-alone norm) */
int ifab_mhc_post_norm(const void* X, const void* branch, long ldb, const void* norm_w, float eps, const float* post, const float* comb, void* Y,
                       int T, int S, int W, void* stream);
/* gated delta rule, one token per row: q, k bf16 [rows, H, dk]; v bf16 [rows, H, dv]; g, beta f32 [rows, H]; state f32 [slots, H, dk, dv] */
int ifab_delta_rule_decode(const void* q, const void* k, const void* v, const float* g, const float* beta, float* state,
                           const int32_t* slots, void* out, int rows, int H, int dk, int dv, void* stream);
/* f32 residual stream with the norm on a sublayer's output; `f32`: activations (xa, gate, y) are f32 instead of bf16; gains f32 */
/* x = table[id] * scale (and once more to copy, when given); xa = x, or rms(x) * w when w is given */
int ifab_embed_rows(const int32_t* ids, const void* table, long ldt, float scale, const float* w, float eps, float* x, long ldx, float* copy, void* xa, long lda,
                    int f32, int T, int D, int vocab, uint32_t* status, void* stream);
/* x += rms(y) * w (y without w, nothing without y) (+ extra), y the sum of `parts` rows part_stride apart; xa = x, or rms(x) * w2 when w2 is given */
int ifab_post_norm_add(const float* y, long ldy, int parts, long part_stride, const float* w, const float* w2, float eps, float* x, long ldx, const float* extra, long lde, void* xa, long lda,
                       int f32, int T, int D, void* stream);
/* y [T, F] = gated unit of gu[:, c] and gu[:, up + c] */
int ifab_gated_rows(const void* gu, long ld, int up, int unit, float limit, float alpha, void* y, long ldy, int f32, int T, int F, void* stream);
int ifab_rms_rows(const float* x, long ldx, const int32_t* rows, const float* w, float eps, void* y, long ldy, int f32, int T, int D, void* stream);
int ifab_group_norm_gate(const float* o, long ldo, const float* w, float eps, const void* gate, long ldg, int act, void* y, long ldy, int f32, int T,
                         int groups, int n, void* stream);
int ifab_gate_rows(const void* o, long ldo, int head_stride, const void* gate, long ldg, int act, void* y, long ldy, int f32, int T, int H, int n,
                   void* stream);
/* decode linears whose prologue finishes the previous sublayer. ..._post_norm: x_out = x_in + rms(y) * w (one CTA column writes it), then
 * z = act(bf16(x_out) W^T), or of bf16(rms(x_out) * norm2_w) when norm2_w is given; ..._group_norm: z = act(bf16((o / rms per group [* gain]) * gate_act(gate)) W^T) */
int ifab_gemv_post_norm(const float* y, long ldy, const float* norm_w, const float* norm2_w, float eps, const float* x_in, float* x_out, long ldx,
                        const void* w, void* z, long ldz, int out_f32, int act, int T, int N, int K, void* stream);
/* the same with both norms as a router: xn = the operand, f32 logits, then ids / wts (and shared_w = sigmoid(logits[:, E]) when N = E + 1), T <= 8 */
int ifab_router_post_norm(const float* y, long ldy, const float* norm_w, const float* norm2_w, float eps, const float* x_in, float* x_out, long ldx, void* xn,
                          long ldn, const void* w, float* logits, long ldz, const float* bias, int E, int topk, int scoring, int renorm, float scale,
                          int32_t* ids, float* wts, float* shared_w, uint32_t* ticket, int T, int N, int K, void* stream);
int ifab_gemv_group_norm(const float* o, long ldo, const float* gain, float eps, int groups, const void* gate, long ldg, int gate_act, const void* w,
                         void* z, long ldz, int out_f32, int act, int T, int N, int K, void* stream);
/* z = act(x W^T + bias + addend), bias and addend (f32 rows, may be z) or null */
int ifab_gemv_act(const void* x, long ldx, const void* w, const float* bias, const float* addend, long ldadd, void* z, long ldz, int out_f32, int act, int T, int N,
                  int K, void* stream);
/* front of a layer with parallel sublayers, T <= 2: x_out = x_in (+ y) (+ extra), h = rms(x_out) * norm_w -> projection z = h W^T + bias, gated unit of
 * [gate | up] rows, router logits and selection */
int ifab_parallel_in_decode(const float* y, long ldy, const float* extra, long lde, const float* norm_w, float eps, const float* x_in, float* x_out, long ldx,
                            void* xn, long ldn, const void* w, const float* bias, void* z, long ldz, int N, const void* w_gu, int F, int unit, float limit,
                            float alpha, void* unit_out, long ldu, const void* w_router, float* logits, long ldl, const float* correction, int E, int topk,
                            int scoring, int renorm, float scale, int groups, int keep, int32_t* ids, float* wts, uint32_t* ticket, int T, int K, void* stream);
/* linear attention with a fixed decay per head over a packed projection row (linear_attn.cu); state f32 [slots, H, e, d], powers f32 [H, 129],
 * rope float2 [T, rot / 2] of ifab_rope_table */
int ifab_rope_table(const int32_t* positions, const double* freq, void* cs, int T, int pairs, void* stream);
int ifab_la_step(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved, const void* rope,
                 int act, float k_scale, const float* powers, float* state, const int32_t* positions, const int32_t* slots, float* o, long ldo, int T,
                 void* stream);
int ifab_la_prepare(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved,
                    const void* rope, int act, float k_scale, float* q, float* k, float* v, int T, void* stream);
int ifab_la_chunks(const float* q, const float* k, const float* v, const int32_t* chunks, int n, const int32_t* positions, int H, int d, int e,
                   const float* powers, float* cstate, uint64_t cstate_bytes, float* state, float* o, long ldo, void* stream);
int ifab_la_tiles(const void* proj, long ldp, int q_off, int k_off, int v_off, int H, int d, int e, int rot, int interleaved, const void* rope, int act,
                  float k_scale, const float* powers, const int32_t* chunks, int n, const int32_t* positions, float* cstate, uint64_t cstate_bytes,
                  float* state, float* o, long ldo, const void* gate, long ldg, int gate_act, void* y, long ldy, float eps, uint32_t* status, void* stream);
/* norm per head (or, `whole`, over all heads of q and of k with a gain per column) + rotation + cache write, and attention over a window or a chunk of the
 * pages with score caps, distance biases, sinks and gates (attn_rule.cuh), any head sizes (window_attn.cu) */
int ifab_qk_norm_rope_write(const void* proj, long ldp, int f32, int q_off, int k_off, int v_off, const float* q_gain, const float* k_gain, float eps,
                            int H, int G, int d, int e, int rot, int interleaved, const void* rope, const int32_t* positions, const int32_t* slots,
                            const int32_t* page_table, int max_pages, int page_tokens, int num_pages, void* q_out, long ldq, int q_stride, void* k_cache,
                            void* v_cache, int whole, int T, uint32_t* status, void* stream);
int ifab_window_attn(const void* q, long ldq, int q_stride, const void* k_cache, const void* v_cache, int f32, const int32_t* positions, const int32_t* slots,
                     const int32_t* page_table, int max_pages, int page_tokens, int num_pages, int H, int G, int d, int e, int window, float scale, float cap,
                     const float* slopes, int chunked, const float* sink, const void* gate, long ldg, int gate_act, int gate_per_head, int keep, int pool,
                     const void* pool_k, const void* pool_v, float factor, void* out, long ldo, int T, uint32_t* status, void* stream);
/* means of the blocks of `pool` positions that end with a row of the step, into pool_k / pool_v [pages, ceil(page_tokens / pool), G, .] */
int ifab_pool_write(const void* k_cache, const void* v_cache, int f32, const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                    int page_tokens, int num_pages, int G, int d, int e, int pool, void* pool_k, void* pool_v, int T, uint32_t* status, void* stream);
/* residual streams side by side with a convolution ahead of every sublayer (hyper_streams.cu) */
int ifab_embed_norm(const int32_t* ids, const void* table, long ldt, const float* gain, float eps, float* x, long ldx, int f32, int T, int D, int vocab,
                    uint32_t* status, void* stream);
int ifab_step_epoch(const int32_t* slots, int32_t* epoch, int T, void* stream);
int ifab_streams_rows(const float* x_in, long ldr_in, long lds_in, float* x_out, long ldr_out, long lds_out, const float* y, long ldy, int parts,
                      long part_stride, const float* mix, const float* out, const float* in, const float* gain, float eps, const float* taps_w, int taps,
                      float* history, const int32_t* epoch, const int32_t* positions, const int32_t* slots, float* sum, long ldsum, void* xa, long lda, int f32,
                      int T, int S, int D, int block, void* stream);
/* recurrences with a decay per token (gated_recurrence.cu, gated_delta.cu). kind: 0 state-space duality, 1 delta rule, 2 matrix memory. q, k [T, G, d] and
 * v [T, H, e] in the activation type, qs / ks [T, G]: factors of their rows or null; the state [slots, H, e (+ 1 for kind 2), d] */
int ifab_gr_prepare(const void* proj, long ldp, int f32, const int32_t* sections, void* q, void* k, void* v, float* q_factors, float* k_factors, float q_factor,
                    const float* taps_w, const float* bias, int taps, int C, void* history, const int32_t* epoch, int kind, int H, int decay_col,
                    int weight_col, const float* a_log, const float* decay_bias, const float* weight_bias, float cap, float* log_decay, float* weight,
                    const int32_t* positions, const int32_t* slots, int T, void* stream);
int ifab_gr_step(const void* q, const void* k, const void* v, int f32, const float* qs, const float* ks, float q_factor, const float* log_decay,
                 const float* weight, int kind, int H, int G, int d, int e, float* state, float* m_state, const int32_t* epoch, float* m_rows,
                 const int32_t* positions, const int32_t* slots, float* o, long ldo, int T, void* stream);
int ifab_gr_chunks(const void* q, const void* k, const void* v, int f32, const float* qs, const float* ks, float q_factor, const float* log_decay,
                   const float* weight, int kind, int H, int G, int d, int e, const int32_t* chunks, int n, const int32_t* positions, float* cstate,
                   uint64_t cstate_bytes, float* cdecay, float* w_rows, float* u_rows, float* state, float* m_state, const int32_t* epoch, float* m_rows,
                   float* o, long ldo, void* stream);
int ifab_gr_tiles(const void* q, const void* k, const void* v, const float* qs, const float* ks, float q_factor, const float* log_decay, const float* weight, int kind,
                  int H, int G, int d, int e, const int32_t* chunks, int n, const int32_t* positions, float* cstate, uint64_t cstate_bytes, float* cdecay, float* u,
                  void* images, uint64_t image_bytes_given, float* state, float* m_state, const int32_t* epoch, float* m_rows, float* o, long ldo,
                  const void* gate, long ldg, int gate_act, const float* gain, float eps, void* y, long ldy, uint32_t* status, void* stream);
/* one or two decode rows (decode_hyper.cu): a linear behind the streams, a linear behind a recurrence, convolution + gates + step in one */
int ifab_gemv_streams(const float* x_in, long ldr_in, long lds_in, float* x_out, long ldr_out, long lds_out, const float* y, long ldy, const float* mix,
                      const float* out, const float* in, const float* gain, float eps, const float* taps_w, int taps, float* history, const int32_t* epoch,
                      const int32_t* positions, const int32_t* slots, int S, const void* w, void* z, long ldz, int out_f32, int act, int T, int N, int K,
                      void* stream);
int ifab_gemv_mixed(const void* x, long ldx, int K1, const float* o, long ldo, int H, int e, int E, const float* m, const void* v, const float* skip,
                    const void* gate, long ldg, int gate_act, int gate_first, int groups, float eps, const float* gain, const void* w, float* z, long ldz, int T,
                    int N, int K, void* stream);
int ifab_gr_decode(const void* proj, long ldp, const int32_t* cols, const int32_t* channels, int unit, float q_factor, const float* taps_w, const float* bias, int taps,
                   int C, void* history, int kind, int H, int G, int d, int e, int decay_col, int weight_col, const float* a_log, const float* decay_bias,
                   const float* weight_bias, float cap, float* state, float* m_state, const int32_t* epoch, void* v, float* m_rows, const int32_t* positions,
                   const int32_t* slots, float* o, long ldo, int T, void* stream);
int ifab_gr_finish(const float* o, long ldo, int H, int e, int E, const float* m, const void* v, const float* skip, const void* gate, long ldg, int act,
                   int gate_first, int groups, float eps, const float* gain, void* y, long ldy, int f32, int T, void* stream);
/* operands of the tensor-core windowed attention: keys / values first .. first + n - 1 of a sequence, heads zero-padded to dp / 128 columns */
int ifab_ctx_gather_pad(const void* k_cache, const void* v_cache, const int32_t* page_table, int slot, int max_pages, int page_tokens, int num_pages,
                        int first, int n, int rows, int keep, int pool, const void* pool_k, const void* pool_v, int n_ahead, int ahead_rows, int G, int d, int dp, int e, void* k,
                        void* vt, long ldvt, uint32_t* status, void* stream);
int ifab_fa_window_bf16(const void* q, long ldq, const void* k, long ldk, const void* k2, long ldk2, int d2, const void* vt, long ldvt, void* out, long ldo,
                        int m, int ctx, int H, int kv_group, int d, int e, int pos0, int window, float scale, float cap, const float* slopes, int chunked,
                        const float* sink, const void* gate, long ldg, int gate_act, int gate_per_head, int keep, int pool, int ahead_rows, int base, float factor,
                        uint32_t* status, void* stream);
/* latent attention over paged rows [latent padded to Lp | rotated key part padded to Rp], any sizes, bf16 or f32 (latent_attn.cu). splits <= 64, the last
 * takes what is left of the keys a row sees; scratch f32 [T, H, splits, Lp + 2] */
int ifab_latent_prepare(const void* proj, long ldp, int f32, int q_off, int q_rank, int kv_off, int kv_rank, int rot_dim, const float* q_gain,
                        const float* kv_gain, float eps, const void* rope, int rot, const int32_t* positions, const int32_t* slots, const int32_t* page_table,
                        int max_pages, int page_tokens, int num_pages, void* cq, long ldc, void* cache, int Lp, int Rp, int T, uint32_t* status, void* stream);
int ifab_latent_query(const void* proj, long ldp, int q_off, int q_rank, int kv_off, int kv_rank, int rot_dim, const void* q_gain, const float* kv_gain,
                      float eps, const void* rope, int rot, const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                      int page_tokens, int num_pages, void* cache, int Lp, int Rp, const void* w_uq, int N, void* q, long ldq, int T, uint32_t* status,
                      void* stream);
int ifab_rotate_heads(void* q, long ldq, int f32, int head_stride, int off, int H, int rot, const void* rope, int T, void* stream);
int ifab_latent_absorb(void* q, long ldq, int head_stride, int rot_off, const void* w_uk, const void* rope, int rot, float* q_lat, int T, int H, int d, int Lp,
                       void* stream);
int ifab_latent_split(const float* q_lat, const void* q_rot, long ldq, int head_stride, const void* cache, int f32, int Lp, int Rp, const int32_t* positions,
                      const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, int num_pages, int window, float scale, int T, int H,
                      int kps, int splits, float* scratch, uint64_t scratch_bytes, uint32_t* status, void* stream);
/* for many rows: splits * sub partials (sub warps of a CTA share four heads; 1 from 17 heads on) */
int ifab_latent_batch(const float* q_lat, const void* q_rot, long ldq, int head_stride, const void* cache, int Lp, int Rp, const int32_t* positions,
                      const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, int num_pages, int window, float scale, int T, int H,
                      int kps, int splits, int sub, float* scratch, uint64_t scratch_bytes, uint32_t* status, void* stream);
int ifab_latent_merge(const float* scratch, const int32_t* positions, int window, int kps, int splits, int sub, const void* gate, long ldg, int f32, int T, int H, int Lp,
                      void* o_lat, long ldo, void* stream);
int ifab_latent_merge_vup(const float* scratch, const int32_t* positions, int window, int kps, int splits, const void* gate, long ldg, int T, int H, int Lp,
                          const void* w_uv, int vdim, void* out, long ldo, void* stream);
int ifab_latent_gather(const void* cache, const int32_t* page_table, int slot, int max_pages, int page_tokens, int num_pages, int first, int n, int rows, int Lp,
                       int Rp, int tile, void* lat, void* rot, uint32_t* status, void* stream);
int ifab_gqa_window_attention(const void* q, long ldq, const void* k_cache, const void* v_cache, const int32_t* positions, const int32_t* slots,
                              const int32_t* page_table, int max_pages, int page_tokens, int num_pages, float scale, int window, float cap, const float* slopes,
                              int chunked, const float* sink, const void* gate, long ldg, int gate_act, int gate_per_head, int keep, int pool, const void* pool_k, const void* pool_v,
                              float factor, int T, int Hq, int Hkv, int head_dim, int keys_per_split, int max_splits, float* scratch, uint64_t scratch_bytes, void* out, long ldo, uint32_t* status, void* stream);
/* indexer: q bf16 [T, heads, dim], w f32 [T, heads], keys paged bf16 [pages, page_tokens, dim]; scores = scratch f32 [T, ctx];
 * out int32 [T, topk]: the top-k key positions (<= the query position) in ascending order, -1 padded */
int ifab_sparse_index(const void* q, const float* w, const void* keys, const int32_t* positions, const int32_t* slots,
                      const int32_t* page_table, int max_pages, int page_tokens, int num_pages, float* scores, int ctx, int T,
                      int heads, int dim, int topk, int32_t* out, uint32_t* status, void* stream);
/* the same over an int8 index cache (keys int8 [pages, page_tokens, dim], one half-precision scale per row; the query heads are
 * quantised the same way before scoring) and the append that fills it */
int ifab_sparse_index_q8(const void* q, const float* w, const void* keys, const void* key_scales, const int32_t* positions, const int32_t* slots,
                         const int32_t* page_table, int max_pages, int page_tokens, int num_pages, float* scores, int ctx, int T, int heads, int dim,
                         int topk, int32_t* out, uint32_t* status, void* stream);
int ifab_index_cache_append_q8(const void* key, long ldk, const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                               int page_tokens, int num_pages, void* cache, void* scales, int T, int dim, uint32_t* status, void* stream);
/* bf16 index keys [T, dim] into the paged bf16 index cache [pages, page_tokens, dim] */
int ifab_index_cache_append(const void* key, long ldk, const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                            int page_tokens, int num_pages, void* cache, int T, int dim, uint32_t* status, void* stream);
/* the general selector: gains f32 [T, heads] (w_bf16 = 0, ldw = heads) or bf16 rows of stride ldw (w_bf16 = 1); key_scales null = bf16 keys */
int ifab_sparse_index_general(const void* q, const void* w, long ldw, int w_bf16, const void* keys, const void* key_scales, const int32_t* positions,
                              const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, int num_pages, float* scores, int ctx,
                              int T, int heads, int dim, int topk, int32_t* out, uint32_t* status, void* stream);
/* split-KV attention restricted to `indices` (int32 [T, n_index], ascending key positions padded with -1; null = every causal key);
 * rope < 0: the cache holds packed int8 rows (656 bytes) */
int ifab_mla_decode_attention_indexed(const void* q_lat, const void* cache, const int32_t* positions, const int32_t* slots, const int32_t* page_table,
                                      int max_pages, int page_tokens, int num_pages, const void* sinks, int n_sinks, int window, float scale, int T,
                                      int H, int latent, int rope, int keys_per_split, int max_splits, float* scratch, uint64_t scratch_bytes,
                                      const void* w_kvb, int nope, int vdim, void* out, long ldo, uint32_t* status, const int32_t* indices, int n_index,
                                      void* stream);

/* ---- packed int8 latent cache (656-byte rows: 512 int8 | 64 bf16 rope | 4 f32 tile scales) and activation quantisation ----
 * Attention over a packed cache: ifab_mla_decode_attention with rope = -64 and `cache` pointing at the packed rows. */
int ifab_mla_kv_write_q8(const void* kv, long ldkv, const void* norm_w, float eps, float theta, const int32_t* positions,
                         const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens, void* cache,
                         int num_pages, int T, uint32_t* status, void* stream);
int ifab_mla_kv_write_q8_split(const void* latent_rows, long ldl, const void* rope_rows, long ldr, const void* norm_w, float eps, float theta,
                               const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages, int page_tokens,
                               void* cache, int num_pages, int T, uint32_t* status, void* stream);
int ifab_kv_dequantize_q8(const void* cache, void* out /* bf16 [rows, 576] */, long rows, void* stream);
/* symmetric int8, ties away from zero; group_cols = K: per-row scale, 128: per-tile scales [T, ceil(K/128)] */
int ifab_quantize_int8(const void* x, long ldx, void* q, long ldq, float* scales, long lds, int T, int K, int group_cols,
                       void* stream);

/* ---- GQA decode path (dense models) ---- */
int ifab_gqa_rope_kv_write(void* qkv, long ld, const int32_t* positions, const int32_t* slots,
                           const int32_t* page_table, int max_pages, int page_tokens, void* k_cache, void* v_cache,
                           int num_pages, int T, int Hq, int Hkv, int head_dim, int rotary_dim, float theta,
                           uint32_t* status, void* stream);
/* Split-KV decode attention. Split s covers keys [s * keys_per_split, (s + 1) * keys_per_split); the LAST split also covers
 * every key beyond max_splits * keys_per_split, so any context is attended in full (contexts longer than that product
 * only lose parallelism). scratch: T * Hq * max_splits * (head_dim + 2) floats. */
int ifab_gqa_decode_attention(const void* q, long ldq, const void* k_cache, const void* v_cache,
                              const int32_t* positions, const int32_t* slots, const int32_t* page_table, int max_pages,
                              int page_tokens, int num_pages, float scale, int T, int Hq, int Hkv, int head_dim,
                              int keys_per_split, int max_splits, float* scratch, uint64_t scratch_bytes, void* out,
                              long ldo, uint32_t* status, void* stream);

/* ---- GQA decode attention without any allocation (this entry point has no counterpart in the reference) ----
 * Same computation and same results as ifab_gqa_decode_attention, but the split-partials workspace is a
 * fixed array inside the library, so neither the caller nor the library calls cudaMalloc / cudaFree or any
 * allocating routine. Meant for C / C++ hosts that link the library without a tensor framework and cannot
 * allocate where they call it: all free device memory already belongs to their KV cache, they run under an
 * allocator lock, or an allocation could stall the device in a latency-critical loop.
 *   - limit: T * Hq * max_splits * (head_dim + 2) * 4 bytes must not exceed IFAB_GQA_STATIC_SCRATCH_BYTES;
 *     a larger call returns IFAB_ERR_STATIC_SCRATCH, launches nothing and explains itself in `err`
 *   - every call looks up the array's address on the current device (cudaGetSymbolAddress: a host-side query that
 *     allocates nothing, and is right again after a device reset); the first call on a device may load the module, so
 *     make that first call before any stream capture begins
 *   - all calls on a device share the one array: calls that may overlap on the GPU race on it, so keep them
 *     on one stream or order them. The array keeps the previous call's contents; each call overwrites
 *     everything it reads, so nothing has to be cleared
 *   - `err` (optional, `err_len` bytes) receives a NUL-terminated message when the result is not 0
 *   - ifab_gqa_static_scratch_bytes() / ifab_err_static_scratch() return the two constants below to callers that do not
 *     include this header (bindings) */
#define IFAB_GQA_STATIC_SCRATCH_BYTES (8u << 20)
#define IFAB_ERR_STATIC_SCRATCH (-6)
uint64_t ifab_gqa_static_scratch_bytes(void);
int ifab_err_static_scratch(void);
int ifab_gqa_decode_attention_static(const void* q, long ldq, const void* k_cache, const void* v_cache,
                                     const int32_t* positions, const int32_t* slots, const int32_t* page_table,
                                     int max_pages, int page_tokens, int num_pages, float scale, int T, int Hq, int Hkv,
                                     int head_dim, int keys_per_split, int max_splits, void* out, long ldo,
                                     uint32_t* status, void* stream, char* err, uint64_t err_len);

#ifdef __cplusplus
}
#endif
