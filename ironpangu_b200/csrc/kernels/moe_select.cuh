// Top-k expert selection of one token row from its router logits, by one warp.
//
// Softmax scoring (0): probabilities over all experts, the k largest, optionally renormalised to sum 1.
// Sigmoid scoring (1): sigmoid scores, selection on score + bias, weights = score / sum of the selected scores.
// Biased-logit scoring (2): selection on logit + bias, weights = softmax over the selected ones only.
// Free sigmoid scoring (3): sigmoid scores, selection on score + bias, weights = score, divided by their sum only on request.
// With groups of neighbours only experts of the `keep` best groups can be selected; a group is worth its two largest selection scores
// together (its only one when it has one).
// Ties go to the lower expert index, so the result does not depend on lane order. Supports up to 256 experts.
#pragma once
#include "common.cuh"

namespace ifab {

constexpr int MAX_TOPK = 16;

// all 32 lanes of the calling warp take part; lane l holds the logits of experts l, l + 32, ... in score[] (-inf beyond E);
// lane 0 writes ids[0..topk) and wts[0..topk)
constexpr int SELECT_PER_LANE = 8;

// selection scores of all but the best `keep` of `groups` groups become -inf
__device__ __forceinline__ void close_groups(float (&sel)[SELECT_PER_LANE], int E, int groups, int keep) {
  const int lane = threadIdx.x & 31, n = E / groups;
  constexpr int PER = SELECT_PER_LANE;
  int group[PER];
  float value[PER];             // of groups lane, lane + 32, ...
  bool open[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    group[i] = lane + 32 * i < E ? (lane + 32 * i) / n : -1;
    value[i] = -INFINITY;
    open[i] = false;
  }
  for (int g = 0; g < groups; ++g) {
    float a = -INFINITY, b = -INFINITY;      // the two largest
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      if (group[i] != g) continue;
      b = fmaxf(b, fminf(a, sel[i]));
      a = fmaxf(a, sel[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
      b = fmaxf(fminf(a, oa), fmaxf(b, ob));
      a = fmaxf(a, oa);
    }
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i == g) value[i] = n > 1 ? a + b : a;
  }
  for (int k = 0; k < keep; ++k) {
    float bv = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (value[i] > bv || (value[i] == bv && lane + 32 * i < bi)) { bv = value[i]; bi = lane + 32 * i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      if (lane + 32 * i == bi) value[i] = -INFINITY;
      if (group[i] == bi) open[i] = true;
    }
  }
#pragma unroll
  for (int i = 0; i < PER; ++i)
    if (!open[i]) sel[i] = -INFINITY;
}

__device__ __forceinline__ void select_topk_scores(float (&score)[SELECT_PER_LANE], const float* bias, int E, int topk, int scoring,
                                                   int renorm, float scale, int32_t* ids, float* wts, int groups = 1, int keep = 1) {
  const int lane = threadIdx.x & 31;
  constexpr int PER = SELECT_PER_LANE;
  float sel[PER];
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < PER; ++i) mx = fmaxf(mx, score[i]);
  mx = warp_max(mx);
  float denom = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int ei = lane + 32 * i;
    if (ei < E) {
      if (scoring == 0) {
        score[i] = __expf(score[i] - mx);
        denom += score[i];
        sel[i] = score[i];
      } else if (scoring == 2) {
        if (bias) score[i] += bias[ei];
        sel[i] = score[i];
      } else if (scoring == 3) {
        score[i] = 1.f / (1.f + expf(-score[i]));
        sel[i] = score[i] + (bias ? bias[ei] : 0.f);
      } else {
        score[i] = 1.f / (1.f + __expf(-score[i]));
        sel[i] = score[i] + (bias ? bias[ei] : 0.f);
      }
    } else {
      score[i] = 0.f;
      sel[i] = -INFINITY;
    }
  }
  denom = warp_sum(denom);
  if (groups > 1) close_groups(sel, E, groups, keep);
  float picked_w[MAX_TOPK];
  int picked_e[MAX_TOPK];
  float wsum = 0.f, top = 0.f;
  for (int k = 0; k < topk; ++k) {
    float bv = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int ei = lane + 32 * i;
      if (sel[i] > bv || (sel[i] == bv && ei < bi)) { bv = sel[i]; bi = ei; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    // the owning lane reports the raw score and retires the expert
    float raw = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      if (lane + 32 * i == bi) { raw = score[i]; sel[i] = -INFINITY; }
    }
    raw = warp_sum(raw);
    picked_e[k] = bi;
    picked_w[k] = (scoring == 0) ? raw / denom : scoring == 2 ? expf(raw - (k ? top : raw)) : raw;
    if (k == 0) top = raw;
    wsum += picked_w[k];
  }
  if (lane == 0) {
    for (int k = 0; k < topk; ++k) {
      float w = picked_w[k];
      if (scoring == 0 || scoring == 3) { if (renorm) w = w / wsum; }
      else if (scoring == 2) w = w / wsum;
      else w = w / (wsum + 1e-20f);
      ids[k] = picked_e[k];
      wts[k] = w * scale;
    }
  }
}

// the same from logits in global memory
__device__ __forceinline__ void select_topk_row(const float* logits, const float* bias, int E, int topk, int scoring,
                                                int renorm, float scale, int32_t* ids, float* wts, int groups = 1, int keep = 1) {
  const int lane = threadIdx.x & 31;
  float score[SELECT_PER_LANE];
#pragma unroll
  for (int i = 0; i < SELECT_PER_LANE; ++i) {
    const int ei = lane + 32 * i;
    score[i] = (ei < E) ? __ldcg(logits + ei) : -INFINITY;
  }
  select_topk_scores(score, bias, E, topk, scoring, renorm, scale, ids, wts, groups, keep);
}

// sizes the selection takes
__host__ __forceinline__ bool select_ok(int E, int topk, int scoring, int groups, int keep) {
  return E >= 1 && E <= 32 * SELECT_PER_LANE && topk >= 1 && topk <= MAX_TOPK && topk <= E && scoring >= 0 && scoring <= 3 && groups >= 1 && E % groups == 0 &&
         keep >= 1 && keep <= groups && topk <= keep * (E / groups);
}

}  // namespace ifab
