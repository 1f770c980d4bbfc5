// The router's choice for one row, run by one full warp: scores (the sigmoid of each logit, or the softmax over all
// experts' logits), the top-k of score + bias (the bias for the choice only), weights = chosen scores, divided by
// (their sum + floor) when normalised, times scale.
// Ties go to the lower expert id; a NaN score is chosen only when nothing else is left.
// (engine/models/lfm2_moe/ref.py:185-197, engine/models/lfm2_moe/kernels.py:265-287 of the reference; the softmax
// scoring is what its other routed families use, engine/models/flashnext/ref.py:479-487)
// The third scoring function takes the bias as part of the logit: the k largest logits + bias are chosen, and their weights are
// the softmax over the chosen ones only (computed from the row's largest logit, which is always chosen).
//
// The launchers' `normalize` argument carries the router's choices: bit 0 = divide the chosen weights by their sum,
// bits 1..3 = the scoring function (TL_SCORE_SIGMOID 0, TL_SCORE_SOFTMAX 1, TL_SCORE_CHOSEN 2), bits 4..9 = the number of expert groups
// (0: the choice is free) and bits 10..15 = how many of them are kept.
//
// Group-limited choice: the experts form `groups` equal groups of neighbours; a group's score is the sum of its two
// largest choice scores (score + bias); only the experts of the `keep` best groups (ties to the lower group) can be
// chosen: the others' choice scores count as minus infinity.
#pragma once

#include "common.cuh"

namespace tl {

#define TL_SCORE_SIGMOID 0
#define TL_SCORE_SOFTMAX 1
#define TL_SCORE_CHOSEN 2
#define TL_SCORE_LAST 2
#define TL_ROUTE_SCORING(flags) (((flags) >> 1) & 7)
#define TL_ROUTE_GROUPS(flags) (((flags) >> 4) & 63)
#define TL_ROUTE_KEEP(flags) (((flags) >> 10) & 63)
#define TL_ROUTE_MAX_GROUPS 32

constexpr int MAX_EXPERTS = 1024;
constexpr int MAX_TOP_K = 32;

// `lg`: the row's E <= 32 PER logits (global or shared memory). Lanes 0..k-1 write ids[lane] and wts[lane], in the
// order of the choice (best first). PER: experts a lane holds.
template <int PER>
__device__ __forceinline__ void warp_route_sized(const float* lg, const float* __restrict__ bias, int E, int k,
                                                 int normalize, float floor_, float scale, int* ids, float* wts) {
  const int lane = threadIdx.x & 31;
  const int scoring = TL_ROUTE_SCORING(normalize);
  const int n_groups = TL_ROUTE_GROUPS(normalize), keep_groups = TL_ROUTE_KEEP(normalize);
  normalize &= 1;
  if (scoring == TL_SCORE_CHOSEN) {
    normalize = 1;
    floor_ = 0.f;
  }
  float score[PER], choice[PER];
  float top = -INFINITY, denom = 1.f;
  if (scoring == TL_SCORE_SOFTMAX) {        // the row's largest logit and the sum of exponentials, over the whole warp
#pragma unroll
    for (int t = 0; t < PER; ++t)
      if (lane + 32 * t < E) top = fmaxf(top, lg[lane + 32 * t]);
    top = warp_max(top);
    float part = 0.f;
#pragma unroll
    for (int t = 0; t < PER; ++t)
      if (lane + 32 * t < E) part += expf(lg[lane + 32 * t] - top);
    denom = warp_sum(part);
  }
  if (scoring == TL_SCORE_CHOSEN) {
#pragma unroll
    for (int t = 0; t < PER; ++t) {
      const int e = lane + 32 * t;
      if (e < E) top = fmaxf(top, bias ? lg[e] + bias[e] : lg[e]);
    }
    top = warp_max(top);
  }
#pragma unroll
  for (int t = 0; t < PER; ++t) {
    const int e = lane + 32 * t;
    if (e < E) {
      if (scoring == TL_SCORE_CHOSEN) {
        choice[t] = bias ? lg[e] + bias[e] : lg[e];
        score[t] = expf(choice[t] - top);
      } else {
        const float s = scoring == TL_SCORE_SOFTMAX ? expf(lg[e] - top) / denom : 1.f / (1.f + expf(-lg[e]));
        score[t] = s;
        choice[t] = bias ? s + bias[e] : s;
      }
      if (!(choice[t] == choice[t])) choice[t] = -INFINITY;
    } else {
      score[t] = 0.f;
      choice[t] = -INFINITY;
    }
  }
  if (n_groups > 1 && keep_groups < n_groups) {
    // lane g ends up with group g's score (at most 32 groups); every lane learns which groups are kept
    const int per = E / n_groups;
    float mine = -INFINITY;
    for (int g = 0; g < n_groups; ++g) {
      float a = -INFINITY, b = -INFINITY;           // the two largest choice scores of group g seen by this lane
#pragma unroll
      for (int t = 0; t < PER; ++t) {
        const int e = lane + 32 * t;
        if (e < E && e / per == g) {
          const float c = choice[t];
          if (c > a) { b = a; a = c; }
          else if (c > b) b = c;
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
        const float hi = fmaxf(a, oa), lo = fminf(a, oa);
        b = fmaxf(lo, fmaxf(b, ob));
        a = hi;
      }
      const float gs = b == -INFINITY ? a : a + b;
      if (lane == g) mine = gs;
    }
    int rank = 0;
    for (int g = 0; g < n_groups; ++g) {
      const float other = __shfl_sync(0xffffffffu, mine, g);
      rank += (other > mine) || (other == mine && g < lane);
    }
    const unsigned kept = __ballot_sync(0xffffffffu, lane < n_groups && rank < keep_groups);
#pragma unroll
    for (int t = 0; t < PER; ++t) {
      const int e = lane + 32 * t;
      if (e < E && !((kept >> (e / per)) & 1u)) choice[t] = -INFINITY;
    }
  }
  float sum = 0.f, my_w = 0.f;
  int my_id = 0;
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY;
    int best_e = 0x7fffffff;
    float best_s = 0.f;
#pragma unroll
    for (int t = 0; t < PER; ++t) {
      const int e = lane + 32 * t;
      if (e < E && choice[t] != -INFINITY && (choice[t] > best || (choice[t] == best && e < best_e))) {
        best = choice[t];
        best_e = e;
        best_s = score[t];
      }
    }
    if (best_e == 0x7fffffff) {     // nothing but -inf left in this lane: offer its lowest untaken id
#pragma unroll
      for (int t = 0; t < PER; ++t) {
        const int e = lane + 32 * t;
        if (e < E && score[t] != -1.f && e < best_e) {
          best_e = e;
          best_s = score[t];
        }
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, best_e, o);
      const float os = __shfl_xor_sync(0xffffffffu, best_s, o);
      if (ob > best || (ob == best && oe < best_e)) {
        best = ob;
        best_e = oe;
        best_s = os;
      }
    }
    if ((best_e & 31) == lane) {    // the owner retires the winner
#pragma unroll
      for (int t = 0; t < PER; ++t)
        if (lane + 32 * t == best_e) {
          choice[t] = -INFINITY;
          score[t] = -1.f;
        }
    }
    sum += best_s;
    if (lane == j) {
      my_id = best_e;
      my_w = best_s;
    }
  }
  if (lane < k) {
    float w = my_w;
    if (normalize) w = w / (sum + floor_);
    ids[lane] = my_id;
    wts[lane] = w * scale;
  }
}

__device__ __forceinline__ void warp_route(const float* lg, const float* __restrict__ bias, int E, int k, int normalize,
                                           float floor_, float scale, int* ids, float* wts) {
  if (E <= 32) warp_route_sized<1>(lg, bias, E, k, normalize, floor_, scale, ids, wts);
  else if (E <= 128) warp_route_sized<4>(lg, bias, E, k, normalize, floor_, scale, ids, wts);
  else warp_route_sized<MAX_EXPERTS / 32>(lg, bias, E, k, normalize, floor_, scale, ids, wts);
}

}  // namespace tl
