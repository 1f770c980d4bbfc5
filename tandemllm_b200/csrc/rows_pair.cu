// The residual add of two branches fused with two RMS norms of the new row (add_rmsnorm.cuh, NORM_PAIR): what stands in front of
// a layer whose mixer and feed-forward both read the residual as it was before either.
//
//   residual[r] += first branch's output + second branch's output
//   normed[r] = weight * row / rms(row);  normed2[r] = weight2 * row / rms(row);  the router (optional) reads normed2's rows
//
// The first branch comes as a tensor or partial sums, the second as a tensor, partial sums or a routed layer's expert rows.
#include "add_rmsnorm.cuh"

using namespace tl;

// See NormParams. `delta2` and `expert_rows` are two forms of the second branch; weight2 null: one norm only.
extern "C" int tl_add_rmsnorm_pair(float* residual, const float* delta, int parts, long long part_stride, const float* delta2,
                                   int parts2, long long part_stride2, const float* expert_rows, int expert_parts,
                                   long long expert_part_stride, const int* pos_of_pair, const int* ids, const float* wts,
                                   int top_k, const float* weight, void* normed, const float* weight2, void* normed2,
                                   const int* gather, int out_rows, int hidden, float eps, int dtype, const float* router_w,
                                   const float* router_bias, int E, int route_k, int normalize, float floor_, float scale,
                                   int* route_ids, float* route_wts, cudaStream_t stream) {
  if (out_rows == 0) return 0;
  TL_REQUIRE(!delta2 || parts2 >= 1, "add_rmsnorm_pair: %d parts", parts2);
  TL_REQUIRE((weight2 != nullptr) == (normed2 != nullptr), "add_rmsnorm_pair: a second norm wants a weight and a place for its rows");
  NormParams p = {};
  p.residual = residual; p.delta = delta; p.parts = parts; p.part_stride = part_stride;
  p.delta2 = delta2; p.parts2 = parts2; p.part_stride2 = part_stride2; p.expert_rows = expert_rows;
  p.expert_parts = expert_parts < 1 ? 1 : expert_parts; p.expert_part_stride = expert_part_stride;
  p.pos_of_pair = pos_of_pair; p.ids = ids; p.wts = wts; p.top_k = top_k; p.weight = weight; p.eps = eps;
  p.normed = normed; p.weight2 = weight2; p.normed2 = normed2; p.gather = gather; p.hidden = hidden; p.out_rows = out_rows;
  p.router_w = router_w; p.router_bias = router_bias; p.E = E; p.route_k = route_k; p.normalize = normalize;
  p.floor_ = floor_; p.scale = scale; p.route_ids = route_ids; p.route_wts = route_wts;
  return launch_add_rmsnorm<NORM_PAIR>(p, dtype, stream);
}
