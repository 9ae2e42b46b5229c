// Routing by corrected scores: s = softmax(z) over all outputs (experts first, then identity experts,
// whose output is their input), the top k of s + correction are chosen, and the weights are the chosen
// experts' own s, not renormalised. Everything in fp32; nothing leaves the device.
//
// The routed experts' histogram and offsets serve the grouped expert products; the chosen identity
// experts appear only as one summed weight per token. The other rule (kRouteChosen) has no identity experts: the
// top k of z + bias, weighted by the softmax over the chosen ones alone. kRouteGrouped chooses by sigmoids among the best
// groups' experts and puts the experts that every token uses behind the chosen ones: they have T rows each, in token order.
#include "../common/launch.cuh"
#include "../common/route.cuh"
#include "../common/rows.cuh"

namespace rb {

template <RouteRule RULE>
__global__ void __launch_bounds__(256)
route_kernel(const float* __restrict__ logits, int ldl, const float* __restrict__ correction,
                       int* __restrict__ idx, float* __restrict__ weights, float* __restrict__ identity,
                       int* __restrict__ counts, int T, int experts, int outputs, int top_k, RouteGroups groups) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), slots = top_k + groups.always;
  if (t < T)
    warp_route<RULE>(logits + size_t(t) * ldl, correction, experts, outputs, top_k, idx + size_t(t) * slots,
                     weights + size_t(t) * slots, identity ? identity + t : nullptr, counts, groups);
}

// offsets[e] = counts before e, offsets[E] = their sum; counts become running cursors. The experts from `counted` on have
// T rows each. One warp.
__global__ void route_offsets_kernel(int* __restrict__ counts, int* __restrict__ offsets, int E, int counted, int T) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x;
  int carry = 0;
  for (int base = 0; base < E; base += 32) {
    const int e = base + lane;
    const int c = e < counted ? counts[e] : e < E ? T : 0;
    int inc = c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int n = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += n;
    }
    if (e < E) { offsets[e] = carry + inc - c; counts[e] = carry + inc - c; }
    carry += __shfl_sync(0xffffffffu, inc, 31);
  }
  if (lane == 0) offsets[E] = carry;
}

// Rows of x sorted by expert: one warp per (token, slot) copies the token's row to the next free place
// of its expert. Identity experts get row -1 and no copy. Which place a token takes inside its expert
// does not matter to any result.
template <class T>
__global__ void __launch_bounds__(256)
route_scatter_kernel(const T* __restrict__ x, int ldx, const int* __restrict__ idx, int* __restrict__ cursors,
                     T* __restrict__ xs, int* __restrict__ row_of_pair, int pairs, int top_k, int experts, int counted) {
  pdl_launch_dependents();
  pdl_wait();
  const int p = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (p >= pairs) return;
  int row = -1;
  if (lane == 0) {
    const int e = idx[p];
    if (e < counted) row = atomicAdd(cursors + e, 1);
    else if (e < experts) row = cursors[e] + p / top_k;
    row_of_pair[p] = row;
  }
  row = __shfl_sync(0xffffffffu, row, 0);
  if (row < 0 || row >= pairs) return;              // (row >= pairs: cursors that belong to another choice)
  const uint4* src = reinterpret_cast<const uint4*>(x + size_t(p / top_k) * ldx);
  uint4* dst = reinterpret_cast<uint4*>(xs + size_t(row) * ldx);
  const int units = ldx * int(sizeof(T)) / 16;
  for (int i = lane; i < units; i += 32) dst[i] = src[i];
}

}  // namespace rb

using namespace rb;
RB_BOUNDS_REGISTER("moe_route.cu")

extern "C" int rmlx_route_max_outputs() { return kRouteMaxOutputs; }
extern "C" int rmlx_route_max_top() { return kRouteMaxTop; }

template <RouteRule RULE>
static int launch_route(const float* logits, int ldl, const float* correction, int* idx, float* weights, float* identity,
                        int* counts, int* offsets, int T, int experts, int outputs, int top_k, int pdl, cudaStream_t st,
                        const RouteGroups& groups = RouteGroups{}) {
  if (T < 1 || experts < 1 || outputs < experts || outputs > kRouteMaxOutputs || top_k < 1 || top_k > kRouteMaxTop ||
      top_k > outputs || ldl < outputs || (!counts) != (!offsets) || (!correction && RULE != kRouteGrouped))
    return -2;
  if (counts) RB_CHECK(cudaMemsetAsync(counts, 0, sizeof(int) * experts, st));
  const int rc = launch(route_kernel<RULE>, dim3((T + 7) / 8), dim3(256), 0, st, pdl != 0 && !counts, logits, ldl,
                        correction, idx, weights, identity, counts, T, experts, outputs, top_k, groups);
  if (rc || !counts) return rc;
  return launch(route_offsets_kernel, dim3(1), dim3(32), 0, st, pdl != 0, counts, offsets, experts + groups.always, experts, T);
}

// logits fp32 [T, ldl], correction fp32 [outputs]; idx, weights [T, top_k], identity [T]; counts
// [experts] (becomes the scatter's cursors) and offsets [experts + 1], both or neither.
extern "C" int rmlx_route_corrected(const float* logits, int ldl, const float* correction, int* idx, float* weights,
                                    float* identity, int* counts, int* offsets, int T, int experts, int outputs,
                                    int top_k, int pdl, cudaStream_t st) {
  if (!identity) return -2;
  return launch_route<kRouteCorrected>(logits, ldl, correction, idx, weights, identity, counts, offsets, T, experts, outputs,
                                       top_k, pdl, st);
}

// The rule without identity experts: bias fp32 [experts], the rest as above.
extern "C" int rmlx_route_chosen(const float* logits, int ldl, const float* bias, int* idx, float* weights, int* counts,
                                 int* offsets, int T, int experts, int top_k, int pdl, cudaStream_t st) {
  return launch_route<kRouteChosen>(logits, ldl, bias, idx, weights, nullptr, counts, offsets, T, experts, experts, top_k, pdl,
                                    st);
}

// Sigmoid scores, the `keep` best of `groups` groups, weights times `scale`; idx and weights [T, top_k + always], counts
// [experts + always], offsets one more.
extern "C" int rmlx_route_grouped(const float* logits, int ldl, int* idx, float* weights, int* counts, int* offsets, int T,
                                  int experts, int top_k, int groups, int keep, int always, float scale, int pdl,
                                  cudaStream_t st) {
  RouteGroups g;
  g.count = groups; g.keep = keep; g.always = always; g.scale = scale;
  if (!route_groups_ok(g, experts, top_k)) return -2;
  return launch_route<kRouteGrouped>(logits, ldl, nullptr, idx, weights, nullptr, counts, offsets, T, experts, experts, top_k,
                                     pdl, st, g);
}

// x [T, ldx] -> xs [T * top_k, ldx]; ldx a multiple of eight; cursors as the choice left them. The `always` last of the
// experts have every token's row.
extern "C" int rmlx_route_scatter(const void* x, int ldx, const int* idx, int* cursors, void* xs, int* row_of_pair,
                                  int T, int top_k, int experts, int always, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || top_k < 1 || ldx % 8 || always < 0 || always >= experts) return -2;
  const int counted = experts - always;
  const int pairs = T * top_k;
  const dim3 grid((pairs + 7) / 8);
  if (f32)
    return launch(route_scatter_kernel<float>, grid, dim3(256), 0, st, pdl != 0, static_cast<const float*>(x), ldx, idx,
                  cursors, static_cast<float*>(xs), row_of_pair, pairs, top_k, experts, counted);
  return launch(route_scatter_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(x), ldx, idx, cursors, static_cast<__nv_bfloat16*>(xs), row_of_pair,
                pairs, top_k, experts, counted);
}
