// Expert choice for one token by one full warp (see moe_route.cu).
#pragma once
#include "ptx.cuh"

namespace rb {

constexpr int kRouteMaxOutputs = 512;
constexpr int kRouteMaxTop = 32;

enum RouteRule {
  kRouteCorrected = 0,      // by softmax + correction; weights: the softmax over all outputs
  kRouteChosen = 1,         // by logit + correction (a bias); weights: the softmax over the chosen ones alone
};

// N: outputs a lane holds. logits, correction: fp32 [outputs], the first `experts` of them with weights of their own. Ties go to
// the lower index. counts (may be null) gets one more for every chosen expert.
template <int N, RouteRule RULE>
__device__ __forceinline__ void warp_route_n(const float* logits, const float* correction, int experts, int outputs,
                                             int top_k, int* idx, float* weights, float* identity, int* counts) {
  const int lane = threadIdx.x & 31;
  float s[N], c[N], m = -INFINITY;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int e = i * 32 + lane;
    s[i] = e < outputs ? logits[e] : -INFINITY;
    m = fmaxf(m, s[i]);
  }
  if (RULE == kRouteCorrected) {
    m = warp_max(m);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) { s[i] = expf(s[i] - m); sum += s[i]; }
    sum = warp_sum(sum);
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = s[i] / sum;
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int e = i * 32 + lane;
    c[i] = e < outputs ? s[i] + correction[e] : -INFINITY;
    if (RULE == kRouteChosen) s[i] = c[i];
  }
  float my_w = 0.f, id_w = 0.f;
  int my_e = 0;
  for (int r = 0; r < top_k; ++r) {
    float best = -INFINITY, w = 0.f;
    int be = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (c[i] > best) { best = c[i]; be = i * 32 + lane; w = s[i]; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o), ow = __shfl_xor_sync(0xffffffffu, w, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; w = ow; }
    }
    if (be >= outputs) { be = outputs - 1; w = 0.f; }      // scores that are no numbers choose nothing
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (i * 32 + lane == be) c[i] = -INFINITY;
    if (lane == r) { my_e = be; my_w = w; }
    if (be >= experts) id_w += w;
  }
  if (RULE == kRouteChosen) {                              // the first choice has the largest logit
    const float top = __shfl_sync(0xffffffffu, my_w, 0);   // (by the whole warp)
    my_w = lane < top_k ? expf(my_w - top) : 0.f;
    my_w = my_w / warp_sum(my_w);
  }
  if (lane < top_k) {
    idx[lane] = my_e;
    weights[lane] = my_w;
    if (counts && my_e < experts) atomicAdd(counts + my_e, 1);
  }
  if (lane == 0 && identity) *identity = id_w;
}

template <RouteRule RULE>
__device__ __forceinline__ void warp_route(const float* logits, const float* correction, int experts, int outputs, int top_k,
                                           int* idx, float* weights, float* identity, int* counts) {
  if (outputs <= 64) warp_route_n<2, RULE>(logits, correction, experts, outputs, top_k, idx, weights, identity, counts);
  else if (outputs <= 256) warp_route_n<8, RULE>(logits, correction, experts, outputs, top_k, idx, weights, identity, counts);
  else warp_route_n<kRouteMaxOutputs / 32, RULE>(logits, correction, experts, outputs, top_k, idx, weights, identity, counts);
}

}  // namespace rb
