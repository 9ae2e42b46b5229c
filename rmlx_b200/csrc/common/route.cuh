// Expert choice for one token by one full warp (see moe_route.cu).
#pragma once
#include "ptx.cuh"

namespace rb {

constexpr int kRouteMaxOutputs = 512;
constexpr int kRouteMaxTop = 32;

enum RouteRule {
  kRouteCorrected = 0,      // by softmax + correction; weights: the softmax over all outputs
  kRouteChosen = 1,         // by logit + correction (a bias); weights: the softmax over the chosen ones alone
  kRouteGrouped = 2,        // by sigmoid, only from the groups with the best pairs; weights: the sigmoids times `scale`
};

// kRouteGrouped: the outputs form `count` equal groups of neighbours (1: one group); the `keep` of them whose two largest
// scores have the largest sums are open. Behind a token's top_k choices come the experts outputs .. outputs + always - 1,
// with weight one: every token uses them.
struct RouteGroups {
  int count = 1, keep = 1, always = 0;
  float scale = 1.f;
};
constexpr int kRouteMaxGroups = 128;

// N: outputs a lane holds. logits, correction: fp32 [outputs], the first `experts` of them with weights of their own. Ties go to
// the lower index. counts (may be null) gets one more for every chosen expert.
template <int N, RouteRule RULE>
__device__ __forceinline__ void warp_route_n(const float* logits, const float* correction, int experts, int outputs,
                                             int top_k, int* idx, float* weights, float* identity, int* counts,
                                             const RouteGroups& groups) {
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
  if (RULE == kRouteGrouped) {
    constexpr int G = kRouteMaxGroups / 32;
    uint32_t open[G];                                      // a bit per group
    // a lane per group (in turns): the sum of its two largest scores
    const int per = outputs / groups.count;
    float gs[G];
#pragma unroll
    for (int j = 0; j < G; ++j) {
      gs[j] = -INFINITY;
      open[j] = 0u;
      const int g = j * 32 + lane;
      if (g < groups.count) {
        float a = 0.f, b = 0.f;                            // sigmoids are positive
        for (int i = 0; i < per; ++i) {
          const float v = 1.f / (1.f + expf(-logits[g * per + i]));
          if (v > a) { b = a; a = v; }
          else if (v > b) b = v;
        }
        gs[j] = a + b;
      }
    }
    for (int r = 0; r < groups.keep; ++r) {
      float best = -INFINITY;
      int bg = 0x7fffffff;
#pragma unroll
      for (int j = 0; j < G; ++j)
        if (gs[j] > best) { best = gs[j]; bg = j * 32 + lane; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int og = __shfl_xor_sync(0xffffffffu, bg, o);
        if (ob > best || (ob == best && og < bg)) { best = ob; bg = og; }
      }
#pragma unroll
      for (int j = 0; j < G; ++j) {
        if (bg >> 5 == j) open[j] |= 1u << (bg & 31);
        if (bg == j * 32 + lane) gs[j] = -INFINITY;
      }
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int e = i * 32 + lane, g = e < outputs ? e / per : 0;
      uint32_t word = 0u;
#pragma unroll
      for (int j = 0; j < G; ++j)
        if (g >> 5 == j) word = open[j];
      s[i] = 1.f / (1.f + expf(-s[i]));
      c[i] = e < outputs && (word >> (g & 31) & 1u) ? s[i] : -INFINITY;
      s[i] *= groups.scale;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int e = i * 32 + lane;
      c[i] = e < outputs ? s[i] + correction[e] : -INFINITY;
      if (RULE == kRouteChosen) s[i] = c[i];
    }
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
  if (RULE == kRouteGrouped && lane >= top_k && lane < top_k + groups.always) {
    idx[lane] = outputs + lane - top_k;                    // (their rows need no counting)
    weights[lane] = 1.f;
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
                                           int* idx, float* weights, float* identity, int* counts,
                                           const RouteGroups& groups = RouteGroups{}) {
  if (outputs <= 64) warp_route_n<2, RULE>(logits, correction, experts, outputs, top_k, idx, weights, identity, counts, groups);
  else if (outputs <= 256) warp_route_n<8, RULE>(logits, correction, experts, outputs, top_k, idx, weights, identity, counts, groups);
  else warp_route_n<kRouteMaxOutputs / 32, RULE>(logits, correction, experts, outputs, top_k, idx, weights, identity, counts, groups);
}
// Whether a routing by groups is possible.
__host__ __device__ inline bool route_groups_ok(const RouteGroups& g, int outputs, int top_k) {
  return g.count >= 1 && g.count <= kRouteMaxGroups && outputs % g.count == 0 && g.keep >= 1 && g.keep <= g.count &&
         top_k <= g.keep * (outputs / g.count) && g.always >= 0 && top_k + g.always <= kRouteMaxTop;
}

}  // namespace rb
