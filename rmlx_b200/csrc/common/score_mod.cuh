// Attention-score modifiers shared by the attention kernels that take them: what happens to q . k
// between the product and the softmax. Every part is optional, so designs pick what they need:
//
//   s = (q . k) * scale * temp[h]               per-head temperature (temp == nullptr: 1)
//   s = softcap * tanh(s / softcap)             logit soft cap       (softcap <= 0: none)
//   s = s - r1[h] * ln(1 + r2[h] * (i - j))     logarithmic distance bias (r1 == nullptr: none)
//   weights = exp(s) / (sum exp(s) + exp(sink[h]))    sink without key or value (nullptr: none)
//   o = o * sigmoid(gate[t, h])                 output gate, one logit per token and head (nullptr: none)
//
// Differential attention: a head has two maps, each a query and a key of its own over the same values, and
//   d = softmax(map 1) v - weight * softmax(map 2) v,   o = scale * d / sqrt(mean(d^2) + eps)     (MapDiff)
//
// The tensor-core kernels work in base 2 (scores times log2 e), which leaves one ex2 per weight.
#pragma once
#include "ptx.cuh"

namespace rb {

constexpr float kLog2e = 1.4426950408889634f;

struct ScoreMod {
  float scale = 1.f;
  float softcap = 0.f;
  const float* temp = nullptr;
  const float* r1 = nullptr;
  const float* r2 = nullptr;
  const float* sink = nullptr;
};

struct MapDiff {
  float weight = 0.f, scale = 1.f, eps = 0.f;
};

// The first key a query at position `pos` sees: the last `window` keys (> 0), only its own chunk of `chunk`
// positions counted from 0 (> 0), or every key before it.
__device__ __forceinline__ int first_key(int pos, int window, int chunk) {
  int first = window > 0 ? max(0, pos - window + 1) : 0;
  if (chunk > 0) first = max(first, pos - pos % chunk);
  return first;
}

// Gate logits of token t, head h at gate[t * ld + h], in the activations' type.
struct HeadGate {
  const void* gate = nullptr;
  int ld = 0;
};
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
template <class T>
__device__ __forceinline__ float head_gate(const HeadGate& g, size_t t, int h) {
  return g.gate ? sigmoid_f(float(static_cast<const T*>(g.gate)[t * g.ld + h])) : 1.f;
}

// tanh(u) / u as a polynomial in u^2, |u| <= kTanhPolyMax: Chebyshev interpolation of degree 4 in
// u^2, largest relative error 1.6e-7 (fp32 evaluation included).
constexpr float kTanhPolyMax = 0.625f;
constexpr float kTanhP0 = 0.9999998807907104f, kTanhP1 = -0.33331942558288574f,
                kTanhP2 = 0.1330437958240509f, kTanhP3 = -0.05181591212749481f,
                kTanhP4 = 0.015043356455862522f;

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// tanh for |u| <= kTanhPolyMax.
__device__ __forceinline__ float tanh_near(float u) {
  const float w = u * u;
  return u * fmaf(fmaf(fmaf(fmaf(kTanhP4, w, kTanhP3), w, kTanhP2), w, kTanhP1), w, kTanhP0);
}
// tanh with small relative error everywhere: the polynomial near zero, 1 - 2 / (1 + e^(2u)) beyond
// (which saturates to +-1 without overflow trouble).
__device__ __forceinline__ float tanh_any(float u) {
  const float far = 1.f - __fdividef(2.f, 1.f + ex2_approx(fminf(u, 40.f) * (2.f * kLog2e)));
  return fabsf(u) <= kTanhPolyMax ? tanh_near(u) : far;
}

// One head's modifiers, in base-2 units.
struct HeadScore {
  float lin;       // scale * temp * log2 e without a cap, else 0
  float inner;     // scale * temp / softcap, 0 without a cap
  float capl;      // softcap * log2 e, 0 without a cap
  float r1, r2;    // r1 as given: r1 * log2(1 + r2 d) is already r1 * ln(..) in base-2 units
  float sink;      // sink * log2 e; -inf without one
};

__device__ __forceinline__ HeadScore head_score(const ScoreMod& m, int h) {
  HeadScore s;
  const float st = m.scale * (m.temp ? m.temp[h] : 1.f);
  s.lin = m.softcap > 0.f ? 0.f : st * kLog2e;
  s.inner = m.softcap > 0.f ? st / m.softcap : 0.f;
  s.capl = m.softcap > 0.f ? m.softcap * kLog2e : 0.f;
  s.r1 = m.r1 ? m.r1[h] : 0.f;
  s.r2 = m.r1 ? m.r2[h] : 0.f;
  s.sink = m.sink ? m.sink[h] * kLog2e : -INFINITY;
  return s;
}

__device__ __forceinline__ float distance_bias(const HeadScore& s, float dist) {
  return s.r1 * __log2f(fmaf(s.r2, dist, 1.f));
}

// Base-2 scores of N dot products of one head at distances dist[i] (i - j, taken as 0 where
// negative), in place and without branches per score. `near`: every |dot * inner| is within the
// polynomial's range.
template <int N>
__device__ __forceinline__ void scores_base2(float* dot, const HeadScore& s, const float* dist, bool near) {
  float th[N];
  if (near) {
#pragma unroll
    for (int i = 0; i < N; ++i) th[i] = tanh_near(dot[i] * s.inner);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) th[i] = tanh_any(dot[i] * s.inner);
  }
#pragma unroll
  for (int i = 0; i < N; ++i)
    dot[i] = fmaf(s.capl, th[i], dot[i] * s.lin) - distance_bias(s, fmaxf(dist[i], 0.f));
}

}  // namespace rb
