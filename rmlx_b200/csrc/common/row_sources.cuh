// What a row kernel adds to the residual: a sublayer's output rows, or the weighted rows of a token's experts.
#pragma once
#include "rows.cuh"

namespace rb {

// Eight consecutive values of row t from column c * 8 on.
template <class TY>
struct RowSource {
  const TY* y;
  int ldy;
  __device__ __forceinline__ void prepare(int) {}
  __device__ __forceinline__ void load(int t, int c, const float (&)[8], float (&f)[8]) const {
    load8(y + size_t(t) * ldy + c * 8, f);
  }
};
// Routed experts: sum over the token's slots of weight * expert output row (identity experts, and
// slots without a row, have row -1), plus the summed identity weight times the input itself.
template <class TY>
struct ExpertSource {
  const TY* y;
  int ldy;
  const int* row_of_pair;     // [T, top_k]
  const float* weights;       // [T, top_k]
  const float* identity;      // [T] summed weight of the identity experts, or null
  int top_k;
  float id_w;
  int rows[4];                // the first four slots
  float wts[4];
  __device__ __forceinline__ void prepare(int t) {
    id_w = identity ? identity[t] : 0.f;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      rows[u] = u < top_k ? row_of_pair[t * top_k + u] : -1;
      wts[u] = u < top_k ? weights[t * top_k + u] : 0.f;
    }
  }
  __device__ __forceinline__ void load(int t, int c, const float (&x)[8], float (&f)[8]) const {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = id_w * x[i];
    float g[4][8];
#pragma unroll
    for (int u = 0; u < 4; ++u) {                      // four slots' rows in flight
      if (rows[u] >= 0) {
        load8(y + size_t(rows[u]) * ldy + c * 8, g[u]);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) g[u][i] = 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = fmaf(wts[u], g[u][i], f[i]);
    for (int s = 4; s < top_k; ++s) {
      const int row = row_of_pair[t * top_k + s];
      if (row < 0) continue;
      const float a = weights[t * top_k + s];
      load8(y + size_t(row) * ldy + c * 8, g[0]);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = fmaf(a, g[0][i], f[i]);
    }
  }
};

}  // namespace rb
