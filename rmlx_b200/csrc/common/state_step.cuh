// One decode token of a recurrent layer: a block holds some columns of a head's fp32 state [n, d], its threads a few rows of
// one column each.
#pragma once
#include "gemv_core.cuh"
#include "launch.cuh"

namespace rb {

__device__ __forceinline__ float step_silu(float z) { return z / (1.f + expf(-z)); }

// State rows of one thread: rows i0 .. i0 + ROWS - 1 (below i1) of one column. They belong to the calling kernel alone
// within a step, so they are asked for before the wait (the step's first kernel has waited for everything before it).
template <int ROWS>
__device__ __forceinline__ void load_state(const float* sp, int d, int i0, int i1, bool live, float (&s)[ROWS]) {
#pragma unroll
  for (int q = 0; q < ROWS; ++q) s[q] = (live && i0 + q < i1) ? __ldcg(sp + size_t(i0 + q) * d) : 0.f;
}
// Their part of S^T r, and S <- w S + k v (w: per row, or one for all).
template <int ROWS, bool ONE>
__device__ __forceinline__ float step_state(float* sp, int d, int i0, int i1, const float (&s)[ROWS], const float* r, const float* k,
                                            const float* w, float one, float v) {
  float o = 0.f;
#pragma unroll
  for (int q = 0; q < ROWS; ++q) {
    const int i = i0 + q;
    if (i < i1) {
      o = fmaf(r[i], s[q], o);
      sp[size_t(i) * d] = fmaf(ONE ? one : w[i], s[q], k[i] * v);
    }
  }
  return o;
}


// Launches a (column blocks, heads, rows) grid with the column blocks of a head as one cluster.
template <class P>
static int launch_columns(void (*kern)(P), const P& p, int blocks, int H, int B, size_t smem, bool cluster, int pdl,
                          cudaStream_t st) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(blocks, H, B);
  cfg.blockDim = dim3(kGemvThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (cluster && blocks > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = blocks; attr[n].val.clusterDim.y = 1; attr[n].val.clusterDim.z = 1;
    ++n;
  }
  if (pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
    prefer_max_shared(kern);
  }
  cfg.attrs = attr; cfg.numAttrs = n;
  const cudaError_t e = cudaLaunchKernelEx(&cfg, kern, p);
  if (e != cudaSuccess) (void)cudaGetLastError();
  return static_cast<int>(e);
}

// The instance for n state rows and d columns: CALL(COLS, ROWS); clusters hold at most eight blocks.
#define RB_STATE_DISPATCH(n_, d_, CALL)                        \
  if ((d_) <= 256) {                                     \
    if ((n_) <= 32) { CALL(32, 4); }                     \
    if ((n_) <= 64) { CALL(32, 8); }                     \
    if ((n_) <= 128) { CALL(32, 16); }                   \
    CALL(32, 32);                                        \
  }                                                      \
  if ((n_) <= 64) { CALL(64, 16); }                      \
  if ((n_) <= 128) { CALL(64, 32); }                     \
  CALL(64, 64)

}  // namespace rb
