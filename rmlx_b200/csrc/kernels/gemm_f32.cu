// fp32 GEMM on the CUDA cores: C[M,N] = A[M,K] W[N,K]^T in true 32-bit (FFMA, no reduced-precision
// tensor mode), for models run in 32-bit. A block owns a 64 x 64 tile, a thread 4 x 4 of it; K goes by
// in steps of 16 through shared memory, double-buffered in registers.
//
// Epilogues: plain store; split (columns before n_raw stored as they are, the others through xIELU
// into a second matrix); scaled accumulate (X[m, n] += s[n] * C[m, n], a layer scale and the
// residual sum). Grouped form: rows sorted by expert, blockIdx.z picks the expert's matrix and rows.
#include "../common/ptx.cuh"
#include "../common/launch.cuh"
#include "../common/xielu.cuh"

namespace rb {

constexpr int kSgTile = 64, kSgK = 16;
enum SgemmEpi : int { kSgPlain = 0, kSgSplit = 1, kSgAccumulate = 2 };

struct SgemmOut {
  float* c; int ldc;
  float* act; int ldact;      // split
  int n_raw;
  float ap, an;
  const float* scale;         // accumulate
  const int* offsets;         // grouped: rows offsets[z] .. offsets[z + 1] take matrix z of the stack
};

template <int EPI>
__global__ void __launch_bounds__(256)
sgemm_kernel(const float* __restrict__ A, int lda, const float* __restrict__ W, int ldw, int M, int N, int K,
             SgemmOut o) {
  __shared__ float sA[kSgK][kSgTile + 4], sW[kSgK][kSgTile + 4];
  pdl_launch_dependents();
  pdl_wait();
  if (o.offsets) {
    const int at = o.offsets[blockIdx.z];
    M = o.offsets[blockIdx.z + 1] - at;
    A += size_t(at) * lda;
    W += size_t(blockIdx.z) * N * ldw;
    o.c += size_t(at) * o.ldc;
  }
  const int m0 = blockIdx.y * kSgTile, n0 = blockIdx.x * kSgTile;
  if (m0 >= M) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  // loader: thread i brings four consecutive k of row i / 4
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float fa[4], fw[4];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      fa[i] = (m0 + lr < M && k < K) ? A[size_t(m0 + lr) * lda + k] : 0.f;
      fw[i] = (n0 + lr < N && k < K) ? W[size_t(n0 + lr) * ldw + k] : 0.f;
    }
  };
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  fetch(0);
  for (int k0 = 0; k0 < K; k0 += kSgK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) { sA[lk + i][lr] = fa[i]; sW[lk + i][lr] = fw[i]; }
    __syncthreads();
    if (k0 + kSgK < K) fetch(k0 + kSgK);
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sW[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      const float v = acc[i][j];
      if (EPI == kSgAccumulate) {
        o.c[size_t(m) * o.ldc + n] += o.scale[n] * v;
      } else if (EPI == kSgSplit && n >= o.n_raw) {
        o.act[size_t(m) * o.ldact + n - o.n_raw] = xielu(v, o.ap, o.an);
      } else {
        o.c[size_t(m) * o.ldc + n] = v;
      }
    }
  }
}

template <int EPI>
static int launch_sgemm(const float* A, int lda, const float* W, int ldw, int M, int N, int K, SgemmOut o,
                        int pdl, cudaStream_t st, int groups = 1) {
  const dim3 grid((N + kSgTile - 1) / kSgTile, (M + kSgTile - 1) / kSgTile, groups);
  if (grid.y > 65535u) return -2;
  return launch(sgemm_kernel<EPI>, grid, dim3(256), 0, st, pdl != 0, A, lda, W, ldw, M, N, K, o);
}

}  // namespace rb

using namespace rb;

// c[M, N] = A W^T, fp32 throughout.
extern "C" int rmlx_sgemm(const float* A, int lda, const float* W, int ldw, float* c, int ldc, int M, int N,
                          int K, int pdl, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1) return -2;
  SgemmOut o{}; o.c = c; o.ldc = ldc;
  return launch_sgemm<kSgPlain>(A, lda, W, ldw, M, N, K, o, pdl, st);
}

// Columns before n_raw to c, the others through xIELU to act (column n - n_raw).
extern "C" int rmlx_sgemm_split_xielu(const float* A, int lda, const float* W, int ldw, float* c, int ldc,
                                      int n_raw, float* act, int ldact, float ap, float an, int M, int N, int K,
                                      int pdl, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1 || n_raw < 0 || n_raw > N || (n_raw < N && !act)) return -2;
  SgemmOut o{}; o.c = c; o.ldc = ldc; o.act = act; o.ldact = ldact; o.n_raw = n_raw; o.ap = ap; o.an = an;
  return launch_sgemm<kSgSplit>(A, lda, W, ldw, M, N, K, o, pdl, st);
}

// x[m, n] += scale[n] * (A W^T)[m, n].
extern "C" int rmlx_sgemm_scaled_add(const float* A, int lda, const float* W, int ldw, const float* scale,
                                     float* x, int ldx, int M, int N, int K, int pdl, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1 || !scale) return -2;
  SgemmOut o{}; o.c = x; o.ldc = ldx; o.scale = scale;
  return launch_sgemm<kSgAccumulate>(A, lda, W, ldw, M, N, K, o, pdl, st);
}

// Grouped: A's rows are sorted by expert, W is the stack [E, N, ldw], offsets int32 [E + 1] on the device;
// M bounds the rows of one expert.
extern "C" int rmlx_sgemm_grouped(const float* A, int lda, const float* W, int ldw, const int* offsets, int E,
                                  float* c, int ldc, int M, int N, int K, int pdl, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1 || E < 1 || E > 65535 || !offsets) return -2;
  SgemmOut o{}; o.c = c; o.ldc = ldc; o.offsets = offsets;
  return launch_sgemm<kSgPlain>(A, lda, W, ldw, M, N, K, o, pdl, st, E);
}
