// Decode projections of a parallel block (one norm, attention and feed-forward side by side, fp32
// residual stream), one warp per weight-row pair as in decode_gemv.cu:
//
//   parallel_in   y = W rmsnorm(x), W = [q; k; v; up]: rows before n_raw go out as fp32 (attention
//                 normalises and appends them), rows from n_raw on through xIELU to bf16. Also the
//                 final norm + LM head (all rows fp32).
//   parallel_out  x += ls1 * (Wo a) + ls2 * (Wdown act): both sublayers' down projections, their
//                 layer scales and the residual sum in one kernel.
//
// A parallel block is thus three launches per decoded token: parallel_in, attention, parallel_out.
#include "../common/gemv_core.cuh"
#include "../common/launch.cuh"
#include "../common/xielu.cuh"

namespace rb {

constexpr int kPgRows = 2;        // weight rows a warp accumulates together

template <int B>
__global__ void __launch_bounds__(kGemvThreads)
parallel_in_kernel(Matrix<WBf16> W, const float* __restrict__ x, int x_stride,
                   const float* __restrict__ norm_w, float eps, int D, float* __restrict__ raw,
                   int raw_stride, int n_raw, __nv_bfloat16* __restrict__ act, int act_stride, int N,
                   float ap, float an) {
  extern __shared__ __align__(16) char smem[];
  __shared__ float red[kGemvWarps];
  __shared__ float inv_rms[B];
  const int K = W.K;
  const size_t bstride = XStage<WBf16>::bytes(K);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int n0 = (blockIdx.x * kGemvWarps + warp) * kPgRows;
  RowBf16 rows[kPgRows];
  Tile<RowBf16, kPgRows> t0;
  if (n0 < N) {                 // weights wait for nothing: ask for the first tile at once
#pragma unroll
    for (int r = 0; r < kPgRows; ++r) rows[r] = W.row(min(n0 + r, N - 1));
    load_tile<kPgRows>(rows, K, 0, t0);
  }
  pdl_launch_dependents();
  pdl_wait();
#pragma unroll
  for (int b = 0; b < B; ++b) {
    XLoadF32 ld{x + size_t(b) * x_stride, norm_w, 0.f};
    XStage<WBf16>::stage_with(smem + b * bstride, K, ld);
    const float ssq = block_sum_256(ld.ssq, red);
    if (threadIdx.x == 0) inv_rms[b] = 1.f / sqrtf(ssq / float(D) + eps);
  }
  __syncthreads();
  for (bool first = true; n0 < N; n0 += gridDim.x * kGemvWarps * kPgRows, first = false) {
    if (!first) {
#pragma unroll
      for (int r = 0; r < kPgRows; ++r) rows[r] = W.row(min(n0 + r, N - 1));
      load_tile<kPgRows>(rows, K, 0, t0);
    }
    float acc[kPgRows][B];
#pragma unroll
    for (int r = 0; r < kPgRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) acc[r][b] = 0.f;
    warp_dot<kPgRows, B, RowBf16>(rows, smem, bstride, K, acc, t0);
#pragma unroll
    for (int r = 0; r < kPgRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const float v = warp_sum(acc[r][b]) * inv_rms[b];
        const int n = n0 + r;
        if (lane == r * B + b && n < N) {
          if (n < n_raw) raw[size_t(b) * raw_stride + n] = v;
          else act[size_t(b) * act_stride + n - n_raw] = __float2bfloat16_rn(xielu(v, ap, an));
        }
      }
  }
}

template <int B>
__global__ void __launch_bounds__(kGemvThreads)
parallel_out_kernel(Matrix<WBf16> Wo, Matrix<WBf16> Wd, const __nv_bfloat16* __restrict__ a, int a_stride,
                    const __nv_bfloat16* __restrict__ act, int act_stride, const float* __restrict__ ls1,
                    const float* __restrict__ ls2, float* __restrict__ x, int x_stride, int N) {
  extern __shared__ __align__(16) char smem[];
  const int K1 = Wo.K, K2 = Wd.K;        // K2 == 0: no feed-forward in this layer
  const size_t s1 = XStage<WBf16>::bytes(K1), s2 = XStage<WBf16>::bytes(K2);
  char* sm_act = smem + B * s1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int n0 = (blockIdx.x * kGemvWarps + warp) * kPgRows;
  RowBf16 ro[kPgRows], rd[kPgRows];
  Tile<RowBf16, kPgRows> t0;
  auto point = [&]() {
#pragma unroll
    for (int r = 0; r < kPgRows; ++r) {
      ro[r] = Wo.row(min(n0 + r, N - 1));
      rd[r] = Wd.row(min(n0 + r, N - 1));
    }
  };
  if (n0 < N) {
    point();
    load_tile<kPgRows>(ro, K1, 0, t0);
  }
  pdl_launch_dependents();
  pdl_wait();
#pragma unroll
  for (int b = 0; b < B; ++b) {
    XLoadBf16 la{a + size_t(b) * a_stride, nullptr, 0.f};
    XStage<WBf16>::stage_part(smem + b * s1, K1, la, threadIdx.x, kGemvThreads);
    if (K2 > 0) {
      XLoadBf16 lf{act + size_t(b) * act_stride, nullptr, 0.f};
      XStage<WBf16>::stage_part(sm_act + b * s2, K2, lf, threadIdx.x, kGemvThreads);
    }
  }
  __syncthreads();
  for (bool first = true; n0 < N; n0 += gridDim.x * kGemvWarps * kPgRows, first = false) {
    if (!first) {
      point();
      load_tile<kPgRows>(ro, K1, 0, t0);
    }
    float acc1[kPgRows][B], acc2[kPgRows][B];
#pragma unroll
    for (int r = 0; r < kPgRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) acc1[r][b] = acc2[r][b] = 0.f;
    warp_dot<kPgRows, B, RowBf16>(ro, smem, s1, K1, acc1, t0);
    if (K2 > 0) warp_dot<kPgRows, B, RowBf16>(rd, sm_act, s2, K2, acc2);
#pragma unroll
    for (int r = 0; r < kPgRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const float m = warp_sum(acc1[r][b]);
        const float f = K2 > 0 ? warp_sum(acc2[r][b]) : 0.f;
        const int n = n0 + r;
        if (lane == r * B + b && n < N) {
          float delta = ls1[n] * m;
          if (K2 > 0) delta += ls2[n] * f;
          float* dst = x + size_t(b) * x_stride + n;
          *dst = __ldcg(dst) + delta;
        }
      }
  }
}

static int pg_grid(int rows) {
  const int per = kGemvWarps * kPgRows;
  const int want = (rows + per - 1) / per, cap = sm_count() * 8;
  return want < cap ? (want > 0 ? want : 1) : cap;
}

template <int B>
static int launch_parallel_in(const void* w, const float* x, int x_stride, const float* norm_w, float eps,
                              int D, float* raw, int raw_stride, int n_raw, void* act, int act_stride,
                              int N, int K, float ap, float an, int pdl, cudaStream_t st) {
  const size_t smem = XStage<WBf16>::bytes(K) * B;
  auto kern = parallel_in_kernel<B>;
  RB_CHECK(set_max_smem(kern, smem));
  return launch(kern, dim3(pg_grid(N)), dim3(kGemvThreads), smem, st, pdl != 0,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(w), K}, x, x_stride, norm_w, eps, D, raw,
                raw_stride, n_raw, static_cast<__nv_bfloat16*>(act), act_stride, N, ap, an);
}

template <int B>
static int launch_parallel_out(const void* wo, const void* wd, const void* a, int a_stride, const void* act,
                               int act_stride, const float* ls1, const float* ls2, float* x, int x_stride,
                               int N, int K1, int K2, int pdl, cudaStream_t st) {
  const size_t smem = (XStage<WBf16>::bytes(K1) + XStage<WBf16>::bytes(K2)) * B;
  auto kern = parallel_out_kernel<B>;
  RB_CHECK(set_max_smem(kern, smem));
  return launch(kern, dim3(pg_grid(N)), dim3(kGemvThreads), smem, st, pdl != 0,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(wo), K1},
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(wd), K2},
                static_cast<const __nv_bfloat16*>(a), a_stride, static_cast<const __nv_bfloat16*>(act),
                act_stride, ls1, ls2, x, x_stride, N);
}

constexpr size_t kPgMaxSmem = 220 * 1024;

}  // namespace rb

using namespace rb;

// Rows (activation vectors) one launch takes for staged widths adding up to K values: at most four,
// fewer when the fp32 staging would not fit a block's shared memory, 0 when one row does not.
extern "C" int rmlx_parallel_gemv_max_rows(int K) {
  const size_t per = size_t(K) * 4;
  int b = 4;
  while (b > 0 && per * b > kPgMaxSmem) --b;
  return b;
}

#define RB_PG_DISPATCH(B_, CALL)                     \
  switch (B_) {                                      \
    case 1: { constexpr int kB = 1; return CALL; }   \
    case 2: { constexpr int kB = 2; return CALL; }   \
    case 3: { constexpr int kB = 3; return CALL; }   \
    case 4: { constexpr int kB = 4; return CALL; }   \
    default: return -2;                              \
  }

// W bf16 [N, K]; x fp32 [B, x_stride]; norm_w fp32 [K]; the mean square is taken over D <= K values
// (columns from D on are zero). Rows n < n_raw: fp32 into raw [B, raw_stride]; the others:
// xIELU(row) in bf16 into act [B, act_stride] at column n - n_raw.
extern "C" int rmlx_parallel_in(const void* w, const float* x, int x_stride, const float* norm_w, float eps,
                                int D, float* raw, int raw_stride, int n_raw, void* act, int act_stride,
                                int B, int N, int K, float ap, float an, int pdl, cudaStream_t st) {
  if (K < 8 || K % 8 || x_stride % 4 || D < 1 || D > K || N < 1 || n_raw < 0 || n_raw > N ||
      (n_raw > 0 && !raw) || (n_raw < N && !act) || B > rmlx_parallel_gemv_max_rows(K))
    return -2;
  RB_PG_DISPATCH(B, (launch_parallel_in<kB>(w, x, x_stride, norm_w, eps, D, raw, raw_stride, n_raw, act,
                                            act_stride, N, K, ap, an, pdl, st)))
}

// Wo bf16 [N, K1], Wdown bf16 [N, K2] (K2 == 0: none); a bf16 [B, a_stride], act bf16 [B, act_stride];
// x fp32 [B, x_stride] is updated in place.
extern "C" int rmlx_parallel_out(const void* wo, const void* wd, const void* a, int a_stride, const void* act,
                                 int act_stride, const float* ls1, const float* ls2, float* x, int x_stride,
                                 int B, int N, int K1, int K2, int pdl, cudaStream_t st) {
  if (K1 < 8 || K1 % 8 || K2 < 0 || K2 % 8 || a_stride % 8 || act_stride % 8 || N < 1 ||
      B > rmlx_parallel_gemv_max_rows(K1 + K2))
    return -2;
  RB_PG_DISPATCH(B, (launch_parallel_out<kB>(wo, wd, a, a_stride, act, act_stride, ls1, ls2, x, x_stride, N,
                                             K1, K2, pdl, st)))
}
