// Decode projections whose input is finished while it is staged, one warp per weight-row pair as in decode_gemv.cu, and the
// state step of heads with a constant decay:
//
//   poly_out        y = W (a N(z) + b N(z^2) + c N(z^3) + e), N: division by the row's root mean square
//   gated_out       y = W (o / rms(o) * w * sigmoid(gate))
//   lightning_step  one token: q, k, v through silu, S <- decay S + k v^T, o = S^T q
//
// Everything is fp32 beside bf16 weights; lightning_step also takes bf16 rows (larger batches, whose projections are GEMMs).
#include <type_traits>

#include "../common/gemv_core.cuh"
#include "../common/launch.cuh"
#include "../common/state_step.cuh"

namespace rb {

constexpr int kSwRows = 2;        // weight rows a warp accumulates together
constexpr size_t kSwMaxSmem = 220 * 1024;

__device__ __forceinline__ void sw_load8(const float* p, int c, float (&f)[8]) {
  const float4 a = __ldcg(reinterpret_cast<const float4*>(p + c * 8));
  const float4 e = __ldcg(reinterpret_cast<const float4*>(p + c * 8 + 4));
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = e.x; f[5] = e.y; f[6] = e.z; f[7] = e.w;
}

// Both stage row b (split-chunk layout of gemv_core.cuh, 256 threads) and return what the products are multiplied by.
struct PolySource {
  const float* z;           // [B, ld], the first D values of a row
  const float* act;         // [4]
  float eps;
  int ld, D;
  __device__ __forceinline__ float stage(int b, int K, char* xs, float* red) const {
    const int chunks = K >> 3;
    float4* dst = reinterpret_cast<float4*>(xs);
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
#pragma unroll 4
    for (int c = threadIdx.x; c < chunks; c += kGemvThreads) {
      float f[8];
      sw_load8(z + size_t(b) * ld, c, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (c * 8 + i >= D) f[i] = 0.f;
        const float q = f[i] * f[i], q2 = q * q;
        s2 += q;
        s4 += q2;
        s6 = fmaf(q2, q, s6);
      }
      dst[c] = make_float4(f[0], f[1], f[2], f[3]);
      dst[chunks + c] = make_float4(f[4], f[5], f[6], f[7]);
    }
    const float k0 = act[0] / sqrtf(block_sum_256(s2, red) / float(D) + eps);
    const float k1 = act[1] / sqrtf(block_sum_256(s4, red) / float(D) + eps);
    const float k2 = act[2] / sqrtf(block_sum_256(s6, red) / float(D) + eps);
    const float e = act[3];
    auto poly = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, k2, k1), k0), e); };
    for (int c = threadIdx.x; c < chunks; c += kGemvThreads) {     // (this thread wrote them; past D the weights are zero)
      const float4 a = dst[c], o = dst[chunks + c];
      dst[c] = make_float4(poly(a.x), poly(a.y), poly(a.z), poly(a.w));
      dst[chunks + c] = make_float4(poly(o.x), poly(o.y), poly(o.z), poly(o.w));
    }
    return 1.f;
  }
};
struct GatedSource {
  const float* o;           // [B, ld]
  const float* gate;        // [B, ld_g]
  const float* w;           // [D]
  float eps;
  int ld, ld_g, D;
  __device__ __forceinline__ float stage(int b, int K, char* xs, float* red) const {
    const int chunks = K >> 3;
    float4* dst = reinterpret_cast<float4*>(xs);
    float ssq = 0.f;
#pragma unroll 2
    for (int c = threadIdx.x; c < chunks; c += kGemvThreads) {
      float f[8], g[8];
      sw_load8(o + size_t(b) * ld, c, f);
      sw_load8(gate + size_t(b) * ld_g, c, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const bool in = c * 8 + i < D;
        ssq += in ? f[i] * f[i] : 0.f;
        f[i] = in ? __fdividef(f[i] * w[c * 8 + i], 1.f + __expf(fminf(-g[i], 80.f))) : 0.f;
      }
      dst[c] = make_float4(f[0], f[1], f[2], f[3]);
      dst[chunks + c] = make_float4(f[4], f[5], f[6], f[7]);
    }
    return 1.f / sqrtf(block_sum_256(ssq, red) / float(D) + eps);
  }
};

// y[b, n] = factor_b * W[n] . staged row b, n < N; the blocks walk the rows.
template <int B, class SRC>
__global__ void __launch_bounds__(kGemvThreads, 2)
staged_out_kernel(Matrix<WBf16> W, SRC src, float* __restrict__ y, int ld_y, int N) {
  extern __shared__ __align__(16) char smem[];
  __shared__ float red[kGemvWarps];
  const int K = W.K, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t bstride = XStage<WBf16>::bytes(K);
  int n0 = (blockIdx.x * kGemvWarps + warp) * kSwRows;
  RowBf16 rows[kSwRows];
  Tile<RowBf16, kSwRows> t0;
  auto point = [&]() {
#pragma unroll
    for (int r = 0; r < kSwRows; ++r) rows[r] = W.row(min(n0 + r, N - 1));
    load_tile<kSwRows>(rows, K, 0, t0);
  };
  if (n0 < N) point();          // weights wait for nothing: ask for the first tile at once
  pdl_launch_dependents();
  pdl_wait();
  float factor[B];
#pragma unroll
  for (int b = 0; b < B; ++b) factor[b] = src.stage(b, K, smem + b * bstride, red);
  __syncthreads();
  for (bool first = true; n0 < N; n0 += gridDim.x * kGemvWarps * kSwRows, first = false) {
    if (!first) point();
    float acc[kSwRows][B];
#pragma unroll
    for (int r = 0; r < kSwRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) acc[r][b] = 0.f;
    warp_dot<kSwRows, B, RowBf16>(rows, smem, bstride, K, acc, t0);
#pragma unroll
    for (int r = 0; r < kSwRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const float v = warp_sum(acc[r][b]);
        if (lane == r * B + b && n0 + r < N) y[size_t(b) * ld_y + n0 + r] = v * factor[b];
      }
  }
}

// Past the first-level cache: the launch before wrote them.
__device__ __forceinline__ float step_load(const float* p) { return __ldcg(p); }
__device__ __forceinline__ float step_load(const __nv_bfloat16* p) {
  return __uint_as_float(uint32_t(__ldcg(reinterpret_cast<const unsigned short*>(p))) << 16);
}

template <class T>
struct LightningStep {
  const T* raw;               // [B, ld_raw]: q at 0, k and v at their columns
  int ld_raw, at_k, at_v;
  const float* decay;             // [H]
  const int* slots;
  float* state;                   // slot s: state + s * stride, [H, n, d]
  long long stride;
  float* out;                     // [B, ld_out]
  int ld_out, n, d;
};

// grid (column blocks, heads, batch rows); COLS columns a block.
template <int COLS, int ROWS, class T>
__global__ void __launch_bounds__(kGemvThreads)
lightning_step_kernel(LightningStep<T> p) {
  constexpr int G = kGemvThreads / COLS;
  extern __shared__ float sm[];
  float* sr = sm;                    // [n] q, k
  float* sk = sr + p.n;
  __shared__ float part[kGemvThreads];
  __shared__ float red[kGemvWarps];
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, n = p.n, d = p.d;
  const int g = tid / COLS, col = blockIdx.x * COLS + tid % COLS;
  const int per = (n + G - 1) / G, i0 = g * per, i1 = min(i0 + per, n);
  float* sp = p.state + size_t(p.slots[b]) * p.stride + size_t(h) * n * d + col;
  float s[ROWS];
  load_state<ROWS>(sp, d, i0, i1, col < d, s);
  const float decay = p.decay[h];
  pdl_launch_dependents();
  pdl_wait();
  const T* row = p.raw + size_t(b) * p.ld_raw;
  float own = 0.f;
  if (tid < n) {
    const float q = step_silu(step_load(row + h * n + tid)), k = step_silu(step_load(row + p.at_k + h * n + tid));
    sr[tid] = q;
    sk[tid] = k;
    own = q * k;
  }
  const float v = col < d ? step_silu(step_load(row + p.at_v + h * d + col)) : 0.f;
  own = block_sum_256(own, red);     // sr and sk are visible, too
  part[tid] = col < d ? step_state<ROWS, true>(sp, d, i0, i1, s, sr, sk, nullptr, decay, v) : 0.f;
  __syncthreads();
  if (tid < COLS && col < d) {
    float o = 0.f;
#pragma unroll
    for (int u = 0; u < G; ++u) o += part[u * COLS + tid];
    p.out[size_t(b) * p.ld_out + h * d + col] = fmaf(decay, o, own * v);
  }
}

template <int B, class SRC>
static int launch_staged(const void* w, const SRC& src, float* y, int ld_y, int N, int K, int pdl, cudaStream_t st) {
  const size_t smem = XStage<WBf16>::bytes(K) * B;
  auto kern = staged_out_kernel<B, SRC>;
  RB_CHECK(set_max_smem(kern, smem));
  int per_sm = 1;
  RB_CHECK(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kern, kGemvThreads, smem));
  const int cap = sm_count() * (per_sm > 0 ? per_sm : 1), tiles = (N + kGemvWarps * kSwRows - 1) / (kGemvWarps * kSwRows);
  const int passes = (tiles + cap - 1) / cap;
  return launch(kern, dim3((tiles + passes - 1) / passes), dim3(kGemvThreads), smem, st, pdl != 0,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(w), K}, src, y, ld_y, N);
}
template <class SRC>
static int run_staged(const void* w, const SRC& src, float* y, int ld_y, int N, int K, int B, int pdl, cudaStream_t st) {
  if (N < 1 || K < 8 || K % 8 || ld_y < N || B < 1 || B > 4 || XStage<WBf16>::bytes(K) * B > kSwMaxSmem) return -2;
  if (B == 1) return launch_staged<1>(w, src, y, ld_y, N, K, pdl, st);
  if (B == 2) return launch_staged<2>(w, src, y, ld_y, N, K, pdl, st);
  if (B == 3) return launch_staged<3>(w, src, y, ld_y, N, K, pdl, st);
  return launch_staged<4>(w, src, y, ld_y, N, K, pdl, st);
}

}  // namespace rb

using namespace rb;

// w bf16 [N, K] (zero from column D on); z fp32 [B, ld >= K], ld a multiple of four; act fp32 [4]; y fp32 [B, ld_y]. B as
// rmlx_postnorm_max_rows(K) allows.
extern "C" int rmlx_poly_out(const void* w, const float* z, int ld, const float* act, float eps, float* y, int ld_y, int B, int N,
                             int K, int D, int pdl, cudaStream_t st) {
  if (D < 1 || D > K || ld < K || ld % 4 || !act) return -2;
  return run_staged(w, PolySource{z, act, eps, ld, D}, y, ld_y, N, K, B, pdl, st);
}

// w bf16 [N, K]; o fp32 [B, ld_o >= K], gate fp32 [B, ld_g >= K] (16-byte aligned, strides multiples of four), norm fp32 [D].
extern "C" int rmlx_gated_out(const void* w, const float* o, int ld_o, const float* gate, int ld_g, const float* norm, float eps,
                              float* y, int ld_y, int B, int N, int K, int D, int pdl, cudaStream_t st) {
  if (D < 1 || D > K || ld_o < K || ld_g < K || (ld_o | ld_g) % 4 || (reinterpret_cast<uintptr_t>(gate) & 15)) return -2;
  return run_staged(w, GatedSource{o, gate, norm, eps, ld_o, ld_g, D}, y, ld_y, N, K, B, pdl, st);
}

// raw fp32 (f32) or bf16 [B, ld_raw] with q at 0; out fp32 [B, ld_out]; n <= 256.
extern "C" int rmlx_lightning_step(const void* raw, int ld_raw, int at_k, int at_v, const float* decay, const int* slots, float* state,
                                   long long stride, float* out, int ld_out, int B, int H, int n, int d, int f32, int pdl,
                                   cudaStream_t st) {
  if (B < 1 || B > 65535 || H < 1 || H > 65535 || n < 1 || n > 256 || d < 1 || !slots || !decay || at_k < H * n || ld_out < H * d ||
      ld_raw < at_v + H * d || ld_raw < at_k + H * n)
    return -2;
  const size_t smem = size_t(2 * n) * sizeof(float);
  auto run = [&](auto* rows) -> int {
    using T = std::remove_const_t<std::remove_pointer_t<decltype(rows)>>;
    const LightningStep<T> p{rows, ld_raw, at_k, at_v, decay, slots, state, stride, out, ld_out, n, d};
    // a head's columns need not meet in one block
#define RB_LS(C_, R_) return launch_columns(lightning_step_kernel<C_, R_, T>, p, (d + C_ - 1) / C_, H, B, smem, false, pdl, st)
    RB_STATE_DISPATCH(n, 1, RB_LS);
#undef RB_LS
  };
  return f32 ? run(static_cast<const float*>(raw)) : run(static_cast<const __nv_bfloat16*>(raw));
}
