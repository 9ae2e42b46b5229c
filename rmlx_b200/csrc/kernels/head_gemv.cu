// Per-head products of a few rows: out[t, h, :] = W[h] in[t, h, :], W [H, N, K]. The two sides of
// absorbed latent attention: queries into the latent space (W = the transposed key up-projection) and
// attended latents to values. A block owns a tile of one head's output channels for up to four rows,
// staged as fp32 in shared memory; L lanes share a weight row. fp32 accumulation.
#include "../common/launch.cuh"
#include "../common/rows.cuh"

namespace rb {

constexpr int kHgRows = 4;          // rows of the batch per block
constexpr int kHgWarps = 8;

// TILE: output channels per block (few rows: small tiles, so that the weights come from many SMs at once).
template <class T, int L, int TILE>
__global__ void __launch_bounds__(kHgWarps * 32)
head_gemv_kernel(const T* __restrict__ w, const T* __restrict__ in, int in_t, int in_h, T* __restrict__ out, int out_t,
                 int out_h, const int* __restrict__ row_ids, int rows, int N, int K) {
  extern __shared__ __align__(16) float xs[];       // [kHgRows][2][K / 2]: first and second halves of the chunks
  const int h = blockIdx.y, n0 = blockIdx.x * TILE, t0 = blockIdx.z * kHgRows;
  const int nt = min(kHgRows, rows - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, chunks = K >> 3;
  constexpr int PER = 32 / L;                        // weight rows a warp holds at once
  const int sub = lane / L, sl = lane % L;
  float f0[8];                                       // weights wait for nothing: the first chunk is asked for at once
  load8(w + (size_t(h) * N + min(n0 + warp * PER + sub, N - 1)) * K + min(sl, chunks - 1) * 8, f0);
  pdl_launch_dependents();
  pdl_wait();
  for (int i = threadIdx.x; i < kHgRows * chunks; i += kHgWarps * 32) {
    const int b = i / chunks, c = i - b * chunks;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (b < nt) {
      const int t = row_ids ? row_ids[t0 + b] : t0 + b;
      load8(in + size_t(t) * in_t + size_t(h) * in_h + c * 8, f);
    }
    float4* d = reinterpret_cast<float4*>(xs + b * K);
    d[c] = make_float4(f[0], f[1], f[2], f[3]);
    d[chunks + c] = make_float4(f[4], f[5], f[6], f[7]);
  }
  __syncthreads();
  for (int r = warp * PER + sub; r < TILE; r += kHgWarps * PER) {
    const int n = n0 + r;                            // the lanes of a row leave the loop together with their warp
    const T* row = w + (size_t(h) * N + min(n, N - 1)) * K;
    float acc[kHgRows] = {0.f, 0.f, 0.f, 0.f};
    for (int c = sl; c < chunks; c += L) {
      float f[8];
      if (r == warp * PER + sub && c == sl) {
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = f0[i];
      } else {
        load8(row + c * 8, f);
      }
#pragma unroll
      for (int b = 0; b < kHgRows; ++b) {
        const float4* d = reinterpret_cast<const float4*>(xs + b * K);
        const float4 a = d[c], e = d[chunks + c];
        acc[b] = fmaf(f[0], a.x, acc[b]); acc[b] = fmaf(f[1], a.y, acc[b]);
        acc[b] = fmaf(f[2], a.z, acc[b]); acc[b] = fmaf(f[3], a.w, acc[b]);
        acc[b] = fmaf(f[4], e.x, acc[b]); acc[b] = fmaf(f[5], e.y, acc[b]);
        acc[b] = fmaf(f[6], e.z, acc[b]); acc[b] = fmaf(f[7], e.w, acc[b]);
      }
    }
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1)
#pragma unroll
      for (int b = 0; b < kHgRows; ++b) acc[b] += __shfl_xor_sync(0xffffffffu, acc[b], o);
    if (sl < nt && n < N) {
      float v = acc[0];
#pragma unroll
      for (int b = 1; b < kHgRows; ++b) v = sl == b ? acc[b] : v;
      const int t = row_ids ? row_ids[t0 + sl] : t0 + sl;
      out[size_t(t) * out_t + size_t(h) * out_h + n] = from_f32<T>(v);
    }
  }
}

template <class T, int TILE>
static int launch_head_gemv(const T* w, const T* in, int in_t, int in_h, T* out, int out_t, int out_h,
                            const int* row_ids, int rows, int H, int N, int K, int pdl, cudaStream_t st) {
  const dim3 grid((N + TILE - 1) / TILE, H, (rows + kHgRows - 1) / kHgRows);
  const size_t smem = size_t(kHgRows) * K * sizeof(float);
  auto go = [&](auto kern) -> int {
    RB_CHECK(set_max_smem(kern, smem));
    return launch(kern, grid, dim3(kHgWarps * 32), smem, st, pdl != 0, w, in, in_t, in_h, out, out_t, out_h, row_ids,
                  rows, N, K);
  };
  if (K <= 64) return go(head_gemv_kernel<T, 8, TILE>);
  if (K <= 128) return go(head_gemv_kernel<T, 16, TILE>);
  return go(head_gemv_kernel<T, 32, TILE>);
}

}  // namespace rb

using namespace rb;

// w [H, N, K]; row t, head h of `in` at in + t * in_t + h * in_h (K values), of `out` likewise (N values);
// strides and K multiples of eight. row_ids: the rows to run (null: 0 .. rows - 1).
extern "C" int rmlx_head_gemv(const void* w, const void* in, int in_t, int in_h, void* out, int out_t, int out_h,
                              const int* row_ids, int rows, int H, int N, int K, int f32, int pdl, cudaStream_t st) {
  if (rows < 1 || (rows + kHgRows - 1) / kHgRows > 65535 || H < 1 || H > 65535 || N < 1 || K < 8 || K % 8 || in_t % 8 ||
      in_h % 8 || K > 8192)
    return -2;
#define RB_HG(T_, TILE_)                                                                                            \
  return launch_head_gemv<T_, TILE_>(static_cast<const T_*>(w), static_cast<const T_*>(in), in_t, in_h,            \
                                     static_cast<T_*>(out), out_t, out_h, row_ids, rows, H, N, K, pdl, st)
  if (f32) RB_HG(float, 64);
  if (rows <= 2 * kHgRows) RB_HG(__nv_bfloat16, 32);
  RB_HG(__nv_bfloat16, 64);
#undef RB_HG
}
