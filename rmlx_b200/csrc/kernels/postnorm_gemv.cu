// Decode projections of decoders with norms on the sublayers' outputs (x <- x + norm(y), fp32 residual),
// one warp per weight-row pair as in decode_gemv.cu. The kernels that read the residual take the previous
// sublayer's output y along and finish that sublayer first: every block forms x + norm(y) while it stages
// its activations (a few thousand values from L2), and block 0 writes it to a second residual buffer.
//
//   postnorm_in       out = W x: fp32 rows, or (gated) the activation of row pairs (i, n + i) in bf16, or
//                     (shift) row segments that each read their own token-shift mix of x
//   postnorm_router   router logits and the choice of experts by one of route.cuh's rules (the last block to finish chooses)
//   postnorm_expert   gate / up projections of each token's chosen experts with the gated activation
//   expert_out        y = sum over slots of weight * Wdown[e] act + identity weight * x
//   matvec_out        y = W a
//   wkv_decode        one token of the WKV recurrence: decay from its low-rank projection, state update,
//                     head norm, output gate
#include "../common/gated.cuh"
#include "../common/gemv_core.cuh"
#include "../common/launch.cuh"
#include "../common/route.cuh"

namespace rb {

constexpr int kPnRows = 2;        // weight rows a warp accumulates together
constexpr size_t kPnMaxSmem = 220 * 1024;

// The residual a kernel reads: x + y / rms(y) * w (y == nullptr: x itself), D real columns of ldx.
struct PostNormIn {
  const float* x;
  const float* y;
  const float* w;
  float eps;
  int D, ldx;
  float* x_out;                   // written by block 0; not x itself (null: y is null, too, and x is only read)
};
// Token shift: rows seg * seg_rows .. of W read x + (prev - x) * mu[seg].
struct ShiftIn {
  const float* mu;                // [5, ldx]
  const float* prev;              // slot s: prev + s * stride
  const int* slots;
  long long stride;
  int seg_rows;                   // rows of the first four segments; the rest is the fifth
};

// Stages row b of the residual into `xs` (split-chunk layout of gemv_core.cuh). 256 threads.
__device__ __forceinline__ void stage_post_norm(const PostNormIn& in, int b, char* xs, float* red, bool write,
                                                const float* mu, const float* prev) {
  constexpr int kKeep = 4;
  const int chunks = in.ldx >> 3;
  const float* x = in.x + size_t(b) * in.ldx;
  const float* y = in.y ? in.y + size_t(b) * in.ldx : nullptr;
  float4* dst = reinterpret_cast<float4*>(xs);
  auto ld = [](const float* p, int c, float (&f)[8]) {
    const float4 a = __ldcg(reinterpret_cast<const float4*>(p + c * 8));
    const float4 e = __ldcg(reinterpret_cast<const float4*>(p + c * 8 + 4));
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = e.x; f[5] = e.y; f[6] = e.z; f[7] = e.w;
  };
  float fy[kKeep][8], fx[kKeep][8];
  float ssq = 0.f;
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kGemvThreads + threadIdx.x;
    if (c < chunks) {
      ld(x, c, fx[u]);
      if (y) {
        ld(y, c, fy[u]);
#pragma unroll
        for (int i = 0; i < 8; ++i) ssq += fy[u][i] * fy[u][i];
      }
    }
  }
  float inv = 0.f;
  if (y) {
    for (int c = kKeep * kGemvThreads + threadIdx.x; c < chunks; c += kGemvThreads) {
      float f[8];
      ld(y, c, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) ssq += f[i] * f[i];
    }
    inv = 1.f / sqrtf(block_sum_256(ssq, red) / float(in.D) + in.eps);
  }
  auto put = [&](int c, float (&a)[8], const float (&e)[8]) {
    if (y) {
      float g[8];
      ld(in.w, c, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] = fmaf(e[i] * inv, g[i], a[i]);
    }
    if (write) {
      float4* o = reinterpret_cast<float4*>(in.x_out + size_t(b) * in.ldx + c * 8);
      o[0] = make_float4(a[0], a[1], a[2], a[3]);
      o[1] = make_float4(a[4], a[5], a[6], a[7]);
    }
    if (mu) {
      float m[8], p[8];
      ld(mu, c, m);
      ld(prev, c, p);
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] = fmaf(p[i] - a[i], m[i], a[i]);
    }
    dst[c] = make_float4(a[0], a[1], a[2], a[3]);
    dst[chunks + c] = make_float4(a[4], a[5], a[6], a[7]);
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kGemvThreads + threadIdx.x;
    if (c < chunks) put(c, fx[u], fy[u]);
  }
  for (int c = kKeep * kGemvThreads + threadIdx.x; c < chunks; c += kGemvThreads) {
    float a[8], e[8];
    ld(x, c, a);
    if (y) ld(y, c, e);
    put(c, a, e);
  }
}

// GATED: N counts output columns, W has 2 N rows (gate then up). Blocks stay and walk the rows (the norm and
// the staging are paid once per block); grid y: the shift segment whose rows a block takes.
template <int B, bool GATED>
__global__ void __launch_bounds__(kGemvThreads, 2)
postnorm_in_kernel(Matrix<WBf16> W, PostNormIn in, ShiftIn sh, float* __restrict__ out, int ld_out,
                   __nv_bfloat16* __restrict__ act, int ld_act, int N, float limit) {
  extern __shared__ __align__(16) char smem[];
  __shared__ float red[kGemvWarps];
  constexpr int R = GATED ? 2 * kPnRows : kPnRows;
  const int K = W.K, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t bstride = XStage<WBf16>::bytes(K);
  const int seg = blockIdx.y, n_lo = sh.mu ? seg * sh.seg_rows : 0, n_hi = sh.mu && seg < 4 ? n_lo + sh.seg_rows : N;
  int n0 = n_lo + (blockIdx.x * kGemvWarps + warp) * kPnRows;
  if (n_lo + int(blockIdx.x) * kGemvWarps * kPnRows >= n_hi) return;        // a short segment
  RowBf16 rows[R];
  Tile<RowBf16, R> t0;
  auto point = [&]() {
#pragma unroll
    for (int r = 0; r < kPnRows; ++r) {
      const int n = min(n0 + r, N - 1);
      rows[r] = W.row(n);
      if (GATED) rows[kPnRows + r] = W.row(size_t(N) + n);
    }
    load_tile<R>(rows, K, 0, t0);
  };
  if (n0 < n_hi) point();       // weights wait for nothing: ask for the first tile at once
  pdl_launch_dependents();
  pdl_wait();
  const float* mu = sh.mu ? sh.mu + size_t(seg) * in.ldx : nullptr;
#pragma unroll
  for (int b = 0; b < B; ++b)
    stage_post_norm(in, b, smem + b * bstride, red, blockIdx.x == 0 && seg == 0 && in.x_out, mu,
                    mu ? sh.prev + sh.slots[b] * sh.stride : nullptr);
  __syncthreads();
  for (bool first = true; n0 < n_hi; n0 += gridDim.x * kGemvWarps * kPnRows, first = false) {
    if (!first) point();
    float acc[R][B];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) acc[r][b] = 0.f;
    warp_dot<R, B, RowBf16>(rows, smem, bstride, K, acc, t0);
#pragma unroll
    for (int r = 0; r < kPnRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const float v = warp_sum(acc[r][b]);
        const float u = GATED ? warp_sum(acc[GATED ? kPnRows + r : r][b]) : 0.f;
        const int n = n0 + r;
        if (lane == r * B + b && n < n_hi) {
          if (GATED) act[size_t(b) * ld_act + n] = __float2bfloat16_rn(gated_act_fast(v, u, limit));
          else out[size_t(b) * ld_out + n] = v;
        }
      }
  }
}

// One block per router output, its warps share the row; the last block to arrive chooses for every token.
template <int B, RouteRule RULE>
__global__ void __launch_bounds__(kGemvThreads)
postnorm_router_kernel(Matrix<WBf16> W, PostNormIn in, const float* __restrict__ correction, float* __restrict__ logits,
                       int* __restrict__ idx, float* __restrict__ weights, float* __restrict__ identity,
                       unsigned int* __restrict__ ticket, int experts, int outputs, int top_k, RouteGroups groups) {
  extern __shared__ __align__(16) char smem[];
  __shared__ float red[kGemvWarps];
  __shared__ float part[kGemvWarps][B];
  __shared__ unsigned int last;
  const int K = W.K, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, chunks = K >> 3;
  const size_t bstride = XStage<WBf16>::bytes(K);
  const int n = blockIdx.x;
  const __nv_bfloat16* row = W.w + size_t(n) * K;
  constexpr int kKeep = 4;
  uint4 wv[kKeep];
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kGemvThreads + threadIdx.x;
    wv[u] = c < chunks ? ldg_stream(row + (size_t(c) << 3)) : make_uint4(0u, 0u, 0u, 0u);
  }
  pdl_launch_dependents();
  pdl_wait();
#pragma unroll
  for (int b = 0; b < B; ++b) stage_post_norm(in, b, smem + b * bstride, red, n == 0 && in.x_out, nullptr, nullptr);
  __syncthreads();
  float acc[B];
#pragma unroll
  for (int b = 0; b < B; ++b) acc[b] = 0.f;
  auto dot = [&](int c, const uint4& w) {
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const float4* xs = reinterpret_cast<const float4*>(smem + b * bstride);
      const float4 x0 = xs[c], x1 = xs[chunks + c];
      float a = acc[b];
      a = fmaf(bf16lo(w.x), x0.x, a); a = fmaf(bf16hi(w.x), x0.y, a);
      a = fmaf(bf16lo(w.y), x0.z, a); a = fmaf(bf16hi(w.y), x0.w, a);
      a = fmaf(bf16lo(w.z), x1.x, a); a = fmaf(bf16hi(w.z), x1.y, a);
      a = fmaf(bf16lo(w.w), x1.z, a); a = fmaf(bf16hi(w.w), x1.w, a);
      acc[b] = a;
    }
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kGemvThreads + threadIdx.x;
    if (c < chunks) dot(c, wv[u]);
  }
  for (int c = kKeep * kGemvThreads + threadIdx.x; c < chunks; c += kGemvThreads) dot(c, ldg_stream(row + (size_t(c) << 3)));
#pragma unroll
  for (int b = 0; b < B; ++b) {
    const float v = warp_sum(acc[b]);
    if (lane == 0) part[warp][b] = v;
  }
  __syncthreads();
  if (threadIdx.x < B) {
    float v = 0.f;
#pragma unroll
    for (int q = 0; q < kGemvWarps; ++q) v += part[q][threadIdx.x];
    logits[size_t(threadIdx.x) * outputs + n] = v;
    __threadfence();
  }
  __syncthreads();
  if (threadIdx.x == 0) last = (atomicAdd(ticket, 1u) == gridDim.x - 1) ? 1u : 0u;
  __syncthreads();
  if (last) {
    __threadfence();
    for (int b = warp; b < B; b += kGemvWarps) {
      // through L2: other blocks wrote the logits
      float* z = reinterpret_cast<float*>(smem) + b * outputs;
      for (int i = lane; i < outputs; i += 32) z[i] = __ldcg(logits + size_t(b) * outputs + i);
      __syncwarp();
      const int slots = top_k + groups.always;
      warp_route<RULE>(z, correction, experts, outputs, top_k, idx + size_t(b) * slots, weights + size_t(b) * slots,
                       identity ? identity + b : nullptr, nullptr, groups);
    }
    if (threadIdx.x == 0) *ticket = 0u;
  }
}

// grid (column blocks, token * slot). x: the finished residual.
__global__ void __launch_bounds__(kGemvThreads, 2)
postnorm_expert_kernel(const __nv_bfloat16* __restrict__ w, int K, const float* __restrict__ x, int ldx,
                       const int* __restrict__ idx, __nv_bfloat16* __restrict__ act, int ld_act, int N, int top_k,
                       int experts, float limit) {
  extern __shared__ __align__(16) char smem[];
  constexpr int R = 2 * kPnRows;
  const int pair = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int e = idx[pair];
  if (e >= experts) return;                           // an identity expert has no tensors
  Matrix<WBf16> W{w + size_t(e) * 2 * N * K, K};
  const int n0 = (blockIdx.x * kGemvWarps + warp) * kPnRows;
  RowBf16 rows[R];
  Tile<RowBf16, R> t0;
  if (n0 < N) {
#pragma unroll
    for (int r = 0; r < kPnRows; ++r) {
      const int n = min(n0 + r, N - 1);
      rows[r] = W.row(n);
      rows[kPnRows + r] = W.row(size_t(N) + n);
    }
    load_tile<R>(rows, K, 0, t0);
  }
  const float* src = x + size_t(pair / top_k) * ldx;
  auto ld = [&](int c, float (&f)[8]) {
    const float4 a = __ldcg(reinterpret_cast<const float4*>(src + c * 8));
    const float4 b = __ldcg(reinterpret_cast<const float4*>(src + c * 8 + 4));
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  };
  XStage<WBf16>::stage_with(smem, K, ld);
  if (n0 >= N) return;
  float acc[R][1];
#pragma unroll
  for (int r = 0; r < R; ++r) acc[r][0] = 0.f;
  warp_dot<R, 1, RowBf16>(rows, smem, 0, K, acc, t0);
#pragma unroll
  for (int r = 0; r < kPnRows; ++r) {
    const float g = warp_sum(acc[r][0]), u = warp_sum(acc[kPnRows + r][0]);
    if (lane == r && n0 + r < N) act[size_t(pair) * ld_act + n0 + r] = __float2bfloat16_rn(gated_act_fast(g, u, limit));
  }
}

// grid (row blocks, tokens): y[b, n] = sum_s weight_s * (Wdown[e_s] act_s)[n] + identity * x[b, n], n < N (identity null:
// without the last term). y may be x.
__global__ void __launch_bounds__(kGemvThreads, 2)
expert_out_kernel(const __nv_bfloat16* __restrict__ w, int rows_e, int K, const __nv_bfloat16* __restrict__ act, int ld_act,
                  const int* __restrict__ idx, const float* __restrict__ weights, const float* __restrict__ identity,
                  const float* x, float* y, int ldx, int N, int top_k, int experts) {
  extern __shared__ __align__(16) char smem[];        // [top_k] staged activations
  __shared__ int s_e[kRouteMaxTop];
  __shared__ float s_w[kRouteMaxTop];
  const int b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t bstride = XStage<WBf16>::bytes(K);
  pdl_launch_dependents();
  pdl_wait();
  if (threadIdx.x < top_k) {
    const int e = idx[b * top_k + threadIdx.x];
    s_e[threadIdx.x] = e < experts ? e : -1;
    s_w[threadIdx.x] = weights[b * top_k + threadIdx.x];
  }
  __syncthreads();
  auto next = [&](int s) { while (s < top_k && s_e[s] < 0) ++s; return s; };
  const int n0 = (blockIdx.x * kGemvWarps + warp) * kPnRows;
  int s = next(0);
  RowBf16 rows[kPnRows];
  Tile<RowBf16, kPnRows> cur;
  auto point = [&](int slot, RowBf16 (&r)[kPnRows]) {
#pragma unroll
    for (int i = 0; i < kPnRows; ++i) r[i] = RowBf16{w + (size_t(s_e[slot]) * rows_e + min(n0 + i, N - 1)) * K};
  };
  if (n0 < N && s < top_k) { point(s, rows); load_tile<kPnRows>(rows, K, 0, cur); }
  for (int q = 0; q < top_k; ++q) {
    if (s_e[q] < 0) continue;
    XLoadBf16 ld{act + size_t(b * top_k + q) * ld_act, nullptr, 0.f};
    XStage<WBf16>::stage_part(smem + q * bstride, K, ld, threadIdx.x, kGemvThreads);
  }
  __syncthreads();
  if (n0 >= N) return;
  float tot[kPnRows];
#pragma unroll
  for (int r = 0; r < kPnRows; ++r) tot[r] = 0.f;
  while (s < top_k) {                                  // the next expert's first tile is asked for early
    const int sn = next(s + 1);
    RowBf16 rn[kPnRows];
    Tile<RowBf16, kPnRows> nxt;
    if (sn < top_k) { point(sn, rn); load_tile<kPnRows>(rn, K, 0, nxt); }
    float acc[kPnRows][1];
#pragma unroll
    for (int r = 0; r < kPnRows; ++r) acc[r][0] = 0.f;
    warp_dot<kPnRows, 1, RowBf16>(rows, smem + s * bstride, 0, K, acc, cur);
#pragma unroll
    for (int r = 0; r < kPnRows; ++r) tot[r] = fmaf(s_w[s], acc[r][0], tot[r]);
    if (sn < top_k) {
      cur = nxt;
#pragma unroll
      for (int r = 0; r < kPnRows; ++r) rows[r] = rn[r];
    }
    s = sn;
  }
#pragma unroll
  for (int r = 0; r < kPnRows; ++r) {
    const float v = warp_sum(tot[r]);
    const int n = n0 + r;
    if (lane == r && n < N) y[size_t(b) * ldx + n] = identity ? fmaf(identity[b], __ldcg(x + size_t(b) * ldx + n), v) : v;
  }
}

template <int B>
__global__ void __launch_bounds__(kGemvThreads)
matvec_out_kernel(Matrix<WBf16> W, const __nv_bfloat16* __restrict__ a, int ld_a, float* __restrict__ y, int ld_y, int N) {
  extern __shared__ __align__(16) char smem[];
  const int K = W.K, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t bstride = XStage<WBf16>::bytes(K);
  const int n0 = (blockIdx.x * kGemvWarps + warp) * kPnRows;
  RowBf16 rows[kPnRows];
  Tile<RowBf16, kPnRows> t0;
  if (n0 < N) {
#pragma unroll
    for (int r = 0; r < kPnRows; ++r) rows[r] = W.row(min(n0 + r, N - 1));
    load_tile<kPnRows>(rows, K, 0, t0);
  }
  pdl_launch_dependents();
  pdl_wait();
#pragma unroll
  for (int b = 0; b < B; ++b) {
    XLoadBf16 ld{a + size_t(b) * ld_a, nullptr, 0.f};
    XStage<WBf16>::stage_part(smem + b * bstride, K, ld, threadIdx.x, kGemvThreads);
  }
  __syncthreads();
  if (n0 >= N) return;
  float acc[kPnRows][B];
#pragma unroll
  for (int r = 0; r < kPnRows; ++r)
#pragma unroll
    for (int b = 0; b < B; ++b) acc[r][b] = 0.f;
  warp_dot<kPnRows, B, RowBf16>(rows, smem, bstride, K, acc, t0);
#pragma unroll
  for (int r = 0; r < kPnRows; ++r)
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const float v = warp_sum(acc[r][b]);
      if (lane == r * B + b && n0 + r < N) y[size_t(b) * ld_y + n0 + r] = v;
    }
}

// raw row b = [r | k | v | g: `inner` values apart | low: rank]. One block per (head, row). ROWS: state rows a
// thread holds; they belong to this kernel alone within a step, so they are asked for before the wait (the
// step's first kernel has waited for everything before it).
template <int ROWS>
__global__ void __launch_bounds__(256)
wkv_decode_kernel(const float* __restrict__ raw, int ld_raw, int inner, const __nv_bfloat16* __restrict__ w2, int rank,
                  const float* __restrict__ w0, const float* __restrict__ u, const float* __restrict__ norm, float eps,
                  const int* __restrict__ slots, float* __restrict__ state, float* __restrict__ prev, long long stride,
                  const float* __restrict__ x, int ldx, __nv_bfloat16* __restrict__ a, int ld_a, int dim, int dim_pad) {
  extern __shared__ float sm[];
  float* sr = sm;                    // [dim_pad] r, k, decay
  float* sk = sr + dim_pad;
  float* sw = sk + dim_pad;
  float* low = sw + dim_pad;         // [rank] tanh
  float* part = low + rank;          // [256]
  __shared__ float red[8];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int slot = slots[b];
  // the column this thread works on and its group's share of the rows
  const int groups = 256 / dim_pad, g = tid / dim_pad, col = tid - g * dim_pad;
  const int per = (dim + groups - 1) / groups, i0 = g * per, i1 = min(i0 + per, dim);
  float* sp = state + size_t(slot) * stride + size_t(h) * dim * dim + col;
  float s[ROWS];
#pragma unroll
  for (int q = 0; q < ROWS; ++q) s[q] = (col < dim && i0 + q < i1) ? __ldcg(sp + size_t(i0 + q) * dim) : 0.f;
  pdl_launch_dependents();
  pdl_wait();
  const float* row = raw + size_t(b) * ld_raw;
  for (int i = tid; i < rank; i += 256) low[i] = tanhf(__ldcg(row + 4 * inner + i));
  float ruk = 0.f;
  if (tid < dim) {
    const float r = __ldcg(row + h * dim + tid), k = __ldcg(row + inner + h * dim + tid);
    sr[tid] = r;
    sk[tid] = k;
    ruk = r * u[h * dim + tid] * k;
  }
  const float v = col < dim ? __ldcg(row + 2 * inner + h * dim + col) : 0.f;
  ruk = block_sum_256(ruk, red);     // low, sr and sk are visible, too
  {                                  // decay of row `col`, the rank's chunks dealt to the groups
    float d = 0.f;
    if (col < dim) {
      const __nv_bfloat16* wr = w2 + size_t(h * dim + col) * rank;
      for (int j = g * 8; j < rank; j += groups * 8) {
        const uint4 q = *reinterpret_cast<const uint4*>(wr + j);
        d = fmaf(bf16lo(q.x), low[j], d); d = fmaf(bf16hi(q.x), low[j + 1], d);
        d = fmaf(bf16lo(q.y), low[j + 2], d); d = fmaf(bf16hi(q.y), low[j + 3], d);
        d = fmaf(bf16lo(q.z), low[j + 4], d); d = fmaf(bf16hi(q.z), low[j + 5], d);
        d = fmaf(bf16lo(q.w), low[j + 6], d); d = fmaf(bf16hi(q.w), low[j + 7], d);
      }
    }
    part[tid] = d;
    __syncthreads();
    if (tid < dim) {
      d = w0[h * dim + tid];
      for (int q = 0; q < groups; ++q) d += part[q * dim_pad + tid];
      sw[tid] = expf(-expf(d));
    }
    __syncthreads();
  }
  float o = 0.f;
  if (col < dim) {
#pragma unroll
    for (int q = 0; q < ROWS; ++q) {
      const int i = i0 + q;
      if (i < i1) {
        o = fmaf(sr[i], s[q], o);
        sp[size_t(i) * dim] = fmaf(sw[i], s[q], sk[i] * v);
      }
    }
  }
  part[tid] = o;
  __syncthreads();
  float ssq = 0.f;
  if (tid < dim) {                   // tid is this thread's column
    o = ruk * v;
    for (int q = 0; q < groups; ++q) o += part[q * dim_pad + tid];
    ssq = o * o;
  }
  ssq = block_sum_256(ssq, red);
  if (tid < dim) {
    const float inv = 1.f / sqrtf(ssq / float(dim) + eps);
    const float z = __ldcg(row + 3 * inner + h * dim + tid);
    a[size_t(b) * ld_a + h * dim + tid] = __float2bfloat16_rn(o * inv * norm[h * dim + tid] * (z / (1.f + expf(-z))));
  }
  if (h == 0) {
    float* keep = prev + size_t(slot) * stride;
    for (int i = tid; i < ldx; i += 256) keep[i] = __ldcg(x + size_t(b) * ldx + i);
  }
}

static int pn_grid(int rows) { return (rows + kGemvWarps * kPnRows - 1) / (kGemvWarps * kPnRows); }

}  // namespace rb

using namespace rb;

// Rows one launch takes for K staged values: at most four, fewer when the fp32 staging would not fit.
extern "C" int rmlx_postnorm_max_rows(int K) {
  int b = 4;
  while (b > 0 && size_t(K) * 4 * b > kPnMaxSmem) --b;
  return b;
}

#define RB_PN_DISPATCH(B_, CALL)                     \
  switch (B_) {                                      \
    case 1: { constexpr int kB = 1; return CALL; }   \
    case 2: { constexpr int kB = 2; return CALL; }   \
    case 3: { constexpr int kB = 3; return CALL; }   \
    case 4: { constexpr int kB = 4; return CALL; }   \
    default: return -2;                              \
  }

template <int B, bool GATED>
static int launch_in(const void* w, const PostNormIn& in, const ShiftIn& sh, float* out, int ld_out, void* act, int ld_act,
                     int N, float limit, int pdl, cudaStream_t st) {
  const size_t smem = XStage<WBf16>::bytes(in.ldx) * B;
  auto kern = postnorm_in_kernel<B, GATED>;
  RB_CHECK(set_max_smem(kern, smem));
  // as many blocks as stay resident, the rows spread evenly over them
  int per_sm = 1;
  RB_CHECK(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kern, kGemvThreads, smem));
  const int segs = sh.mu ? 5 : 1, longest = sh.mu ? sh.seg_rows : N;
  const int cap = sm_count() * (per_sm > 0 ? per_sm : 1) / (sh.mu ? 4 : 1), tiles = pn_grid(longest);
  const int passes = (tiles + cap - 1) / cap;
  return launch(kern, dim3((tiles + passes - 1) / passes, segs), dim3(kGemvThreads), smem, st, pdl != 0,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(w), in.ldx}, in, sh, out, ld_out,
                static_cast<__nv_bfloat16*>(act), ld_act, N, limit);
}

// w bf16 [N, ldx]; x, y (or null) and x_out (or, with y, null) fp32 [B, ldx], norm_w fp32 [ldx]; out fp32 [B, ld_out]. mu (or
// null): fp32 [5, ldx], prev rows `stride` apart by slots [B]; then w's rows are four segments of seg_rows (a
// multiple of 16) and a fifth.
extern "C" int rmlx_postnorm_in(const void* w, const float* x, const float* y, const float* norm_w, float eps, float* x_out,
                                int D, int ldx, const float* mu, const float* prev, const int* slots, long long stride,
                                int seg_rows, float* out, int ld_out, int B, int N, int pdl, cudaStream_t st) {
  if (ldx < 8 || ldx % 8 || D < 1 || D > ldx || N < 1 || ld_out < N || (!x_out && y) || x_out == x || B > rmlx_postnorm_max_rows(ldx) ||
      (y && !norm_w) || (mu && (!prev || !slots || stride % 4 || seg_rows < 16 || seg_rows % 16)))
    return -2;
  const PostNormIn in{x, y, norm_w, eps, D, ldx, x_out};
  const ShiftIn sh{mu, prev, slots, stride, mu ? seg_rows : 1};
  RB_PN_DISPATCH(B, (launch_in<kB, false>(w, in, sh, out, ld_out, nullptr, 0, N, 0.f, pdl, st)))
}

// w bf16 [2 N, ldx] = [gate; up]; act bf16 [B, ld_act].
extern "C" int rmlx_postnorm_gated(const void* w, const float* x, const float* y, const float* norm_w, float eps,
                                   float* x_out, int D, int ldx, void* act, int ld_act, int B, int N, float limit, int pdl,
                                   cudaStream_t st) {
  if (ldx < 8 || ldx % 8 || D < 1 || D > ldx || N < 1 || ld_act < N || !x_out || x_out == x || B > rmlx_postnorm_max_rows(ldx) ||
      (y && !norm_w))
    return -2;
  const PostNormIn in{x, y, norm_w, eps, D, ldx, x_out};
  const ShiftIn sh{nullptr, nullptr, nullptr, 0, 1};
  RB_PN_DISPATCH(B, (launch_in<kB, true>(w, in, sh, nullptr, 0, act, ld_act, N, limit, pdl, st)))
}

template <int B, RouteRule RULE>
static int launch_router(const void* w, const PostNormIn& in, const float* correction, float* logits, int* idx,
                         float* weights, float* identity, unsigned int* ticket, int experts, int outputs, int top_k, int pdl,
                         cudaStream_t st, const RouteGroups& groups = RouteGroups{}) {
  size_t smem = XStage<WBf16>::bytes(in.ldx) * B;
  if (smem < size_t(B) * outputs * 4) smem = size_t(B) * outputs * 4;
  auto kern = postnorm_router_kernel<B, RULE>;
  RB_CHECK(set_max_smem(kern, smem));
  return launch(kern, dim3(outputs), dim3(kGemvThreads), smem, st, pdl != 0,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(w), in.ldx}, in, correction, logits, idx, weights, identity,
                ticket, experts, outputs, top_k, groups);
}

// w bf16 [outputs, ldx]; logits fp32 [B, outputs] scratch; ticket: one word, zero on entry and on exit.
extern "C" int rmlx_postnorm_router(const void* w, const float* x, const float* y, const float* norm_w, float eps,
                                    float* x_out, int D, int ldx, const float* correction, float* logits, int* idx,
                                    float* weights, float* identity, unsigned int* ticket, int B, int experts, int outputs,
                                    int top_k, int pdl, cudaStream_t st) {
  if (ldx < 8 || ldx % 8 || D < 1 || D > ldx || !x_out || x_out == x || (y && !norm_w) || experts < 1 || outputs < experts ||
      outputs > kRouteMaxOutputs || top_k < 1 || top_k > kRouteMaxTop || top_k > outputs || B > rmlx_postnorm_max_rows(ldx))
    return -2;
  const PostNormIn in{x, y, norm_w, eps, D, ldx, x_out};
  RB_PN_DISPATCH(B, (launch_router<kB, kRouteCorrected>(w, in, correction, logits, idx, weights, identity, ticket, experts,
                                                        outputs, top_k, pdl, st)))
}

// Routing by sigmoids and groups of finished rows h fp32 [B, ldx]; idx and weights [B, top_k + always], the rest as above.
extern "C" int rmlx_grouped_router(const void* w, const float* h, int ldx, float* logits, int* idx, float* weights,
                                   unsigned int* ticket, int B, int experts, int top_k, int groups, int keep, int always,
                                   float scale, int pdl, cudaStream_t st) {
  RouteGroups g;
  g.count = groups; g.keep = keep; g.always = always; g.scale = scale;
  if (ldx < 8 || ldx % 8 || experts < 1 || experts > kRouteMaxOutputs || top_k < 1 || !route_groups_ok(g, experts, top_k) ||
      B > rmlx_postnorm_max_rows(ldx))
    return -2;
  const PostNormIn in{h, nullptr, nullptr, 0.f, ldx, ldx, nullptr};
  RB_PN_DISPATCH(B, (launch_router<kB, kRouteGrouped>(w, in, nullptr, logits, idx, weights, nullptr, ticket, experts, experts,
                                                      top_k, pdl, st, g)))
}

// w bf16 [experts, 2 N, ldx]; x fp32 [B, ldx]; idx [B, top_k]; act bf16 [B * top_k, ld_act].
extern "C" int rmlx_postnorm_expert(const void* w, const float* x, int ldx, const int* idx, void* act, int ld_act, int B,
                                    int top_k, int N, int experts, float limit, int pdl, cudaStream_t st) {
  if (B < 1 || top_k < 1 || B * top_k > 65535 || ldx < 8 || ldx % 8 || N < 1 || ld_act < N || experts < 1 ||
      XStage<WBf16>::bytes(ldx) > kPnMaxSmem)
    return -2;
  const size_t smem = XStage<WBf16>::bytes(ldx);
  RB_CHECK(set_max_smem(postnorm_expert_kernel, smem));
  return launch(postnorm_expert_kernel, dim3(pn_grid(N), B * top_k), dim3(kGemvThreads), smem, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(w), ldx, x, ldx, idx, static_cast<__nv_bfloat16*>(act), ld_act, N, top_k,
                experts, limit);
}

// w bf16 [experts, rows_e, K], N <= rows_e; act bf16 [B * top_k, ld_act >= K]; x, y fp32 [B, ldx].
extern "C" int rmlx_expert_out(const void* w, int rows_e, int K, const void* act, int ld_act, const int* idx,
                               const float* weights, const float* identity, const float* x, float* y, int ldx, int B, int N,
                               int top_k, int experts, int pdl, cudaStream_t st) {
  if (B < 1 || B > 65535 || top_k < 1 || top_k > kRouteMaxTop || K < 8 || K % 8 || ld_act % 8 || ld_act < K || N < 1 ||
      N > rows_e || N > ldx || XStage<WBf16>::bytes(K) * top_k > kPnMaxSmem)
    return -2;
  const size_t smem = XStage<WBf16>::bytes(K) * top_k;
  RB_CHECK(set_max_smem(expert_out_kernel, smem));
  return launch(expert_out_kernel, dim3(pn_grid(N), B), dim3(kGemvThreads), smem, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(w), rows_e, K, static_cast<const __nv_bfloat16*>(act), ld_act, idx, weights,
                identity, x, y, ldx, N, top_k, experts);
}

template <int B>
static int launch_matvec(const void* w, const void* a, int ld_a, float* y, int ld_y, int N, int K, int pdl, cudaStream_t st) {
  const size_t smem = XStage<WBf16>::bytes(K) * B;
  auto kern = matvec_out_kernel<B>;
  RB_CHECK(set_max_smem(kern, smem));
  return launch(kern, dim3(pn_grid(N)), dim3(kGemvThreads), smem, st, pdl != 0,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(w), K}, static_cast<const __nv_bfloat16*>(a), ld_a, y, ld_y, N);
}

// w bf16 [N, K], a bf16 [B, ld_a], y fp32 [B, ld_y].
extern "C" int rmlx_matvec_out(const void* w, const void* a, int ld_a, float* y, int ld_y, int B, int N, int K, int pdl,
                               cudaStream_t st) {
  if (K < 8 || K % 8 || ld_a % 8 || ld_a < K || N < 1 || ld_y < N || B > rmlx_postnorm_max_rows(K)) return -2;
  RB_PN_DISPATCH(B, (launch_matvec<kB>(w, a, ld_a, y, ld_y, N, K, pdl, st)))
}

// raw fp32 [B, ld_raw] = [r | k | v | g] `inner` apart, then `rank` values (a multiple of eight); w2 bf16
// [>= H * dim, rank]; a bf16 [B, ld_a]; state / prev as in rmlx_wkv_scan; x fp32 [B, ldx] what the layer read.
extern "C" int rmlx_wkv_decode(const float* raw, int ld_raw, int inner, const void* w2, int rank, const float* w0,
                               const float* u, const float* norm, float eps, const int* slots, float* state, float* prev,
                               long long stride, const float* x, int ldx, void* a, int ld_a, int B, int H, int dim, int pdl,
                               cudaStream_t st) {
  if (B < 1 || B > 65535 || H < 1 || dim < 1 || dim > 256 || inner < H * dim || rank < 8 || rank % 8 ||
      ld_raw < 4 * inner + rank || ld_a < H * dim || !slots || rank > 4096 || w2 == nullptr)
    return -2;
  int dim_pad = 8;
  while (dim_pad < dim) dim_pad *= 2;
  const size_t smem = size_t(3 * dim_pad + rank + 256) * sizeof(float);
  const int groups = 256 / dim_pad, per = (dim + groups - 1) / groups;
  auto go = [&](auto kern) -> int {
    RB_CHECK(set_max_smem(kern, smem));
    return launch(kern, dim3(H, B), dim3(256), smem, st, pdl != 0, raw, ld_raw, inner,
                  static_cast<const __nv_bfloat16*>(w2), rank, w0, u, norm, eps, slots, state, prev, stride, x, ldx,
                  static_cast<__nv_bfloat16*>(a), ld_a, dim, dim_pad);
  };
  if (per <= 4) return go(wkv_decode_kernel<4>);
  if (per <= 16) return go(wkv_decode_kernel<16>);
  if (per <= 64) return go(wkv_decode_kernel<64>);
  return go(wkv_decode_kernel<256>);
}
