// Decode steps of decoders whose mixer and feed-forward read the same fp32 residual row through norms of their own, one
// warp per weight-row pair as in decode_gemv.cu:
//
//   twin_in       one launch for everything that reads the residual: the mixer's projection of norm1(x) (fp32 rows out)
//                 beside, on blocks of their own, the gate / up projection of norm2(x) with the gated activation, or
//                 the router's logits of norm2(x) (the last of its blocks chooses the experts)
//   gla_decode    one token of gated linear attention: decay from its low-rank projection, state update, head norm,
//                 output gate; a head's value columns are spread over a cluster
//   ssd_decode    one token of the state-space heads: convolution, step size, state update
//   ssd_finish    gate, grouped norm, and the convolution's carried inputs
//
// The output projections run on parallel_gemv.cu (two terms into the residual) and postnorm_gemv.cu (experts).
#include <cooperative_groups.h>

#include "../common/gated.cuh"
#include "../common/gemv_core.cuh"
#include "../common/launch.cuh"
#include "../common/route.cuh"
#include "../common/rows.cuh"
#include "../common/state_step.cuh"

namespace cg = cooperative_groups;

namespace rb {

constexpr int kTnRows = 2;        // weight rows a warp accumulates together
constexpr size_t kTnMaxSmem = 220 * 1024;
enum TwinSecond { kTwinNone = 0, kTwinGated = 1, kTwinRouter = 2 };

struct TwinIn {
  const float* x;                 // [B, ldx] residual
  const float* w1;                // norm weights [ldx]
  const float* w2;
  float eps;
  int D, ldx;
};
struct TwinFf {
  const __nv_bfloat16* w;         // gated: [2 N, ldx] (gate, up); router: [N, ldx]
  int N;
  __nv_bfloat16* act;             // gated: [B, ld_act]
  int ld_act;
  float limit;
  const float* bias;              // router: [N]
  float* logits;                  // router: [B, N] scratch
  float* h2;                      // router: [B, ldx], norm2(x) for the experts
  int* idx;                       // router: [B, top_k]
  float* weights;
  unsigned int* ticket;           // one word, zero on entry and on exit
  int top_k;
};

// Rows n0, n0 + step, .. of W times the staged rows; put(n, b, value, second value) for each.
template <int B, bool GATED, class PUT>
__device__ __forceinline__ void twin_rows(const Matrix<WBf16>& W, int N, int n0, int step, const char* smem, size_t bstride,
                                          RowBf16 (&rows)[GATED ? 2 * kTnRows : kTnRows],
                                          Tile<RowBf16, GATED ? 2 * kTnRows : kTnRows>& t0, PUT put) {
  constexpr int R = GATED ? 2 * kTnRows : kTnRows;
  const int K = W.K, lane = threadIdx.x & 31;
  for (bool first = true; n0 < N; n0 += step, first = false) {
    if (!first) {
#pragma unroll
      for (int r = 0; r < kTnRows; ++r) {
        const int n = min(n0 + r, N - 1);
        rows[r] = W.row(n);
        if (GATED) rows[kTnRows + r] = W.row(size_t(N) + n);
      }
      load_tile<R>(rows, K, 0, t0);
    }
    float acc[R][B];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) acc[r][b] = 0.f;
    warp_dot<R, B, RowBf16>(rows, smem, bstride, K, acc, t0);
#pragma unroll
    for (int r = 0; r < kTnRows; ++r)
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const float v = warp_sum(acc[r][b]);
        const float u = GATED ? warp_sum(acc[GATED ? kTnRows + r : r][b]) : 0.f;
        if (lane == r * B + b && n0 + r < N) put(n0 + r, b, v, u);
      }
  }
}

// Blocks 0 .. g1 - 1: out = Wm norm1(x); the rest: the second part.
template <int B, int SECOND>
__global__ void __launch_bounds__(kGemvThreads, 2)
twin_in_kernel(TwinIn in, Matrix<WBf16> Wm, int N1, float* __restrict__ out, int ld_out, int g1, TwinFf ff) {
  extern __shared__ __align__(16) char smem[];
  __shared__ float red[kGemvWarps];
  __shared__ float inv_rms[B];
  const int K = in.ldx, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, chunks = K >> 3;
  const size_t bstride = XStage<WBf16>::bytes(K);
  // norm weights times x, unnormed; the sum of squares beside it
  auto stage = [&](const float* nw) {
#pragma unroll
    for (int b = 0; b < B; ++b) {
      XLoadF32 ld{in.x + size_t(b) * K, nw, 0.f};
      XStage<WBf16>::stage_part(smem + b * bstride, K, ld, threadIdx.x, kGemvThreads);
      const float ssq = block_sum_256(ld.ssq, red);
      if (threadIdx.x == 0) inv_rms[b] = 1.f / sqrtf(ssq / float(in.D) + in.eps);
    }
    __syncthreads();
  };
  if (int(blockIdx.x) < g1) {
    const int n0 = (blockIdx.x * kGemvWarps + warp) * kTnRows, step = g1 * kGemvWarps * kTnRows;
    RowBf16 rows[kTnRows];
    Tile<RowBf16, kTnRows> t0;
    if (n0 < N1) {              // weights wait for nothing: ask for the first tile at once
#pragma unroll
      for (int r = 0; r < kTnRows; ++r) rows[r] = Wm.row(min(n0 + r, N1 - 1));
      load_tile<kTnRows>(rows, K, 0, t0);
    }
    pdl_launch_dependents();
    pdl_wait();
    stage(in.w1);
    twin_rows<B, false>(Wm, N1, n0, step, smem, bstride, rows, t0,
                        [&](int n, int b, float v, float) { out[size_t(b) * ld_out + n] = v * inv_rms[b]; });
    return;
  }
  const int blk = blockIdx.x - g1;
  if (SECOND == kTwinGated) {
    const Matrix<WBf16> W{ff.w, K};
    const int g2 = gridDim.x - g1, n0 = (blk * kGemvWarps + warp) * kTnRows, step = g2 * kGemvWarps * kTnRows;
    RowBf16 rows[2 * kTnRows];
    Tile<RowBf16, 2 * kTnRows> t0;
    if (n0 < ff.N) {
#pragma unroll
      for (int r = 0; r < kTnRows; ++r) {
        const int n = min(n0 + r, ff.N - 1);
        rows[r] = W.row(n);
        rows[kTnRows + r] = W.row(size_t(ff.N) + n);
      }
      load_tile<2 * kTnRows>(rows, K, 0, t0);
    }
    pdl_launch_dependents();
    pdl_wait();
    stage(in.w2);
    twin_rows<B, true>(W, ff.N, n0, step, smem, bstride, rows, t0, [&](int n, int b, float g, float u) {
      ff.act[size_t(b) * ff.ld_act + n] = __float2bfloat16_rn(gated_act_fast(g * inv_rms[b], u * inv_rms[b], ff.limit));
    });
  } else if (SECOND == kTwinRouter) {
    // one block per router output, its warps share the row
    __shared__ float part[kGemvWarps][B];
    __shared__ unsigned int last;
    const __nv_bfloat16* row = ff.w + size_t(blk) * K;
    constexpr int kKeep = 4;
    uint4 wv[kKeep];
#pragma unroll
    for (int u = 0; u < kKeep; ++u) {
      const int c = u * kGemvThreads + threadIdx.x;
      wv[u] = c < chunks ? ldg_stream(row + (size_t(c) << 3)) : make_uint4(0u, 0u, 0u, 0u);
    }
    pdl_launch_dependents();
    pdl_wait();
    stage(in.w2);
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
        if (blk == 0) {           // the experts read norm2(x)
          float4* o = reinterpret_cast<float4*>(ff.h2 + size_t(b) * K + c * 8);
          const float s = inv_rms[b];
          o[0] = make_float4(x0.x * s, x0.y * s, x0.z * s, x0.w * s);
          o[1] = make_float4(x1.x * s, x1.y * s, x1.z * s, x1.w * s);
        }
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
      ff.logits[size_t(threadIdx.x) * ff.N + blk] = v * inv_rms[threadIdx.x];
      __threadfence();
    }
    __syncthreads();
    if (threadIdx.x == 0) last = (atomicAdd(ff.ticket, 1u) == unsigned(ff.N - 1)) ? 1u : 0u;
    __syncthreads();
    if (last) {
      __threadfence();
      for (int b = warp; b < B; b += kGemvWarps) {
        float* z = reinterpret_cast<float*>(smem) + b * ff.N;          // through L2: other blocks wrote the logits
        for (int i = lane; i < ff.N; i += 32) z[i] = __ldcg(ff.logits + size_t(b) * ff.N + i);
        __syncwarp();
        warp_route<kRouteChosen>(z, ff.bias, ff.N, ff.N, ff.top_k, ff.idx + size_t(b) * ff.top_k,
                                 ff.weights + size_t(b) * ff.top_k, nullptr, nullptr);
      }
      if (threadIdx.x == 0) *ff.ticket = 0u;
    }
  }
}

__device__ __forceinline__ float tn_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct GlaStep {
  const float* raw;               // [B, ld_raw]: q, k, v, g and the decay rank at their columns
  int ld_raw, at_k, at_v, at_g, at_low;
  const __nv_bfloat16* a2;        // [H * n, rank]
  int rank;
  const float* bias;              // [H * n]
  float inv_tau, scale;
  const float* norm;              // [H * d]
  float eps;
  const int* slots;
  float* state;                   // slot s: state + s * stride, [H, n, d]
  long long stride;
  __nv_bfloat16* a;               // [B, ld_a]
  int ld_a, n, d;
};

// grid (column blocks = one cluster, heads, batch rows); COLS columns a block.
template <int COLS, int ROWS>
__global__ void __launch_bounds__(kGemvThreads)
gla_decode_kernel(GlaStep p) {
  constexpr int G = kGemvThreads / COLS;
  extern __shared__ float sm[];
  float* sr = sm;                    // [n] r, k, decay
  float* sk = sr + p.n;
  float* sw = sk + p.n;
  float* low = sw + p.n;             // [rank]
  __shared__ float part[kGemvThreads];
  __shared__ float red[kGemvWarps];
  __shared__ float s_ssq;
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, n = p.n, d = p.d;
  const int g = tid / COLS, col = blockIdx.x * COLS + tid % COLS;
  const int per = (n + G - 1) / G, i0 = g * per, i1 = min(i0 + per, n);
  float* sp = p.state + size_t(p.slots[b]) * p.stride + size_t(h) * n * d + col;
  float s[ROWS];
  load_state<ROWS>(sp, d, i0, i1, col < d, s);
  pdl_launch_dependents();
  pdl_wait();
  const float* row = p.raw + size_t(b) * p.ld_raw;
  for (int i = tid; i < p.rank; i += kGemvThreads) low[i] = __ldcg(row + p.at_low + i);
  float own = 0.f, q = 0.f;
  if (tid < n) {
    q = __ldcg(row + h * n + tid) * p.scale;
    const float k = __ldcg(row + p.at_k + h * n + tid);
    sk[tid] = k;
    own = q * k;
  }
  const float v = col < d ? __ldcg(row + p.at_v + h * d + col) : 0.f;
  own = block_sum_256(own, red);     // low is visible, too
  if (tid < n) {
    float z = p.bias[h * n + tid];
    const __nv_bfloat16* wr = p.a2 + size_t(h * n + tid) * p.rank;
    for (int j = 0; j < p.rank; j += 8) {
      const uint4 w = *reinterpret_cast<const uint4*>(wr + j);
      z = fmaf(bf16lo(w.x), low[j], z); z = fmaf(bf16hi(w.x), low[j + 1], z);
      z = fmaf(bf16lo(w.y), low[j + 2], z); z = fmaf(bf16hi(w.y), low[j + 3], z);
      z = fmaf(bf16lo(w.z), low[j + 4], z); z = fmaf(bf16hi(w.z), low[j + 5], z);
      z = fmaf(bf16lo(w.w), low[j + 6], z); z = fmaf(bf16hi(w.w), low[j + 7], z);
    }
    const float alpha = expf(-tn_softplus(-z) * p.inv_tau);
    sw[tid] = alpha;
    sr[tid] = q * alpha;
  }
  __syncthreads();
  part[tid] = col < d ? step_state<ROWS, false>(sp, d, i0, i1, s, sr, sk, sw, 0.f, v) : 0.f;
  __syncthreads();
  float o = 0.f;
  if (tid < COLS && col < d) {
    o = own * v;
#pragma unroll
    for (int u = 0; u < G; ++u) o += part[u * COLS + tid];
  }
  float ssq = block_sum_256(o * o, red);
  if (gridDim.x > 1) {               // the head's other columns
    cg::cluster_group cluster = cg::this_cluster();
    if (tid == 0) s_ssq = ssq;
    cluster.sync();
    ssq = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) ssq += *cluster.map_shared_rank(&s_ssq, r);
    cluster.sync();                  // nobody leaves while a neighbour still reads its shared memory
  }
  if (tid < COLS && col < d) {
    const float inv = 1.f / sqrtf(ssq / float(d) + p.eps);
    p.a[size_t(b) * p.ld_a + h * d + col] =
        __float2bfloat16_rn(o * inv * p.norm[h * d + col] * step_silu(__ldcg(row + p.at_g + h * d + col)));
  }
}

struct SsdStep {
  const float* raw;               // [B, ld_raw]: z at 0, x | B | C at x_at, dt at dt_at
  int ld_raw, x_at, dt_at;
  const float* conv_w;            // [taps, channels]
  const float* conv_b;
  int taps;
  float* carried;                 // slot s: carried + s * stride, [taps - 1, channels]
  const float* dt_bias; const float* a_log; const float* skip;
  const int* slots;
  float* state;                   // [H, n, d]
  long long stride;
  float* out;                     // [B, ld_out] fp32
  int ld_out, H, G, n, d;
};
// Channel c's convolution without the current token.
__device__ __forceinline__ float past_conv(const SsdStep& p, const float* before, int ch, int c) {
  float a = p.conv_b[c];
#pragma unroll 4
  for (int j = 0; j < p.taps - 1; ++j) a = fmaf(p.conv_w[size_t(j) * ch + c], __ldcg(before + size_t(j) * ch + c), a);
  return a;
}

template <int COLS, int ROWS>
__global__ void __launch_bounds__(kGemvThreads)
ssd_decode_kernel(SsdStep p) {
  constexpr int G = kGemvThreads / COLS;
  extern __shared__ float sm[];
  float* sB = sm;                    // [n]
  float* sC = sB + p.n;
  __shared__ float sx[COLS];
  __shared__ float part[kGemvThreads];
  __shared__ float red[kGemvWarps];
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, n = p.n, d = p.d, inner = p.H * d, ch = inner + 2 * p.G * n;
  const int g = tid / COLS, c0 = blockIdx.x * COLS, col = c0 + tid % COLS;
  const int per = (n + G - 1) / G, i0 = g * per, i1 = min(i0 + per, n);
  const size_t slot = size_t(p.slots[b]) * p.stride;
  float* sp = p.state + slot + size_t(h) * n * d + col;
  float s[ROWS];
  load_state<ROWS>(sp, d, i0, i1, col < d, s);
  // B and C of the head's group, then x of the block's columns: what earlier tokens contribute waits for nothing, either
  const int grp = h / (p.H / p.G), last = p.taps - 1;
  const float* before = p.carried + slot;
  auto channel = [&](int i) {
    if (i < n) return inner + grp * n + i;
    if (i < 2 * n) return inner + p.G * n + grp * n + i - n;
    return i - 2 * n < COLS && c0 + i - 2 * n < d ? h * d + c0 + i - 2 * n : -1;
  };
  constexpr int kKeep = 2;
  float past[kKeep], now_w[kKeep];
  int chan[kKeep];
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    chan[u] = channel(u * kGemvThreads + tid);
    past[u] = chan[u] >= 0 ? past_conv(p, before, ch, chan[u]) : 0.f;
    now_w[u] = chan[u] >= 0 ? p.conv_w[size_t(last) * ch + chan[u]] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  const float* row = p.raw + size_t(b) * p.ld_raw;
  auto keep = [&](int i, float v) {
    if (i < 2 * n) sm[i] = v;
    else sx[i - 2 * n] = v;
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u)
    if (chan[u] >= 0) keep(u * kGemvThreads + tid, step_silu(fmaf(now_w[u], __ldcg(row + p.x_at + chan[u]), past[u])));
  for (int i = kKeep * kGemvThreads + tid; i < 2 * n + COLS; i += kGemvThreads) {
    const int c = channel(i);
    if (c >= 0) keep(i, step_silu(fmaf(p.conv_w[size_t(last) * ch + c], __ldcg(row + p.x_at + c), past_conv(p, before, ch, c))));
  }
  const float dt = tn_softplus(__ldcg(row + p.dt_at + h) + p.dt_bias[h]), decay = expf(-expf(p.a_log[h]) * dt);
  __syncthreads();
  const float own = block_sum_256(tid < n ? sB[tid] * sC[tid] : 0.f, red);
  const float x = col < d ? sx[tid % COLS] : 0.f;
  part[tid] = col < d ? step_state<ROWS, true>(sp, d, i0, i1, s, sC, sB, nullptr, decay, dt * x) : 0.f;
  __syncthreads();
  if (tid < COLS && col < d) {
    float o = 0.f;
#pragma unroll
    for (int u = 0; u < G; ++u) o += part[u * COLS + tid];
    p.out[size_t(b) * p.ld_out + h * d + col] = fmaf(decay, o, fmaf(own * dt, x, p.skip[h] * x));
  }
}

// grid (norm groups + blocks of channels, batch rows): f = y silu(z), f / rms(f over the group) * norm; the channels'
// blocks move the row's conv inputs up.
__global__ void __launch_bounds__(kGemvThreads)
ssd_finish_kernel(SsdStep p, const float* __restrict__ norm, float eps, int groups, int size, __nv_bfloat16* __restrict__ a,
                  int ld_a) {
  constexpr int kKeep = 16;
  __shared__ float red[kGemvWarps];
  const int b = blockIdx.y, at = blockIdx.x * size, tid = threadIdx.x;
  const float* row = p.raw + size_t(b) * p.ld_raw;
  pdl_launch_dependents();
  pdl_wait();
  if (int(blockIdx.x) >= groups) {
    const int ch = p.H * p.d + 2 * p.G * p.n, c = (blockIdx.x - groups) * kGemvThreads + tid;
    if (c >= ch) return;
    float* st = p.carried + size_t(p.slots[b]) * p.stride + c;
#pragma unroll 4
    for (int j = 0; j + 2 < p.taps; ++j) st[size_t(j) * ch] = st[size_t(j + 1) * ch];
    st[size_t(p.taps - 2) * ch] = __ldcg(row + p.x_at + c);
    return;
  }
  const float* y = p.out + size_t(b) * p.ld_out + at;
  float f[kKeep], ssq = 0.f;
  auto value = [&](int i) { return __ldcg(y + i) * step_silu(__ldcg(row + at + i)); };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = u * kGemvThreads + tid;
    f[u] = i < size ? value(i) : 0.f;
    ssq += f[u] * f[u];
  }
  for (int i = kKeep * kGemvThreads + tid; i < size; i += kGemvThreads) { const float v = value(i); ssq += v * v; }
  const float inv = 1.f / sqrtf(block_sum_256(ssq, red) / float(size) + eps);
  __nv_bfloat16* dst = a + size_t(b) * ld_a + at;
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = u * kGemvThreads + tid;
    if (i < size) dst[i] = __float2bfloat16_rn(f[u] * inv * norm[at + i]);
  }
  for (int i = kKeep * kGemvThreads + tid; i < size; i += kGemvThreads) dst[i] = __float2bfloat16_rn(value(i) * inv * norm[at + i]);
}

}  // namespace rb

using namespace rb;

#define RB_TN_DISPATCH(B_, CALL)                     \
  switch (B_) {                                      \
    case 1: { constexpr int kB = 1; return CALL; }   \
    case 2: { constexpr int kB = 2; return CALL; }   \
    case 3: { constexpr int kB = 3; return CALL; }   \
    case 4: { constexpr int kB = 4; return CALL; }   \
    default: return -2;                              \
  }

template <int B, int SECOND>
static int launch_twin_in(const TwinIn& in, const void* w, int N1, float* out, int ld_out, const TwinFf& ff, int pdl,
                          cudaStream_t st) {
  size_t smem = XStage<WBf16>::bytes(in.ldx) * B;
  if (SECOND == kTwinRouter && smem < size_t(B) * ff.N * 4) smem = size_t(B) * ff.N * 4;
  if (smem > kTnMaxSmem) return -2;
  auto kern = twin_in_kernel<B, SECOND>;
  RB_CHECK(set_max_smem(kern, smem));
  // as many blocks as stay resident; each part's blocks walk its rows, in step with the bytes they read
  int per_sm = 1;
  RB_CHECK(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kern, kGemvThreads, smem));
  constexpr int kTile = kGemvWarps * kTnRows;
  const int second = SECOND == kTwinRouter ? ff.N : 0;
  const int cap = sm_count() * (per_sm > 0 ? per_sm : 1);
  const int t1 = (N1 + kTile - 1) / kTile, t2 = SECOND == kTwinGated ? (ff.N + kTile - 1) / kTile : 0;
  const int room = cap - second > cap / 2 ? cap - second : cap / 2, passes = (t1 + 2 * t2 + room - 1) / room;
  const int g1 = (t1 + passes - 1) / passes;
  int g2 = (2 * t2 + passes - 1) / passes;
  if (g2 > t2) g2 = t2;
  return launch(kern, dim3(g1 + g2 + second), dim3(kGemvThreads), smem, st, pdl != 0, in,
                Matrix<WBf16>{static_cast<const __nv_bfloat16*>(w), in.ldx}, N1, out, ld_out, g1, ff);
}

static bool twin_in_ok(const float* x, const float* w1, int D, int ldx, int N1, int ld_out, int B) {
  return x && w1 && ldx >= 8 && ldx % 8 == 0 && D >= 1 && D <= ldx && N1 >= 1 && ld_out >= N1 && B >= 1 && B <= 4;
}

// Most batch rows one launch takes for rows of ldx values (0: none).
extern "C" int rmlx_twin_in_max_rows(int ldx) {
  int b = 4;
  while (b > 0 && XStage<WBf16>::bytes(ldx) * b > kTnMaxSmem) --b;
  return b;
}

// x fp32 [B, ldx], norm weights fp32 [ldx], w bf16 [N1, ldx], out fp32 [B, ld_out]; w_ff (or null) bf16 [2 N, ldx] =
// [gate; up], act bf16 [B, ld_act].
extern "C" int rmlx_twin_in_gated(const float* x, const float* w1, const float* w2, float eps, int D, int ldx, const void* w,
                                  int N1, float* out, int ld_out, const void* w_ff, int N, void* act, int ld_act, float limit,
                                  int B, int pdl, cudaStream_t st) {
  if (!twin_in_ok(x, w1, D, ldx, N1, ld_out, B) || (w_ff && (!w2 || N < 1 || ld_act < N))) return -2;
  const TwinIn in{x, w1, w2, eps, D, ldx};
  TwinFf ff{};
  ff.w = static_cast<const __nv_bfloat16*>(w_ff); ff.N = N; ff.act = static_cast<__nv_bfloat16*>(act); ff.ld_act = ld_act;
  ff.limit = limit;
  if (!w_ff) { RB_TN_DISPATCH(B, (launch_twin_in<kB, kTwinNone>(in, w, N1, out, ld_out, ff, pdl, st))) }
  RB_TN_DISPATCH(B, (launch_twin_in<kB, kTwinGated>(in, w, N1, out, ld_out, ff, pdl, st)))
}

// The same with a router: w_r bf16 [N, ldx], bias fp32 [N]; logits fp32 [B, N] scratch, h2 fp32 [B, ldx]; ticket: one
// word, zero on entry and on exit.
extern "C" int rmlx_twin_in_router(const float* x, const float* w1, const float* w2, float eps, int D, int ldx, const void* w,
                                   int N1, float* out, int ld_out, const void* w_r, const float* bias, int N, float* logits,
                                   float* h2, int* idx, float* weights, int top_k, unsigned int* ticket, int B, int pdl,
                                   cudaStream_t st) {
  if (!twin_in_ok(x, w1, D, ldx, N1, ld_out, B) || !w2 || !w_r || !bias || N < 1 || N > kRouteMaxOutputs || top_k < 1 ||
      top_k > kRouteMaxTop || top_k > N || !ticket)
    return -2;
  const TwinIn in{x, w1, w2, eps, D, ldx};
  TwinFf ff{};
  ff.w = static_cast<const __nv_bfloat16*>(w_r); ff.N = N; ff.bias = bias; ff.logits = logits; ff.h2 = h2; ff.idx = idx;
  ff.weights = weights; ff.ticket = ticket; ff.top_k = top_k;
  RB_TN_DISPATCH(B, (launch_twin_in<kB, kTwinRouter>(in, w, N1, out, ld_out, ff, pdl, st)))
}

// 1 when the decode kernel of gated linear attention takes a state of n x d.
extern "C" int rmlx_gla_decode_supported(int n, int d) { return n >= 1 && n <= 256 && d >= 1 && d <= 512; }

// raw fp32 [B, ld_raw] with q at 0; rank a multiple of eight, a2 rows 16-byte aligned; a bf16 [B, ld_a].
extern "C" int rmlx_gla_decode(const float* raw, int ld_raw, int at_k, int at_v, int at_g, int at_low, const void* a2, int rank,
                               const float* bias, float inv_tau, float scale, const float* norm, float eps, const int* slots,
                               float* state, long long stride, void* a, int ld_a, int B, int H, int n, int d, int pdl,
                               cudaStream_t st) {
  if (B < 1 || B > 65535 || H < 1 || H > 65535 || !rmlx_gla_decode_supported(n, d) || rank < 8 || rank % 8 || rank > 4096 ||
      !slots || ld_a < H * d || ld_raw < at_low + rank || ld_raw < at_g + H * d || (reinterpret_cast<uintptr_t>(a2) & 15))
    return -2;
  const GlaStep p{raw, ld_raw, at_k, at_v, at_g, at_low, static_cast<const __nv_bfloat16*>(a2), rank, bias, inv_tau, scale,
                  norm, eps, slots, state, stride, static_cast<__nv_bfloat16*>(a), ld_a, n, d};
  const size_t smem = size_t(3 * n + rank) * sizeof(float);
#define RB_GD(C_, R_) return launch_columns(gla_decode_kernel<C_, R_>, p, (d + C_ - 1) / C_, H, B, smem, true, pdl, st)
  RB_STATE_DISPATCH(n, d, RB_GD);
#undef RB_GD
}

// raw fp32 [B, ld_raw] with the gate at 0; out fp32 [B, ld_out] scratch; a bf16 [B, ld_a]. Two launches.
extern "C" int rmlx_ssd_decode(const float* raw, int ld_raw, int x_at, int dt_at, const float* conv_w, const float* conv_b,
                               int taps, float* carried, const float* dt_bias, const float* a_log, const float* skip,
                               const int* slots, float* state, long long stride, float* out, int ld_out, const float* norm,
                               float eps, int norm_groups, void* a, int ld_a, int B, int H, int G, int n, int d, int pdl,
                               cudaStream_t st) {
  if (B < 1 || B > 65535 || H < 1 || H > 65535 || G < 1 || H % G || n < 1 || n > 256 || d < 1 || taps < 1 || !slots ||
      norm_groups < 1 || (H * d) % norm_groups || ld_a < H * d || ld_out < H * d || ld_raw < dt_at + H ||
      ld_raw < x_at + H * d + 2 * G * n || x_at < H * d || (taps > 1 && !carried))
    return -2;
  const SsdStep p{raw, ld_raw, x_at, dt_at, conv_w, conv_b, taps, carried, dt_bias, a_log, skip, slots, state, stride, out,
                  ld_out, H, G, n, d};
  const size_t smem = size_t(2 * n) * sizeof(float);
  const int rc = [&]() -> int {
    // a head's columns need not meet in one block here
#define RB_SD(C_, R_) return launch_columns(ssd_decode_kernel<C_, R_>, p, (d + C_ - 1) / C_, H, B, smem, false, pdl, st)
    RB_STATE_DISPATCH(n, 1, RB_SD);
#undef RB_SD
  }();
  if (rc) return rc;
  const int movers = taps > 1 ? (H * d + 2 * G * n + kGemvThreads - 1) / kGemvThreads : 0;
  return launch(ssd_finish_kernel, dim3(norm_groups + movers, B), dim3(kGemvThreads), 0, st, pdl != 0, p, norm, eps, norm_groups,
                H * d / norm_groups, static_cast<__nv_bfloat16*>(a), ld_a);
}
