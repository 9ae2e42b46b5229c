// Row kernels of decoders with a layer norm before and after each sublayer, x <- x + norm_b(f(conv(norm(x)))), x in fp32:
//
//   sandwich_norm  x += LN(y) (y: a sublayer's rows, or the weighted rows of a token's experts) and h = LN(x) for the
//                  sublayer that follows, in one pass
//   short_conv     h + causal depthwise convolution of h over time, the last inputs carried per sequence
//   poly_norm      a N(z) + b N(z^2) + c N(z^3) + e, N: division by the row's root mean square
//   sandwich_step  decode rows through both of the first two in one launch
//
// LN(v) = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w + b. Activations are bf16 (serving) or fp32 (the all-32-bit
// mode); norms, convolutions and the residual are fp32 in both.
#include <type_traits>

#include "../common/launch.cuh"
#include "../common/row_sources.cuh"
#include "../common/rows.cuh"

namespace rb {

// Weight and bias of a norm: [2, ld] fp32.
struct Affine {
  const float* w;
  int ld;
  __device__ __forceinline__ void load(int c, float (&g)[8], float (&b)[8]) const {
    load8(w + c * 8, g);
    load8(w + ld + c * 8, b);
  }
};

// A warp's share of a row: how many values, their mean, and the sum of their squared deviations from it. Shares of several
// warps are joined by the deviations of the means, so nothing cancels and a block needs one barrier per norm.
struct Share {
  float n, mean, m2;
};
template <int WARPS>
__device__ __forceinline__ void join_shares(const Share (&s)[WARPS], float total, float eps, float& mean, float& inv) {
  float m = 0.f, q = 0.f;
#pragma unroll
  for (int w = 0; w < WARPS; ++w) m = fmaf(s[w].n, s[w].mean, m);
  mean = m / total;
#pragma unroll
  for (int w = 0; w < WARPS; ++w) {
    const float d = s[w].mean - mean;
    q += fmaf(s[w].n * d, d, s[w].m2);
  }
  inv = 1.f / sqrtf(q / total + eps);
}

// Eight values as they are stored; rows pass through once, so their loads leave the first-level cache to the weights.
template <class T>
struct Packed;
template <>
struct Packed<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = __ldcs(reinterpret_cast<const uint4*>(p)); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = bf16lo(v.x); f[1] = bf16hi(v.x); f[2] = bf16lo(v.y); f[3] = bf16hi(v.y);
    f[4] = bf16lo(v.z); f[5] = bf16hi(v.z); f[6] = bf16lo(v.w); f[7] = bf16hi(v.w);
  }
};
template <>
struct Packed<float> {
  float v[8];
  __device__ __forceinline__ void load(const float* p) {
    const float4 a = __ldcs(reinterpret_cast<const float4*>(p)), b = __ldcs(reinterpret_cast<const float4*>(p + 4));
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = v[i];
  }
};

// What a thread keeps of the rows it norms.
template <class SRC>
struct Kept {
  Packed<float> p;
  __device__ __forceinline__ void load(const SRC& src, int t, int c) {
    const float none[8] = {};
    src.load(t, c, none, p.v);
  }
};
template <class TY>
struct Kept<RowSource<TY>> {
  Packed<TY> p;
  __device__ __forceinline__ void load(const RowSource<TY>& src, int t, int c) { p.load(src.y + size_t(t) * src.ldy + c * 8); }
};

// x[t] += LN(source; wy); h[t] = LN(x[t]; wh) (h may be null) for R rows a block. Columns past D are zero in the source, x
// and the weights, so they stay zero, add nothing to a sum, and mean^2 each to a sum of squared deviations. KEEP chunks of
// eight a thread keeps; rows wider than KEEP * 8 * 256 are read again.
template <class SRC, bool ADD, class T, int KEEP, int R, int BLOCKS>
__global__ void __launch_bounds__(kRowThreads, BLOCKS)
sandwich_norm_kernel(SRC src, Affine wy, float* __restrict__ x, Affine wh, T* __restrict__ h, float eps, int rows, int D, int ldx) {
  constexpr int kWarps = kRowThreads / 32;
  __shared__ Share part[2][R][kWarps];
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * R, chunks = ldx >> 3;
  auto row = [&](int r) { return min(t0 + r, rows - 1); };         // (past the last row: done once more, not stored)
  auto chunk = [&](int u) { return u * kRowThreads + threadIdx.x; };
  SRC from[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    from[r] = src;
    if constexpr (ADD) from[r].prepare(row(r));
  }
  Packed<float> f[R][KEEP];
  float count = 0.f, pads = 0.f;
  for (int c = threadIdx.x; c < chunks; c += kRowThreads) {
    const int n = max(0, min(8, D - c * 8));
    count += float(n);
    pads += float(8 - n);
  }
  count = warp_sum(count);
  pads = warp_sum(pads);
  // mean and 1 / deviation of the rows; keep[] holds a row's first chunks, get(r, c, .) gives the others
  auto moments = [&](auto& keep, auto get, Share (&mine)[R][kWarps], float (&mean)[R], float (&inv)[R]) {
    float v[R];
    auto each = [&](auto use) {
#pragma unroll
      for (int u = 0; u < KEEP; ++u)
        if (chunk(u) < chunks) {
#pragma unroll
          for (int r = 0; r < R; ++r) {
            float a[8];
            keep(r, u, a);
            use(r, a);
          }
        }
      for (int c = chunk(KEEP); c < chunks; c += kRowThreads)
#pragma unroll
        for (int r = 0; r < R; ++r) {
          float a[8];
          get(r, c, a);
          use(r, a);
        }
    };
#pragma unroll
    for (int r = 0; r < R; ++r) v[r] = 0.f;
    each([&](int r, const float (&a)[8]) {
#pragma unroll
      for (int i = 0; i < 8; ++i) v[r] += a[i];
    });
#pragma unroll
    for (int r = 0; r < R; ++r) mean[r] = count > 0.f ? warp_sum(v[r]) / count : 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) v[r] = 0.f;
    each([&](int r, const float (&a)[8]) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float d = a[i] - mean[r];
        v[r] = fmaf(d, d, v[r]);
      }
    });
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float q = fmaf(-pads * mean[r], mean[r], warp_sum(v[r]));
      if ((threadIdx.x & 31) == 0) mine[r][threadIdx.x >> 5] = Share{count, mean[r], q};
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < R; ++r) join_shares<kWarps>(mine[r], float(D), eps, mean[r], inv[r]);
  };
  auto scaled = [&](const float (&g)[8], const float (&b)[8], const float (&a)[8], float mean, float inv, float (&o)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = fmaf((a[i] - mean) * inv, g[i], b[i]);
  };
  float mean[R], inv[R];
  if constexpr (ADD) {
    Kept<SRC> y[R][KEEP];
#pragma unroll
    for (int u = 0; u < KEEP; ++u)
      if (chunk(u) < chunks) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
          y[r][u].load(from[r], row(r), chunk(u));
          f[r][u].load(x + size_t(row(r)) * ldx + chunk(u) * 8);
        }
      }
    auto again = [&](int r, int c, float (&a)[8]) {
      Kept<SRC> k;
      k.load(from[r], row(r), c);
      k.p.get(a);
    };
    auto kept = [&](int r, int u, float (&a)[8]) { y[r][u].p.get(a); };
    moments(kept, again, part[0], mean, inv);
    auto add = [&](int r, int c, const float (&g)[8], const float (&b)[8], const float (&a)[8], float (&v)[8]) {
      float o[8];
      scaled(g, b, a, mean[r], inv[r], o);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] += o[i];
      if (r == 0 || t0 + r < rows) store8(x + size_t(row(r)) * ldx + c * 8, v);
    };
#pragma unroll
    for (int u = 0; u < KEEP; ++u)
      if (chunk(u) < chunks) {
        float g[8], b[8];
        wy.load(chunk(u), g, b);
#pragma unroll
        for (int r = 0; r < R; ++r) {
          float a[8];
          kept(r, u, a);
          add(r, chunk(u), g, b, a, f[r][u].v);
        }
      }
    for (int c = chunk(KEEP); c < chunks; c += kRowThreads) {
      float g[8], b[8];
      wy.load(c, g, b);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float a[8], v[8];
        again(r, c, a);
        load8(x + size_t(row(r)) * ldx + c * 8, v);
        add(r, c, g, b, a, v);
      }
    }
  } else {
#pragma unroll
    for (int u = 0; u < KEEP; ++u)
      if (chunk(u) < chunks) {
#pragma unroll
        for (int r = 0; r < R; ++r) f[r][u].load(x + size_t(row(r)) * ldx + chunk(u) * 8);
      }
  }
  if (!h) return;
  // (a thread reads again what it has written itself)
  auto kept_x = [&](int r, int u, float (&a)[8]) { f[r][u].get(a); };
  moments(kept_x, [&](int r, int c, float (&a)[8]) { load8(x + size_t(row(r)) * ldx + c * 8, a); }, part[1], mean, inv);
  auto put = [&](int c, auto value) {
    float g[8], b[8], o[8];
    wh.load(c, g, b);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      scaled(g, b, value(r), mean[r], inv[r], o);
      if (r == 0 || t0 + r < rows) store8(h + size_t(row(r)) * ldx + c * 8, o);
    }
  };
#pragma unroll
  for (int u = 0; u < KEEP; ++u)
    if (chunk(u) < chunks) put(chunk(u), [&](int r) -> const float (&)[8] { return f[r][u].v; });
  for (int c = chunk(KEEP); c < chunks; c += kRowThreads) {
    float a[R][8];
#pragma unroll
    for (int r = 0; r < R; ++r) load8(x + size_t(row(r)) * ldx + c * 8, a[r]);
    put(c, [&](int r) -> const float (&)[8] { return a[r]; });
  }
}

// out[t] = h[t] + sum_j w[j] h[t - taps + 1 + j] within a sequence. A thread owns eight columns. Blocks y < strips: `strip`
// rows each (kConvRows at a time), of which those with all their inputs in the batch are done; the others: one run of rows each, its first
// taps - 1 rows with the help of the carried inputs, which it then replaces by the run's last ones. So a sequence's carried
// inputs are read and written by one thread alone.
constexpr int kConvRows = 4;
template <class T, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_kernel(const T* __restrict__ h, T* __restrict__ out, int ldx, const float* __restrict__ w, int n_taps,
                  float* __restrict__ carried, long long stride, const int4* __restrict__ runs, const int* __restrict__ slots,
                  int T_rows, int strip, int strips) {
  pdl_launch_dependents();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : n_taps, keep = taps - 1;
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= ldx) return;
  auto put = [&](int t, const float (&a)[8]) { store8(out + size_t(t) * ldx + c, a); };
  if (int(blockIdx.y) < strips) {
    const int t0 = blockIdx.y * strip, n = min(strip, T_rows - t0);
    if constexpr (TAPS > 0) {
      constexpr int K = TAPS - 1;
      Packed<T> v[kConvRows + K];
      float g[TAPS][8];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) load8(w + size_t(j) * ldx + c, g[j]);
#pragma unroll
      for (int i = 0; i < K; ++i)
        if (t0 + i >= K) v[i].load(h + size_t(t0 + i - K) * ldx + c);
      // rows of one sequence are neighbours: with both ends its own, the strip is one sequence's
      const bool inside = t0 >= K && (K == 0 || slots[max(t0 - K, 0)] == slots[t0 + n - 1]);
      for (int at = t0; at < t0 + n; at += kConvRows) {
#pragma unroll
        for (int i = 0; i < kConvRows; ++i)
          if (at + i < T_rows) v[K + i].load(h + size_t(at + i) * ldx + c);
#pragma unroll
        for (int i = 0; i < kConvRows; ++i) {
          const int t = at + i;
          if (t >= t0 + n || (!inside && (t < K || (K > 0 && slots[t - K] != slots[t])))) continue;
          float a[8], s[8] = {};
#pragma unroll
          for (int j = 0; j < TAPS; ++j) {
            v[i + j].get(a);
#pragma unroll
            for (int e = 0; e < 8; ++e) s[e] = fmaf(g[j][e], a[e], s[e]);
          }
#pragma unroll
          for (int e = 0; e < 8; ++e) a[e] += s[e];          // (the last one read is the row itself)
          put(t, a);
        }
#pragma unroll
        for (int i = 0; i < K; ++i) v[i] = v[kConvRows + i];
      }
    } else {
      for (int t = t0; t < t0 + n; ++t) {
        if (t < keep || (keep > 0 && slots[t - keep] != slots[t])) continue;
        float a[8], x[8], g[8];
        load8(h + size_t(t) * ldx + c, a);
        float s[8] = {};
        for (int j = 0; j < taps; ++j) {
          load8(h + size_t(t - keep + j) * ldx + c, x);
          load8(w + size_t(j) * ldx + c, g);
#pragma unroll
          for (int e = 0; e < 8; ++e) s[e] = fmaf(g[e], x[e], s[e]);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) a[e] += s[e];
        put(t, a);
      }
    }
    return;
  }
  const int r = blockIdx.y - strips;
  int row0 = r, len = 1, slot;
  if (runs) {
    const int4 q = runs[r];
    row0 = q.x; len = q.y; slot = q.z;
  } else {
    slot = slots[r];
  }
  float* past = carried + size_t(slot) * stride + c;             // [keep, ldx], oldest first
  for (int i = 0; i < min(len, keep); ++i) {
    float a[8], x[8], g[8], s[8] = {};
    load8(h + size_t(row0 + i) * ldx + c, a);
    for (int j = 0; j < taps; ++j) {
      const int k = i - keep + j;                                // row of the run; below 0: carried
      if (k >= 0) load8(h + size_t(row0 + k) * ldx + c, x);
      else load8(past + size_t(keep + k) * ldx, x);
      load8(w + size_t(j) * ldx + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) s[e] = fmaf(g[e], x[e], s[e]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) a[e] += s[e];
    put(row0 + i, a);
  }
  for (int m = 0; m < keep; ++m) {                               // ascending, reading ahead of what is written
    const int i = len - keep + m;
    float x[8];
    if (i >= 0) load8(h + size_t(row0 + i) * ldx + c, x);
    else load8(past + size_t(m + len) * ldx, x);
    store8(past + size_t(m) * ldx, x);
  }
}

// out[t] = a N(z) + b N(z^2) + c N(z^3) + e over the first D columns; the rest is zero.
template <class T, int KEEP>
__global__ void __launch_bounds__(kRowThreads)
poly_norm_kernel(const T* __restrict__ z, const float* __restrict__ act, float eps, T* __restrict__ out, int D, int ld) {
  __shared__ float red[3][kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int chunks = ld >> 3;
  const T* row = z + size_t(blockIdx.x) * ld;
  T* dst = out + size_t(blockIdx.x) * ld;
  Packed<T> f[KEEP];
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto take = [&](int c, const Packed<T>& p) {
    float a[8];
    p.get(a);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (c * 8 + i >= D) a[i] = 0.f;
      const float q = a[i] * a[i], q2 = q * q;
      s2 += q;
      s4 += q2;
      s6 = fmaf(q2, q, s6);
    }
  };
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) f[u].load(row + c * 8);
  }
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) take(c, f[u]);
  }
  for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    Packed<T> p;
    p.load(row + c * 8);
    take(c, p);
  }
  s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = s2; red[1][threadIdx.x >> 5] = s4; red[2][threadIdx.x >> 5] = s6; }
  __syncthreads();
  float k[3];
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < kRowThreads / 32; ++w) v += red[i][w];
    k[i] = act[i] / sqrtf(v / float(D) + eps);
  }
  const float e = act[3];
  auto put = [&](int c, const Packed<T>& p) {
    float a[8], o[8];
    p.get(a);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = c * 8 + i < D ? fmaf(a[i], fmaf(a[i], fmaf(a[i], k[2], k[1]), k[0]), e) : 0.f;
    store8(dst + c * 8, o);
  };
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) put(c, f[u]);
  }
  for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    Packed<T> p;
    p.load(row + c * 8);
    put(c, p);
  }
}

// ------------------------------------------------------------------ decode
constexpr int kStepThreads = 512;

template <class SRC, class T>
struct SandwichStep {
  SRC src;                  // finished sublayer
  int add;                  // 0: there is none
  float* x;                 // [B, ldx]
  Affine wy, wh;
  T* h;                     // [B, ldx]
  const float* conv;        // [taps, ldx], or null: no convolution
  int taps;
  float* carried;           // slot s: carried + s * stride, [taps - 1, ldx]
  long long stride;
  const int* slots;
  float eps;
  int D, ldx;
};

__device__ __forceinline__ void step_copy32(float* dst, const float* src) {      // 32 bytes, asynchronously
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + 4)), "l"(src + 4) : "memory");
}

// One block per row, E chunks of eight columns a thread. What no kernel of the step writes is asked for before the wait: the
// weights go to shared memory (every thread its own columns'), the carried inputs move up, and their share of the
// convolution is taken.
template <int E, class SRC, class T>
__global__ void __launch_bounds__(kStepThreads)
sandwich_step_kernel(SandwichStep<SRC, T> p) {
  constexpr int kWarps = kStepThreads / 32;
  extern __shared__ __align__(16) float sw[];          // [5][chunks][8]: weight, bias of both norms, the current token's tap
  __shared__ Share part[2][kWarps];
  const int b = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, chunks = p.ldx >> 3;
  auto chunk = [&](int e) { return e * kStepThreads + tid; };
  auto own = [&](int k, int c) { return sw + (size_t(k) * chunks + c) * 8; };
  float* st = p.conv && p.taps > 1 ? p.carried + size_t(p.slots[b]) * p.stride : nullptr;
  float count = 0.f, pads = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int c = chunk(e);
    if (c >= chunks) continue;
    const int n = max(0, min(8, p.D - c * 8));
    count += float(n);
    pads += float(8 - n);
    if (p.add) {
      step_copy32(own(0, c), p.wy.w + c * 8);
      step_copy32(own(1, c), p.wy.w + p.ldx + c * 8);
    }
    step_copy32(own(2, c), p.wh.w + c * 8);
    step_copy32(own(3, c), p.wh.w + p.ldx + c * 8);
    if (p.conv) step_copy32(own(4, c), p.conv + size_t(p.taps - 1) * p.ldx + c * 8);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  float past[E][8];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int c = chunk(e);
#pragma unroll
    for (int i = 0; i < 8; ++i) past[e][i] = 0.f;
    if (c >= chunks || !p.conv) continue;
#pragma unroll 3
    for (int j = 0; j < p.taps - 1; ++j) {
      float w[8], v[8];
      load8(p.conv + size_t(j) * p.ldx + c * 8, w);
      load8(st + size_t(j) * p.ldx + c * 8, v);
      if (j > 0) store8(st + size_t(j - 1) * p.ldx + c * 8, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) past[e][i] = fmaf(w[i], v[i], past[e][i]);
    }
  }
  count = warp_sum(count);
  pads = warp_sum(pads);
  pdl_launch_dependents();
  pdl_wait();
  if (p.add) p.src.prepare(b);
  const float none[8] = {};
  float x[E][8], y[E][8];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    if (chunk(e) < chunks) {
      load8(p.x + size_t(b) * p.ldx + chunk(e) * 8, x[e]);
      if (p.add) p.src.load(b, chunk(e), none, y[e]);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) x[e][i] = y[e][i] = 0.f;
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  // mean and 1 / deviation over the row (columns past D are zero)
  auto moments = [&](const float (&v)[E][8], Share (&mine)[kWarps], float& mean, float& inv) {
    float s = 0.f, q = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e)
#pragma unroll
      for (int i = 0; i < 8; ++i) s += v[e][i];
    mean = count > 0.f ? warp_sum(s) / count : 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e)
      if (chunk(e) < chunks) {
#pragma unroll
        for (int i = 0; i < 8; ++i) q = fmaf(v[e][i] - mean, v[e][i] - mean, q);
      }
    q = fmaf(-pads * mean, mean, warp_sum(q));
    if (lane == 0) mine[warp] = Share{count, mean, q};
    __syncthreads();
    join_shares<kWarps>(mine, float(p.D), p.eps, mean, inv);
  };
  float mean, inv;
  if (p.add) {
    moments(y, part[0], mean, inv);
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int c = chunk(e);
      if (c >= chunks) continue;
      float g[8], o[8];
      load8(own(0, c), g);
      load8(own(1, c), o);
#pragma unroll
      for (int i = 0; i < 8; ++i) x[e][i] += fmaf((y[e][i] - mean) * inv, g[i], o[i]);
      store8(p.x + size_t(b) * p.ldx + c * 8, x[e]);
    }
  }
  moments(x, part[1], mean, inv);
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int c = chunk(e);
    if (c >= chunks) continue;
    float g[8], o[8], a[8];
    load8(own(2, c), g);
    load8(own(3, c), o);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] = o[i] = fmaf((x[e][i] - mean) * inv, g[i], o[i]);
    if (p.conv) {
      load8(own(4, c), g);
#pragma unroll
      for (int i = 0; i < 8; ++i) o[i] += fmaf(g[i], a[i], past[e][i]);
      if (p.taps > 1) store8(st + size_t(p.taps - 2) * p.ldx + c * 8, a);
    }
    store8(p.h + size_t(b) * p.ldx + c * 8, o);
  }
}

template <class SRC, bool ADD, class TH>
static int launch_sandwich(SRC src, const float* wy, float* x, const float* wh, TH* h, float eps, int T, int D, int ldx, int pdl,
                           cudaStream_t st) {
  const Affine ay{wy, ldx}, ah{wh, ldx};
  auto go = [&](auto kern, int per) -> int {
    return launch(kern, dim3((T + per - 1) / per), dim3(kRowThreads), 0, st, pdl != 0, src, ay, x, ah, h, eps, T, D, ldx);
  };
  // where rows are plenty, several a block share its weights and barriers; else as many blocks as the registers allow
  const int keep = (ldx + 8 * kRowThreads - 1) / (8 * kRowThreads);
  const bool some = T >= 8 * sm_count(), many = T >= 16 * sm_count();
  if constexpr (sizeof(TH) == 4) {
    return keep <= 2 ? go(sandwich_norm_kernel<SRC, ADD, TH, 2, 1, 2>, 1) : go(sandwich_norm_kernel<SRC, ADD, TH, 4, 1, 2>, 1);
  } else if constexpr (!std::is_same<SRC, RowSource<float>>::value && !std::is_same<SRC, RowSource<__nv_bfloat16>>::value) {
    if (keep > 2) return go(sandwich_norm_kernel<SRC, ADD, TH, 4, 1, 2>, 1);
    if (keep > 1) return some ? go(sandwich_norm_kernel<SRC, ADD, TH, 2, 2, 2>, 2) : go(sandwich_norm_kernel<SRC, ADD, TH, 2, 1, 2>, 1);
    return some ? go(sandwich_norm_kernel<SRC, ADD, TH, 1, 2, 3>, 2) : go(sandwich_norm_kernel<SRC, ADD, TH, 1, 1, 3>, 1);
  } else {
    if (keep > 2) return go(sandwich_norm_kernel<SRC, ADD, TH, 4, 1, 2>, 1);
    if (keep > 1) return many ? go(sandwich_norm_kernel<SRC, ADD, TH, 2, 2, 3>, 2) : go(sandwich_norm_kernel<SRC, ADD, TH, 2, 1, 4>, 1);
    return many ? go(sandwich_norm_kernel<SRC, ADD, TH, 1, 4, 3>, 4)
           : some ? go(sandwich_norm_kernel<SRC, ADD, TH, 1, 2, 4>, 2) : go(sandwich_norm_kernel<SRC, ADD, TH, 1, 1, 4>, 1);
  }
}

template <class SRC, class T>
static int launch_step(const SandwichStep<SRC, T>& p, int B, int pdl, cudaStream_t st) {
  const int pieces = (p.ldx + 8 * kStepThreads - 1) / (8 * kStepThreads);
  auto kern = pieces <= 1 ? sandwich_step_kernel<1, SRC, T> : pieces <= 2 ? sandwich_step_kernel<2, SRC, T>
                                                                           : sandwich_step_kernel<3, SRC, T>;
  const size_t smem = size_t(5) * p.ldx * sizeof(float);
  RB_CHECK(set_max_smem(kern, smem));
  return launch(kern, dim3(B), dim3(kStepThreads), smem, st, pdl != 0, p);
}

}  // namespace rb

using namespace rb;

// x fp32 [T, ldx]; wy, wh fp32 [2, ldx] = (weight, bias). y (or null: nothing is added) in the compute type, rows ldy apart:
// the sublayer's rows, or (row_of_pair) expert rows with weights [T, top_k]. h [T, ldx] fp32 (f32) or bf16, or null. ldx, ldy
// multiples of eight.
extern "C" int rmlx_sandwich_norm(float* x, const void* y, int ldy, const int* row_of_pair, const float* weights, int top_k,
                                  const float* wy, const float* wh, void* h, float eps, int T, int D, int ldx, int f32, int pdl,
                                  cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || ldx % 8 || (h && !wh) || (!h && !y)) return -2;
  if (y && (ldy % 8 || ldy < ldx || !wy || (row_of_pair && (!weights || top_k < 1)))) return -2;
  auto run = [&](auto* p) -> int {
    using TY = std::remove_const_t<std::remove_pointer_t<decltype(p)>>;
    TY* out = static_cast<TY*>(h);
    if (!p) return launch_sandwich<RowSource<TY>, false, TY>(RowSource<TY>{p, 0}, nullptr, x, wh, out, eps, T, D, ldx, pdl, st);
    if (row_of_pair)
      return launch_sandwich<ExpertSource<TY>, true, TY>(ExpertSource<TY>{p, ldy, row_of_pair, weights, nullptr, top_k}, wy, x, wh,
                                                         out, eps, T, D, ldx, pdl, st);
    return launch_sandwich<RowSource<TY>, true, TY>(RowSource<TY>{p, ldy}, wy, x, wh, out, eps, T, D, ldx, pdl, st);
  };
  return f32 ? run(static_cast<const float*>(y)) : run(static_cast<const __nv_bfloat16*>(y));
}

// h, out [T, ldx] fp32 (f32) or bf16, not the same; w fp32 [taps, ldx], the last row is the current token's. carried: slot s
// at carried + s * stride (stride a multiple of four), fp32 [taps - 1, ldx]; slots int32 [T]: every row's slot (one tap: or null); runs int32
// [n_runs, 4] = (first row, rows, slot, -), 16-byte aligned, the runs' rows in order and without gaps, no slot twice, or
// null: every row is a run.
extern "C" int rmlx_short_conv(const void* h, void* out, int ldx, const float* w, int taps, float* carried, long long stride,
                               const int* runs, const int* slots, int n_runs, int T, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || ldx < 8 || ldx % 8 || taps < 1 || taps > 64 || h == out || n_runs < 1 || n_runs > T || (!runs && n_runs != T) ||
      (taps > 1 && (!carried || !slots || stride % 4 || (reinterpret_cast<uintptr_t>(carried) & 15))) || (reinterpret_cast<uintptr_t>(runs) & 15))
    return -2;
  // longer strips read fewer rows and weights twice, as far as there is work for every SM
  const int wide = (ldx / 8 + 127) / 128;
  int strip = kConvRows;
  while (strip < 4 * kConvRows && (long long)wide * ((T + 2 * strip - 1) / (2 * strip)) >= 12 * sm_count()) strip *= 2;
  const int strips = runs || taps == 1 ? (T + strip - 1) / strip : 0, tails = taps > 1 ? n_runs : 0;
  if (strips + tails > 65535) return -2;
  const dim3 grid(wide, strips + tails);
  auto go = [&](auto* type) -> int {
    using T_ = std::remove_pointer_t<decltype(type)>;
    auto kern = taps == 4 ? short_conv_kernel<T_, 4> : taps == 3 ? short_conv_kernel<T_, 3>
                : taps == 2 ? short_conv_kernel<T_, 2> : short_conv_kernel<T_, 0>;
    return launch(kern, grid, dim3(128), 0, st, pdl != 0, static_cast<const T_*>(h), static_cast<T_*>(out), ldx, w, taps, carried,
                  stride, reinterpret_cast<const int4*>(runs), slots, T, strip, strips);
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// z, out [T, ld] fp32 (f32) or bf16 (may be the same), ld a multiple of eight; act fp32 [4] = a, b, c, e.
extern "C" int rmlx_poly_norm(const void* z, const float* act, float eps, void* out, int T, int D, int ld, int f32, int pdl,
                              cudaStream_t st) {
  if (T < 1 || D < 1 || ld < D || ld % 8 || !act) return -2;
  auto go = [&](auto kern, auto* type) -> int {
    using T_ = std::remove_pointer_t<decltype(type)>;
    return launch(kern, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, static_cast<const T_*>(z), act, eps, static_cast<T_*>(out),
                  D, ld);
  };
  const int keep = (ld + 8 * kRowThreads - 1) / (8 * kRowThreads);
  if (f32) {
    float* type = nullptr;
    return keep <= 2 ? go(poly_norm_kernel<float, 2>, type) : go(poly_norm_kernel<float, 6>, type);
  }
  __nv_bfloat16* type = nullptr;
  return keep <= 4 ? go(poly_norm_kernel<__nv_bfloat16, 4>, type) : keep <= 7 ? go(poly_norm_kernel<__nv_bfloat16, 7>, type)
                                                                               : go(poly_norm_kernel<__nv_bfloat16, 12>, type);
}

// Widest row the decode step takes.
extern "C" int rmlx_sandwich_step_max_width() { return 44 * 1024 / 4; }      // five fp32 rows of shared memory

// x fp32 [B, ldx] += LN(y; wy) (y null: nothing), h = LN(x; wh), with conv (fp32 [taps, ldx]) h + its convolution. y and h
// [B, ldx] fp32 (f32) or bf16, y's rows ldy apart or (row_of_pair) expert rows with weights [B, top_k]; carried and slots [B] as in rmlx_short_conv.
extern "C" int rmlx_sandwich_step(float* x, const void* y, int ldy, const int* row_of_pair, const float* weights,
                                  int top_k, const float* wy, const float* wh, void* h, int f32, const float* conv, int taps,
                                  float* carried, long long stride, const int* slots, float eps, int B, int D, int ldx, int pdl,
                                  cudaStream_t st) {
  if (B < 1 || D < 1 || ldx < D || ldx % 8 || ldx > rmlx_sandwich_step_max_width() || !x || !wh || !h || h == x ||
      (y && (!wy || ldy % 8 || ldy < ldx)) || (row_of_pair && (!y || !weights || top_k < 1)) ||
      (conv && (taps < 1 || (taps > 1 && (!carried || !slots || stride % 4)))))
    return -2;
  auto run = [&](auto src, auto* out) -> int {
    using SRC = decltype(src);
    using T = std::remove_pointer_t<decltype(out)>;
    return launch_step(SandwichStep<SRC, T>{src, y != nullptr, x, Affine{wy, ldx}, Affine{wh, ldx}, out, conv, taps, carried, stride,
                                            slots, eps, D, ldx}, B, pdl, st);
  };
  auto from = [&](auto* rows, auto* out) -> int {
    using TY = std::remove_const_t<std::remove_pointer_t<decltype(rows)>>;
    if (row_of_pair) return run(ExpertSource<TY>{rows, ldy, row_of_pair, weights, nullptr, top_k}, out);
    return run(RowSource<TY>{rows, ldy}, out);
  };
  return f32 ? from(static_cast<const float*>(y), static_cast<float*>(h))
             : from(static_cast<const __nv_bfloat16*>(y), static_cast<__nv_bfloat16*>(h));
}
