// Row kernels of decoders with a layer norm before and after each sublayer, x <- x + norm_b(f(conv(norm(x)))), x in fp32:
//
//   sandwich_norm  x += LN(y) (y: a sublayer's rows, or the weighted rows of a token's experts) and h = LN(x) for the
//                  sublayer that follows, in one pass
//   short_conv     h + causal depthwise convolution of h over time, the last inputs carried per sequence
//   poly_norm      a N(z) + b N(z^2) + c N(z^3) + e, N: division by the row's root mean square
//   sandwich_step  a decode row through all of the first two: a cluster per row
//
// LN(v) = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w + b. Activations are bf16 (serving) or fp32 (the all-32-bit
// mode); norms, convolutions and the residual are fp32 in both.
#include <cooperative_groups.h>
#include <type_traits>

#include "../common/launch.cuh"
#include "../common/row_sources.cuh"
#include "../common/rows.cuh"

namespace cg = cooperative_groups;

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

// x[t] += LN(source; wy); h[t] = LN(x[t]; wh) (h may be null). Columns past D are zero. KEEP chunks of eight a thread keeps;
// rows wider than KEEP * 8 * 256 are read again.
template <class SRC, bool ADD, class T, int KEEP>
__global__ void __launch_bounds__(kRowThreads)
sandwich_norm_kernel(SRC src, Affine wy, float* __restrict__ x, Affine wh, T* __restrict__ h, float eps, int D, int ldx) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, chunks = ldx >> 3;
  float* row = x + size_t(t) * ldx;
  if constexpr (ADD) src.prepare(t);
  const float none[8] = {};
  float f[KEEP][8];
  // mean and 1 / deviation of the values that get(c, .) gives; keep[] holds the first ones
  auto moments = [&](float (&keep)[KEEP][8], auto get, float& mean, float& inv) {
    float sum = 0.f;
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
      const int c = u * kRowThreads + threadIdx.x;
      if (c < chunks) {
#pragma unroll
        for (int i = 0; i < 8; ++i) sum += c * 8 + i < D ? keep[u][i] : 0.f;
      }
    }
    for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
      float a[8];
      get(c, a);
#pragma unroll
      for (int i = 0; i < 8; ++i) sum += c * 8 + i < D ? a[i] : 0.f;
    }
    mean = row_block_sum(sum, red) / float(D);
    float ssq = 0.f;
    auto dev = [&](int c, const float (&a)[8]) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float d = a[i] - mean;
        ssq += c * 8 + i < D ? d * d : 0.f;
      }
    };
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
      const int c = u * kRowThreads + threadIdx.x;
      if (c < chunks) dev(c, keep[u]);
    }
    for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
      float a[8];
      get(c, a);
      dev(c, a);
    }
    inv = 1.f / sqrtf(row_block_sum(ssq, red) / float(D) + eps);
  };
  auto scaled = [&](const Affine& w, int c, const float (&a)[8], float mean, float inv, float (&o)[8]) {
    float g[8], b[8];
    w.load(c, g, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = c * 8 + i < D ? fmaf((a[i] - mean) * inv, g[i], b[i]) : 0.f;
  };
  float mean, inv;
  if constexpr (ADD) {
    float y[KEEP][8];
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
      const int c = u * kRowThreads + threadIdx.x;
      if (c < chunks) {
        src.load(t, c, none, y[u]);
        load8(row + c * 8, f[u]);
      }
    }
    moments(y, [&](int c, float (&a)[8]) { src.load(t, c, none, a); }, mean, inv);
    auto add = [&](int c, const float (&a)[8], float (&v)[8]) {
      float o[8];
      scaled(wy, c, a, mean, inv, o);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] += o[i];
      store8(row + c * 8, v);
    };
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
      const int c = u * kRowThreads + threadIdx.x;
      if (c < chunks) add(c, y[u], f[u]);
    }
    for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
      float a[8], v[8];
      src.load(t, c, none, a);
      load8(row + c * 8, v);
      add(c, a, v);
    }
  } else {
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
      const int c = u * kRowThreads + threadIdx.x;
      if (c < chunks) load8(row + c * 8, f[u]);
    }
  }
  if (!h) return;
  moments(f, [&](int c, float (&a)[8]) { load8(row + c * 8, a); }, mean, inv);   // (this thread wrote them)
  T* dst = h + size_t(t) * ldx;
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) {
      float o[8];
      scaled(wh, c, f[u], mean, inv, o);
      store8(dst + c * 8, o);
    }
  }
  for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float a[8], o[8];
    load8(row + c * 8, a);
    scaled(wh, c, a, mean, inv, o);
    store8(dst + c * 8, o);
  }
}

// out[t] = h[t] + sum_j w[j] h[t - taps + 1 + j] within a sequence. A thread owns eight columns. Blocks y < strips: kStrip
// rows each, of which those with all their inputs in the batch are done; the others: one run of rows each, its first
// taps - 1 rows with the help of the carried inputs, which it then replaces by the run's last ones. So a sequence's carried
// inputs are read and written by one thread alone.
constexpr int kConvStrip = 8;
template <class T, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_kernel(const T* __restrict__ h, T* __restrict__ out, int ldx, const float* __restrict__ w, int n_taps,
                  float* __restrict__ carried, long long stride, const int4* __restrict__ runs, const int* __restrict__ slots,
                  int T_rows, int strips) {
  pdl_launch_dependents();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : n_taps, keep = taps - 1;
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= ldx) return;
  auto put = [&](int t, const float (&a)[8]) { store8(out + size_t(t) * ldx + c, a); };
  if (int(blockIdx.y) < strips) {
    const int t0 = blockIdx.y * kConvStrip, n = min(kConvStrip, T_rows - t0);
    if constexpr (TAPS > 0) {
      float v[kConvStrip + TAPS - 1][8], g[TAPS][8];
#pragma unroll
      for (int i = 0; i < kConvStrip + TAPS - 1; ++i) {
        const int t = t0 + i - (TAPS - 1);
        if (t >= 0 && t < T_rows) load8(h + size_t(t) * ldx + c, v[i]);
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j) load8(w + size_t(j) * ldx + c, g[j]);
#pragma unroll
      for (int i = 0; i < kConvStrip; ++i) {
        const int t = t0 + i;
        if (i >= n || t < keep || (keep > 0 && slots[t - keep] != slots[t])) continue;
        float a[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          float s = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) s = fmaf(g[j][e], v[i + j][e], s);
          a[e] = v[i + TAPS - 1][e] + s;
        }
        put(t, a);
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
  float f[KEEP][8], s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto take = [&](int c, float (&a)[8]) {
    load8(row + c * 8, a);
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
    if (c < chunks) take(c, f[u]);
  }
  for (int c = KEEP * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float a[8];
    take(c, a);
  }
  s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = s2; red[1][threadIdx.x >> 5] = s4; red[2][threadIdx.x >> 5] = s6; }
  __syncthreads();
  float k[3];
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const float v = (threadIdx.x & 31) < kRowThreads / 32 ? red[i][threadIdx.x & 31] : 0.f;
    k[i] = act[i] / sqrtf(warp_sum(v) / float(D) + eps);
  }
  const float e = act[3];
  auto put = [&](int c, const float (&a)[8]) {
    float o[8];
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
    float a[8];
    load8(row + c * 8, a);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] = c * 8 + i < D ? a[i] : 0.f;
    put(c, a);
  }
}

// ------------------------------------------------------------------ decode
constexpr int kStepThreads = 128, kStepCols = kStepThreads * 4;

struct SandwichStep {
  float* x;                 // [B, ldx]
  const float* y;           // [B, ldx] finished sublayer, or null
  const float* wy;          // [2, ldx]
  const float* wh;          // [2, ldx]
  float* h;                 // [B, ldx]
  const float* conv;        // [taps, ldx], or null: no convolution
  int taps;
  float* carried;           // slot s: carried + s * stride, [taps - 1, ldx]
  long long stride;
  const int* slots;
  float eps;
  int D, ldx;
};

// A count, a mean and a sum of squared deviations, joined without cancellation.
struct Moments {
  float n, mean, m2;
};
__device__ __forceinline__ Moments join(const Moments& a, const Moments& b) {
  const float n = a.n + b.n;
  if (n == 0.f) return a;
  const float d = b.mean - a.mean, f = b.n / n;
  return Moments{n, fmaf(d, f, a.mean), a.m2 + b.m2 + d * d * a.n * f};
}

// grid (column blocks = one cluster, rows). E float4 pieces a thread holds.
template <int E>
__global__ void __launch_bounds__(kStepThreads)
sandwich_step_kernel(SandwichStep p) {
  __shared__ Moments warp_part[kStepThreads / 32];
  __shared__ Moments part[2];
  const int b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int col0 = (blockIdx.x * kStepThreads + tid) * 4, step = gridDim.x * kStepCols;
  auto ld = [](const float* q) { return __ldcg(reinterpret_cast<const float4*>(q)); };
  auto at = [&](int e) { return col0 + e * step; };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // what no kernel of this step writes before: norm weights, and the convolution's share of the carried inputs
  float4 gy[E], by[E], gh[E], bh[E], past[E], now[E];
  float* st = p.conv && p.taps > 1 ? p.carried + size_t(p.slots[b]) * p.stride : nullptr;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    gy[e] = by[e] = gh[e] = bh[e] = past[e] = now[e] = zero;
    if (at(e) >= p.ldx) continue;
    if (p.y) { gy[e] = ld(p.wy + at(e)); by[e] = ld(p.wy + p.ldx + at(e)); }
    gh[e] = ld(p.wh + at(e));
    bh[e] = ld(p.wh + p.ldx + at(e));
    if (p.conv) {
      now[e] = ld(p.conv + size_t(p.taps - 1) * p.ldx + at(e));
      for (int j = 0; j < p.taps - 1; ++j) {
        const float4 w = ld(p.conv + size_t(j) * p.ldx + at(e)), v = ld(st + size_t(j) * p.ldx + at(e));
        past[e].x = fmaf(w.x, v.x, past[e].x); past[e].y = fmaf(w.y, v.y, past[e].y);
        past[e].z = fmaf(w.z, v.z, past[e].z); past[e].w = fmaf(w.w, v.w, past[e].w);
      }
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  float4 x[E], y[E];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const bool in = at(e) < p.ldx;
    x[e] = in ? ld(p.x + size_t(b) * p.ldx + at(e)) : zero;
    y[e] = in && p.y ? ld(p.y + size_t(b) * p.ldx + at(e)) : zero;
  }
  cg::cluster_group cluster = cg::this_cluster();
  // mean and 1 / deviation over the row
  auto moments = [&](const float4 (&v)[E], Moments* mine, float& mean, float& inv) {
    Moments m{0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int n = max(0, min(4, p.D - at(e)));
      const float f[4] = {v[e].x, v[e].y, v[e].z, v[e].w};
      float s = 0.f, q = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) s += i < n ? f[i] : 0.f;
      const float mu = n > 0 ? s / float(n) : 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) q += i < n ? (f[i] - mu) * (f[i] - mu) : 0.f;
      m = join(m, Moments{float(n), mu, q});
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
      m = join(m, Moments{__shfl_xor_sync(0xffffffffu, m.n, o), __shfl_xor_sync(0xffffffffu, m.mean, o),
                          __shfl_xor_sync(0xffffffffu, m.m2, o)});
    if (lane == 0) warp_part[warp] = m;
    __syncthreads();
    m = warp_part[0];
#pragma unroll
    for (int q = 1; q < kStepThreads / 32; ++q) m = join(m, warp_part[q]);
    if (gridDim.x > 1) {
      if (tid == 0) *mine = m;
      cluster.sync();
      m = *cluster.map_shared_rank(mine, 0);
      for (unsigned r = 1; r < gridDim.x; ++r) m = join(m, *cluster.map_shared_rank(mine, r));
    } else {
      __syncthreads();                                 // warp_part is written again
    }
    mean = m.mean;
    inv = 1.f / sqrtf(m.m2 / float(p.D) + p.eps);
  };
  auto norm4 = [&](int e, const float4& v, float mean, float inv, const float4& g, const float4& o) {
    const int n = p.D - at(e);
    return make_float4(n > 0 ? fmaf((v.x - mean) * inv, g.x, o.x) : 0.f, n > 1 ? fmaf((v.y - mean) * inv, g.y, o.y) : 0.f,
                       n > 2 ? fmaf((v.z - mean) * inv, g.z, o.z) : 0.f, n > 3 ? fmaf((v.w - mean) * inv, g.w, o.w) : 0.f);
  };
  float mean, inv;
  if (p.y) {
    moments(y, part, mean, inv);
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const float4 a = norm4(e, y[e], mean, inv, gy[e], by[e]);
      x[e].x += a.x; x[e].y += a.y; x[e].z += a.z; x[e].w += a.w;
      if (at(e) < p.ldx) *reinterpret_cast<float4*>(p.x + size_t(b) * p.ldx + at(e)) = x[e];
    }
  }
  moments(x, part + 1, mean, inv);
#pragma unroll
  for (int e = 0; e < E; ++e) {
    if (at(e) >= p.ldx) continue;
    const float4 a = norm4(e, x[e], mean, inv, gh[e], bh[e]);
    float4 o = a;
    if (p.conv) {
      o.x += fmaf(now[e].x, a.x, past[e].x); o.y += fmaf(now[e].y, a.y, past[e].y);
      o.z += fmaf(now[e].z, a.z, past[e].z); o.w += fmaf(now[e].w, a.w, past[e].w);
      float* q = st + at(e);
      for (int j = 0; j + 2 < p.taps; ++j) *reinterpret_cast<float4*>(q + size_t(j) * p.ldx) = ld(q + size_t(j + 1) * p.ldx);
      if (p.taps > 1) *reinterpret_cast<float4*>(q + size_t(p.taps - 2) * p.ldx) = a;
    }
    *reinterpret_cast<float4*>(p.h + size_t(b) * p.ldx + at(e)) = o;
  }
  if (gridDim.x > 1) cluster.sync();                   // nobody leaves while a neighbour still reads its shared memory
}

template <class SRC, bool ADD>
static int launch_sandwich(SRC src, const float* wy, float* x, const float* wh, void* h, float eps, int T, int D, int ldx, int f32,
                           int pdl, cudaStream_t st) {
  const Affine ay{wy, ldx}, ah{wh, ldx};
  auto go = [&](auto kern, auto* out) -> int {
    return launch(kern, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, src, ay, x, ah, out, eps, D, ldx);
  };
  const bool narrow = ldx <= 2 * 8 * kRowThreads;
  if (f32) {
    float* out = static_cast<float*>(h);
    return narrow ? go(sandwich_norm_kernel<SRC, ADD, float, 2>, out) : go(sandwich_norm_kernel<SRC, ADD, float, 4>, out);
  }
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(h);
  return narrow ? go(sandwich_norm_kernel<SRC, ADD, __nv_bfloat16, 2>, out)
                : go(sandwich_norm_kernel<SRC, ADD, __nv_bfloat16, 4>, out);
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
  if (!y) return launch_sandwich<RowSource<float>, false>(RowSource<float>{nullptr, 0}, nullptr, x, wh, h, eps, T, D, ldx, f32, pdl, st);
  if (ldy % 8 || ldy < ldx || !wy || (row_of_pair && (!weights || top_k < 1))) return -2;
  auto run = [&](auto* p) -> int {
    using TY = std::remove_const_t<std::remove_pointer_t<decltype(p)>>;
    if (row_of_pair)
      return launch_sandwich<ExpertSource<TY>, true>(ExpertSource<TY>{p, ldy, row_of_pair, weights, nullptr, top_k}, wy, x, wh, h,
                                                     eps, T, D, ldx, f32, pdl, st);
    return launch_sandwich<RowSource<TY>, true>(RowSource<TY>{p, ldy}, wy, x, wh, h, eps, T, D, ldx, f32, pdl, st);
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
  const int strips = runs || taps == 1 ? (T + kConvStrip - 1) / kConvStrip : 0, tails = taps > 1 ? n_runs : 0;
  if (strips + tails > 65535) return -2;
  const dim3 grid((ldx / 8 + 127) / 128, strips + tails);
  auto go = [&](auto* type) -> int {
    using T_ = std::remove_pointer_t<decltype(type)>;
    auto kern = taps == 4 ? short_conv_kernel<T_, 4> : taps == 3 ? short_conv_kernel<T_, 3>
                : taps == 2 ? short_conv_kernel<T_, 2> : short_conv_kernel<T_, 0>;
    return launch(kern, grid, dim3(128), 0, st, pdl != 0, static_cast<const T_*>(h), static_cast<T_*>(out), ldx, w, taps, carried,
                  stride, reinterpret_cast<const int4*>(runs), slots, T, strips);
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
  const bool narrow = ld <= 2 * 8 * kRowThreads;
  if (f32)
    return narrow ? go(poly_norm_kernel<float, 2>, static_cast<float*>(nullptr)) : go(poly_norm_kernel<float, 8>, static_cast<float*>(nullptr));
  return narrow ? go(poly_norm_kernel<__nv_bfloat16, 2>, static_cast<__nv_bfloat16*>(nullptr))
                : go(poly_norm_kernel<__nv_bfloat16, 8>, static_cast<__nv_bfloat16*>(nullptr));
}

// Widest row the decode step takes.
extern "C" int rmlx_sandwich_step_max_width() { return 8 * kStepCols * 4; }

// x += LN(y; wy) (y null: nothing), h = LN(x; wh), with conv (fp32 [taps, ldx]) h + its convolution; everything fp32 [B, ldx],
// carried and slots [B] as in rmlx_short_conv.
extern "C" int rmlx_sandwich_step(float* x, const float* y, const float* wy, const float* wh, float* h, const float* conv, int taps,
                                  float* carried, long long stride, const int* slots, float eps, int B, int D, int ldx, int pdl,
                                  cudaStream_t st) {
  if (B < 1 || B > 65535 || D < 1 || ldx < D || ldx % 8 || ldx > rmlx_sandwich_step_max_width() || !x || !wh || !h || h == x ||
      (y && !wy) || (conv && (taps < 1 || (taps > 1 && (!carried || !slots || stride % 4)))))
    return -2;
  int blocks = 1;
  while (blocks < 8 && blocks * kStepCols < ldx) blocks *= 2;
  const int pieces = (ldx + blocks * kStepCols - 1) / (blocks * kStepCols);
  const SandwichStep p{x, y, wy, wh, h, conv, taps, carried, stride, slots, eps, D, ldx};
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(blocks, B);
  cfg.blockDim = dim3(kStepThreads);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int n = 0;
  attr[n].id = cudaLaunchAttributeClusterDimension;
  attr[n].val.clusterDim.x = blocks; attr[n].val.clusterDim.y = 1; attr[n].val.clusterDim.z = 1;
  ++n;
  auto kern = pieces <= 1 ? sandwich_step_kernel<1> : pieces <= 2 ? sandwich_step_kernel<2> : sandwich_step_kernel<4>;
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
