// Linear recurrences beside attention, on common/scan.cuh (token by token, fp32 state):
//
//   gla   gated linear attention: a decay per key channel, alpha = sigmoid(z + bias)^(1 / tau);
//         S <- diag(alpha) S + k v^T, o = S^T (q scale)
//   ssd   state-space heads: x, B and C through a causal depthwise convolution and silu, dt = softplus(.),
//         S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; `H / G` heads share a group's B and C
//   lightning  one constant decay per head; q, k and v through silu; S <- decay S + k v^T, o = S^T q
//
// and what surrounds them: the convolution's carried inputs, and the norm of the outputs over equal groups of
// columns with a silu or sigmoid gate before or after it. Decays, step sizes and their exponentials are fp32.
#include "../common/launch.cuh"
#include "../common/rows.cuh"
#include "../common/scan.cuh"
#include <type_traits>

namespace rb {

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <class T>
struct GlaIn {
  const T* q; const T* k; const T* v;
  int ld;
  const float* z;
  int ld_z;
  const float* bias;
  float inv_tau, scale;
  int dim, vdim;
  __device__ __forceinline__ void rows4(int t, int h, int i, float (&fr)[4], float (&fk)[4], float (&fw)[4], float (&fb)[4]) const {
    const bool vec = dim % 4 == 0 && ld % 4 == 0;
    const size_t at = size_t(t) * ld + h * dim;
    const float* zp = z + size_t(t) * ld_z + h * dim;
    scan_load4(q + at, i, dim, vec, fb);
    scan_load4(k + at, i, dim, vec, fk);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const bool in = i + j < dim;
      const int c = in ? i + j : 0;
      fw[j] = in ? expf(-softplus_f(-(zp[c] + bias[h * dim + c])) * inv_tau) : 1.f;
      fb[j] *= scale;
      fr[j] = fb[j] * fw[j];
    }
  }
  __device__ __forceinline__ void cols4(int t, int h, int i, float (&fv)[4]) const {
    scan_load4(v + size_t(t) * ld + h * vdim, i, vdim, vdim % 4 == 0 && ld % 4 == 0, fv);
  }
};

// What a state-space layer reads: rows [.. | x: H*d | B: G*n | C: G*n at x_at | .. | dt: H at dt_at | ..].
template <class T>
struct SsdIn {
  const T* raw;
  int ld, x_at, dt_at;
  const float* conv_w;      // [taps, channels], the last row is the current token's
  const float* conv_b;      // [channels]
  int taps;
  const float* before;      // slot s: before + s * stride, [taps - 1, channels]: inputs carried over, newest last
  long long stride;
  const int* slots;         // [rows]
  int each_row;             // no two rows share a sequence
  const float* dt_bias; const float* a_log; const float* skip;      // [H]
  int H, G, n, d;
  __host__ __device__ __forceinline__ int channels() const { return H * d + 2 * G * n; }
};

// Two consecutive inputs, 4- or 8-byte aligned.
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf16lo(v), bf16hi(v));
}

// All channels' convolutions and the step sizes of a block's TOKENS tokens into shared memory, then the records. Where the
// block and the taps before it lie in one sequence, a thread asks for a pair of channels' inputs of all tokens at once
// (TAPS 0, or elsewhere: one by one).
template <class T, int ROWS, int LANES, int TAPS, int TOKENS>
__global__ void __launch_bounds__(kRowThreads)
ssd_prepare_kernel(SsdIn<T> in, float* __restrict__ rec, float* __restrict__ col, int rows, int shift) {
  constexpr int kRows = ROWS * LANES, tokens = TOKENS;
  extern __shared__ __align__(16) float sm[];
  const int t0 = blockIdx.x * tokens, nt = min(tokens, rows - t0), inner = in.H * in.d, gn = in.G * in.n, ch = inner + 2 * gn;
  const int taps = in.taps;
  float* s_own = sm + tokens * ch;         // [tokens, G] C . B
  float* s_dt = s_own + tokens * in.G;     // [tokens, H]
  float* s_a = s_dt + tokens * in.H;       // [tokens, H]
  pdl_launch_dependents();
  pdl_wait();
  const bool inside = TAPS > 0 && !in.each_row && nt == tokens && t0 >= TAPS - 1 &&
                      in.slots[t0 - (TAPS > 0 ? TAPS - 1 : 0)] == in.slots[t0 + tokens - 1] && ((ch | in.ld | in.x_at) & 1) == 0;
  if (inside) {
    constexpr int W = TAPS > 0 ? TAPS : 1;
    const T* base = in.raw + size_t(t0 - (W - 1)) * in.ld + in.x_at;
    for (int c = threadIdx.x * 2; c < ch; c += kRowThreads * 2) {
      float2 x[tokens + W - 1], w[W];
#pragma unroll
      for (int i = 0; i < tokens + W - 1; ++i) x[i] = load2(base + size_t(i) * in.ld + c);
#pragma unroll
      for (int j = 0; j < W; ++j) w[j] = load2(in.conv_w + size_t(j) * ch + c);
      const float2 bias = load2(in.conv_b + c);
#pragma unroll
      for (int i = 0; i < tokens; ++i) {
        float2 a = bias;
#pragma unroll
        for (int j = 0; j < W; ++j) { a.x = fmaf(w[j].x, x[i + j].x, a.x); a.y = fmaf(w[j].y, x[i + j].y, a.y); }
        *reinterpret_cast<float2*>(sm + i * ch + c) = make_float2(silu_f(a.x), silu_f(a.y));
      }
    }
  } else {
    for (int i = 0; i < nt; ++i) {
      const int t = t0 + i;
      int back = 0;                        // how many of the rows before t are its sequence's (at most taps - 1)
      if (!in.each_row)
        while (back < taps - 1 && t - back - 1 >= 0 && in.slots[t - back - 1] == in.slots[t]) ++back;
      const float* before = in.before + size_t(in.slots[t]) * in.stride;
      for (int c = threadIdx.x; c < ch; c += kRowThreads) {
        float a = in.conv_b[c];
        for (int j = taps - 1; j >= 0; --j) {              // j tokens back
          const float x = j <= back ? to_f32(in.raw[size_t(t - j) * in.ld + in.x_at + c]) : before[size_t(taps - 1 - (j - back)) * ch + c];
          a = fmaf(in.conv_w[size_t(taps - 1 - j) * ch + c], x, a);
        }
        sm[i * ch + c] = silu_f(a);
      }
    }
  }
  for (int u = threadIdx.x; u < nt * in.H; u += kRowThreads) {
    const int i = u / in.H, h = u - i * in.H;
    const float dt = softplus_f(to_f32(in.raw[size_t(t0 + i) * in.ld + in.dt_at + h]) + in.dt_bias[h]);
    s_dt[u] = dt;
    s_a[u] = expf(-expf(in.a_log[h]) * dt);
  }
  __syncthreads();
  for (int u = threadIdx.x >> 5; u < nt * in.G; u += kRowThreads / 32) {
    const int i = u / in.G, g = u - i * in.G;
    const float* B = sm + i * ch + inner + g * in.n;
    float s = 0.f;
    for (int j = threadIdx.x & 31; j < in.n; j += 32) s = fmaf(B[j], B[gn + j], s);
    s = warp_sum(s);
    if ((threadIdx.x & 31) == 0) s_own[u] = s;
  }
  for (int u = threadIdx.x; u < nt * in.G * kRows; u += kRowThreads) {
    const int q = u / kRows, j = u - q * kRows, i = q / in.G, g = q - i * in.G;
    const float* B = sm + i * ch + inner + g * in.n;
    float* o = rec + (size_t(g) * rows + t0 + i) * (2 * kRows) + scan_at<ROWS, LANES>(j);
    o[0] = j < in.n ? B[gn + j] : 0.f;
    o[kRows] = j < in.n ? B[j] : 0.f;
  }
  __syncthreads();
  // column records of a block's tokens are neighbours: four values a thread, tokens before column blocks
  const int cols = 1 << shift, nb = (in.d + cols - 1) >> shift, per = in.H / in.G, quads = (cols + 4) >> 2;
  for (int u = threadIdx.x; u < in.H * nb * tokens * quads; u += kRowThreads) {
    const int v = u / quads, q = u - v * quads, i = v % tokens, hb = v / tokens, h = nb == 1 ? hb : hb / nb;
    const int c0 = ((hb - h * nb) << shift) + q * 4;
    if (i >= nt) continue;
    float4 f;
    if (q == quads - 1) {
      const float dt = s_dt[i * in.H + h];
      f = make_float4(s_a[i * in.H + h], dt, fmaf(s_own[i * in.G + h / per], dt, in.skip[h]), 0.f);
    } else {
      const float* x = sm + i * ch + h * in.d + c0;
      f = make_float4(c0 < in.d ? x[0] : 0.f, c0 + 1 < in.d ? x[1] : 0.f, c0 + 2 < in.d ? x[2] : 0.f, c0 + 3 < in.d ? x[3] : 0.f);
    }
    *reinterpret_cast<float4*>(col + (size_t(hb) * rows + t0 + i) * (cols + 4) + q * 4) = f;
  }
}

template <class T>
struct LightIn {
  const T* q; const T* k; const T* v;
  int ld;
  const float* decay;       // [H]
  int dim, vdim;
};
// Records of heads with a constant decay, LU lanes per (token, head).
template <class T, int ROWS, int LANES, int LU>
__global__ void __launch_bounds__(kRowThreads)
lightning_prepare_kernel(LightIn<T> in, float* __restrict__ rec, float* __restrict__ col, int rows, int H, int shift) {
  constexpr int kRows = ROWS * LANES;
  pdl_launch_dependents();
  pdl_wait();
  const int unit = (blockIdx.x * kRowThreads + threadIdx.x) / LU, lane = threadIdx.x % LU;
  const bool live = unit < rows * H;                 // the lanes of a warp stay together for the sum
  const int t = live ? unit / H : 0, h = live ? unit - t * H : 0;
  const bool vec = in.dim % 4 == 0 && in.ld % 4 == 0, vec_v = in.vdim % 4 == 0 && in.ld % 4 == 0;
  const size_t row = size_t(t) * in.ld;
  float* out = rec + (size_t(h) * rows + t) * 2 * kRows;
  float own = 0.f;
  for (int i = lane * 4; i < kRows; i += LU * 4) {
    float r[4], k[4];
    scan_load4(in.q + row + h * in.dim, i, in.dim, vec, r);
    scan_load4(in.k + row + h * in.dim, i, in.dim, vec, k);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      r[j] = silu_f(r[j]);
      k[j] = silu_f(k[j]);
      own = fmaf(r[j], k[j], own);
    }
    if (live) {
      float* o = out + scan_at<ROWS, LANES>(i);
      *reinterpret_cast<float4*>(o) = make_float4(r[0], r[1], r[2], r[3]);
      *reinterpret_cast<float4*>(o + kRows) = make_float4(k[0], k[1], k[2], k[3]);
    }
  }
  own = group_sum<LU>(own);
  if (!live) return;
  const int cols = 1 << shift, nb = (in.vdim + cols - 1) >> shift;
  for (int i = lane * 4; i < nb << shift; i += LU * 4) {
    float v[4];
    scan_load4(in.v + row + h * in.vdim, i, in.vdim, vec_v, v);
    const int at = i & (cols - 1);
    float* o = col + ((size_t(h) * nb + (i >> shift)) * rows + t) * (cols + 4) + at;
    *reinterpret_cast<float4*>(o) = make_float4(silu_f(v[0]), silu_f(v[1]), silu_f(v[2]), silu_f(v[3]));
    if (at == 0) *reinterpret_cast<float4*>(o + cols) = make_float4(in.decay[h], 1.f, own, 0.f);
  }
}

// The last taps - 1 inputs of every segment's sequence become its carried ones. A thread owns a channel; it
// writes in ascending order and reads ahead of what it writes.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
conv_carry_kernel(const T* __restrict__ raw, int ld, int x_at, float* __restrict__ carried, long long stride,
                  const int4* __restrict__ segs, const int* __restrict__ slots, int ch, int keep) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * kRowThreads + threadIdx.x;
  if (c >= ch) return;
  int row0 = blockIdx.y, len = 1, slot;
  if (segs) {
    const int4 s = segs[blockIdx.y];
    row0 = s.x; len = s.y; slot = s.z;
  } else {
    slot = slots[blockIdx.y];
  }
  float* st = carried + size_t(slot) * stride + c;
  for (int m = 0; m < keep; ++m) {
    const int i = len - keep + m;
    st[size_t(m) * ch] = i >= 0 ? to_f32(raw[size_t(row0 + i) * ld + x_at + c]) : st[size_t(m + len) * ch];
  }
}

// silu (or sigmoid) of an output gate; with the hardware exponential and division where the result is rounded to bf16.
template <class T>
__device__ __forceinline__ float gate_value(float z, bool sigmoid) {
  const float n = sigmoid ? 1.f : z;
  return sizeof(T) == 2 ? __fdividef(n, 1.f + __expf(fminf(-z, 80.f))) : n / (1.f + expf(-z));
}

// out[t, c] over equal groups of columns, g: silu or sigmoid: FIRST: f = o g(gate), f / rms(f over the group) * w;
// else o / rms(o over the group) * w * g(gate). L lanes (256: a block) per (row, group), KEEP chunks of eight a lane
// keeps; what is left is read again. VEC: sizes and strides are multiples of eight.
template <class T, int L, int KEEP, bool FIRST, bool VEC>
__global__ void __launch_bounds__(kRowThreads)
gated_norm_kernel(const float* __restrict__ o, int ld_o, const T* __restrict__ gate, int ld_g, const float* __restrict__ w,
                  float eps, T* __restrict__ out, int ld_out, int rows, int groups, int size, bool sigmoid) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int unit = (blockIdx.x * kRowThreads + threadIdx.x) / L, lane = threadIdx.x % L;
  const bool live = unit < rows * groups;              // the lanes of a warp stay together for the sums
  const int t = live ? unit / groups : 0, at = live ? (unit - t * groups) * size : 0;
  const float* op = o + size_t(t) * ld_o + at;
  const T* gp = gate + size_t(t) * ld_g + at;
  float f[KEEP][8], g[KEEP][8], ssq = 0.f;
  auto load = [&](int i0, float (&a)[8]) {
    load8_upto(op + i0, size - i0, VEC, a);
    if (FIRST) {
      float z[8];
      load8_upto(gp + i0, size - i0, VEC, z);
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] *= gate_value<T>(z[i], sigmoid);
    }
  };
  auto factor = [&](int i0, float (&a)[8]) {           // what the normed values are multiplied by
    load8_upto(w + at + i0, size - i0, VEC, a);
    if (!FIRST) {
      float z[8];
      load8_upto(gp + i0, size - i0, VEC, z);
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] *= gate_value<T>(z[i], sigmoid);
    }
  };
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int i0 = (u * L + lane) * 8;
    if (i0 < size) {
      load(i0, f[u]);
      factor(i0, g[u]);
#pragma unroll
      for (int i = 0; i < 8; ++i) ssq += f[u][i] * f[u][i];
    }
  }
  for (int i0 = (KEEP * L + lane) * 8; i0 < size; i0 += L * 8) {
    float a[8];
    load(i0, a);
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += a[i] * a[i];
  }
  if (L <= 32) ssq = group_sum<L <= 32 ? L : 32>(ssq);
  else ssq = row_block_sum(ssq, red);
  if (!live) return;
  const float inv = 1.f / sqrtf(ssq / float(size) + eps);
  T* dst = out + size_t(t) * ld_out + at;
  auto put = [&](int i0, float (&a)[8], const float (&m)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] *= inv * m[i];
    if (VEC) {
      store8(dst + i0, a);
    } else {
      for (int i = 0; i < 8 && i0 + i < size; ++i) dst[i0 + i] = from_f32<T>(a[i]);
    }
  };
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int i0 = (u * L + lane) * 8;
    if (i0 < size) put(i0, f[u], g[u]);
  }
  for (int i0 = (KEEP * L + lane) * 8; i0 < size; i0 += L * 8) {
    float a[8], m[8];
    load(i0, a);
    factor(i0, m);
    put(i0, a, m);
  }
}

template <class T>
static int run_gla(const GlaIn<T>& in, const ScanParams& p, float* rec, int n, int pdl, cudaStream_t st) {
#define RB_GLA(R_, L_) return launch_row_scan<GlaIn<T>, R_, L_>(in, p, rec, n, pdl, st)
  RB_SCAN_DISPATCH(p.n, RB_GLA);
#undef RB_GLA
  return -2;
}

template <class T, int ROWS, int LANES>
static int launch_ssd(const SsdIn<T>& in, ScanParams p, float* rec, int n_segs, int pdl, cudaStream_t st) {
  const size_t per_token = size_t(in.channels() + in.G + 2 * in.H) * sizeof(float);
  if (per_token > 200 * 1024) return -2;
  const int th = scan_threads(LANES, p.d, p.H, n_segs);
  float* col = rec + size_t(in.G) * p.rows * 2 * ROWS * LANES;
  auto prepare = [&](auto kern, int tokens) -> int {
    const size_t smem = per_token * tokens;
    RB_CHECK(set_max_smem(kern, smem));
    return launch(kern, dim3((p.rows + tokens - 1) / tokens), dim3(kRowThreads), smem, st, pdl != 0, in, rec, col, p.rows,
                  scan_col_shift(LANES, th));
  };
  const bool one = per_token * 4 > 200 * 1024;
  const int rc = one ? prepare(ssd_prepare_kernel<T, ROWS, LANES, 0, 1>, 1)
                     : in.taps == 4 ? prepare(ssd_prepare_kernel<T, ROWS, LANES, 4, 4>, 4)
                                    : prepare(ssd_prepare_kernel<T, ROWS, LANES, 0, 4>, 4);
  if (rc) return rc;
  p.rec = rec; p.col = col; p.per = in.H / in.G;
  return launch_scan<ROWS, LANES, true>(p, th, n_segs, pdl, st);
}
template <class T, int ROWS, int LANES>
static int launch_lightning(const LightIn<T>& in, ScanParams p, float* rec, int n_segs, int pdl, cudaStream_t st) {
  constexpr int kRows = ROWS * LANES, LU = kRows >= 128 ? 32 : kRows / 4;
  const long long threads = 1LL * p.rows * p.H * LU;
  if (threads > 0x7fffffffLL) return -2;
  const int th = scan_threads(LANES, p.d, p.H, n_segs);
  float* col = rec + size_t(p.H) * p.rows * 2 * kRows;
  const int rc = launch(lightning_prepare_kernel<T, ROWS, LANES, LU>, dim3(unsigned((threads + kRowThreads - 1) / kRowThreads)),
                        dim3(kRowThreads), 0, st, pdl != 0, in, rec, col, p.rows, p.H, scan_col_shift(LANES, th));
  if (rc) return rc;
  p.rec = rec; p.col = col; p.per = 1;
  return launch_scan<ROWS, LANES, true>(p, th, n_segs, pdl, st);
}
template <class T>
static int run_lightning(const LightIn<T>& in, const ScanParams& p, float* rec, int n, int pdl, cudaStream_t st) {
#define RB_LI(R_, L_) return launch_lightning<T, R_, L_>(in, p, rec, n, pdl, st)
  RB_SCAN_DISPATCH(p.n, RB_LI);
#undef RB_LI
  return -2;
}
template <class T>
static int run_ssd(const SsdIn<T>& in, const ScanParams& p, float* rec, int n, int pdl, cudaStream_t st) {
#define RB_SSD(R_, L_) return launch_ssd<T, R_, L_>(in, p, rec, n, pdl, st)
  RB_SCAN_DISPATCH(p.n, RB_SSD);
#undef RB_SSD
  return -2;
}

static bool scan_args_ok(int rows, const int* segs, const int* slots, int n_segs, const float* rec, int H, int n, int d) {
  return rows >= 1 && n_segs >= 1 && n_segs <= 65535 && H >= 1 && H <= 65535 && n >= 1 && n <= kScanMaxRows && d >= 1 &&
         (segs || slots) && !((reinterpret_cast<uintptr_t>(segs) | reinterpret_cast<uintptr_t>(rec)) & 15);
}

}  // namespace rb

using namespace rb;

extern "C" int rmlx_scan_max_rows() { return kScanMaxRows; }
// Floats of the scratch records of one (token, head); one != 0: heads with a single decay, `per` of which share
// their row record.
extern "C" long long rmlx_scan_record(int n, int d, int one, int per) {
  if (per < 1) return 0;
#define RB_REC(R_, L_) return scan_row_floats((R_) * (L_), L_, one ? 2 : 3, d, one ? per : 1)
  RB_SCAN_DISPATCH(n, RB_REC);
#undef RB_REC
  return 0;
}

// q, k [rows, ld] (H x dim), v (H x vdim) fp32 (f32) or bf16, 16-byte aligned; z fp32 [rows, ld_z], bias fp32
// [H * dim]; out fp32 [rows, ld_out] (H x vdim); state fp32, slot s at state + s * stride, [H, dim, vdim]; rec:
// scratch, rows * H records; segs int32 [n_segs, 4] = (first row, rows, slot, -), 16-byte aligned, or null with
// slots [n_segs]: then every row is a segment. No slot occurs twice except one that nobody reads.
extern "C" int rmlx_gla_scan(const void* q, const void* k, const void* v, int ld, const float* z, int ld_z, const float* bias,
                             float inv_tau, float scale, float* rec, int rows, const int* segs, const int* slots, int n_segs,
                             float* state, long long stride, float* out, int ld_out, int H, int dim, int vdim, int f32,
                             int* status, int pdl, cudaStream_t st) {
  if (!scan_args_ok(rows, segs, slots, n_segs, rec, H, dim, vdim) || ld < H * dim || ld < H * vdim || ld_z < H * dim ||
      ld_out < H * vdim ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15))
    return -2;
  ScanParams p{};
  p.rows = rows; p.segs = reinterpret_cast<const int4*>(segs); p.slots = slots;
  p.state = state; p.stride = stride; p.out = out; p.ld_out = ld_out;
  p.H = H; p.n = dim; p.d = vdim; p.status = status;
  auto run = [&](auto* type) {
    using T = std::remove_pointer_t<decltype(type)>;
    return run_gla<T>(GlaIn<T>{static_cast<const T*>(q), static_cast<const T*>(k), static_cast<const T*>(v), ld, z, ld_z, bias,
                               inv_tau, scale, dim, vdim}, p, rec, n_segs, pdl, st);
  };
  return f32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
}

// raw fp32 (f32) or bf16 [rows, ld] with x | B | C at column x_at and dt at dt_at; conv_w fp32 [taps, channels],
// conv_b [channels], dt_bias, a_log, skip [H]; carried: slot s at carried + s * stride, fp32 [taps - 1, channels];
// state [H, n, d]; row_slots int32 [rows]: the slot of every row; segs / slots as above. Updates state and carried.
extern "C" int rmlx_ssd_scan(const void* raw, int ld, int x_at, int dt_at, const float* conv_w, const float* conv_b, int taps,
                             float* carried, const float* dt_bias, const float* a_log, const float* skip, float* rec, int rows,
                             const int* segs, const int* row_slots, int n_segs, float* state, long long stride, float* out,
                             int ld_out, int H, int G, int n, int d, int f32, int* status, int pdl, cudaStream_t st) {
  if (!scan_args_ok(rows, segs, row_slots, n_segs, rec, H, n, d) || !row_slots || G < 1 || H % G || taps < 1 || ld_out < H * d ||
      x_at < 0 || dt_at < 0 || ld < x_at + H * d + 2 * G * n || ld < dt_at + H || (taps > 1 && !carried))
    return -2;
  ScanParams p{};
  p.rows = rows; p.segs = reinterpret_cast<const int4*>(segs); p.slots = row_slots;
  p.state = state; p.stride = stride; p.out = out; p.ld_out = ld_out;
  p.H = H; p.n = n; p.d = d; p.status = status;
  auto run = [&](auto* type) -> int {
    using T = std::remove_pointer_t<decltype(type)>;
    const SsdIn<T> in{static_cast<const T*>(raw), ld, x_at, dt_at, conv_w, conv_b, taps, carried, stride, row_slots, !segs,
                      dt_bias, a_log, skip, H, G, n, d};
    const int rc = run_ssd<T>(in, p, rec, n_segs, pdl, st);
    if (rc || taps == 1) return rc;
    const int ch = H * d + 2 * G * n;
    return launch(conv_carry_kernel<T>, dim3((ch + kRowThreads - 1) / kRowThreads, n_segs), dim3(kRowThreads), 0, st, pdl != 0,
                  in.raw, ld, x_at, carried, stride, p.segs, row_slots, ch, taps - 1);
  };
  return f32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
}

// q, k, v and the other arguments as in rmlx_gla_scan; decay fp32 [H]. rec: rmlx_scan_record(dim, vdim, 1, 1) floats per
// (token, head).
extern "C" int rmlx_lightning_scan(const void* q, const void* k, const void* v, int ld, const float* decay, float* rec, int rows,
                                   const int* segs, const int* slots, int n_segs, float* state, long long stride, float* out,
                                   int ld_out, int H, int dim, int vdim, int f32, int* status, int pdl, cudaStream_t st) {
  if (!scan_args_ok(rows, segs, slots, n_segs, rec, H, dim, vdim) || !decay || ld < H * dim || ld < H * vdim || ld_out < H * vdim ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15))
    return -2;
  ScanParams p{};
  p.rows = rows; p.segs = reinterpret_cast<const int4*>(segs); p.slots = slots;
  p.state = state; p.stride = stride; p.out = out; p.ld_out = ld_out;
  p.H = H; p.n = dim; p.d = vdim; p.status = status;
  auto run = [&](auto* type) {
    using T = std::remove_pointer_t<decltype(type)>;
    return run_lightning<T>(LightIn<T>{static_cast<const T*>(q), static_cast<const T*>(k), static_cast<const T*>(v), ld, decay,
                                       dim, vdim}, p, rec, n_segs, pdl, st);
  };
  return f32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
}

// o fp32 [rows, ld_o], gate and out [rows, ..] fp32 (f32) or bf16, w fp32 [groups * size].
extern "C" int rmlx_gated_norm(const float* o, int ld_o, const void* gate, int ld_g, const float* w, float eps, void* out,
                               int ld_out, int rows, int groups, int size, int gate_first, int sigmoid, int f32, int pdl,
                               cudaStream_t st) {
  if (rows < 1 || groups < 1 || size < 1 || ld_o < groups * size || ld_g < groups * size || ld_out < groups * size) return -2;
  const int lanes = size <= 64 ? 8 : size <= 128 ? 16 : size <= 256 ? 32 : 256;
  const long long units = 1LL * rows * groups, blocks = (units * lanes + kRowThreads - 1) / kRowThreads;
  if (units * lanes > 0x7fffffffLL) return -2;
  const dim3 grid{unsigned(blocks)};
  const bool vec = size % 8 == 0 && ld_o % 8 == 0 && ld_g % 8 == 0 && ld_out % 8 == 0 &&
                   !((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out) |
                      reinterpret_cast<uintptr_t>(w)) & 15);
#define RB_GN(T_, L_, K_, F_, V_)                                                                                      \
  return launch(gated_norm_kernel<T_, L_, K_, F_, V_>, grid, dim3(kRowThreads), 0, st, pdl != 0, o, ld_o,              \
                static_cast<const T_*>(gate), ld_g, w, eps, static_cast<T_*>(out), ld_out, rows, groups, size, sigmoid != 0)
#define RB_GNL(T_, F_, V_)                          \
  {                                                 \
    if (lanes == 8) RB_GN(T_, 8, 1, F_, V_);        \
    if (lanes == 16) RB_GN(T_, 16, 1, F_, V_);      \
    if (lanes == 32) RB_GN(T_, 32, 1, F_, V_);      \
    if (size <= 2048) RB_GN(T_, 256, 1, F_, V_);    \
    RB_GN(T_, 256, 2, F_, V_);                      \
  }
#define RB_GNV(T_)                                    \
  {                                                   \
    if (gate_first && vec) RB_GNL(T_, true, true)     \
    if (gate_first) RB_GNL(T_, true, false)           \
    if (vec) RB_GNL(T_, false, true)                  \
    RB_GNL(T_, false, false)                          \
  }
  if (f32) RB_GNV(float)
  RB_GNV(__nv_bfloat16)
#undef RB_GNV
#undef RB_GNL
#undef RB_GN
}
