// RWKV-style time mixing: token shift, the WKV recurrence with its fp32 state, and the per-head norm
// with the output gate.
//
// Per head, with S [dim, dim] (rows: key channels, columns: value channels) carried per sequence:
//     o_t = (S + diag(u) k_t v_t^T)^T r_t,   S <- diag(w_t) S + k_t v_t^T,
//     w_t = exp(-exp(dl_t + w0))
// Columns are independent of each other. A block owns one (sequence, head, group of columns) and walks
// the sequence's new tokens. A thread holds ROWS rows of four columns in registers (each r, k and w read from
// shared memory then serves four columns: shared-memory wavefronts, not arithmetic, are what one column per
// thread is bound by); LANES threads share a column and add their parts by a transposing butterfly. Half of the
// block's warps fetch tokens ahead, take the exponentials and r . (u k), and stage the next chunk while the
// other half runs the current one. Arithmetic on the state runs on pairs (fma.rn.f32x2).
//
// The state of a sequence lives in its slot's row of a flat fp32 pool, beside the last token's
// residual row, which the token shift of the sequence's next token needs.
#include "../common/launch.cuh"
#include "../common/rows.cuh"

namespace rb {

constexpr int kShiftParts = 5;            // r, k, v, g, w

// out[s][t] = x[t] + (prev[t] - x[t]) * mu[s]; prev: the row before in the batch, or for a sequence's
// first row of the batch the row kept in its slot. slots [T]; each_row: no two rows share a sequence.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
token_shift_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ mu, const float* __restrict__ prev,
                   long long prev_stride, const int* __restrict__ slots, int each_row, T* __restrict__ out, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const bool first = each_row || t == 0 || slots[t - 1] != slots[t];
  const float* before = first ? prev + size_t(slots[t]) * prev_stride : x + size_t(t - 1) * ldx;
  const float* row = x + size_t(t) * ldx;
  for (int c = threadIdx.x; c < ldx >> 3; c += kRowThreads) {
    float a[8], b[8];
    load8(row + c * 8, a);
    load8(before + c * 8, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) b[i] -= a[i];
#pragma unroll
    for (int s = 0; s < kShiftParts; ++s) {
      float m[8];
      load8(mu + s * ldx + c * 8, m);
#pragma unroll
      for (int i = 0; i < 8; ++i) m[i] = fmaf(b[i], m[i], a[i]);
      store8(out + (size_t(s) * rows + t) * ldx + c * 8, m);
    }
  }
}

__device__ __forceinline__ uint64_t wk_pair(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void wk_unpair(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t wk_fma(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t wk_mul(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

struct WkvParams {
  const void* r;            // [rows, ld] each, head h at column h * dim
  const void* k;
  const void* v;
  int ld;
  const float* dl;          // [rows, ld_dl] decay logits before w0
  int ld_dl;
  const float* w0;          // [H * dim]
  const float* u;           // [H * dim]
  const int4* segs;         // {first row, rows, slot, -}; null: segment i is row i with slot slots[i]
  const int* slots;
  float* state;             // slot s: state + s * stride, [H, dim, dim]
  float* prev;              // slot s: prev + s * stride, [ldx]
  long long stride;
  const float* x;           // [rows, ldx] what the sublayer read
  int ldx;
  float* out;               // [rows, ld_out] fp32
  int ld_out;
  int H, dim;
};

constexpr int kWkHalf = 64, kWkCols = 4;            // compute (and staging) threads; columns per thread
template <int ROWS, int LANES>
struct WkCfg {
  static constexpr int kDim = ROWS * LANES;          // padded rows of the state
  static constexpr int kCols = kWkHalf / LANES * kWkCols;        // columns per block
  static constexpr int kChunk = kDim > 128 ? 4 : kDim > 64 ? 8 : 16;   // tokens per chunk
  static constexpr int kTok = 3 * kDim + kCols + 4;              // r, k, w, v, r . (u k)
  static constexpr int kSmem = 2 * kChunk * kTok * 4;
};

template <class T, int ROWS, int LANES>
__global__ void __launch_bounds__(2 * kWkHalf) wkv_scan_kernel(WkvParams p) {
  using C = WkCfg<ROWS, LANES>;
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, col0 = blockIdx.x * C::kCols;
  int row0, len, slot;
  if (p.segs) {
    const int4 s = p.segs[blockIdx.z];
    row0 = s.x; len = s.y; slot = s.z;
  } else {
    row0 = blockIdx.z; len = 1; slot = p.slots[blockIdx.z];
  }
  const int dim = p.dim, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int SW = kWkHalf / 32;                               // staging warps
  const bool stager = warp >= SW;
  const int chunks = (len + C::kChunk - 1) / C::kChunk;

  // A stager warp holds the raw values of its tokens of one chunk: they are asked for one chunk before they
  // are converted, so that the loads run beside the recurrence.
  constexpr int M = (C::kDim + 31) / 32;                         // key channels per lane
  constexpr int VM = (C::kCols + 31) / 32;
  constexpr int PER = C::kChunk / SW;                            // tokens per warp
  T fr[PER][M], fk[PER][M], fv[PER][VM];
  float fd[PER][M], w0[M], uu[M];
  const T* rp = static_cast<const T*>(p.r) + h * dim;
  const T* kp = static_cast<const T*>(p.k) + h * dim;
  const T* vp = static_cast<const T*>(p.v) + h * dim + col0;
  const float* dp = p.dl + h * dim;
  auto fetch = [&](int ch) {
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      const int t = ch * C::kChunk + q * SW + (warp - SW);
      const size_t row = size_t(row0 + min(t, len - 1));
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int i = min(m * 32 + lane, dim - 1);               // always in bounds; masked below
        fr[q][m] = rp[row * p.ld + i];
        fk[q][m] = kp[row * p.ld + i];
        fd[q][m] = dp[row * p.ld_dl + i];
      }
#pragma unroll
      for (int m = 0; m < VM; ++m) fv[q][m] = vp[row * p.ld + min(m * 32 + lane, dim - 1 - col0)];
    }
  };
  auto convert = [&](int ch) {
    float* buf = smem + (ch & 1) * C::kChunk * C::kTok;
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      const int tok = q * SW + (warp - SW);
      const bool there = ch * C::kChunk + tok < len;             // tokens past the end leave the state as it is
      float* b = buf + tok * C::kTok;
      float ruk = 0.f;
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int i = m * 32 + lane;
        if (C::kDim < 32 && i >= C::kDim) continue;
        // row group g's values four at a time: 16-byte pieces of consecutive groups are neighbours
        const int at = (i % ROWS) / 4 * (LANES * 4) + i / ROWS * 4 + i % 4;
        const bool in = there && i < dim;
        const float r = in ? to_f32(fr[q][m]) : 0.f, k = in ? to_f32(fk[q][m]) : 0.f;
        b[at] = r;
        b[C::kDim + at] = k;
        b[2 * C::kDim + at] = in ? __expf(-__expf(fd[q][m] + w0[m])) : 1.f;
        ruk = fmaf(r * uu[m], k, ruk);
      }
#pragma unroll
      for (int m = 0; m < VM; ++m) {
        const int c = m * 32 + lane;
        if (c < C::kCols) b[3 * C::kDim + c] = there && col0 + c < dim ? to_f32(fv[q][m]) : 0.f;
      }
      ruk = warp_sum(ruk);
      if (lane == 0) b[3 * C::kDim + C::kCols] = ruk;
    }
  };

  // compute threads: rows g * ROWS .. of columns c0 .. c0 + 3 (of the block)
  const int g = threadIdx.x % LANES, c0 = (threadIdx.x & (kWkHalf - 1)) / LANES * kWkCols;
  uint64_t s2[ROWS / 2][kWkCols];
  float* sp = p.state + size_t(slot) * p.stride + size_t(h) * dim * dim;
  if (!stager) {
#pragma unroll
    for (int i = 0; i < ROWS / 2; ++i)
#pragma unroll
      for (int c = 0; c < kWkCols; ++c) {
        const int r0 = g * ROWS + 2 * i, col = col0 + c0 + c;
        s2[i][c] = wk_pair((r0 < dim && col < dim) ? sp[size_t(r0) * dim + col] : 0.f,
                           (r0 + 1 < dim && col < dim) ? sp[size_t(r0 + 1) * dim + col] : 0.f);
      }
  } else {
    fetch(0);
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const bool in = m * 32 + lane < dim;
      w0[m] = in ? p.w0[h * dim + m * 32 + lane] : 0.f;
      uu[m] = in ? p.u[h * dim + m * 32 + lane] : 0.f;
    }
    convert(0);
    if (chunks > 1) fetch(1);
  }
  __syncthreads();
  // after the butterfly, the lanes of a column group hold column `mine` of the four
  const int mine = (g & (LANES / 2) ? 2 : 0) + (g & (LANES / 4) ? 1 : 0);
  const bool writer = g % (LANES / 4) == 0 && col0 + c0 + mine < dim;
  float* op = p.out + size_t(row0) * p.ld_out + h * dim + col0 + c0 + mine;
  for (int ch = 0; ch < chunks; ++ch) {
    if (stager) {
      if (ch + 1 < chunks) {
        convert(ch + 1);
        if (ch + 2 < chunks) fetch(ch + 2);
      }
    } else {
      const float* buf = smem + (ch & 1) * C::kChunk * C::kTok;
      const int n = min(C::kChunk, len - ch * C::kChunk);
      constexpr int TU = 4;                                      // tokens whose sums are in flight together
      for (int t0 = 0; t0 < n; t0 += TU) {
        float o[TU][kWkCols];
#pragma unroll
        for (int q = 0; q < TU; ++q) {
          const float* b = buf + (t0 + q) * C::kTok;
          const float4 v = *reinterpret_cast<const float4*>(b + 3 * C::kDim + c0);
          const uint64_t v2[kWkCols] = {wk_pair(v.x, v.x), wk_pair(v.y, v.y), wk_pair(v.z, v.z), wk_pair(v.w, v.w)};
          uint64_t acc[kWkCols] = {0, 0, 0, 0};
#pragma unroll
          for (int i = 0; i < ROWS / 4; ++i) {
            const int at = i * (LANES * 4) + g * 4;
            const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(b + at);
            const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(b + C::kDim + at);
            const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(b + 2 * C::kDim + at);
#pragma unroll
            for (int c = 0; c < kWkCols; ++c) {
              acc[c] = wk_fma(r.x, s2[2 * i][c], acc[c]);
              acc[c] = wk_fma(r.y, s2[2 * i + 1][c], acc[c]);
              s2[2 * i][c] = wk_fma(w.x, s2[2 * i][c], wk_mul(k.x, v2[c]));
              s2[2 * i + 1][c] = wk_fma(w.y, s2[2 * i + 1][c], wk_mul(k.y, v2[c]));
            }
          }
#pragma unroll
          for (int c = 0; c < kWkCols; ++c) {
            float lo, hi;
            wk_unpair(acc[c], lo, hi);
            o[q][c] = lo + hi;
          }
        }
        float sum[TU];
#pragma unroll
        for (int q = 0; q < TU; ++q) {
          const bool up = g & (LANES / 2), up2 = g & (LANES / 4);
          const float k0 = up ? o[q][2] : o[q][0], k1 = up ? o[q][3] : o[q][1];
          const float x0 = up ? o[q][0] : o[q][2], x1 = up ? o[q][1] : o[q][3];
          const float y0 = k0 + __shfl_xor_sync(0xffffffffu, x0, LANES / 2);
          const float y1 = k1 + __shfl_xor_sync(0xffffffffu, x1, LANES / 2);
          sum[q] = (up2 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, up2 ? y0 : y1, LANES / 4);
        }
#pragma unroll
        for (int off = LANES / 8; off > 0; off >>= 1)
#pragma unroll
          for (int q = 0; q < TU; ++q) sum[q] += __shfl_xor_sync(0xffffffffu, sum[q], off);
        if (writer) {
#pragma unroll
          for (int q = 0; q < TU; ++q) {
            const float* b = buf + (t0 + q) * C::kTok + 3 * C::kDim;
            if (t0 + q < n) op[size_t(ch * C::kChunk + t0 + q) * p.ld_out] = fmaf(b[C::kCols], b[c0 + mine], sum[q]);
          }
        }
      }
    }
    __syncthreads();
  }
  if (!stager) {
#pragma unroll
    for (int i = 0; i < ROWS / 2; ++i)
#pragma unroll
      for (int c = 0; c < kWkCols; ++c) {
        const int r0 = g * ROWS + 2 * i, col = col0 + c0 + c;
        float lo, hi;
        wk_unpair(s2[i][c], lo, hi);
        if (col < dim) {
          if (r0 < dim) sp[size_t(r0) * dim + col] = lo;
          if (r0 + 1 < dim) sp[size_t(r0 + 1) * dim + col] = hi;
        }
      }
  } else if (blockIdx.x == 0 && h == 0) {
    const float* last = p.x + size_t(row0 + len - 1) * p.ldx;
    float* keep = p.prev + size_t(slot) * p.stride;
    for (int i = threadIdx.x - kWkHalf; i < p.ldx; i += kWkHalf) keep[i] = last[i];
  }
}

// a[t, h*dim + i] = o / rms(o over the head) * norm * silu(gate). L lanes per (row, head).
template <class T, int L>
__global__ void __launch_bounds__(kRowThreads)
wkv_finish_kernel(const float* __restrict__ o, int ld_o, const T* __restrict__ gate, int ld_g,
                  const float* __restrict__ norm, float eps, T* __restrict__ a, int ld_a, int rows, int H, int dim) {
  pdl_launch_dependents();
  pdl_wait();
  const int unit = (blockIdx.x * kRowThreads + threadIdx.x) / L, lane = threadIdx.x % L;
  const bool live = unit < rows * H;                   // the lanes of a warp stay together for the sums
  const int t = live ? unit / H : 0, h = live ? unit - t * H : 0;
  const int at = h * dim + lane * 8, n = dim - lane * 8;
  const bool vec = dim % 8 == 0 && ld_o % 8 == 0 && ld_g % 8 == 0 && ld_a % 8 == 0 && n > 0;
  float f[8], ssq = 0.f;
  load8_upto(o + size_t(t) * ld_o + at, n, vec, f);
#pragma unroll
  for (int i = 0; i < 8; ++i) ssq += f[i] * f[i];
  ssq = group_sum<L>(ssq);
  if (!live || n <= 0) return;
  const float inv = 1.f / sqrtf(ssq / float(dim) + eps);
  float z[8], w[8];
  load8_upto(gate + size_t(t) * ld_g + at, n, vec, z);
  load8_upto(norm + at, n, vec, w);
#pragma unroll
  for (int i = 0; i < 8; ++i) f[i] = f[i] * inv * w[i] * (z[i] / (1.f + expf(-z[i])));
  T* dst = a + size_t(t) * ld_a + at;
  if (vec) {
    store8(dst, f);
  } else {
    for (int i = 0; i < 8 && i < n; ++i) dst[i] = from_f32<T>(f[i]);
  }
}

template <class T, int ROWS, int LANES>
static int launch_wkv(const WkvParams& p, int n_segs, int pdl, cudaStream_t st) {
  using C = WkCfg<ROWS, LANES>;
  auto kern = wkv_scan_kernel<T, ROWS, LANES>;
  RB_CHECK(set_max_smem(kern, C::kSmem));
  return launch(kern, dim3((p.dim + C::kCols - 1) / C::kCols, p.H, n_segs), dim3(2 * kWkHalf), C::kSmem, st, pdl != 0, p);
}
template <class T>
static int dispatch_wkv(const WkvParams& p, int n, int pdl, cudaStream_t st) {
  if (p.dim <= 16) return launch_wkv<T, 4, 4>(p, n, pdl, st);
  if (p.dim <= 32) return launch_wkv<T, 4, 8>(p, n, pdl, st);
  if (p.dim <= 64) return launch_wkv<T, 4, 16>(p, n, pdl, st);
  if (p.dim <= 128) return launch_wkv<T, 4, 32>(p, n, pdl, st);
  if (p.dim <= 256) return launch_wkv<T, 8, 32>(p, n, pdl, st);
  return -2;
}

}  // namespace rb

using namespace rb;

// Largest head size of the recurrence.
extern "C" int rmlx_wkv_max_dim() { return 256; }

// x fp32 [T, ldx], mu fp32 [5, ldx], out [5, T, ldx] fp32 (f32) or bf16; ldx a multiple of eight, prev
// rows 16-byte aligned. slots int32 [T].
extern "C" int rmlx_token_shift(const float* x, int ldx, const float* mu, const float* prev, long long prev_stride,
                                const int* slots, int each_row, void* out, int T, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || ldx < 8 || ldx % 8 || prev_stride % 4 || !slots) return -2;
  if (f32)
    return launch(token_shift_kernel<float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, x, ldx, mu, prev, prev_stride,
                  slots, each_row, static_cast<float*>(out), T);
  return launch(token_shift_kernel<__nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, x, ldx, mu, prev,
                prev_stride, slots, each_row, static_cast<__nv_bfloat16*>(out), T);
}

// r, k, v [rows, ld] fp32 (f32) or bf16; dl fp32 [rows, ld_dl]; segs int32 [n_segs, 4] (16-byte aligned) or
// null with slots [n_segs]: then every row is a segment. No slot occurs twice except one that nobody reads.
extern "C" int rmlx_wkv_scan(const void* r, const void* k, const void* v, int ld, const float* dl, int ld_dl,
                             const float* w0, const float* u, const int* segs, const int* slots, int n_segs,
                             float* state, float* prev, long long stride, const float* x, int ldx, float* out,
                             int ld_out, int H, int dim, int f32, int pdl, cudaStream_t st) {
  if (n_segs < 1 || n_segs > 65535 || H < 1 || H > 65535 || dim < 1 || ld < H * dim || ld_dl < H * dim ||
      ld_out < H * dim || (!segs && !slots) || (reinterpret_cast<uintptr_t>(segs) & 15))
    return -2;
  WkvParams p;
  p.r = r; p.k = k; p.v = v; p.ld = ld; p.dl = dl; p.ld_dl = ld_dl; p.w0 = w0; p.u = u;
  p.segs = reinterpret_cast<const int4*>(segs); p.slots = slots;
  p.state = state; p.prev = prev; p.stride = stride; p.x = x; p.ldx = ldx; p.out = out; p.ld_out = ld_out;
  p.H = H; p.dim = dim;
  return f32 ? dispatch_wkv<float>(p, n_segs, pdl, st) : dispatch_wkv<__nv_bfloat16>(p, n_segs, pdl, st);
}

extern "C" int rmlx_wkv_finish(const float* o, int ld_o, const void* gate, int ld_g, const float* norm, float eps,
                               void* a, int ld_a, int rows, int H, int dim, int f32, int pdl, cudaStream_t st) {
  const long long units = 1LL * rows * H;
  if (rows < 1 || H < 1 || dim < 1 || units > 0x7fffffffLL) return -2;
  const int lanes = dim <= 64 ? 8 : dim <= 128 ? 16 : 32;
  if (dim > 256 || units * lanes > 0x7fffffffLL) return -2;
  const dim3 grid(unsigned((units * lanes + kRowThreads - 1) / kRowThreads));
#define RB_WF(T_, L_)                                                                                              \
  return launch(wkv_finish_kernel<T_, L_>, grid, dim3(kRowThreads), 0, st, pdl != 0, o, ld_o,                      \
                static_cast<const T_*>(gate), ld_g, norm, eps, static_cast<T_*>(a), ld_a, rows, H, dim)
#define RB_WFL(T_)                 \
  {                                \
    if (lanes == 8) RB_WF(T_, 8);  \
    if (lanes == 16) RB_WF(T_, 16); \
    RB_WF(T_, 32);                 \
  }
  if (f32) RB_WFL(float)
  RB_WFL(__nv_bfloat16)
#undef RB_WFL
#undef RB_WF
}
