// RWKV-style time mixing: token shift, the WKV recurrence with its fp32 state, and the per-head norm
// with the output gate.
//
// Per head, with S [dim, dim] (rows: key channels, columns: value channels) carried per sequence:
//     o_t = (S + diag(u) k_t v_t^T)^T r_t,   S <- diag(w_t) S + k_t v_t^T,
//     w_t = exp(-exp(dl_t + w0))
// The recurrence runs on common/scan.cuh.
//
// The state of a sequence lives in its slot's row of a flat fp32 pool, beside the last token's
// residual row, which the token shift of the sequence's next token needs.
#include "../common/launch.cuh"
#include "../common/rows.cuh"
#include "../common/scan.cuh"

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

// Rows of the scan: r, k and the decay; the new token's own share is r . (u k) v.
template <class T>
struct WkvIn {
  const T* r; const T* k; const T* v;
  int ld;
  const float* dl;
  int ld_dl;
  const float* w0; const float* u;
  int dim;
  __device__ __forceinline__ void rows4(int t, int h, int i, float (&fr)[4], float (&fk)[4], float (&fw)[4], float (&fb)[4]) const {
    const bool vec = dim % 4 == 0 && ld % 4 == 0;
    const size_t at = size_t(t) * ld + h * dim;
    const float* dp = dl + size_t(t) * ld_dl + h * dim;
    scan_load4(r + at, i, dim, vec, fr);
    scan_load4(k + at, i, dim, vec, fk);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const bool in = i + j < dim;
      fw[j] = in ? expf(-expf(dp[in ? i + j : 0] + w0[h * dim + (in ? i + j : 0)])) : 1.f;
      fb[j] = fr[j] * (in ? u[h * dim + i + j] : 0.f);
    }
  }
  __device__ __forceinline__ void cols4(int t, int h, int i, float (&fv)[4]) const {
    scan_load4(v + size_t(t) * ld + h * dim, i, dim, dim % 4 == 0 && ld % 4 == 0, fv);
  }
};

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

template <class T>
static int dispatch_wkv(const WkvIn<T>& in, const ScanParams& p, float* rec, int n, int pdl, cudaStream_t st) {
#define RB_WKV(R_, L_) return launch_row_scan<WkvIn<T>, R_, L_>(in, p, rec, n, pdl, st)
  RB_SCAN_DISPATCH(p.n, RB_WKV);
#undef RB_WKV
  return -2;
}

}  // namespace rb

using namespace rb;

// Largest head size of the recurrence.
extern "C" int rmlx_wkv_max_dim() { return kScanMaxRows; }
// Floats of the scratch records of one (token, head).
extern "C" int rmlx_wkv_record(int dim) {
#define RB_WKV(R_, L_) return int(scan_row_floats((R_) * (L_), L_, 3, dim, 1))
  RB_SCAN_DISPATCH(dim, RB_WKV);
#undef RB_WKV
  return 0;
}

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

// r, k, v [rows, ld] fp32 (f32) or bf16; dl fp32 [rows, ld_dl]; rec: scratch, rows * H records,
// 16-byte aligned; segs int32 [n_segs, 4] (16-byte aligned) or null with slots [n_segs]: then every row is a segment.
// No slot occurs twice except one that nobody reads. status: set when a wait for a chunk gave up.
extern "C" int rmlx_wkv_scan(const void* r, const void* k, const void* v, int ld, const float* dl, int ld_dl,
                             const float* w0, const float* u, float* rec, int rows, const int* segs, const int* slots,
                             int n_segs, float* state, float* prev, long long stride, const float* x, int ldx, float* out,
                             int ld_out, int H, int dim, int f32, int* status, int pdl, cudaStream_t st) {
  if (rows < 1 || n_segs < 1 || n_segs > 65535 || H < 1 || H > 65535 || dim < 1 || ld < H * dim || ld_dl < H * dim ||
      ld_out < H * dim || (!segs && !slots) || ((reinterpret_cast<uintptr_t>(segs) | reinterpret_cast<uintptr_t>(rec)) & 15) ||
      ((reinterpret_cast<uintptr_t>(r) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) |
        reinterpret_cast<uintptr_t>(dl)) & 15))
    return -2;
  ScanParams p{};
  p.rows = rows;
  p.segs = reinterpret_cast<const int4*>(segs); p.slots = slots;
  p.state = state; p.prev = prev; p.stride = stride; p.x = x; p.ldx = ldx; p.out = out; p.ld_out = ld_out;
  p.H = H; p.n = p.d = dim; p.status = status;
  auto run = [&](auto* type) {
    using T = std::remove_pointer_t<decltype(type)>;
    return dispatch_wkv<T>(WkvIn<T>{static_cast<const T*>(r), static_cast<const T*>(k), static_cast<const T*>(v), ld, dl, ld_dl,
                                    w0, u, dim}, p, rec, n_segs, pdl, st);
  };
  return f32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
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
