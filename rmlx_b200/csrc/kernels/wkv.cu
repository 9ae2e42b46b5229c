// RWKV-style time mixing: token shift, the WKV recurrence with its fp32 state, and the per-head norm
// with the output gate.
//
// Per head, with S [dim, dim] (rows: key channels, columns: value channels) carried per sequence:
//     o_t = (S + diag(u) k_t v_t^T)^T r_t,   S <- diag(w_t) S + k_t v_t^T,
//     w_t = exp(-exp(dl_t + w0))
// Columns are independent of each other. wkv_prepare takes the exponentials once per head and writes one fp32
// record per (head, token): r, k, w, v and r . (u k), the records of a head in token order. wkv_scan: a block
// owns one (sequence, head, group of columns) and walks the sequence's new tokens, whose records arrive in
// shared memory by one bulk copy per chunk, two chunks ahead: no instruction of the scan is spent on staging
// (when the block converted its own inputs, that took more issue slots than the recurrence). A thread holds
// ROWS rows of four columns in registers, so that each r, k and w it reads serves four columns; LANES threads
// share a column and add their parts by a transposing butterfly. Arithmetic on the state runs on pairs
// (fma.rn.f32x2).
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

constexpr int kWkThreads = 64, kWkCols = 4, kWkStages = 3;       // columns per thread; chunks in flight
template <int ROWS, int LANES>
struct WkCfg {
  static constexpr int kDim = ROWS * LANES;          // padded rows of the state
  static constexpr int kCols = kWkThreads / LANES * kWkCols;     // columns per block
  static constexpr int kChunk = kDim > 128 ? 8 : 16;             // tokens per chunk
  static constexpr int kV = (kDim + kCols - 1) / kCols * kCols;  // padded columns
  static constexpr int kRec = 3 * kDim + kV + 4;                 // floats of a record
  static constexpr int kSmem = kWkStages * kChunk * kRec * 4 + 64;
};

// Where value i of r, k or w sits in a record: row group g's values four at a time, so that the 16-byte pieces
// of consecutive groups are neighbours.
template <int ROWS, int LANES>
__device__ __forceinline__ int wk_at(int i) {
  return (i % ROWS) / 4 * (LANES * 4) + i / ROWS * 4 + i % 4;
}

// rec[h][t] of all heads and rows. LU lanes per record, four values each per turn.
template <class T, int ROWS, int LANES, int LU>
__global__ void __launch_bounds__(kRowThreads)
wkv_prepare_kernel(const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, int ld,
                   const float* __restrict__ dl, int ld_dl, const float* __restrict__ w0, const float* __restrict__ u,
                   float* __restrict__ rec, int rows, int H, int dim) {
  using C = WkCfg<ROWS, LANES>;
  pdl_launch_dependents();
  pdl_wait();
  const int unit = (blockIdx.x * kRowThreads + threadIdx.x) / LU, lane = threadIdx.x % LU;
  const bool live = unit < rows * H;                 // the lanes of a warp stay together for the sum
  const int t = live ? unit / H : 0, h = live ? unit - t * H : 0;
  float* out = rec + (size_t(h) * rows + t) * C::kRec;
  const bool vec = dim % 4 == 0 && ld % 4 == 0 && ld_dl % 4 == 0;
  auto load4 = [&](const T* p, int i, float (&f)[4]) {
    if (vec && i < dim) {
      if (sizeof(T) == 2) {
        const uint2 q = *reinterpret_cast<const uint2*>(p + i);
        f[0] = bf16lo(q.x); f[1] = bf16hi(q.x); f[2] = bf16lo(q.y); f[3] = bf16hi(q.y);
      } else {
        const float4 q = *reinterpret_cast<const float4*>(p + i);
        f[0] = q.x; f[1] = q.y; f[2] = q.z; f[3] = q.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) f[j] = i + j < dim ? to_f32(p[i + j]) : 0.f;
    }
  };
  const size_t at = size_t(t) * ld + h * dim;
  const float* dp = dl + size_t(t) * ld_dl + h * dim;
  float ruk = 0.f;
  for (int i = lane * 4; i < C::kV || i < C::kDim; i += LU * 4) {
    float fr[4], fk[4], fv[4], fw[4];
    load4(r + at, i, fr);
    load4(k + at, i, fk);
    load4(v + at, i, fv);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const bool in = i + j < dim;
      fw[j] = in ? expf(-expf(dp[in ? i + j : 0] + w0[h * dim + (in ? i + j : 0)])) : 1.f;
      ruk = fmaf(fr[j] * (in ? u[h * dim + i + j] : 0.f), fk[j], ruk);
    }
    if (live) {
      if (i < C::kDim) {
        float* o = out + wk_at<ROWS, LANES>(i);
        *reinterpret_cast<float4*>(o) = make_float4(fr[0], fr[1], fr[2], fr[3]);
        *reinterpret_cast<float4*>(o + C::kDim) = make_float4(fk[0], fk[1], fk[2], fk[3]);
        *reinterpret_cast<float4*>(o + 2 * C::kDim) = make_float4(fw[0], fw[1], fw[2], fw[3]);
      }
      if (i < C::kV) *reinterpret_cast<float4*>(out + 3 * C::kDim + i) = make_float4(fv[0], fv[1], fv[2], fv[3]);
    }
  }
  ruk = group_sum<LU>(ruk);
  if (live && lane == 0) *reinterpret_cast<float4*>(out + 3 * C::kDim + C::kV) = make_float4(ruk, 0.f, 0.f, 0.f);
}

struct WkvParams {
  const float* rec;         // [H, rows, kRec]
  int rows;
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
  int* status;
};

template <int ROWS, int LANES>
__global__ void __launch_bounds__(kWkThreads) wkv_scan_kernel(WkvParams p) {
  using C = WkCfg<ROWS, LANES>;
  extern __shared__ __align__(128) float smem[];
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + kWkStages * C::kChunk * C::kRec);      // [stages]
  __shared__ uint32_t gave_up;
  const int h = blockIdx.y, col0 = blockIdx.x * C::kCols, dim = p.dim;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kWkStages; ++i) mbar_init(full + i, 1);
    gave_up = 0u;
    fence_mbar_init();
  }
  pdl_launch_dependents();
  pdl_wait();
  int row0, len, slot;
  if (p.segs) {
    const int4 s = p.segs[blockIdx.z];
    row0 = s.x; len = s.y; slot = s.z;
  } else {
    row0 = blockIdx.z; len = 1; slot = p.slots[blockIdx.z];
  }
  __syncthreads();                                   // the barriers are initialised
  const int chunks = (len + C::kChunk - 1) / C::kChunk;
  const float* src = p.rec + (size_t(h) * p.rows + row0) * C::kRec;
  auto issue = [&](int ch) {
    const int n = min(C::kChunk, len - ch * C::kChunk), st = ch % kWkStages;
    const uint32_t bytes = uint32_t(n) * C::kRec * 4;
    mbar_arrive_expect_tx(full + st, bytes);
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                     smem_u32(smem + st * C::kChunk * C::kRec)),
                 "l"(src + size_t(ch) * C::kChunk * C::kRec), "r"(bytes), "r"(smem_u32(full + st))
                 : "memory");
  };
  if (threadIdx.x == 0)
    for (int ch = 0; ch < kWkStages && ch < chunks; ++ch) issue(ch);

  // rows g * ROWS .. of columns c0 .. c0 + 3 (of the block)
  const int g = threadIdx.x % LANES, c0 = threadIdx.x / LANES * kWkCols;
  uint64_t s2[ROWS / 2][kWkCols];
  float* sp = p.state + size_t(slot) * p.stride + size_t(h) * dim * dim;
#pragma unroll
  for (int i = 0; i < ROWS / 2; ++i)
#pragma unroll
    for (int c = 0; c < kWkCols; ++c) {
      const int r0 = g * ROWS + 2 * i, col = col0 + c0 + c;
      s2[i][c] = wk_pair((r0 < dim && col < dim) ? sp[size_t(r0) * dim + col] : 0.f,
                         (r0 + 1 < dim && col < dim) ? sp[size_t(r0 + 1) * dim + col] : 0.f);
    }
  // after the butterfly, the lanes of a column group hold column `mine` of the four
  const int mine = (g & (LANES / 2) ? 2 : 0) + (g & (LANES / 4) ? 1 : 0);
  const bool writer = g % (LANES / 4) == 0 && col0 + c0 + mine < dim;
  const int at_v = 3 * C::kDim + col0 + c0, at_ruk = 3 * C::kDim + C::kV;
  float* op = p.out + size_t(row0) * p.ld_out + h * dim + col0 + c0 + mine;

  // one token: the state's part of o, then the state's update
  auto token = [&](const float* b, float (&o)[kWkCols]) {
    const float4 v = *reinterpret_cast<const float4*>(b + at_v);
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
      o[c] = lo + hi;
    }
  };
  const bool up = g & (LANES / 2), up2 = g & (LANES / 4);
  auto fold = [&](const float (&o)[kWkCols]) {
    const float k0 = up ? o[2] : o[0], k1 = up ? o[3] : o[1], x0 = up ? o[0] : o[2], x1 = up ? o[1] : o[3];
    const float y0 = k0 + __shfl_xor_sync(0xffffffffu, x0, LANES / 2);
    const float y1 = k1 + __shfl_xor_sync(0xffffffffu, x1, LANES / 2);
    float sum = (up2 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, up2 ? y0 : y1, LANES / 4);
#pragma unroll
    for (int off = LANES / 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    return sum;
  };

  bool ok = true;
  for (int ch = 0; ch < chunks; ++ch) {
    const int st = ch % kWkStages;
    ok = mbar_wait(full + st, uint32_t(ch / kWkStages) & 1u, &gave_up) && ok;
    const float* buf = smem + st * C::kChunk * C::kRec;
    const int n = min(C::kChunk, len - ch * C::kChunk);
    float* oc = op + size_t(ch) * C::kChunk * p.ld_out;
    // groups of TU tokens; a group's sums are taken beside the next group's arithmetic
    constexpr int TU = 4;
    auto put = [&](int t, const float (&o)[TU][kWkCols]) {
      float sum[TU];
#pragma unroll
      for (int q = 0; q < TU; ++q) sum[q] = fold(o[q]);
      if (writer) {
#pragma unroll
        for (int q = 0; q < TU; ++q) {
          const float* b = buf + (t + q) * C::kRec;
          oc[size_t(t + q) * p.ld_out] = fmaf(b[at_ruk], b[at_v + mine], sum[q]);
        }
      }
    };
    int t = 0;
    if (n >= TU) {
      float o[TU][kWkCols];
#pragma unroll
      for (int q = 0; q < TU; ++q) token(buf + q * C::kRec, o[q]);
      for (t = TU; t + TU <= n; t += TU) {
        float next[TU][kWkCols];
#pragma unroll
        for (int q = 0; q < TU; ++q) token(buf + (t + q) * C::kRec, next[q]);
        put(t - TU, o);
#pragma unroll
        for (int q = 0; q < TU; ++q)
#pragma unroll
          for (int c = 0; c < kWkCols; ++c) o[q][c] = next[q][c];
      }
      put(t - TU, o);
    }
    for (; t < n; ++t) {
      const float* b = buf + t * C::kRec;
      float o[kWkCols];
      token(b, o);
      const float sum = fold(o);
      if (writer) oc[size_t(t) * p.ld_out] = fmaf(b[at_ruk], b[at_v + mine], sum);
    }
    __syncthreads();                                 // the stage has been read
    if (threadIdx.x == 0 && ch + kWkStages < chunks) issue(ch + kWkStages);
  }
  if (!ok) {                                         // let the copies in flight land, as far as that goes
    for (int i = 0; threadIdx.x == 0 && i < kWkStages; ++i)
      for (uint32_t k = 0; k < (1u << 16); ++k)
        if (mbar_try_wait(full + i, uint32_t((chunks - 1 - (chunks - 1 - i) % kWkStages) / kWkStages) & 1u)) break;
    if (p.status) atomicExch(p.status, int(kStatusMbarTimeout));
  }
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
  if (blockIdx.x == 0 && h == 0) {
    const float* last = p.x + size_t(row0 + len - 1) * p.ldx;
    float* keep = p.prev + size_t(slot) * p.stride;
    for (int i = threadIdx.x; i < p.ldx; i += kWkThreads) keep[i] = last[i];
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

struct WkvIn {
  const void* r; const void* k; const void* v; int ld;
  const float* dl; int ld_dl; const float* w0; const float* u; float* rec;
};

template <class T, int ROWS, int LANES>
static int launch_wkv(const WkvIn& in, WkvParams p, int n_segs, int pdl, cudaStream_t st) {
  using C = WkCfg<ROWS, LANES>;
  constexpr int LU = C::kDim >= 128 ? 32 : C::kDim / 4;
  const long long threads = 1LL * p.rows * p.H * LU;
  if (threads > 0x7fffffffLL) return -2;
  const int rc = launch(wkv_prepare_kernel<T, ROWS, LANES, LU>, dim3(unsigned((threads + kRowThreads - 1) / kRowThreads)),
                        dim3(kRowThreads), 0, st, pdl != 0, static_cast<const T*>(in.r), static_cast<const T*>(in.k),
                        static_cast<const T*>(in.v), in.ld, in.dl, in.ld_dl, in.w0, in.u, in.rec, p.rows, p.H, p.dim);
  if (rc) return rc;
  auto kern = wkv_scan_kernel<ROWS, LANES>;
  RB_CHECK(set_max_smem(kern, C::kSmem));
  return launch(kern, dim3((p.dim + C::kCols - 1) / C::kCols, p.H, n_segs), dim3(kWkThreads), C::kSmem, st, pdl != 0, p);
}
template <class T>
static int dispatch_wkv(const WkvIn& in, const WkvParams& p, int n, int pdl, cudaStream_t st) {
  if (p.dim <= 16) return launch_wkv<T, 4, 4>(in, p, n, pdl, st);
  if (p.dim <= 32) return launch_wkv<T, 4, 8>(in, p, n, pdl, st);
  if (p.dim <= 64) return launch_wkv<T, 4, 16>(in, p, n, pdl, st);
  if (p.dim <= 128) return launch_wkv<T, 4, 32>(in, p, n, pdl, st);
  if (p.dim <= 256) return launch_wkv<T, 8, 32>(in, p, n, pdl, st);
  return -2;
}

}  // namespace rb

using namespace rb;

// Largest head size of the recurrence.
extern "C" int rmlx_wkv_max_dim() { return 256; }
// Floats of the scratch record of one (token, head).
extern "C" int rmlx_wkv_record(int dim) {
  if (dim <= 16) return WkCfg<4, 4>::kRec;
  if (dim <= 32) return WkCfg<4, 8>::kRec;
  if (dim <= 64) return WkCfg<4, 16>::kRec;
  if (dim <= 128) return WkCfg<4, 32>::kRec;
  return WkCfg<8, 32>::kRec;
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

// r, k, v [rows, ld] fp32 (f32) or bf16; dl fp32 [rows, ld_dl]; rec: scratch, fp32 [H, rows, record], 16-byte
// aligned; segs int32 [n_segs, 4] (16-byte aligned) or null with slots [n_segs]: then every row is a segment.
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
  const WkvIn in{r, k, v, ld, dl, ld_dl, w0, u, rec};
  WkvParams p;
  p.rec = rec; p.rows = rows;
  p.segs = reinterpret_cast<const int4*>(segs); p.slots = slots;
  p.state = state; p.prev = prev; p.stride = stride; p.x = x; p.ldx = ldx; p.out = out; p.ld_out = ld_out;
  p.H = H; p.dim = dim; p.status = status;
  return f32 ? dispatch_wkv<float>(in, p, n_segs, pdl, st) : dispatch_wkv<__nv_bfloat16>(in, p, n_segs, pdl, st);
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
