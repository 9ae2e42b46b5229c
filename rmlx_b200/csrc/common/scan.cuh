// Recurrences with an fp32 matrix state per head, token by token: S [n, d] (rows: key channels, columns: value
// channels) carried per sequence,
//     o_t = scale_t * S^T r_t + own_t * v_t,   S <- diag(w_t) S + k_t v_t^T.
// WKV, gated linear attention and state-space heads are all of this form: what reads the state after its update
// has the decay folded into r (or, when a head has one decay for all its rows, into scale) and adds the new token's
// own share, a multiple of its v.
//
// Columns are independent of each other. A prepare kernel takes the exponentials once and writes fp32 records
// in token order: one per (head, token) with r | k | w - or, with one decay per head (ONE), one per (group of
// heads, token) with r | k - and one per (head, column block, token) with v and own (ONE: x, the decay, which is
// scale, too, the step size dt with v = dt x, and the multiple of x). scan_kernel: a block owns one (sequence, head, group of columns) and walks the sequence's new tokens,
// whose records arrive in shared memory by two bulk copies per chunk, two chunks ahead: no instruction of the
// scan is spent on staging (when the block converted its own inputs, that took more issue slots than the
// recurrence). A thread holds ROWS rows of four columns in registers, so that each r, k and w it reads serves
// four columns; LANES threads share a column and add their parts by a transposing butterfly. Arithmetic on the
// state runs on pairs (fma.rn.f32x2).
#pragma once
#include <type_traits>

#include "launch.cuh"
#include "rows.cuh"

namespace rb {

__device__ __forceinline__ uint64_t scan_pair(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void scan_unpair(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t scan_fma(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t scan_mul(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

constexpr int kScanCols = 4, kScanStages = 3;       // columns per thread; chunks in flight
// TH threads a block: more of them share the row records a block fetches (which L2 bandwidth bounds when every block
// of 64 fetches its own: GLA with 512 blocks at 3.9 TB/s), fewer spread a small problem over more SMs.
template <int ROWS, int LANES, bool ONE, int TH>
struct ScanCfg {
  static constexpr int kRows = ROWS * LANES;                     // padded rows of the state
  static constexpr int kCols = TH / LANES * kScanCols;           // columns per block
  static constexpr int kChunk = kRows > 128 ? 8 : 16;            // tokens per chunk
  static constexpr int kRec = (ONE ? 2 : 3) * kRows;             // floats of a row record
  static constexpr int kCol = kCols + 4;                         // floats of a column record: v | own, or x | decay, dt, own
  static constexpr int kStage = kChunk * (kRec + kCol);
  static constexpr int kSmem = kScanStages * kStage * 4 + 64;
  static constexpr int blocks(int d) { return (d + kCols - 1) / kCols; }
};

// Columns per block, as a power of two: what a column record's layout depends on.
inline int scan_col_shift(int lanes, int threads) {
  int s = 0;
  while ((1 << s) < threads / lanes * kScanCols) ++s;
  return s;
}
inline int scan_blocks(int d, int shift) { return (d + (1 << shift) - 1) >> shift; }
// Threads per block: as many as still leave blocks for most SMs.
inline int scan_threads(int lanes, int d, int H, int n_segs) {
  int th = 64;
  while (th < 256 && (1 << scan_col_shift(lanes, 2 * th)) <= (d + 7) / 8 * 8 &&
         1LL * scan_blocks(d, scan_col_shift(lanes, 2 * th)) * H * n_segs * 10 >= 7LL * sm_count())
    th *= 2;
  return th;
}
// Floats of the records of one token and head whatever the block size; `per` heads share a row record.
inline long long scan_row_floats(int rows, int lanes, int parts, int d, int per) {
  long long widest = 0;
  for (int th = 64; th <= 256; th *= 2) {
    const int sh = scan_col_shift(lanes, th);
    const long long n = 1LL * scan_blocks(d, sh) * ((1 << sh) + 4);
    widest = n > widest ? n : widest;
  }
  return (parts * rows + per - 1) / per + widest;
}

// Where value i of r, k or w sits in a record: row group g's values four at a time, so that the 16-byte pieces
// of consecutive groups are neighbours.
template <int ROWS, int LANES>
__device__ __forceinline__ int scan_at(int i) {
  return (i % ROWS) / 4 * (LANES * 4) + i / ROWS * 4 + i % 4;
}

struct ScanParams {
  const float* rec;         // [H / per, rows, kRec]
  const float* col;         // [H, column blocks, rows, kCol]
  int per;                  // heads that share a row record
  int rows;
  const int4* segs;         // {first row, rows, slot, -}; null: segment i is row i with slot slots[i]
  const int* slots;
  float* state;             // slot s: state + s * stride, [H, n, d]
  long long stride;
  float* out;               // [rows, ld_out] fp32
  int ld_out;
  int H, n, d;
  // the last row of x is kept in the slot's row of `prev` (null: nothing is)
  float* prev;              // slot s: prev + s * stride, [ldx]
  const float* x;           // [rows, ldx]
  int ldx;
  int* status;
};

// Four consecutive values from i on, of which those below `dim` exist. `vec`: i.. is 4-value aligned.
template <class T>
__device__ __forceinline__ void scan_load4(const T* p, int i, int dim, bool vec, float (&f)[4]) {
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
}

// Records of heads with a decay per row. in.rows4(t, h, i, r, k, w, b): rows i .. i + 3 (past the last: r = k =
// b = 0, w = 1), where the new token's own share of the output is (sum of b k) v; in.cols4(t, h, i, v). LU lanes
// per record, four values each per turn.
template <class IN, int ROWS, int LANES, int LU>
__global__ void __launch_bounds__(kRowThreads)
scan_prepare_kernel(IN in, float* __restrict__ rec, float* __restrict__ col, int rows, int H, int d, int shift) {
  constexpr int kRows = ROWS * LANES;
  pdl_launch_dependents();
  pdl_wait();
  const int unit = (blockIdx.x * kRowThreads + threadIdx.x) / LU, lane = threadIdx.x % LU;
  const bool live = unit < rows * H;                 // the lanes of a warp stay together for the sum
  const int t = live ? unit / H : 0, h = live ? unit - t * H : 0;
  float* out = rec + (size_t(h) * rows + t) * 3 * kRows;
  float own = 0.f;
  for (int i = lane * 4; i < kRows; i += LU * 4) {
    float r[4], k[4], w[4], b[4];
    in.rows4(t, h, i, r, k, w, b);
#pragma unroll
    for (int j = 0; j < 4; ++j) own = fmaf(b[j], k[j], own);
    if (live) {
      float* o = out + scan_at<ROWS, LANES>(i);
      *reinterpret_cast<float4*>(o) = make_float4(r[0], r[1], r[2], r[3]);
      *reinterpret_cast<float4*>(o + kRows) = make_float4(k[0], k[1], k[2], k[3]);
      *reinterpret_cast<float4*>(o + 2 * kRows) = make_float4(w[0], w[1], w[2], w[3]);
    }
  }
  own = group_sum<LU>(own);
  if (!live) return;
  const int cols = 1 << shift, nb = (d + cols - 1) >> shift;
  for (int i = lane * 4; i < nb << shift; i += LU * 4) {
    float v[4];
    in.cols4(t, h, i, v);
    const int at = i & (cols - 1);
    float* o = col + ((size_t(h) * nb + (i >> shift)) * rows + t) * (cols + 4) + at;
    *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]);
    if (at == 0) *reinterpret_cast<float4*>(o + cols) = make_float4(own, 0.f, 0.f, 0.f);
  }
}

template <int ROWS, int LANES, bool ONE, int TH>
__global__ void __launch_bounds__(TH) scan_kernel(ScanParams p) {
  using C = ScanCfg<ROWS, LANES, ONE, TH>;
  extern __shared__ __align__(128) float smem[];
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + kScanStages * C::kStage);      // [stages]
  __shared__ uint32_t gave_up;
  const int h = blockIdx.y, col0 = blockIdx.x * C::kCols, n_rows = p.n, dim = p.d;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kScanStages; ++i) mbar_init(full + i, 1);
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
  const float* src = p.rec + (size_t(h / p.per) * p.rows + row0) * C::kRec;
  const float* src_col = p.col + ((size_t(h) * gridDim.x + blockIdx.x) * p.rows + row0) * C::kCol;
  auto copy = [&](float* dst, const float* from, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                     smem_u32(dst)),
                 "l"(from), "r"(bytes), "r"(smem_u32(bar))
                 : "memory");
  };
  auto issue = [&](int ch) {
    const int n = min(C::kChunk, len - ch * C::kChunk), st = ch % kScanStages;
    float* buf = smem + st * C::kStage;
    mbar_arrive_expect_tx(full + st, uint32_t(n) * (C::kRec + C::kCol) * 4);
    copy(buf, src + size_t(ch) * C::kChunk * C::kRec, uint32_t(n) * C::kRec * 4, full + st);
    copy(buf + C::kChunk * C::kRec, src_col + size_t(ch) * C::kChunk * C::kCol, uint32_t(n) * C::kCol * 4, full + st);
  };
  if (threadIdx.x == 0)
    for (int ch = 0; ch < kScanStages && ch < chunks; ++ch) issue(ch);

  // rows g * ROWS .. of columns c0 .. c0 + 3 (of the block)
  const int g = threadIdx.x % LANES, c0 = threadIdx.x / LANES * kScanCols;
  uint64_t s2[ROWS / 2][kScanCols];
  float* sp = p.state + size_t(slot) * p.stride + size_t(h) * n_rows * dim;
#pragma unroll
  for (int i = 0; i < ROWS / 2; ++i)
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
      const int r0 = g * ROWS + 2 * i, col = col0 + c0 + c;
      s2[i][c] = scan_pair((r0 < n_rows && col < dim) ? sp[size_t(r0) * dim + col] : 0.f,
                         (r0 + 1 < n_rows && col < dim) ? sp[size_t(r0 + 1) * dim + col] : 0.f);
    }
  // after the butterfly, the lanes of a column group hold column `mine` of the four
  const int mine = (g & (LANES / 2) ? 2 : 0) + (g & (LANES / 4) ? 1 : 0);
  const bool writer = g % (LANES / 4) == 0 && col0 + c0 + mine < dim;
  const int at_own = C::kCols + (ONE ? 2 : 0);
  float* op = p.out + size_t(row0) * p.ld_out + h * dim + col0 + c0 + mine;

  // one token: the state's part of o, then the state's update
  auto token = [&](const float* b, const float* bc, float (&o)[kScanCols]) {
    float4 v = *reinterpret_cast<const float4*>(bc + c0);
    uint64_t one = 0;
    if (ONE) {
      const float2 a = *reinterpret_cast<const float2*>(bc + C::kCols);      // decay, dt
      one = scan_pair(a.x, a.x);
      v.x *= a.y; v.y *= a.y; v.z *= a.y; v.w *= a.y;
    }
    const uint64_t v2[kScanCols] = {scan_pair(v.x, v.x), scan_pair(v.y, v.y), scan_pair(v.z, v.z), scan_pair(v.w, v.w)};
    uint64_t acc[kScanCols] = {0, 0, 0, 0};
#pragma unroll
    for (int i = 0; i < ROWS / 4; ++i) {
      const int at = i * (LANES * 4) + g * 4;
      const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(b + at);
      const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(b + C::kRows + at);
      const ulonglong2 w = ONE ? make_ulonglong2(one, one) : *reinterpret_cast<const ulonglong2*>(b + (ONE ? 0 : 2 * C::kRows) + at);
#pragma unroll
      for (int c = 0; c < kScanCols; ++c) {
        acc[c] = scan_fma(r.x, s2[2 * i][c], acc[c]);
        acc[c] = scan_fma(r.y, s2[2 * i + 1][c], acc[c]);
        s2[2 * i][c] = scan_fma(w.x, s2[2 * i][c], scan_mul(k.x, v2[c]));
        s2[2 * i + 1][c] = scan_fma(w.y, s2[2 * i + 1][c], scan_mul(k.y, v2[c]));
      }
    }
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
      float lo, hi;
      scan_unpair(acc[c], lo, hi);
      o[c] = lo + hi;
    }
  };
  const bool up = g & (LANES / 2), up2 = g & (LANES / 4);
  auto fold = [&](const float (&o)[kScanCols]) {
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
    const int st = ch % kScanStages;
    ok = mbar_wait(full + st, uint32_t(ch / kScanStages) & 1u, &gave_up) && ok;
    const float* buf = smem + st * C::kStage;
    const float* buf_col = buf + C::kChunk * C::kRec;
    const int n = min(C::kChunk, len - ch * C::kChunk);
    float* oc = op + size_t(ch) * C::kChunk * p.ld_out;
    // groups of TU tokens; a group's sums are taken beside the next group's arithmetic
    constexpr int TU = 4;
    auto put = [&](int t, const float (&o)[TU][kScanCols]) {
      float sum[TU];
#pragma unroll
      for (int q = 0; q < TU; ++q) sum[q] = fold(o[q]);
      if (writer) {
#pragma unroll
        for (int q = 0; q < TU; ++q) {
          const float* bc = buf_col + (t + q) * C::kCol;
          oc[size_t(t + q) * p.ld_out] = fmaf(bc[at_own], bc[c0 + mine], ONE ? bc[C::kCols] * sum[q] : sum[q]);
        }
      }
    };
    int t = 0;
    if (n >= TU) {
      float o[TU][kScanCols];
#pragma unroll
      for (int q = 0; q < TU; ++q) token(buf + q * C::kRec, buf_col + q * C::kCol, o[q]);
      for (t = TU; t + TU <= n; t += TU) {
        float next[TU][kScanCols];
#pragma unroll
        for (int q = 0; q < TU; ++q) token(buf + (t + q) * C::kRec, buf_col + (t + q) * C::kCol, next[q]);
        put(t - TU, o);
#pragma unroll
        for (int q = 0; q < TU; ++q)
#pragma unroll
          for (int c = 0; c < kScanCols; ++c) o[q][c] = next[q][c];
      }
      put(t - TU, o);
    }
    for (; t < n; ++t) {
      const float* bc = buf_col + t * C::kCol;
      float o[kScanCols];
      token(buf + t * C::kRec, bc, o);
      const float sum = fold(o);
      if (writer) oc[size_t(t) * p.ld_out] = fmaf(bc[at_own], bc[c0 + mine], ONE ? bc[C::kCols] * sum : sum);
    }
    __syncthreads();                                 // the stage has been read
    if (threadIdx.x == 0 && ch + kScanStages < chunks) issue(ch + kScanStages);
  }
  if (!ok) {                                         // let the copies in flight land, as far as that goes
    for (int i = 0; threadIdx.x == 0 && i < kScanStages; ++i)
      for (uint32_t k = 0; k < (1u << 16); ++k)
        if (mbar_try_wait(full + i, uint32_t((chunks - 1 - (chunks - 1 - i) % kScanStages) / kScanStages) & 1u)) break;
    if (p.status) atomicExch(p.status, int(kStatusMbarTimeout));
  }
#pragma unroll
  for (int i = 0; i < ROWS / 2; ++i)
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
      const int r0 = g * ROWS + 2 * i, col = col0 + c0 + c;
      float lo, hi;
      scan_unpair(s2[i][c], lo, hi);
      if (col < dim) {
        if (r0 < n_rows) sp[size_t(r0) * dim + col] = lo;
        if (r0 + 1 < n_rows) sp[size_t(r0 + 1) * dim + col] = hi;
      }
    }
  if (p.prev && blockIdx.x == 0 && h == 0) {
    const float* last = p.x + size_t(row0 + len - 1) * p.ldx;
    float* keep = p.prev + size_t(slot) * p.stride;
    for (int i = threadIdx.x; i < p.ldx; i += TH) keep[i] = last[i];
  }
}

// The scan over records that are in place, made for column blocks of th threads.
template <int ROWS, int LANES, bool ONE>
static int launch_scan(const ScanParams& p, int th, int n_segs, int pdl, cudaStream_t st) {
  auto go = [&](auto threads) -> int {
    constexpr int TH = decltype(threads)::value;
    using C = ScanCfg<ROWS, LANES, ONE, TH>;
    auto kern = scan_kernel<ROWS, LANES, ONE, TH>;
    RB_CHECK(set_max_smem(kern, C::kSmem));
    return launch(kern, dim3((p.d + C::kCols - 1) / C::kCols, p.H, n_segs), dim3(TH), C::kSmem, st, pdl != 0, p);
  };
  if (th == 256) return go(std::integral_constant<int, 256>{});
  if (th == 128) return go(std::integral_constant<int, 128>{});
  return go(std::integral_constant<int, 64>{});
}
// Records and scan of heads with a decay per row. rec: scratch, 16-byte aligned.
template <class IN, int ROWS, int LANES>
static int launch_row_scan(const IN& in, ScanParams p, float* rec, int n_segs, int pdl, cudaStream_t st) {
  constexpr int kRows = ROWS * LANES, LU = kRows >= 128 ? 32 : kRows / 4;
  const long long threads = 1LL * p.rows * p.H * LU;
  if (threads > 0x7fffffffLL) return -2;
  const int th = scan_threads(LANES, p.d, p.H, n_segs);
  float* col = rec + size_t(p.H) * p.rows * 3 * kRows;
  const int rc = launch(scan_prepare_kernel<IN, ROWS, LANES, LU>, dim3(unsigned((threads + kRowThreads - 1) / kRowThreads)),
                        dim3(kRowThreads), 0, st, pdl != 0, in, rec, col, p.rows, p.H, p.d, scan_col_shift(LANES, th));
  if (rc) return rc;
  p.rec = rec; p.col = col; p.per = 1;
  return launch_scan<ROWS, LANES, false>(p, th, n_segs, pdl, st);
}

constexpr int kScanMaxRows = 256;
// The instance for a state of n rows: CALL(ROWS, LANES).
#define RB_SCAN_DISPATCH(n_, CALL)        \
  do {                                    \
    if ((n_) <= 16) CALL(4, 4);           \
    if ((n_) <= 32) CALL(4, 8);           \
    if ((n_) <= 64) CALL(4, 16);          \
    if ((n_) <= 128) CALL(4, 32);         \
    if ((n_) <= kScanMaxRows) CALL(8, 32); \
  } while (0)

}  // namespace rb
