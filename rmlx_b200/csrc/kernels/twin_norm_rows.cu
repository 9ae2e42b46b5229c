// Row-wise kernels of decoders whose mixer and feed-forward read the same residual row through norms of their own,
// x <- x + f(norm1(x)) + g(norm2(x)), x in fp32:
//
//   twin_norm           the residual, with the routed experts' weighted rows added if there are any, and both norms
//                       of it in one pass
//   rows_norm           RMS norm of a slice of a projection's rows (the latent that queries go through)
//   rotary_norm_append  bias, rotation (of halves or of neighbours), unweighted per-head norm of queries and keys (or
//                       none), cache append; heads of one or of two maps
//
// Activations are bf16 (serving) or fp32 (the all-32-bit mode); norms, angles and the residual are fp32 in both.
#include "../common/launch.cuh"
#include "../common/row_sources.cuh"
#include "../common/rows.cuh"

namespace rb {

struct NoSource {
  __device__ __forceinline__ void prepare(int) {}
};

// x[t] += source; h1[t] = x[t] / rms * w1, h2[t] = x[t] / rms * w2 (h1, h2 may be null). Columns past D are zero.
template <class SRC, bool ADD, class T>
__global__ void __launch_bounds__(kRowThreads)
twin_norm_kernel(SRC src, float* __restrict__ x, const float* __restrict__ w1, T* __restrict__ h1,
                 const float* __restrict__ w2, T* __restrict__ h2, float eps, int D, int ldx) {
  constexpr int kKeep = 4;                 // chunks of eight a thread keeps in registers
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, chunks = ldx >> 3;
  float* row = x + size_t(t) * ldx;
  src.prepare(t);
  float f[kKeep][8], ssq = 0.f;
  auto take = [&](int c, float (&a)[8]) {
    load8(row + c * 8, a);
    if constexpr (ADD) {
      float b[8];
      src.load(t, c, a, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] = c * 8 + i < D ? a[i] + b[i] : 0.f;
      store8(row + c * 8, a);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += a[i] * a[i];
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) take(c, f[u]);
  }
  for (int c = kKeep * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float a[8];
    take(c, a);
  }
  if (!h1 && !h2) return;
  ssq = row_block_sum(ssq, red);
  const float inv = 1.f / sqrtf(ssq / float(D) + eps);
  auto put = [&](int c, const float (&a)[8]) {
    float g[8], o[8];
    if (h1) {
      load8(w1 + c * 8, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) o[i] = a[i] * inv * g[i];
      store8(h1 + size_t(t) * ldx + c * 8, o);
    }
    if (h2) {
      load8(w2 + c * 8, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) o[i] = a[i] * inv * g[i];
      store8(h2 + size_t(t) * ldx + c * 8, o);
    }
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) put(c, f[u]);
  }
  for (int c = kKeep * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float a[8];
    load8(row + c * 8, a);                 // (this thread wrote them)
    put(c, a);
  }
}

// out[t, :D] = in[t, :D] / rms * w, zeros up to ldo. in rows ld apart.
template <class TR, class T>
__global__ void __launch_bounds__(kRowThreads)
rows_norm_kernel(const TR* __restrict__ in, int ld, const float* __restrict__ w, float eps, T* __restrict__ out, int ldo, int D) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const TR* row = in + size_t(blockIdx.x) * ld;
  const bool vec = D % 8 == 0 && ld % 8 == 0;
  float ssq = 0.f;
  for (int c = threadIdx.x; c < ldo >> 3; c += kRowThreads) {
    float f[8];
    load8_upto(row + c * 8, D - c * 8, vec, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += f[i] * f[i];
  }
  ssq = row_block_sum(ssq, red);
  const float inv = 1.f / sqrtf(ssq / float(D) + eps);
  for (int c = threadIdx.x; c < ldo >> 3; c += kRowThreads) {
    float f[8];
    load8_upto(row + c * 8, D - c * 8, vec, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = c * 8 + i < D ? f[i] * inv * w[c * 8 + i] : 0.f;
    store8(out + size_t(blockIdx.x) * ldo + c * 8, f);
  }
}

// raw row t = [q: Hq*dim | k: Hkv*dim | v: Hkv*vdim | ..], bias (fp32, the same layout) or null. Value i of a query
// or key head turns with value i + dims / 2 by position * inv_freq[i], cos and sin times `grow`; then every query
// and key head is divided by its own root mean square. q goes to q_out [T, Hq, dkp], k and v to the token's slot of
// its sequence's pages. One block per token, or (grid y) several; L lanes per head. neighbours: values 2 i and 2 i + 1 turn
// together instead. norm 0: no division. maps 2 (differential attention): every query and key head is two of `dim`
// values, side by side also in q_out and in a key's cache row; each part turns and is normed on its own.
template <class TR, class T, int L>
__global__ void __launch_bounds__(kRowThreads)
rotary_norm_append_kernel(const TR* __restrict__ raw, int ldraw, const float* __restrict__ bias,
                          const float* __restrict__ inv_freq, int dims, float grow, float eps, T* __restrict__ q_out,
                          T* __restrict__ k_cache, T* __restrict__ v_cache, const int* __restrict__ block_table,
                          const int* __restrict__ positions, const int* __restrict__ token_seq, int Hq, int Hkv, int dim,
                          int vdim, int dkp, int dvp, int max_blocks, int page, int neighbours, int norm, int maps) {
  extern __shared__ __align__(16) float trig[];          // cos [dims / 2], sin [dims / 2]
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, pos = positions[t], half = dims / 2;
  for (int i = threadIdx.x; i < half; i += kRowThreads) {
    float s, c;
    rotary_sincos(pos, inv_freq[i], s, c);
    trig[i] = c * grow;
    trig[half + i] = s * grow;
  }
  __syncthreads();
  const TR* row = raw + size_t(t) * ldraw;
  const int seq = token_seq ? token_seq[t] : t;
  const bool in_table = RB_BOUNDS(pos / page, max_blocks);
  const int blk = in_table ? block_table[size_t(seq) * max_blocks + pos / page] : 0;
  const int nq = Hq * maps, nk = Hkv * maps, per = nq + nk + Hkv, lane = threadIdx.x % L;
  for (int r0 = blockIdx.y * (kRowThreads / L); r0 < per; r0 += gridDim.y * (kRowThreads / L)) {
    const int r = r0 + threadIdx.x / L;
    const bool live = r < per;                         // the lanes of a warp stay together for the sums
    const bool is_q = r < nq, is_v = r >= nq + nk;
    const int head = is_q ? r : is_v ? r - nq - nk : r - nq;
    const int width = !live ? 0 : is_v ? vdim : dim, padded = is_v ? dvp : dkp;
    const int src0 = !live ? 0 : is_v ? (nq + nk) * dim + head * vdim : r * dim;
    const TR* src = row + src0;
    const float* bs = bias ? bias + src0 : nullptr;
    const bool vec = width % 8 == 0 && src0 % 8 == 0 && ldraw % 8 == 0;
    const bool pairs = vec && half % 8 == 0;           // eight values turn with eight
    auto value = [&](int d) { return to_f32(src[d]) + (bs ? bs[d] : 0.f); };
    auto biased = [&](int d0, float (&f)[8]) {
      load8_upto(src + d0, width - d0, vec && d0 < width, f);
      if (!bs) return;
      if (vec && d0 < width) {
        float g[8];
        load8(bs + d0, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += g[i];
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += d0 + i < width ? bs[d0 + i] : 0.f;
      }
    };
    auto load = [&](int d0, float (&f)[8]) {
      biased(d0, f);
      if (is_v || d0 >= dims || !live) return;
      if (neighbours) {
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
          if (d0 + i >= dims) break;
          const float c = trig[(d0 + i) >> 1], s = trig[half + ((d0 + i) >> 1)], u = f[i], v = f[i + 1];
          f[i] = u * c - v * s;
          f[i + 1] = v * c + u * s;
        }
      } else if (pairs) {
        const bool low = d0 < half;
        const int j = low ? d0 : d0 - half;
        float g[8], cs[8], sn[8];
        biased(low ? d0 + half : j, g);
        load8(trig + j, cs);
        load8(trig + half + j, sn);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = fmaf(f[i], cs[i], low ? -g[i] * sn[i] : g[i] * sn[i]);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int d = d0 + i;
          if (d < half) f[i] = f[i] * trig[d] - value(d + half) * trig[half + d];
          else if (d < dims) f[i] = f[i] * trig[d - half] + value(d - half) * trig[d];
        }
      }
    };
    T* dst = nullptr;
    if (is_q) dst = q_out + (size_t(t) * nq + head) * dkp;
    else if (in_table && is_v) dst = v_cache + ((size_t(blk) * Hkv + head) * page + pos % page) * dvp;
    else if (in_table) dst = k_cache + (((size_t(blk) * Hkv + head / maps) * page + pos % page) * maps + head % maps) * dkp;
    float first[8], ssq = 0.f;
    load(lane * 8, first);
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += first[i] * first[i];
    for (int d0 = (lane + L) * 8; d0 < width; d0 += L * 8) {
      float f[8];
      load(d0, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) ssq += f[i] * f[i];
    }
    ssq = group_sum<L>(ssq);
    if (!live || !dst) continue;
    const float inv = is_v || !norm ? 1.f : 1.f / sqrtf(ssq / float(dim) + eps);
    for (int d0 = lane * 8; d0 < padded; d0 += L * 8) {
      float f[8];
      if (d0 == lane * 8) {
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = first[i];
      } else {
        load(d0, f);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= inv;
      store8(dst + d0, f);
    }
  }
}

// The form with neighbours, no norm and no bias: chunks of eight turn on their own, so a block deals those of TOKENS
// tokens to its threads in a row. Source rows, widths and strides are multiples of eight values.
template <class TR, class T, int TOKENS>
__global__ void __launch_bounds__(kRowThreads)
rotary_append_kernel(const TR* __restrict__ raw, int ldraw, const float* __restrict__ inv_freq, int dims, float grow,
                     T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache, const int* __restrict__ block_table,
                     const int* __restrict__ positions, const int* __restrict__ token_seq, int rows, int Hq, int Hkv, int dim,
                     int vdim, int max_blocks, int page, int maps) {
  extern __shared__ __align__(16) float trig[];          // per token: cos [dims / 2], sin [dims / 2]
  __shared__ int s_blk[TOKENS], s_off[TOKENS];
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * TOKENS, n = min(TOKENS, rows - t0), half = dims / 2;
  for (int i = threadIdx.x; i < n * half; i += kRowThreads) {
    const int a = i / half, j = i - a * half;
    float s, c;
    rotary_sincos(positions[t0 + a], inv_freq[j], s, c);
    trig[a * dims + j] = c * grow;
    trig[a * dims + half + j] = s * grow;
  }
  if (threadIdx.x < n) {
    const int t = t0 + threadIdx.x, pos = positions[t];
    const bool in_table = RB_BOUNDS(pos / page, max_blocks);
    s_blk[threadIdx.x] = in_table ? block_table[size_t(token_seq ? token_seq[t] : t) * max_blocks + pos / page] : -1;
    s_off[threadIdx.x] = pos % page;
  }
  __syncthreads();
  const int nq = Hq * maps * dim, nk = Hkv * maps * dim, chunks = (nq + nk + Hkv * vdim) >> 3;
  for (int a = 0; a < n; ++a) {
    const TR* row = raw + size_t(t0 + a) * ldraw;
    const float* cs = trig + a * dims;
#pragma unroll 4
    for (int c = threadIdx.x; c < chunks; c += kRowThreads) {
      const int at = c * 8;
      float f[8];
      load8(row + at, f);
      T* dst;
      if (at < nq + nk) {
        const int r = at / dim, d0 = at - r * dim;         // part (head, map) and place in it
        if (d0 < dims) {
#pragma unroll
          for (int i = 0; i < 8; i += 2) {
            if (d0 + i >= dims) break;
            const float co = cs[(d0 + i) >> 1], si = cs[half + ((d0 + i) >> 1)], u = f[i], v = f[i + 1];
            f[i] = u * co - v * si;
            f[i + 1] = v * co + u * si;
          }
        }
        if (at < nq) {
          dst = q_out + size_t(t0 + a) * nq + at;
        } else {
          if (s_blk[a] < 0) continue;
          const int k = r - Hq * maps;
          dst = k_cache + (((size_t(s_blk[a]) * Hkv + k / maps) * page + s_off[a]) * maps + k % maps) * dim + d0;
        }
      } else {
        if (s_blk[a] < 0) continue;
        const int v = at - nq - nk, g = v / vdim;
        dst = v_cache + ((size_t(s_blk[a]) * Hkv + g) * page + s_off[a]) * vdim + v - g * vdim;
      }
      store8(dst, f);
    }
  }
}

template <class SRC, bool ADD>
static int launch_twin(SRC src, float* x, const float* w1, void* h1, const float* w2, void* h2, float eps, int T, int D, int ldx,
                       int f32, int pdl, cudaStream_t st) {
  if (f32)
    return launch(twin_norm_kernel<SRC, ADD, float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, src, x, w1,
                  static_cast<float*>(h1), w2, static_cast<float*>(h2), eps, D, ldx);
  return launch(twin_norm_kernel<SRC, ADD, __nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, src, x, w1,
                static_cast<__nv_bfloat16*>(h1), w2, static_cast<__nv_bfloat16*>(h2), eps, D, ldx);
}

}  // namespace rb

using namespace rb;
RB_BOUNDS_REGISTER("twin_norm_rows.cu")

// x fp32 [T, ldx]; w1, w2 fp32 [ldx]; h1, h2 [T, ldx] fp32 (f32) or bf16, or null. y (null: nothing is added):
// expert rows [rows, ldy] in the compute type, row_of_pair / weights [T, top_k]. ldx and ldy multiples of eight.
extern "C" int rmlx_twin_norm(float* x, const void* y, int ldy, const int* row_of_pair, const float* weights, int top_k,
                              const float* w1, void* h1, const float* w2, void* h2, float eps, int T, int D, int ldx, int f32,
                              int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || ldx % 8 || (h1 && !w1) || (h2 && !w2)) return -2;
  if (!y) return launch_twin<NoSource, false>(NoSource{}, x, w1, h1, w2, h2, eps, T, D, ldx, f32, pdl, st);
  if (ldy % 8 || ldy < ldx || top_k < 1 || !row_of_pair || !weights) return -2;
  if (f32)
    return launch_twin<ExpertSource<float>, true>(
        ExpertSource<float>{static_cast<const float*>(y), ldy, row_of_pair, weights, nullptr, top_k}, x, w1, h1, w2, h2, eps, T, D,
        ldx, f32, pdl, st);
  return launch_twin<ExpertSource<__nv_bfloat16>, true>(
      ExpertSource<__nv_bfloat16>{static_cast<const __nv_bfloat16*>(y), ldy, row_of_pair, weights, nullptr, top_k}, x, w1, h1, w2,
      h2, eps, T, D, ldx, f32, pdl, st);
}

// in [T, ld] fp32 (in_f32) or bf16, out [T, ldo] fp32 (f32) or bf16; ldo a multiple of eight; w fp32 [D].
extern "C" int rmlx_rows_norm(const void* in, int ld, int in_f32, const float* w, float eps, void* out, int ldo, int T, int D,
                              int f32, int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ld < D || ldo < D || ldo % 8 || (f32 && !in_f32)) return -2;
#define RB_RN(TR_, T_)                                                                                               \
  return launch(rows_norm_kernel<TR_, T_>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, static_cast<const TR_*>(in), ld, w, \
                eps, static_cast<T_*>(out), ldo, D)
  if (f32) RB_RN(float, float);
  if (in_f32) RB_RN(float, __nv_bfloat16);
  RB_RN(__nv_bfloat16, __nv_bfloat16);
#undef RB_RN
}

// f32: q_out and the caches are fp32, else bf16; raw_f32: raw is fp32. dims: how many of a head's values turn (even,
// <= dim); inv_freq fp32 [dims / 2]. maps 2: q_out [T, Hq, 2, dkp], key rows of 2 dkp values.
extern "C" int rmlx_rotary_norm_append(const void* raw, int ldraw, int raw_f32, const float* bias, const float* inv_freq,
                                       int dims, float grow, float eps, void* q_out, void* k_cache, void* v_cache,
                                       const int* block_table, const int* positions, const int* token_seq, int T, int Hq,
                                       int Hkv, int dim, int vdim, int dkp, int dvp, int max_blocks, int page, int neighbours,
                                       int norm, int maps, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || Hq < 1 || Hkv < 1 || dim < 1 || vdim < 1 || dkp % 8 || dvp % 8 || dkp < dim || dvp < vdim || dims < 0 ||
      dims % 2 || dims > dim || maps < 1 || maps > 2 || ldraw < (Hq + Hkv) * maps * dim + Hkv * vdim || (f32 && !raw_f32))
    return -2;
  const size_t smem = size_t(dims) * sizeof(float);
  if (smem > 32 * 1024) return -2;
  if (neighbours && !norm && !bias && dim % 8 == 0 && vdim % 8 == 0 && ldraw % 8 == 0 && dkp == dim && dvp == vdim && dims <= 2048) {
    const int per = T >= 8 * sm_count() ? 4 : 1;          // tokens a block
#define RB_RF(TR_, T_)                                                                                                        \
  return launch(per == 4 ? rotary_append_kernel<TR_, T_, 4> : rotary_append_kernel<TR_, T_, 1>, dim3((T + per - 1) / per),    \
                dim3(kRowThreads), smem * per, st, pdl != 0, static_cast<const TR_*>(raw), ldraw, inv_freq, dims, grow,       \
                static_cast<T_*>(q_out), static_cast<T_*>(k_cache), static_cast<T_*>(v_cache), block_table, positions,        \
                token_seq, T, Hq, Hkv, dim, vdim, max_blocks, page, maps)
    if (f32) RB_RF(float, float);
    if (raw_f32) RB_RF(float, __nv_bfloat16);
    RB_RF(__nv_bfloat16, __nv_bfloat16);
#undef RB_RF
  }
  const int widest = dkp > dvp ? dkp : dvp, lanes = widest <= 64 ? 8 : widest <= 128 ? 16 : 32;
  const int per_block = kRowThreads / lanes, blocks = ((Hq + Hkv) * maps + Hkv + per_block - 1) / per_block;
  const dim3 grid(T, T >= 64 ? 1 : blocks);           // few tokens: several blocks share one
#define RB_RA_L(TR_, T_, L_)                                                                                            \
  return launch(rotary_norm_append_kernel<TR_, T_, L_>, grid, dim3(kRowThreads), smem, st, pdl != 0,                    \
                static_cast<const TR_*>(raw), ldraw, bias, inv_freq, dims, grow, eps, static_cast<T_*>(q_out),          \
                static_cast<T_*>(k_cache), static_cast<T_*>(v_cache), block_table, positions, token_seq, Hq, Hkv, dim, vdim, \
                dkp, dvp, max_blocks, page, neighbours, norm, maps)
#define RB_RA(TR_, T_)                     \
  {                                        \
    if (lanes == 8) RB_RA_L(TR_, T_, 8);   \
    if (lanes == 16) RB_RA_L(TR_, T_, 16); \
    RB_RA_L(TR_, T_, 32);                  \
  }
  if (f32) RB_RA(float, float);
  if (raw_f32) RB_RA(float, __nv_bfloat16);
  RB_RA(__nv_bfloat16, __nv_bfloat16);
#undef RB_RA
#undef RB_RA_L
}
