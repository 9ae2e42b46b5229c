// Row-wise kernels of parallel-block decoders with an fp32 residual stream: embedding with a scale,
// RMSNorm of fp32 rows, and the step between the merged input projection and attention (RMS norm
// over the whole query / key projection, then queries to a buffer and keys / values to their
// pages). Activations are bf16 (serving) or fp32 (the all-32-bit mode); sums of squares and the
// residual are fp32 in both.
//
// Row widths are padded to multiples of eight elements so that tensor maps and 16-byte accesses
// always apply; the kernels keep the padding at zero.
#include "../common/launch.cuh"
#include "../common/rows.cuh"

namespace rb {

// x[t, :] = table[ids[t], :] * scale; columns D .. ldx-1 are zeroed.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
embed_scaled_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ x,
                    float scale, int D, int ldx, int vocab) {
  pdl_launch_dependents();
  pdl_wait();
  int id = ids[blockIdx.x];
  (void)RB_BOUNDS(id, vocab);
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + size_t(id) * D;
  float* dst = x + size_t(blockIdx.x) * ldx;
  for (int i = threadIdx.x; i < ldx; i += kRowThreads) dst[i] = i < D ? to_f32(src[i]) * scale : 0.f;
}

// out[t, :] = x[t, :] / sqrt(mean over D of x^2 + eps) * w. x and w have ldx columns, zero from D on.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
rms_norm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ out,
                    int D, int ldx, float eps) {
  constexpr int kKeep = 4;                 // chunks of eight a thread keeps in registers
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const float* row = x + size_t(blockIdx.x) * ldx;
  const int chunks = ldx >> 3;
  float f[kKeep][8];
  float ssq = 0.f;
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) {
      load8(row + c * 8, f[u]);
#pragma unroll
      for (int i = 0; i < 8; ++i) ssq += f[u][i] * f[u][i];
    }
  }
  for (int c = kKeep * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float g[8];
    load8(row + c * 8, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += g[i] * g[i];
  }
  ssq = row_block_sum(ssq, red);
  const float inv = 1.f / sqrtf(ssq / float(D) + eps);
  T* dst = out + size_t(blockIdx.x) * ldx;
  auto put = [&](int c, float (&v)[8]) {
    float g[8];
    load8(w + c * 8, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = v[i] * inv * g[i];
    store8(dst + c * 8, v);
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) put(c, f[u]);
  }
  for (int c = kKeep * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float g[8];
    load8(row + c * 8, g);
    put(c, g);
  }
}

// raw row t = [q: Hq*dim | k: Hkv*dim | v: Hkv*vdim] (row stride ldraw). Queries and keys are each
// divided by the root mean square of their whole projection and multiplied by q_w / k_w; q goes to
// q_out [T, Hq, dkp], k and v to the token's slot of its sequence's pages
// ([blocks, Hkv, page, dkp] and [.., dvp]). dkp / dvp: dim / vdim rounded up to eight.
template <class TR, class T>
__global__ void __launch_bounds__(kRowThreads)
qk_norm_append_kernel(const TR* __restrict__ raw, int ldraw, const float* __restrict__ q_w,
                      const float* __restrict__ k_w, float eps, T* __restrict__ q_out,
                      T* __restrict__ k_cache, T* __restrict__ v_cache,
                      const int* __restrict__ block_table, const int* __restrict__ positions,
                      const int* __restrict__ token_seq, int Hq, int Hkv, int dim, int vdim, int dkp,
                      int dvp, int max_blocks, int page) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const TR* row = raw + size_t(t) * ldraw;
  const int nq = Hq * dim, nk = Hkv * dim;
  const bool vec = (dim % 8 == 0) && (vdim % 8 == 0) && (ldraw % 8 == 0);
  float sq = 0.f, sk = 0.f;
  if (vec) {
    for (int c = threadIdx.x; c < (nq + nk) >> 3; c += kRowThreads) {
      float f[8];
      load8(row + c * 8, f);
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) s += f[i] * f[i];
      if (c * 8 < nq) sq += s; else sk += s;
    }
  } else {
    for (int i = threadIdx.x; i < nq + nk; i += kRowThreads) {
      const float v = to_f32(row[i]);
      if (i < nq) sq += v * v; else sk += v * v;
    }
  }
  sq = row_block_sum(sq, red);
  sk = row_block_sum(sk, red);
  const float iq = 1.f / sqrtf(sq / float(nq) + eps), ik = 1.f / sqrtf(sk / float(nk) + eps);
  const int pos = positions[t];
  const int seq = token_seq ? token_seq[t] : t;
  const bool in_table = RB_BOUNDS(pos / page, max_blocks);
  const int blk = in_table ? block_table[size_t(seq) * max_blocks + pos / page] : 0;
  const int slot = pos % page;
  const int uk = dkp >> 3, uv = dvp >> 3;             // eight-element units per head
  const int units = (Hq + Hkv) * uk + Hkv * uv;
  for (int u = threadIdx.x; u < units; u += kRowThreads) {
    const bool is_v = u >= (Hq + Hkv) * uk;
    const int per = is_v ? uv : uk, width = is_v ? vdim : dim;
    const int r = is_v ? u - (Hq + Hkv) * uk : u;
    const int head = r / per, d0 = (r - head * per) * 8;
    const int src = (is_v ? nq + nk : 0) + head * width + d0;
    float f[8];
    if (vec) {
      load8(row + src, f);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = d0 + i < width ? to_f32(row[src + i]) : 0.f;
    }
    if (!is_v) {
      const bool is_q = head < Hq;
      const float inv = is_q ? iq : ik;
      const float* w = is_q ? q_w + src : k_w + (src - nq);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = d0 + i < width ? f[i] * inv * w[i] : 0.f;
      if (is_q) {
        store8(q_out + (size_t(t) * Hq + head) * dkp + d0, f);
      } else if (in_table) {
        store8(k_cache + ((size_t(blk) * Hkv + (head - Hq)) * page + slot) * dkp + d0, f);
      }
    } else if (in_table) {
      store8(v_cache + ((size_t(blk) * Hkv + head) * page + slot) * dvp + d0, f);
    }
  }
}

}  // namespace rb

using namespace rb;
RB_BOUNDS_REGISTER("parallel_rows.cu")

// f32: the table is fp32, else bf16. x is always fp32 [T, ldx], ldx >= D.
extern "C" int rmlx_embed_scaled(const void* table, const int* ids, float* x, float scale, int T, int D,
                                 int ldx, int vocab, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || vocab < 1) return -2;
  if (f32)
    return launch(embed_scaled_kernel<float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0,
                  static_cast<const float*>(table), ids, x, scale, D, ldx, vocab);
  return launch(embed_scaled_kernel<__nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(table), ids, x, scale, D, ldx, vocab);
}

// x fp32 [T, ldx] (zero from column D on), w fp32 [ldx]; out [T, ldx] fp32 (f32) or bf16.
extern "C" int rmlx_rms_norm_f32(const float* x, const float* w, void* out, int T, int D, int ldx,
                                 float eps, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || ldx % 8) return -2;
  if (f32)
    return launch(rms_norm_f32_kernel<float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, x, w,
                  static_cast<float*>(out), D, ldx, eps);
  return launch(rms_norm_f32_kernel<__nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, x, w,
                static_cast<__nv_bfloat16*>(out), D, ldx, eps);
}

// f32: raw, q_out and the caches are fp32, else bf16. token_seq: row of the block table per token
// (null: token t belongs to row t).
extern "C" int rmlx_qk_norm_append(const void* raw, int ldraw, const float* q_w, const float* k_w,
                                   float eps, void* q_out, void* k_cache, void* v_cache,
                                   const int* block_table, const int* positions, const int* token_seq,
                                   int T, int Hq, int Hkv, int dim, int vdim, int dkp, int dvp,
                                   int max_blocks, int page, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || Hq < 1 || Hkv < 1 || dim < 1 || vdim < 1 || dkp % 8 || dvp % 8 || dkp < dim ||
      dvp < vdim || ldraw < (Hq + Hkv) * dim + Hkv * vdim)
    return -2;
  if (f32)
    return launch(qk_norm_append_kernel<float, float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0,
                  static_cast<const float*>(raw), ldraw, q_w, k_w, eps, static_cast<float*>(q_out),
                  static_cast<float*>(k_cache), static_cast<float*>(v_cache), block_table, positions,
                  token_seq, Hq, Hkv, dim, vdim, dkp, dvp, max_blocks, page);
  return launch(qk_norm_append_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st,
                pdl != 0, static_cast<const __nv_bfloat16*>(raw), ldraw, q_w, k_w, eps,
                static_cast<__nv_bfloat16*>(q_out), static_cast<__nv_bfloat16*>(k_cache),
                static_cast<__nv_bfloat16*>(v_cache), block_table, positions, token_seq, Hq, Hkv, dim,
                vdim, dkp, dvp, max_blocks, page);
}
