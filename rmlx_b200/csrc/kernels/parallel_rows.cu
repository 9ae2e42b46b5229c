// Row-wise kernels of parallel-block decoders with an fp32 residual stream: embedding with a scale,
// RMSNorm of fp32 rows, and the step between the merged input projection and attention (RMS norm
// over the whole query / key projection, then queries to a buffer and keys / values to their
// pages). Activations are bf16 (serving) or fp32 (the all-32-bit mode); sums of squares and the
// residual are fp32 in both.
//
// Row widths are padded to multiples of eight elements so that tensor maps and 16-byte accesses
// always apply; the kernels keep the padding at zero.
#include "../common/ptx.cuh"
#include "../common/launch.cuh"

namespace rb {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Eight consecutive elements, 16-byte aligned.
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  f[0] = bf16lo(v.x); f[1] = bf16hi(v.x); f[2] = bf16lo(v.y); f[3] = bf16hi(v.y);
  f[4] = bf16lo(v.z); f[5] = bf16hi(v.z); f[6] = bf16lo(v.w); f[7] = bf16hi(v.w);
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 o;
  o.x = pack_bf16(f[0], f[1]); o.y = pack_bf16(f[2], f[3]);
  o.z = pack_bf16(f[4], f[5]); o.w = pack_bf16(f[6], f[7]);
  *reinterpret_cast<uint4*>(p) = o;
}

constexpr int kRowThreads = 256;

__device__ __forceinline__ float row_block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = (threadIdx.x & 31) < kRowThreads / 32 ? red[threadIdx.x & 31] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

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
