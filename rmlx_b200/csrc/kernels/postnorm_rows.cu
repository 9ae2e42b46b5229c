// Row-wise kernels of decoders whose sublayers read the residual stream itself and whose norms sit on
// the sublayers' outputs (x <- x + norm(f(x)), x in fp32): embedding with a norm, the output norm with
// the residual sum, the steps between the input projections and the two kinds of attention (per-head
// query / key norm; latent norm and rotation) with the cache append, and the gated activation.
//
// Activations are bf16 (serving) or fp32 (the all-32-bit mode); norms, rotations and the residual are
// fp32 in both. Residual rows are padded to a multiple of eight; the padding stays zero.
#include "../common/gated.cuh"
#include "../common/launch.cuh"
#include "../common/row_sources.cuh"
#include "../common/rows.cuh"

namespace rb {

// x[t] = table[ids[t]] / rms * w (fp32), h[t] = x[t] in the compute type.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
embed_norm_kernel(const T* __restrict__ table, const int* __restrict__ ids, const float* __restrict__ w,
                  float eps, float* __restrict__ x, T* __restrict__ h, int D, int ldx, int vocab) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  int id = ids[blockIdx.x];
  (void)RB_BOUNDS(id, vocab);
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + size_t(id) * D;
  float ssq = 0.f;
  for (int i = threadIdx.x; i < D; i += kRowThreads) { const float v = to_f32(src[i]); ssq += v * v; }
  ssq = row_block_sum(ssq, red);
  const float inv = 1.f / sqrtf(ssq / float(D) + eps);
  const size_t at = size_t(blockIdx.x) * ldx;
  for (int i = threadIdx.x; i < ldx; i += kRowThreads) {
    const float v = i < D ? to_f32(src[i]) * inv * w[i] : 0.f;
    x[at + i] = v;
    h[at + i] = from_f32<T>(v);
  }
}

// x[t] += y[t] / rms(y[t]) * w, h[t] = x[t] in the compute type (h may be null).
template <class SRC, class T>
__global__ void __launch_bounds__(kRowThreads)
post_norm_add_kernel(SRC src, const float* __restrict__ w, float eps, float* __restrict__ x, T* __restrict__ h,
                     int D, int ldx) {
  constexpr int kKeep = 2;                 // chunks of eight a thread keeps in registers
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  float* row = x + size_t(t) * ldx;
  const int chunks = ldx >> 3;
  src.prepare(t);
  float fy[kKeep][8], fx[kKeep][8];
  float ssq = 0.f;
  // columns past D are zero in every source but experts padded for the tensor cores, whose extra
  // columns lie past ldx
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) {
      load8(row + c * 8, fx[u]);
      src.load(t, c, fx[u], fy[u]);
#pragma unroll
      for (int i = 0; i < 8; ++i) ssq += c * 8 + i < D ? fy[u][i] * fy[u][i] : 0.f;
    }
  }
  for (int c = kKeep * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float a[8], b[8];
    load8(row + c * 8, a);
    src.load(t, c, a, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += c * 8 + i < D ? b[i] * b[i] : 0.f;
  }
  ssq = row_block_sum(ssq, red);
  const float inv = 1.f / sqrtf(ssq / float(D) + eps);
  auto put = [&](int c, float (&a)[8], const float (&b)[8]) {
    float g[8];
    load8(w + c * 8, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] += c * 8 + i < D ? b[i] * inv * g[i] : 0.f;
    store8(row + c * 8, a);
    if (h) store8(h + size_t(t) * ldx + c * 8, a);
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int c = u * kRowThreads + threadIdx.x;
    if (c < chunks) put(c, fx[u], fy[u]);
  }
  for (int c = kKeep * kRowThreads + threadIdx.x; c < chunks; c += kRowThreads) {
    float a[8], b[8];
    load8(row + c * 8, a);
    src.load(t, c, a, b);
    put(c, a, b);
  }
}

// raw row t = [q: Hq*dim | k: Hkv*dim | v: Hkv*vdim | ..]. Every query and key head is divided by its
// own root mean square and multiplied by q_w / k_w [dim]; q goes to q_out [T, Hq, dkp], k and v to the
// token's slot of its sequence's pages. L lanes per head.
template <class TR, class T, int L>
__global__ void __launch_bounds__(kRowThreads)
head_norm_append_kernel(const TR* __restrict__ raw, int ldraw, const float* __restrict__ q_w,
                        const float* __restrict__ k_w, float eps, T* __restrict__ q_out,
                        T* __restrict__ k_cache, T* __restrict__ v_cache, const int* __restrict__ block_table,
                        const int* __restrict__ positions, const int* __restrict__ token_seq, int rows, int Hq,
                        int Hkv, int dim, int vdim, int dkp, int dvp, int max_blocks, int page) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = Hq + 2 * Hkv, units = rows * per;
  const int unit = (blockIdx.x * kRowThreads + threadIdx.x) / L, lane = threadIdx.x % L;
  const bool live = unit < units;                      // the lanes of a warp stay together for the sums
  const int t = live ? unit / per : 0, r = live ? unit - t * per : 0;
  const bool is_q = r < Hq, is_v = r >= Hq + Hkv;
  const int head = is_q ? r : is_v ? r - Hq - Hkv : r - Hq;
  const int width = is_v ? vdim : dim, padded = is_v ? dvp : dkp;
  const int src0 = is_q ? head * dim : is_v ? (Hq + Hkv) * dim + head * vdim : (Hq + head) * dim;
  const TR* src = raw + size_t(t) * ldraw + src0;
  const bool vec = width % 8 == 0 && src0 % 8 == 0 && ldraw % 8 == 0;
  T* dst = nullptr;
  if (is_q) {
    dst = q_out + (size_t(t) * Hq + head) * dkp;
  } else {
    const int pos = positions[t];
    if (RB_BOUNDS(pos / page, max_blocks)) {
      const int seq = token_seq ? token_seq[t] : t;
      const int blk = block_table[size_t(seq) * max_blocks + pos / page];
      dst = (is_v ? v_cache : k_cache) + ((size_t(blk) * Hkv + head) * page + pos % page) * padded;
    }
  }
  float first[8], ssq = 0.f;
  load8_upto(src + lane * 8, width - lane * 8, vec && lane * 8 < width, first);
#pragma unroll
  for (int i = 0; i < 8; ++i) ssq += first[i] * first[i];
  for (int d0 = (lane + L) * 8; d0 < width; d0 += L * 8) {
    float f[8];
    load8_upto(src + d0, width - d0, vec, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) ssq += f[i] * f[i];
  }
  ssq = group_sum<L>(ssq);
  if (!live || !dst) return;
  const float inv = is_v ? 1.f : 1.f / sqrtf(ssq / float(dim) + eps);
  const float* w = is_q ? q_w : k_w;
  auto put = [&](int d0, float (&f)[8]) {
    if (!is_v) {
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = d0 + i < dim ? f[i] * inv * w[d0 + i] : 0.f;
    }
    store8(dst + d0, f);
  };
  if (lane * 8 < padded) put(lane * 8, first);
  for (int d0 = (lane + L) * 8; d0 < padded; d0 += L * 8) {
    float f[8];
    load8_upto(src + d0, width - d0, vec && d0 < width, f);
    put(d0, f);
  }
}

// q row t = [H * (dim + rot)], down row t = [latent: rank | shared key part: rot] (null: the token's cache row is
// another layer's, only the queries are done). Queries go to q_out
// [T, H, dimp + rotp] with their last `rot` values rotated (pairs (2i, 2i+1) of the first `dims` by
// position * inv_freq[i]), the rotated part also behind the latent part of q_abs [T, H, latp + rotp]
// when that is given. The latent is divided by its root mean square, times c_w; it and the rotated
// shared key part form the token's cache row [latp | rotp | ..] of `ldc` elements. One block per token, or (grid y) several.
template <class TR, class T>
__global__ void __launch_bounds__(kRowThreads)
latent_append_kernel(const TR* __restrict__ qraw, int ldq, const TR* __restrict__ draw, int ldd,
                     const float* __restrict__ c_w, float eps,
                     const float* __restrict__ inv_freq, int dims, T* __restrict__ q_out, T* __restrict__ q_abs,
                     T* __restrict__ cache, int ldc, const int* __restrict__ block_table,
                     const int* __restrict__ positions, const int* __restrict__ token_seq, int H, int dim,
                     int rot, int rank, int dimp, int rotp, int latp, int max_blocks, int page) {
  extern __shared__ float trig[];          // cos [dims / 2], sin [dims / 2]
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, pos = positions[t];
  const TR* row = qraw + size_t(t) * ldq;
  const TR* down = draw ? draw + size_t(t) * ldd : nullptr;
  float ssq = 0.f;
  for (int i = threadIdx.x; down && i < rank; i += kRowThreads) { const float v = to_f32(down[i]); ssq += v * v; }
  for (int i = threadIdx.x; i < dims / 2; i += kRowThreads) {
    float s, c;
    rotary_sincos(pos, inv_freq[i], s, c);
    trig[i] = c;
    trig[dims / 2 + i] = s;
  }
  ssq = row_block_sum(ssq, red);           // the angles are in shared memory, too
  const float inv = 1.f / sqrtf(ssq / float(rank) + eps);
  const bool vec = dim % 8 == 0 && rot % 8 == 0 && rank % 8 == 0 && ldq % 8 == 0 && ldd % 8 == 0;
  // values i0 .. i0 + 7 of a vector whose first `dims` values turn
  auto rotate = [&](int i0, float (&f)[8]) {
#pragma unroll
    for (int i = 0; i < 8; i += 2)
      if (i0 + i < dims) {
        const float c = trig[(i0 + i) >> 1], s = trig[dims / 2 + ((i0 + i) >> 1)], u = f[i], v = f[i + 1];
        f[i] = fmaf(u, c, -v * s);
        f[i + 1] = fmaf(v, c, u * s);
      }
  };
  const int seq = token_seq ? token_seq[t] : t;
  const bool in_table = RB_BOUNDS(pos / page, max_blocks);
  const int blk = in_table ? block_table[size_t(seq) * max_blocks + pos / page] : 0;
  T* cdst = cache + (size_t(blk) * page + pos % page) * ldc;
  const int ud = dimp >> 3, uq = (dimp + rotp) >> 3, ul = latp >> 3, uc = (latp + rotp) >> 3;
  for (int u = blockIdx.y * kRowThreads + threadIdx.x; u < H * uq + (down ? uc : 0); u += gridDim.y * kRowThreads) {
    float f[8];
    if (u < H * uq) {                      // a query
      const int h = u / uq, c = u - h * uq;
      const TR* p = row + h * (dim + rot);
      if (c < ud) {
        load8_upto(p + c * 8, dim - c * 8, vec, f);
      } else {
        const int i0 = (c - ud) * 8;
        load8_upto(p + dim + i0, rot - i0, vec, f);
        rotate(i0, f);
        if (q_abs) store8(q_abs + (size_t(t) * H + h) * (latp + rotp) + latp + i0, f);
      }
      store8(q_out + (size_t(t) * H + h) * (dimp + rotp) + c * 8, f);
    } else if (in_table) {                 // the token's cache row
      const int c = u - H * uq;
      if (c < ul) {
        load8_upto(down + c * 8, rank - c * 8, vec, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = c * 8 + i < rank ? f[i] * inv * c_w[c * 8 + i] : 0.f;
      } else {
        const int i0 = (c - ul) * 8;
        load8_upto(down + rank + i0, rot - i0, vec, f);
        rotate(i0, f);
      }
      store8(cdst + c * 8, f);
    }
  }
}

// The latents of whole contexts in position order: page i of the result is page pages[i].y of the sequence
// in row pages[i].x of the block table. One block per page.
__global__ void __launch_bounds__(kRowThreads)
latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, int ldc, const int* __restrict__ block_table, int max_blocks,
                     const int2* __restrict__ pages, __nv_bfloat16* __restrict__ out, int lat, int page) {
  pdl_launch_dependents();
  pdl_wait();
  const int2 pg = pages[blockIdx.x];
  const int blk = RB_BOUNDS(pg.y, max_blocks) ? block_table[size_t(pg.x) * max_blocks + pg.y] : 0;
  const int units = lat / 8;
  for (int i = threadIdx.x; i < page * units; i += kRowThreads) {
    const int r = i / units, c = i - r * units;
    reinterpret_cast<uint4*>(out + (size_t(blockIdx.x) * page + r) * lat)[c] =
        reinterpret_cast<const uint4*>(cache + (size_t(blk) * page + r) * ldc)[c];
  }
}

// out[r, i] = act(in[r, i], in[r, n + i]); n a multiple of eight.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
gated_act_kernel(const T* __restrict__ in, T* __restrict__ out, long long units, int per_row, float limit) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long u = blockIdx.x * (long long)(kRowThreads) + threadIdx.x; u < units;
       u += (long long)(gridDim.x) * kRowThreads) {
    const long long r = u / per_row;
    const int c = int(u - r * per_row);
    float g[8], v[8];
    load8(in + (r * 2 * per_row + c) * 8, g);
    load8(in + (r * 2 * per_row + per_row + c) * 8, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) g[i] = gated_act(g[i], v[i], limit);
    store8(out + u * 8, g);
  }
}

// out = tanh(in) elementwise, fp32 in, compute type out.
template <class T>
__global__ void __launch_bounds__(kRowThreads)
tanh_kernel(const float* __restrict__ in, T* __restrict__ out, long long n) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = blockIdx.x * (long long)(kRowThreads) + threadIdx.x;
  if (i < n) out[i] = from_f32<T>(tanhf(in[i]));
}

template <class SRC>
static int launch_post_norm(SRC src, const float* w, float eps, float* x, void* h, int T, int D, int ldx, int h_f32,
                            int pdl, cudaStream_t st) {
  if (h_f32)
    return launch(post_norm_add_kernel<SRC, float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, src, w, eps, x,
                  static_cast<float*>(h), D, ldx);
  return launch(post_norm_add_kernel<SRC, __nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0, src, w, eps, x,
                static_cast<__nv_bfloat16*>(h), D, ldx);
}

}  // namespace rb

using namespace rb;
RB_BOUNDS_REGISTER("postnorm_rows.cu")

// f32: table and h are fp32, else bf16. x fp32 [T, ldx], h [T, ldx].
extern "C" int rmlx_embed_norm(const void* table, const int* ids, const float* w, float eps, float* x, void* h,
                               int T, int D, int ldx, int vocab, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || vocab < 1) return -2;
  if (f32)
    return launch(embed_norm_kernel<float>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0,
                  static_cast<const float*>(table), ids, w, eps, x, static_cast<float*>(h), D, ldx, vocab);
  return launch(embed_norm_kernel<__nv_bfloat16>, dim3(T), dim3(kRowThreads), 0, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(table), ids, w, eps, x, static_cast<__nv_bfloat16*>(h), D, ldx,
                vocab);
}

// y [T, ldy] fp32 (y_f32) or bf16, w fp32 [ldx], x fp32 [T, ldx] in place, h [T, ldx] fp32 / bf16 or null.
// ldx and ldy multiples of eight, ldy >= ldx.
extern "C" int rmlx_post_norm_add(const void* y, int ldy, int y_f32, const float* w, float eps, float* x, void* h,
                                  int T, int D, int ldx, int h_f32, int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || ldx % 8 || ldy % 8 || ldy < ldx) return -2;
  if (y_f32)
    return launch_post_norm(RowSource<float>{static_cast<const float*>(y), ldy}, w, eps, x, h, T, D, ldx, h_f32, pdl, st);
  return launch_post_norm(RowSource<__nv_bfloat16>{static_cast<const __nv_bfloat16*>(y), ldy}, w, eps, x, h, T, D, ldx,
                          h_f32, pdl, st);
}

// The same for routed experts: y [rows, ldy] in the compute type (f32), row_of_pair / weights [T, top_k],
// identity [T].
extern "C" int rmlx_moe_combine_post_norm(const void* y, int ldy, const int* row_of_pair, const float* weights,
                                          const float* identity, int top_k, const float* w, float eps, float* x,
                                          void* h, int T, int D, int ldx, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || D < 1 || ldx < D || ldx % 8 || ldy % 8 || ldy < ldx || top_k < 1) return -2;
  if (f32)
    return launch_post_norm(ExpertSource<float>{static_cast<const float*>(y), ldy, row_of_pair, weights, identity,
                                                top_k}, w, eps, x, h, T, D, ldx, 1, pdl, st);
  return launch_post_norm(ExpertSource<__nv_bfloat16>{static_cast<const __nv_bfloat16*>(y), ldy, row_of_pair, weights,
                                                      identity, top_k}, w, eps, x, h, T, D, ldx, 0, pdl, st);
}

// f32: q_out and the caches are fp32, else bf16; raw_f32: raw is fp32.
extern "C" int rmlx_head_norm_append(const void* raw, int ldraw, int raw_f32, const float* q_w, const float* k_w,
                                     float eps, void* q_out, void* k_cache, void* v_cache, const int* block_table,
                                     const int* positions, const int* token_seq, int T, int Hq, int Hkv, int dim,
                                     int vdim, int dkp, int dvp, int max_blocks, int page, int f32, int pdl,
                                     cudaStream_t st) {
  if (T < 1 || Hq < 1 || Hkv < 1 || dim < 1 || vdim < 1 || dkp % 8 || dvp % 8 || dkp < dim || dvp < vdim ||
      ldraw < (Hq + Hkv) * dim + Hkv * vdim || (f32 && !raw_f32))
    return -2;
  const long long units = 1LL * T * (Hq + 2 * Hkv);
  if (units * 32 > 0x7fffffffLL) return -2;
  const int widest = dkp > dvp ? dkp : dvp, lanes = widest <= 64 ? 8 : widest <= 128 ? 16 : 32;
  const dim3 grid(unsigned((units * lanes + kRowThreads - 1) / kRowThreads));
#define RB_HN_L(TR_, T_, L_)                                                                                      \
  return launch(head_norm_append_kernel<TR_, T_, L_>, grid, dim3(kRowThreads), 0, st, pdl != 0,                   \
                static_cast<const TR_*>(raw), ldraw, q_w, k_w, eps, static_cast<T_*>(q_out),                      \
                static_cast<T_*>(k_cache), static_cast<T_*>(v_cache), block_table, positions, token_seq, T, Hq,   \
                Hkv, dim, vdim, dkp, dvp, max_blocks, page)
#define RB_HN(TR_, T_)                     \
  {                                        \
    if (lanes == 8) RB_HN_L(TR_, T_, 8);   \
    if (lanes == 16) RB_HN_L(TR_, T_, 16); \
    RB_HN_L(TR_, T_, 32);                  \
  }
  if (f32) RB_HN(float, float);
  if (raw_f32) RB_HN(float, __nv_bfloat16);
  RB_HN(__nv_bfloat16, __nv_bfloat16);
#undef RB_HN
#undef RB_HN_L
}

// Types as above; q_raw rows ldq apart; down rows ldd apart, or null. dims: how many of the rotated part's values turn (even, <= rot); inv_freq fp32 [dims / 2].
extern "C" int rmlx_latent_append(const void* q_raw, int ldq, const void* down, int ldd, int raw_f32, const float* c_w, float eps,
                                  const float* inv_freq, int dims, void* q_out, void* q_abs, void* cache, int ldc,
                                  const int* block_table, const int* positions, const int* token_seq, int T, int H,
                                  int dim, int rot, int rank, int dimp, int rotp, int latp, int max_blocks, int page,
                                  int f32, int pdl, cudaStream_t st) {
  if (T < 1 || H < 1 || dim < 0 || rot < 0 || rank < 1 || dims < 0 || dims % 2 || dims > rot || dimp < dim ||
      rotp < rot || latp < rank || ldc < latp + rotp || ldq < H * (dim + rot) ||
      (down && ldd < rank + rot) || (f32 && !raw_f32))
    return -2;
  const size_t smem = size_t(dims) * sizeof(float);
  if (smem > 32 * 1024) return -2;
  const int work = (H * (dimp + rotp) + latp + rotp) / 8;            // few tokens: several blocks share one
  const int split = T >= 64 ? 1 : (work + kRowThreads - 1) / kRowThreads;
#define RB_LA(TR_, T_)                                                                                            \
  return launch(latent_append_kernel<TR_, T_>, dim3(T, split), dim3(kRowThreads), smem, st, pdl != 0,                    \
                static_cast<const TR_*>(q_raw), ldq, static_cast<const TR_*>(down), ldd, c_w, eps, inv_freq, dims, static_cast<T_*>(q_out),           \
                static_cast<T_*>(q_abs), static_cast<T_*>(cache), ldc, block_table, positions, token_seq, H, dim, \
                rot, rank, dimp, rotp, latp, max_blocks, page)
  if (f32) RB_LA(float, float);
  if (raw_f32) RB_LA(float, __nv_bfloat16);
  RB_LA(__nv_bfloat16, __nv_bfloat16);
#undef RB_LA
}

// cache [.., page, ldc] bf16, pages int32 [n, 2], out bf16 [n * page, lat]; lat and ldc multiples of eight.
extern "C" int rmlx_latent_gather(const void* cache, int ldc, const int* block_table, int max_blocks, const int* pages,
                                  void* out, int n, int lat, int page, int pdl, cudaStream_t st) {
  if (n < 1 || lat < 8 || lat % 8 || ldc % 8 || ldc < lat || page < 1 || (reinterpret_cast<uintptr_t>(pages) & 7)) return -2;
  return launch(latent_gather_kernel, dim3(n), dim3(kRowThreads), 0, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(cache), ldc, block_table, max_blocks,
                reinterpret_cast<const int2*>(pages), static_cast<__nv_bfloat16*>(out), lat, page);
}

// in [R, 2 n] = [gate | up], out [R, n], both fp32 (f32) or bf16; n a multiple of eight.
extern "C" int rmlx_gated_act(const void* in, void* out, int R, int n, float limit, int f32, int pdl,
                              cudaStream_t st) {
  if (R < 1 || n < 8 || n % 8) return -2;
  const long long units = 1LL * R * (n / 8);
  const long long want = (units + kRowThreads - 1) / kRowThreads, cap = 16LL * sm_count();
  const dim3 grid(unsigned(want < cap ? want : cap));
  if (f32)
    return launch(gated_act_kernel<float>, grid, dim3(kRowThreads), 0, st, pdl != 0, static_cast<const float*>(in),
                  static_cast<float*>(out), units, n / 8, limit);
  return launch(gated_act_kernel<__nv_bfloat16>, grid, dim3(kRowThreads), 0, st, pdl != 0,
                static_cast<const __nv_bfloat16*>(in), static_cast<__nv_bfloat16*>(out), units, n / 8, limit);
}

extern "C" int rmlx_tanh_rows(const float* in, void* out, long long n, int f32, int pdl, cudaStream_t st) {
  if (n < 1) return -2;
  const dim3 grid(unsigned((n + kRowThreads - 1) / kRowThreads));
  if (f32) return launch(tanh_kernel<float>, grid, dim3(kRowThreads), 0, st, pdl != 0, in, static_cast<float*>(out), n);
  return launch(tanh_kernel<__nv_bfloat16>, grid, dim3(kRowThreads), 0, st, pdl != 0, in,
                static_cast<__nv_bfloat16*>(out), n);
}
