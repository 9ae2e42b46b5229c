// bf16 GEMM on the 5th-generation tensor cores: C[M,N] = A[M,K] · W[N,K]^T (+ residual), fp32
// accumulation in tensor memory.
//
// Persistent, warp-specialised kernel, one CTA per SM:
//   warp 0      TMA producer: 128x64 A tiles and BNx64 W tiles (128-byte swizzle) into a ring of
//               shared-memory stages, completion on mbarriers
//   warp 1      MMA issuer: one elected thread issues tcgen05.mma (M=128, N=BN, K=16) four times
//               per stage; tcgen05.commit releases the stage back to the producer and, at the end
//               of a tile, hands the accumulator to the epilogue
//   warps 2-5   epilogue: tcgen05.ld the 128xBN fp32 accumulator out of TMEM (each warp owns the
//               32 lanes its position in the warpgroup may touch), add the residual, convert to
//               bf16 and store
// Two accumulators (2 x BN columns of TMEM) let the epilogue of tile i overlap the main loop of
// tile i+1. Rows past M and columns past K are zero-filled by TMA; stores are predicated.
//
// Two more epilogues serve parallel-block decoders (attention and feed-forward side by side, fp32
// residual): kEpiSplit stores the columns before n_raw as bf16 and sends the others through xIELU
// into a second matrix (the merged [q; k; v; up] projection); kEpiDual keeps TWO accumulators per tile, one
// per (A, W) pair, and adds ls1 * A1 W1^T + ls2 * A2 W2^T to the fp32 residual (attention output and
// feed-forward down projections, layer scales and residual sum in one kernel).
//
// Replaces the reference's simdgroup-MMA GEMM family and its tile-selection logic (gemm_mlx_*,
// gemm_nax_*, split-K; crates/rmlx-core/src/ops/matmul.rs:2160-5610,6377-6480) and the residual
// epilogue of matmul_add_residual_into_cb (matmul.rs:7988).
#include <cuda.h>
#include "../common/ptx.cuh"
#include "../common/launch.cuh"
#include "../common/tensormap.cuh"
#include "../common/xielu.cuh"

namespace rb {

constexpr int kBM = 128;
constexpr int kBK = 64;
constexpr int kGemmThreads = 192;

template <int BN>
struct GemmSmem {
  static constexpr int kStageA = kBM * kBK * 2;
  static constexpr int kStageB = BN * kBK * 2;
  static constexpr int kStages = (BN >= 256) ? 4 : (BN >= 128 ? 6 : 8);
  static constexpr int kBytes = kStages * (kStageA + kStageB) + 1024 /*align slack*/ + 256 /*barriers*/;
};

// Epilogues. kEpiF32: the accumulator is stored as fp32 (C is then float*, ldc counts floats): router
// logits and other results that must not be rounded to bf16.
enum GemmEpi : int { kEpiPlain = 0, kEpiResidual = 1, kEpiF32 = 2, kEpiSplit = 3, kEpiDual = 4 };

struct GemmEpiArgs {
  // kEpiSplit
  __nv_bfloat16* act = nullptr; int ldact = 0; int n_raw = 0; float ap = 0.f, an = 0.f;
  // kEpiDual: C is the fp32 residual; K2 == 0: no second product
  const float* s1 = nullptr; const float* s2 = nullptr; int K2 = 0;
};

template <int BN, int EPI>
__global__ void __launch_bounds__(kGemmThreads, 1)
gemm_bf16_tcgen05_kernel(const __grid_constant__ CUtensorMap tmap_a,
                         const __grid_constant__ CUtensorMap tmap_w,
                         const __grid_constant__ CUtensorMap tmap_a2,
                         const __grid_constant__ CUtensorMap tmap_w2,
                         void* __restrict__ Cv, const __nv_bfloat16* __restrict__ residual,
                         int M, int N, int K, int ldc, int* __restrict__ status, GemmEpiArgs ea) {
  constexpr bool RESIDUAL = EPI == kEpiResidual, OUT_F32 = EPI == kEpiF32, DUAL = EPI == kEpiDual;
  __nv_bfloat16* C = static_cast<__nv_bfloat16*>(Cv);
  using S = GemmSmem<BN>;
  constexpr int STAGES = S::kStages;
  constexpr int ACC = DUAL ? 2 * BN : BN;                        // accumulator columns per tile
  static_assert(2 * ACC <= 512, "two accumulators per tile leave room for BN <= 128");
  constexpr uint32_t TMEM_COLS = (2 * ACC <= 32) ? 32 : 2 * ACC;  // power of two: BN in {32,..,256}
  extern __shared__ char smem_raw[];
  // tiles need 1024-byte alignment for the 128-byte swizzle
  char* smem = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  char* sA = smem;
  char* sB = smem + STAGES * S::kStageA;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sB + STAGES * S::kStageB);
  uint64_t* full = bars;                  // [STAGES]
  uint64_t* empty = bars + STAGES;        // [STAGES]
  uint64_t* acc_full = bars + 2 * STAGES; // [2]
  uint64_t* acc_empty = acc_full + 2;     // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile uint32_t* abort_flag = tmem_slot + 1;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tiles_m = (M + kBM - 1) / kBM, tiles_n = (N + BN - 1) / BN;
  const int num_tiles = tiles_m * tiles_n;
  const int num_kb1 = (K + kBK - 1) / kBK;
  const int num_kb = num_kb1 + (DUAL ? (ea.K2 + kBK - 1) / kBK : 0);

  if (threadIdx.x == 0) {
    for (int i = 0; i < STAGES; ++i) { mbar_init(full + i, 1); mbar_init(empty + i, 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(acc_full + i, 1); mbar_init(acc_empty + i, 4); }
    *abort_flag = 0u;
    fence_mbar_init();
  }
  if (warp == 1) {  // this warp owns the TMEM allocation
    tmem_alloc(tmem_slot, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (elect_one()) {
      tma_prefetch_desc(&tmap_a);
      tma_prefetch_desc(&tmap_w);
      pdl_wait();
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        // consecutive CTAs share the same W tile column-block: good L2 reuse of W across M
        const int tm = tile % tiles_m, tn = tile / tiles_m;
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!mbar_wait(empty + stage, phase ^ 1u, abort_flag)) { ok = false; break; }
          mbar_arrive_expect_tx(full + stage, S::kStageA + S::kStageB);
          const bool second = DUAL && kb >= num_kb1;
          const int kx = (second ? kb - num_kb1 : kb) * kBK;
          tma_load_2d(sA + stage * S::kStageA, second ? &tmap_a2 : &tmap_a, full + stage, kx, tm * kBM);
          tma_load_2d(sB + stage * S::kStageB, second ? &tmap_w2 : &tmap_w, full + stage, kx, tn * BN);
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      constexpr uint32_t idesc = umma_idesc_bf16_f32(kBM, BN);
      int stage = 0;
      uint32_t phase = 0;
      int acc = 0;
      uint32_t acc_phase = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        if (!mbar_wait(acc_empty + acc, acc_phase ^ 1u, abort_flag)) { ok = false; break; }
        tc_fence_after_sync();
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!mbar_wait(full + stage, phase, abort_flag)) { ok = false; break; }
          tc_fence_after_sync();
          const uint32_t a_addr = smem_u32(sA + stage * S::kStageA);
          const uint32_t b_addr = smem_u32(sB + stage * S::kStageB);
          const bool second = DUAL && kb >= num_kb1;
          const uint32_t d_tmem = tmem_base + acc * ACC + (second ? BN : 0);
          const int kfirst = second ? kb - num_kb1 : kb;
#pragma unroll
          for (int k = 0; k < kBK / 16; ++k) {
            tc_mma_f16(d_tmem, umma_desc_sw128_kmajor(a_addr + k * 32),
                       umma_desc_sw128_kmajor(b_addr + k * 32), idesc, (kfirst | k) != 0 ? 1u : 0u);
          }
          tc_commit(empty + stage);  // stage is free once these MMAs have read it
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
        if (!ok) break;
        tc_commit(acc_full + acc);   // accumulator complete
        if (++acc == 2) { acc = 0; acc_phase ^= 1u; }
      }
    }
  } else {
    // ------------------------------------------------------------------ epilogue (warps 2..5)
    const int q = warp & 3;  // TMEM lane quarter this warp may access
    int acc = 0;
    uint32_t acc_phase = 0;
    bool ok = true;
    if (RESIDUAL || DUAL) pdl_wait();
    for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
      const int tm = tile % tiles_m, tn = tile / tiles_m;
      if (!mbar_wait(acc_full + acc, acc_phase, abort_flag)) { ok = false; break; }
      tc_fence_after_sync();
      const int row = tm * kBM + q * 32 + lane;
      const uint32_t t_row = tmem_base + acc * ACC + (uint32_t(q * 32) << 16);
#pragma unroll 1
      for (int c = 0; c < BN / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(t_row + c * 32, r);
        const int col0 = tn * BN + c * 32;
        if (DUAL) {
          uint32_t r2[32];
          if (ea.K2 > 0) tmem_ld_32x32(t_row + BN + c * 32, r2);
          tmem_ld_wait();
          if (row < M && col0 < N) {
            float* dst = static_cast<float*>(Cv) + size_t(row) * ldc + col0;
#pragma unroll
            for (int v = 0; v < 8; ++v) {
              if (col0 + v * 4 < N) {                   // N is a multiple of 8 (checked by the launcher)
                float4 x = *reinterpret_cast<const float4*>(dst + v * 4);
                const float4 a = *reinterpret_cast<const float4*>(ea.s1 + col0 + v * 4);
                float4 d = make_float4(a.x * __uint_as_float(r[v * 4]), a.y * __uint_as_float(r[v * 4 + 1]),
                                       a.z * __uint_as_float(r[v * 4 + 2]), a.w * __uint_as_float(r[v * 4 + 3]));
                if (ea.K2 > 0) {
                  const float4 b = *reinterpret_cast<const float4*>(ea.s2 + col0 + v * 4);
                  d.x = fmaf(b.x, __uint_as_float(r2[v * 4]), d.x);
                  d.y = fmaf(b.y, __uint_as_float(r2[v * 4 + 1]), d.y);
                  d.z = fmaf(b.z, __uint_as_float(r2[v * 4 + 2]), d.z);
                  d.w = fmaf(b.w, __uint_as_float(r2[v * 4 + 3]), d.w);
                }
                x.x += d.x; x.y += d.y; x.z += d.z; x.w += d.w;
                *reinterpret_cast<float4*>(dst + v * 4) = x;
              }
            }
          }
          continue;
        }
        tmem_ld_wait();
        if (EPI == kEpiSplit) {
          // n_raw is a multiple of 32: a chunk lies on one side of it
          if (row < M && col0 < N) {
            const bool is_act = col0 >= ea.n_raw;
            __nv_bfloat16* dst = is_act ? ea.act + size_t(row) * ea.ldact + (col0 - ea.n_raw)
                                        : C + size_t(row) * ldc + col0;
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              if (col0 + v * 8 < N) {                   // N is a multiple of 8
                float f[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                  f[j] = __uint_as_float(r[v * 8 + j]);
                  if (is_act) f[j] = xielu_fast(f[j], ea.ap, ea.an);
                }
                uint4 o;
                o.x = pack_bf16(f[0], f[1]); o.y = pack_bf16(f[2], f[3]);
                o.z = pack_bf16(f[4], f[5]); o.w = pack_bf16(f[6], f[7]);
                *reinterpret_cast<uint4*>(dst + v * 8) = o;
              }
            }
          }
          continue;
        }
        if (OUT_F32) {
          if (row < M && col0 < N) {
            float* dstf = static_cast<float*>(Cv) + size_t(row) * ldc + col0;
            if (col0 + 32 <= N && (ldc & 3) == 0 && (reinterpret_cast<uintptr_t>(Cv) & 15) == 0) {
#pragma unroll
              for (int v = 0; v < 8; ++v)
                *reinterpret_cast<float4*>(dstf + v * 4) =
                    make_float4(__uint_as_float(r[v * 4]), __uint_as_float(r[v * 4 + 1]),
                                __uint_as_float(r[v * 4 + 2]), __uint_as_float(r[v * 4 + 3]));
            } else {
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (col0 + j < N) dstf[j] = __uint_as_float(r[j]);
            }
          }
        } else if (row < M && col0 < N) {
          __nv_bfloat16* dst = C + size_t(row) * ldc + col0;
          const __nv_bfloat16* res = RESIDUAL ? residual + size_t(row) * ldc + col0 : nullptr;
          if (col0 + 32 <= N) {
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              float f[8];
#pragma unroll
              for (int j = 0; j < 8; ++j) f[j] = __uint_as_float(r[v * 8 + j]);
              if (RESIDUAL) {
                const uint4 rv = *reinterpret_cast<const uint4*>(res + v * 8);
                f[0] += bf16lo(rv.x); f[1] += bf16hi(rv.x); f[2] += bf16lo(rv.y); f[3] += bf16hi(rv.y);
                f[4] += bf16lo(rv.z); f[5] += bf16hi(rv.z); f[6] += bf16lo(rv.w); f[7] += bf16hi(rv.w);
              }
              uint4 o;
              o.x = pack_bf16(f[0], f[1]); o.y = pack_bf16(f[2], f[3]);
              o.z = pack_bf16(f[4], f[5]); o.w = pack_bf16(f[6], f[7]);
              *reinterpret_cast<uint4*>(dst + v * 8) = o;
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; ++j) {
              if (col0 + j < N) {
                float f = __uint_as_float(r[j]);
                if (RESIDUAL) f += __bfloat162float(res[j]);
                dst[j] = __float2bfloat16_rn(f);
              }
            }
          }
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(acc_empty + acc);
      if (++acc == 2) { acc = 0; acc_phase ^= 1u; }
    }
  }

  // ------------------------------------------------------------------ teardown
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
  if (threadIdx.x == 0 && *abort_flag && status) atomicExch(status, kStatusMbarTimeout);
  pdl_launch_dependents();
}

template <int BN, int EPI>
static int launch_gemm(const CUtensorMap& ta, const CUtensorMap& tw, const CUtensorMap& ta2,
                       const CUtensorMap& tw2, void* C, const void* residual, int M, int N, int K, int ldc,
                       int* status, const GemmEpiArgs& ea, int pdl, cudaStream_t st) {
  auto kern = gemm_bf16_tcgen05_kernel<BN, EPI>;
  constexpr size_t smem = GemmSmem<BN>::kBytes;
  RB_CHECK(set_max_smem(kern, smem));
  const int tiles = ((M + kBM - 1) / kBM) * ((N + BN - 1) / BN);
  const int grid = tiles < sm_count() ? tiles : sm_count();
  return launch(kern, dim3(grid), dim3(kGemmThreads), smem, st, pdl != 0, ta, tw, ta2, tw2, C,
                static_cast<const __nv_bfloat16*>(residual), M, N, K, ldc, status, ea);
}
template <int BN, int EPI>
static int launch_gemm(const CUtensorMap& ta, const CUtensorMap& tw, void* C, const void* residual,
                       int M, int N, int K, int ldc, int* status, int pdl, cudaStream_t st) {
  return launch_gemm<BN, EPI>(ta, tw, ta, tw, C, residual, M, N, K, ldc, status, GemmEpiArgs{}, pdl, st);
}

}  // namespace rb

using namespace rb;

// Tile width heuristic: the widest N tile that still yields about one tile per SM.
extern "C" int rmlx_gemm_pick_bn(int M, int N) {
  const int tm = (M + kBM - 1) / kBM;
  const int sms = sm_count();
  const int cands[4] = {256, 128, 64, 32};
  for (int i = 0; i < 4; ++i) {
    const int bn = cands[i];
    if (tm * ((N + bn - 1) / bn) >= sms || bn == 32) return bn;
  }
  return 32;
}

// C[M,N] (bf16, row stride ldc) = A[M,K] (bf16, row stride lda) * W[N,K]^T (bf16, row stride ldw)
// (+ residual[M,N] with C's stride). K, lda, ldw multiples of 8; A and W 16-byte aligned.
// bn: 0 = choose, else one of 32/64/128/256. status: optional device int set non-zero if a
// pipeline wait gave up.
extern "C" int rmlx_gemm_bf16(const void* A, const void* W, void* C, const void* residual, int M,
                              int N, int K, int lda, int ldw, int ldc, int bn, int* status, int pdl,
                              cudaStream_t st) {
  if (M < 1 || N < 1 || K < 8 || K % 8 || lda % 8 || ldw % 8) return -2;
  if ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(W)) & 15) return -2;
  if (bn == 0) bn = rmlx_gemm_pick_bn(M, N);
  CUtensorMap ta, tw;
  int rc = make_tmap_2d_bf16(&ta, A, uint64_t(K), uint64_t(M), uint64_t(lda) * 2, kBK, kBM);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tw, W, uint64_t(K), uint64_t(N), uint64_t(ldw) * 2, kBK, bn);
  if (rc) return rc;
#define RB_GEMM(BN_)                                                                              \
  case BN_:                                                                                       \
    return residual ? launch_gemm<BN_, kEpiResidual>(ta, tw, C, residual, M, N, K, ldc, status, pdl, st) \
                    : launch_gemm<BN_, kEpiPlain>(ta, tw, C, residual, M, N, K, ldc, status, pdl, st);
  switch (bn) {
    RB_GEMM(256)
    RB_GEMM(128)
    RB_GEMM(64)
    RB_GEMM(32)
    default: return -2;
  }
#undef RB_GEMM
}

// The same product with an fp32 result: C[M,N] float, row stride ldc floats. No residual.
extern "C" int rmlx_gemm_bf16_f32(const void* A, const void* W, void* C, int M, int N, int K, int lda,
                                  int ldw, int ldc, int* status, int pdl, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 8 || K % 8 || lda % 8 || ldw % 8) return -2;
  if ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(W)) & 15) return -2;
  int bn = rmlx_gemm_pick_bn(M, N);
  if (bn < 64) bn = 64;
  CUtensorMap ta, tw;
  int rc = make_tmap_2d_bf16(&ta, A, uint64_t(K), uint64_t(M), uint64_t(lda) * 2, kBK, kBM);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tw, W, uint64_t(K), uint64_t(N), uint64_t(ldw) * 2, kBK, bn);
  if (rc) return rc;
  if (bn == 256) return launch_gemm<256, kEpiF32>(ta, tw, C, nullptr, M, N, K, ldc, status, pdl, st);
  if (bn == 128) return launch_gemm<128, kEpiF32>(ta, tw, C, nullptr, M, N, K, ldc, status, pdl, st);
  return launch_gemm<64, kEpiF32>(ta, tw, C, nullptr, M, N, K, ldc, status, pdl, st);
}

// Merged projection of a parallel block: columns n < n_raw of A W^T to C (bf16, row stride ldc), the
// others through xIELU(ap, an) to act (bf16, row stride ldact, column n - n_raw). n_raw a multiple of
// 32; N, ldc and ldact multiples of 8; C and act 16-byte aligned. bn: 0 = choose, else 32 .. 256.
extern "C" int rmlx_gemm_bf16_split_xielu(const void* A, const void* W, void* C, void* act, int n_raw, float ap,
                                          float an, int M, int N, int K, int lda, int ldw, int ldc, int ldact,
                                          int bn, int* status, int pdl, cudaStream_t st) {
  if (M < 1 || N < 8 || N % 8 || K < 8 || K % 8 || lda % 8 || ldw % 8 || ldc % 8 || ldact % 8 ||
      n_raw < 0 || n_raw % 32 || n_raw > N || (n_raw < N && !act))
    return -2;
  if ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(W) | reinterpret_cast<uintptr_t>(C) |
       reinterpret_cast<uintptr_t>(act)) & 15)
    return -2;
  if (bn == 0) bn = rmlx_gemm_pick_bn(M, N);
  GemmEpiArgs ea;
  ea.act = static_cast<__nv_bfloat16*>(act); ea.ldact = ldact; ea.n_raw = n_raw; ea.ap = ap; ea.an = an;
  CUtensorMap ta, tw;
  int rc = make_tmap_2d_bf16(&ta, A, uint64_t(K), uint64_t(M), uint64_t(lda) * 2, kBK, kBM);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tw, W, uint64_t(K), uint64_t(N), uint64_t(ldw) * 2, kBK, bn);
  if (rc) return rc;
#define RB_GEMM(BN_) \
  case BN_: return launch_gemm<BN_, kEpiSplit>(ta, tw, ta, tw, C, nullptr, M, N, K, ldc, status, ea, pdl, st);
  switch (bn) {
    RB_GEMM(256)
    RB_GEMM(128)
    RB_GEMM(64)
    RB_GEMM(32)
    default: return -2;
  }
#undef RB_GEMM
}

// x[m, n] += s1[n] (A1 W1^T)[m, n] + s2[n] (A2 W2^T)[m, n], x fp32 with row stride ldx (a multiple of
// 4), K2 == 0: first product only. N, K1, K2 and the bf16 strides multiples of 8; every pointer
// 16-byte aligned.
extern "C" int rmlx_gemm_bf16_dual_add(const void* A1, const void* W1, int K1, int lda1, int ldw1,
                                       const void* A2, const void* W2, int K2, int lda2, int ldw2,
                                       const float* s1, const float* s2, float* x, int ldx, int M, int N,
                                       int bn, int* status, int pdl, cudaStream_t st) {
  if (M < 1 || N < 8 || N % 8 || K1 < 8 || K1 % 8 || lda1 % 8 || ldw1 % 8 || ldx % 4 || K2 < 0 || K2 % 8 ||
      (K2 > 0 && (lda2 % 8 || ldw2 % 8 || !A2 || !W2 || !s2)) || !s1)
    return -2;
  if ((reinterpret_cast<uintptr_t>(A1) | reinterpret_cast<uintptr_t>(W1) | reinterpret_cast<uintptr_t>(A2) |
       reinterpret_cast<uintptr_t>(W2) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(s1) |
       reinterpret_cast<uintptr_t>(s2)) & 15)
    return -2;
  if (bn == 0) { bn = rmlx_gemm_pick_bn(M, N); if (bn > 128) bn = 128; }
  GemmEpiArgs ea;
  ea.s1 = s1; ea.s2 = s2; ea.K2 = K2;
  CUtensorMap ta, tw, ta2, tw2;
  int rc = make_tmap_2d_bf16(&ta, A1, uint64_t(K1), uint64_t(M), uint64_t(lda1) * 2, kBK, kBM);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tw, W1, uint64_t(K1), uint64_t(N), uint64_t(ldw1) * 2, kBK, bn);
  if (rc) return rc;
  ta2 = ta; tw2 = tw;
  if (K2 > 0) {
    rc = make_tmap_2d_bf16(&ta2, A2, uint64_t(K2), uint64_t(M), uint64_t(lda2) * 2, kBK, kBM);
    if (rc) return rc;
    rc = make_tmap_2d_bf16(&tw2, W2, uint64_t(K2), uint64_t(N), uint64_t(ldw2) * 2, kBK, bn);
    if (rc) return rc;
  }
#define RB_GEMM(BN_) \
  case BN_: return launch_gemm<BN_, kEpiDual>(ta, tw, ta2, tw2, x, nullptr, M, N, K1, ldx, status, ea, pdl, st);
  switch (bn) {
    RB_GEMM(128)
    RB_GEMM(64)
    RB_GEMM(32)
    default: return -2;
  }
#undef RB_GEMM
}
