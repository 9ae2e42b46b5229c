// Paged causal flash attention for prompt processing on the 5th-generation tensor cores
// (head_dim 128, optional sliding window; other head dimensions use the mma.sync kernel in
// flash_prefill.cu), and its form with score modifiers (score_mod.cuh: temperature, soft cap,
// logarithmic distance bias, sink) over ragged batches, for key and value widths up to 128 each.
//
// KP / VP: 64-column panels of a key / value row. Widths that are not a multiple of 64 cost no extra
// global memory: the tensor maps end at the real width and TMA fills the rest of a panel with zeros.
// Ragged batches come as a table of query tiles ({first row, rows, position of the first row, row of
// the block table}), so prompt portions of several sequences share one launch.
// Latent attention (LAT): the keys and values of the batch's contexts are expanded from their latents
// beforehand, [context rows, H, dim + vdim] in position order, and read through three-dimensional tensor
// maps (a head's columns past its width read as zero); the rotated key part, shared by all heads, is the
// last panel of a key row and comes straight from the latent cache's pages.
// Differential attention (DIFF, score_mod.cuh): the two lanes are the two maps of one query tile. Each has its own
// query tile and, per step, its own key tile; the value tile serves both, so the values cross shared memory once. At the
// end the lanes exchange their sums and take half of the value columns each: difference of the maps, its norm over the
// head, one store.
//
// Score modifiers run between S and the softmax, in base 2: t = P(s) - bias(i - j), where P is
// softcap * tanh(s scale temp / softcap) as s times a polynomial in s^2 with the head's constants
// folded in (all FMA), or, in a step where some |argument| leaves the polynomial's range, by
// ex2 / rcp. The bias depends on the distance only: every softmax warp keeps the values for the
// 95 distances a step can hold in a ring in shared memory (128 entries, stored twice so that a
// step reads a straight run) and adds the 64 new ones of each step. The sink is a first key of
// weight one and no value: it initialises the running maximum and sum.
//
// A CTA owns LANES (1 or 2) tiles of 128 query tokens of one query head and walks the keys 64 at a
// time; the K and V tiles of a step serve every lane. A kernel that allocates tensor memory gets one
// CTA per SM (the occupancy calculator reports 1 for any kernel with tcgen05.alloc), so a second
// lane is the only way to put two softmax warps on each scheduler: each lane has its own softmax
// warpgroup, S and O accumulators and P tile.
//   warp 0      TMA producer: the Q tiles once, then per step four 16-token pages of K and of V
//               (found through the block table) as 64-column panels with the 128-byte swizzle, two
//               stages each
//   warp 1      MMA issuer: per lane S = Q K^T (tcgen05.mma, M 128, N 64 keys, K = head_dim) into
//               one of the lane's two S accumulators in tensor memory, and O += P V (N = head_dim,
//               K = 64 keys, V read in place as an MN-major operand) into the lane's O accumulator.
//               S of step j+1 is issued before P V of step j, so the tensor cores work while step
//               j's softmax runs.
//   warps 2-5   softmax of lane 0 (warps 6-9: lane 1): thread i owns query row i. It reads its row
//               of S from tensor memory, applies the causal mask on the steps that touch the
//               diagonal, exponentiates against a running reference maximum, writes P (bf16) into
//               shared memory in the K-major
//               swizzled operand layout, and keeps the running sum. The reference maximum moves
//               only when a row's maximum has grown by more than 2^8 since it was set (then the O
//               row in tensor memory is rescaled in place), so most steps touch O not at all.
//               At the end the same threads normalise O and store it.
// Every wait is bounded; a wait that gives up sets the CTA's abort word, the roles leave their
// loops, tensor memory is freed and the status word is set.
//
// Replaces sdpa_prefill_mma_* / sdpa_prefill_nax_* (crates/rmlx-core/src/ops/sdpa.rs:1873-2855)
// with attention that reads the paged cache directly
// (crates/rmlx-nn/src/paged_kv_cache.rs:303-305 gathers on the CPU).
#include <cuda.h>
#include "../common/ptx.cuh"
#include "../common/launch.cuh"
#include "../common/tensormap.cuh"
#include "../common/score_mod.cuh"

namespace rb {

constexpr int kTcRows = 128;                  // query rows per lane
constexpr int kTcKeys = 64;                   // keys per step
constexpr int kTcHd = 128;
constexpr int kTcPage = 16;
constexpr int kTcPages = kTcKeys / kTcPage;   // pages per step
constexpr int kTcQPanel = 128 * 128;          // 128 rows x 64 bf16 columns
constexpr int kTcKvPanel = kTcKeys * 128;     // 64 rows x 64 bf16 columns
constexpr int kTcBiasRing = 256;              // floats per softmax warp: 128 distances, twice
constexpr int kTcPTile = kTcQPanel;           // 128 rows x 64 keys bf16
constexpr int kTcPageBytes = kTcPage * 128;   // one page inside a 64-column panel
constexpr float kTcRescaleStep = 8.f;         // log2 of the growth tolerated before O is rescaled

template <int LANES, int KP, int VP, bool MOD, bool DIFF = false>
struct TcCfg {
  static constexpr int kQTile = KP * kTcQPanel;     // 128 query rows
  static constexpr int kKMap = KP * kTcKvPanel;     // 64 keys of one map
  static constexpr int kKTile = (DIFF ? 2 : 1) * kKMap;
  static constexpr int kVTile = VP * kTcKvPanel;
  static constexpr int kThreads = 64 + 128 * LANES;
  // per lane: S0 [0,64) S1 [64,128); then per lane O (VP * 64 columns)
  static constexpr uint32_t kTmemCols = 256 * LANES;
  static constexpr int kBars = 9 + 6 * LANES;
  // Q per lane, K x2, V x2, P per lane, barriers. No slack for alignment: the kernel checks that
  // the dynamic shared-memory window starts on a 1024-byte boundary and refuses to run otherwise.
  static constexpr int kBiasBytes = MOD ? LANES * 4 * kTcBiasRing * 4 : 0;
  static constexpr int kSmem = LANES * kQTile + 2 * kKTile + 2 * kVTile + LANES * kTcPTile + 256 + kBiasBytes;
};

struct TcParams {
  const int* block_table;   // this sequence's pages (with tiles: the whole table)
  __nv_bfloat16* out;       // [T, Hq, dv]
  int T, Hq, Hkv, pos0, n_qt;
  int dk, dv;               // key and value row widths in memory
  const int4* tiles;        // ragged batches: {first row, rows, position of the first row, table row}
  int max_blocks;
  int window;               // > 0: a query sees only its last `window` keys
  int chunk;                // > 0: only the keys of its own chunk of so many positions
  float scale_log2;
  ScoreMod mod;             // MOD instances
  HeadGate gate;            // ragged batches
  // LAT instances: panels of the unrotated key part, where the rotated part starts in a query row and in
  // a cache row, first context row of every tile's sequence
  int kn, q_rot, c_rot;
  const int* tile_ctx;
  // DIFF instances: query rows are [head][map], values of a head that exist
  MapDiff diff;
  int vdim;
  int* status;
};

__device__ __forceinline__ float tc_ex2(float x) { return ex2_approx(x); }

// Pairs of fp32 values in one 64-bit register (one issue slot for two operations).
__device__ __forceinline__ uint64_t pair2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpair2(uint64_t v, uint32_t& lo, uint32_t& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=r"(lo), "=r"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
// Largest of three values / of three magnitudes, one instruction each.
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float max3_abs(float a, float b, float c) {
  float d;
  asm("max.abs.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}

// Barrier `id` among `threads` threads of the block.
__device__ __forceinline__ void named_bar_sync(int id, int threads) {
  asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory");
}

template <int LANES, int KP, int VP, bool MOD, bool LAT, bool DIFF>
__global__ void __launch_bounds__(TcCfg<LANES, KP, VP, MOD, DIFF>::kThreads, 1)
flash_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmap_q,
                        const __grid_constant__ CUtensorMap tmap_k,
                        const __grid_constant__ CUtensorMap tmap_v,
                        const __grid_constant__ CUtensorMap tmap_kr, TcParams p) {
  using C = TcCfg<LANES, KP, VP, MOD, DIFF>;
  static_assert(!DIFF || (LANES == 2 && !MOD && !LAT), "differential attention: one lane per map");
  constexpr int kLaneRows = DIFF ? 0 : kTcRows;     // rows from one lane's tile to the next one's
  extern __shared__ __align__(1024) char smem[];
  if (smem_u32(smem) & 1023u) {       // the swizzled tiles need 1024-byte alignment
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, kStatusBadArgument);
    return;
  }
  char* sQ = smem;                        // one tile per lane
  char* sK = sQ + LANES * C::kQTile;      // two stages
  char* sV = sK + 2 * C::kKTile;          // two stages
  char* sP = sV + 2 * C::kVTile;          // one tile per lane
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + LANES * kTcPTile);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;            // [2]
  uint64_t* k_free = bars + 3;            // [2]
  uint64_t* v_full = bars + 5;            // [2]
  uint64_t* v_free = bars + 7;            // [2]
  uint64_t* lane_bars = bars + 9;         // per lane: s_full[2], s_free[2], p_full, o_done
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + C::kBars);
  volatile uint32_t* abort_flag = tmem_slot + 1;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = int(blockIdx.x) % p.Hq;
  const int kvh = h / (p.Hq / p.Hkv);
  // q0: the block's first query row; rows: how many rows from there on are its sequence's; pos_q0:
  // position of row q0; bt: the sequence's pages
  int q0, rows, pos_q0, ctx0 = 0;
  const int* bt;
  if (p.tiles) {
    pdl_wait();      // the table may have been written by the launch before this one
    const int4 tile = p.tiles[int(blockIdx.x) / p.Hq];
    q0 = tile.x; rows = tile.y; pos_q0 = tile.z;
    bt = p.block_table + size_t(tile.w) * p.max_blocks;
    if (LAT) ctx0 = p.tile_ctx[int(blockIdx.x) / p.Hq];
  } else {
    // long rows of work first: the last query tile walks the most keys
    q0 = (p.n_qt - 1 - int(blockIdx.x) / p.Hq) * (kTcRows * LANES);
    rows = p.T - q0; pos_q0 = p.pos0 + q0;
    bt = p.block_table;
  }
  // steps of lane L: it sees keys [0, kv_end_L); a lane that starts past the last token is idle.
  // With a sliding window or chunks the block's steps start at j0, the step that holds the first key its
  // first row can see (later rows mask what lies before their own first key).
  const int j0 = first_key(pos_q0, p.window, p.chunk) / kTcKeys;
  int n_steps[LANES];
  int n_max = 0, kv_end_max = 1;
#pragma unroll
  for (int L = 0; L < LANES; ++L) {
    const int first = L * kLaneRows;
    const int kv_end = pos_q0 + min(first + kTcRows, rows);
    n_steps[L] = first < rows ? (kv_end + kTcKeys - 1) / kTcKeys - j0 : 0;
    if (n_steps[L] > 0) { n_max = max(n_max, n_steps[L]); kv_end_max = max(kv_end_max, kv_end); }
  }
  const int last_page = (kv_end_max - 1) / kTcPage;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(k_full + i, 1); mbar_init(k_free + i, 1);
      mbar_init(v_full + i, 1); mbar_init(v_free + i, 1);
    }
    for (int L = 0; L < LANES; ++L) {
      uint64_t* lb = lane_bars + 6 * L;
      mbar_init(lb + 0, 1); mbar_init(lb + 1, 1);     // s_full
      mbar_init(lb + 2, 4); mbar_init(lb + 3, 4);     // s_free: one arrival per softmax warp
      mbar_init(lb + 4, 4);                           // p_full
      mbar_init(lb + 5, 1);                           // o_done
    }
    // a wait that gave up earlier in this launch (or one the host has not cleared yet) ends the
    // remaining CTAs at their first wait instead of letting each run out its own polls
    *abort_flag = (p.status && *reinterpret_cast<volatile int*>(p.status) != 0) ? 1u : 0u;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, C::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (elect_one()) {
      tma_prefetch_desc(&tmap_q);
      tma_prefetch_desc(&tmap_k);
      tma_prefetch_desc(&tmap_v);
      pdl_wait();
      int last_k[2] = {-1, -1}, last_v[2] = {-1, -1};   // last step whose loads went to each stage
      const bool q_issued = *abort_flag == 0u;
      if (q_issued) {
        int active = 0;
#pragma unroll
        for (int L = 0; L < LANES; ++L) active += n_steps[L] > 0;
        mbar_arrive_expect_tx(q_full, active * C::kQTile);
#pragma unroll
        for (int L = 0; L < LANES; ++L) {
          if (n_steps[L] == 0) continue;
#pragma unroll
          for (int c = 0; c < KP; ++c)
            tma_load_2d(sQ + L * C::kQTile + c * kTcQPanel, &tmap_q, q_full,
                        (DIFF ? h * 2 + L : h) * p.dk + (LAT && c >= p.kn ? p.q_rot + (c - p.kn) * 64 : c * 64),
                        q0 + L * kLaneRows);
        }
      }
      for (int j = 0; j < n_max; ++j) {
        if (*abort_flag) break;
        const int s = j & 1;
        const uint32_t par = ((j >> 1) & 1) ^ 1;
        int y[kTcPages];
#pragma unroll
        for (int pg = 0; pg < kTcPages; ++pg) {
          // pages past the last one this CTA can see repeat it (their keys are masked)
          const int page = min((j + j0) * kTcPages + pg, last_page);
          y[pg] = (LAT ? bt[page] : bt[page] * p.Hkv + kvh) * kTcPage;
        }
        if (!mbar_wait(k_free + s, par, abort_flag)) break;
        mbar_arrive_expect_tx(k_full + s, C::kKTile);
        last_k[s] = j;
        char* kd = sK + s * C::kKTile;
        if (LAT) {
#pragma unroll
          for (int c = 0; c < KP; ++c) {
            if (c < p.kn) {
              tma_load_3d(kd + c * kTcKvPanel, &tmap_k, k_full + s, c * 64, h, ctx0 + j * kTcKeys);
            } else {
#pragma unroll
              for (int pg = 0; pg < kTcPages; ++pg)
                tma_load_2d(kd + c * kTcKvPanel + pg * kTcPageBytes, &tmap_kr, k_full + s, p.c_rot + (c - p.kn) * 64, y[pg]);
            }
          }
        } else {
#pragma unroll
          for (int pg = 0; pg < kTcPages; ++pg)
#pragma unroll
            for (int c = 0; c < KP; ++c) {
              tma_load_2d(kd + c * kTcKvPanel + pg * kTcPageBytes, &tmap_k, k_full + s, c * 64, y[pg]);
              if (DIFF)          // the second map's columns, through a tensor map of their own
                tma_load_2d(kd + C::kKMap + c * kTcKvPanel + pg * kTcPageBytes, &tmap_kr, k_full + s, c * 64, y[pg]);
            }
        }
        if (!mbar_wait(v_free + s, par, abort_flag)) break;
        mbar_arrive_expect_tx(v_full + s, C::kVTile);
        last_v[s] = j;
        char* vd = sV + s * C::kVTile;
        if (LAT) {
#pragma unroll
          for (int c = 0; c < VP; ++c)
            tma_load_3d(vd + c * kTcKvPanel, &tmap_v, v_full + s, c * 64, h, ctx0 + j * kTcKeys);
        } else {
#pragma unroll
          for (int pg = 0; pg < kTcPages; ++pg)
#pragma unroll
            for (int c = 0; c < VP; ++c)
              tma_load_2d(vd + c * kTcKvPanel + pg * kTcPageBytes, &tmap_v, v_full + s, c * 64, y[pg]);
        }
      }
      if (*abort_flag) {
        // leaving early: let the copies already in flight land before the CTA gives up its
        // shared memory (they complete on their own; the polls are bounded all the same)
        auto drain = [](uint64_t* bar, uint32_t parity) {
          for (uint32_t i = 0; i < (1u << 16); ++i)
            if (mbar_try_wait(bar, parity)) return;
        };
        if (q_issued) drain(q_full, 0);
        for (int s = 0; s < 2; ++s) {
          if (last_k[s] >= 0) drain(k_full + s, (last_k[s] >> 1) & 1);
          if (last_v[s] >= 0) drain(v_full + s, (last_v[s] >> 1) & 1);
        }
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (elect_one()) {
      constexpr uint32_t idesc_s = umma_idesc_bf16_f32(128, kTcKeys);
      constexpr uint32_t idesc_pv = umma_idesc_bf16_f32(128, VP * 64) | kUmmaBMajorMN;
      bool ok = mbar_wait(q_full, 0, abort_flag);
      // S of step j for every lane that still has work
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1;
        const uint32_t u = (j >> 1) & 1;
        if (!mbar_wait(k_full + s, u, abort_flag)) return false;
        const uint32_t k_tile = smem_u32(sK + s * C::kKTile);
#pragma unroll
        for (int L = 0; L < LANES; ++L) {
          if (j >= n_steps[L]) continue;
          const uint32_t k_addr = k_tile + (DIFF ? L * C::kKMap : 0);
          uint64_t* lb = lane_bars + 6 * L;
          if (!mbar_wait(lb + 2 + s, u ^ 1u, abort_flag)) return false;   // s_free
          tc_fence_after_sync();
          const uint32_t q_addr = smem_u32(sQ + L * C::kQTile);
#pragma unroll
          for (int ks = 0; ks < KP * 4; ++ks) {  // 16 of the head dimensions per product
            const uint32_t in_row = (ks & 3) * 32;
            tc_mma_f16(tmem_base + L * 128 + s * kTcKeys,
                       umma_desc_sw128_kmajor(q_addr + (ks >> 2) * kTcQPanel + in_row),
                       umma_desc_sw128_kmajor(k_addr + (ks >> 2) * kTcKvPanel + in_row), idesc_s,
                       ks != 0 ? 1u : 0u);
          }
          tc_commit(lb + s);                      // s_full
        }
        tc_commit(k_free + s);
        return true;
      };
      if (ok && n_max > 0) ok = issue_s(0);
      for (int j = 0; j < n_max && ok; ++j) {
        if (j + 1 < n_max && !issue_s(j + 1)) { ok = false; break; }
        const int s = j & 1;
        if (!mbar_wait(v_full + s, (j >> 1) & 1, abort_flag)) { ok = false; break; }
        const uint32_t v_addr = smem_u32(sV + s * C::kVTile);
#pragma unroll
        for (int L = 0; L < LANES; ++L) {
          if (j >= n_steps[L]) continue;
          uint64_t* lb = lane_bars + 6 * L;
          if (!mbar_wait(lb + 4, j & 1, abort_flag)) { ok = false; break; }   // p_full
          tc_fence_after_sync();
          const uint32_t p_addr = smem_u32(sP + L * kTcPTile);
#pragma unroll
          for (int ks = 0; ks < kTcKeys / 16; ++ks) {       // 16 keys per product
            tc_mma_f16(tmem_base + LANES * 128 + L * (VP * 64), umma_desc_sw128_kmajor(p_addr + ks * 32),
                       umma_desc_sw128_mnmajor(v_addr + ks * 2048, kTcKvPanel), idesc_pv,
                       (j | ks) != 0 ? 1u : 0u);
          }
          tc_commit(lb + 5);                      // o_done
        }
        if (!ok) break;
        tc_commit(v_free + s);
      }
    }
  } else {
    // ---------------------------------------------------------------- softmax warpgroups
    const int L = (warp - 2) >> 2;                     // lane served by this warpgroup
    const int quarter = warp & 3;                      // the 32 TMEM lanes this warp may touch
    const int row = quarter * 32 + lane;
    const uint32_t t_lane = uint32_t(quarter * 32) << 16;
    const uint32_t tmem_s = tmem_base + L * 128 + t_lane;
    const uint32_t tmem_o = tmem_base + LANES * 128 + L * (VP * 64) + t_lane;
    uint64_t* s_full = lane_bars + 6 * L;
    uint64_t* s_free = s_full + 2;
    uint64_t* p_full = s_full + 4;
    uint64_t* o_done = s_full + 5;
    const int lrow = L * kLaneRows + row;              // row inside the block
    const int pos = pos_q0 + lrow, first = first_key(pos, p.window, p.chunk);
    const int my_steps = n_steps[LANES == 1 ? 0 : L];
    const float sc = MOD ? 1.f : p.scale_log2;         // MOD: scores are final, in base 2
    char* prow = sP + L * kTcPTile + row * 128;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    pdl_wait();
    // score modifiers of this head; polynomial coefficients with every constant folded in
    HeadScore hs{};
    float far_in = 0.f;
    uint64_t p0 = 0, p1 = 0, p2 = 0, p3 = 0, p4 = 0;
    float* ring = nullptr;
    int d_low = 0;                                     // smallest distance this warp's step can hold
    if (MOD) {
      hs = head_score(p.mod, h);
      if (hs.capl > 0.f) {
        const float w = hs.inner * hs.inner, f = hs.capl * hs.inner;
        auto both = [](float v) { return pair2(v, v); };
        p0 = both(f * kTanhP0);
        p1 = both(f * w * kTanhP1);
        p2 = both(f * (w * w) * kTanhP2);
        p3 = both(f * (w * w) * w * kTanhP3);
        p4 = both(f * (w * w) * (w * w) * kTanhP4);
        far_in = 2.f * kLog2e * hs.inner;
      } else {
        p0 = pair2(hs.lin, hs.lin);
      }
      if (hs.sink != -INFINITY) { m_used = hs.sink; l = 1.f; }
      ring = reinterpret_cast<float*>(reinterpret_cast<char*>(bars) + 256) + (warp - 2) * kTcBiasRing;
      d_low = pos_q0 + L * kTcRows + quarter * 32 - j0 * kTcKeys - (kTcKeys - 1);
      for (int i = lane; i < 128; i += 32) {
        const int d = d_low + i;
        const float v = -distance_bias(hs, float(max(d, 0)));
        ring[d & 127] = v;
        ring[(d & 127) + 128] = v;
      }
      __syncwarp();
    }
#pragma unroll 1
    for (int j = 0; j < my_steps; ++j) {
      const int sb = j & 1;
      ok = mbar_wait(s_full + sb, (j >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after_sync();
      constexpr int NC = kTcKeys / 32;                 // 32-column chunks of this row of S
      uint32_t r[NC][32];
#pragma unroll
      for (int c = 0; c < NC; ++c) tmem_ld_32x32(tmem_s + sb * kTcKeys + c * 32, r[c]);
      tmem_ld_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(s_free + sb);         // the issuer may overwrite this S now

      const int k0 = (j + j0) * kTcKeys;
      if (MOD) {
        float amax[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int i = 0; i < 32; i += 2)
            amax[(i >> 1) & 3] = max3_abs(amax[(i >> 1) & 3], __uint_as_float(r[c][i]), __uint_as_float(r[c][i + 1]));
        const float top = fmaxf(fmaxf(amax[0], amax[1]), fmaxf(amax[2], amax[3]));
        const float* bias = ring + (d_low & 127) + lane + (kTcKeys - 1);   // bias[-i]: key k0 + i
        if (!__any_sync(0xffffffffu, top * fabsf(hs.inner) > kTanhPolyMax)) {
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const uint64_t a = pair2(__uint_as_float(r[c][i]), __uint_as_float(r[c][i + 1]));
              const uint64_t w = mul2(a, a);
              const uint64_t poly = fma2(fma2(fma2(fma2(p4, w, p3), w, p2), w, p1), w, p0);
              unpair2(fma2(a, poly, pair2(bias[-(c * 32 + i)], bias[-(c * 32 + i + 1)])), r[c][i], r[c][i + 1]);
            }
        } else {
#pragma unroll
          for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const float a = __uint_as_float(r[c][i]);
              const float e = tc_ex2(fminf(a * far_in, 80.f));
              r[c][i] = __float_as_uint(hs.capl - __fdividef(2.f * hs.capl, 1.f + e) + bias[-(c * 32 + i)]);
            }
        }
        // the next step's 64 new distances (all below the ones held)
        __syncwarp();
        d_low -= kTcKeys;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int d = d_low + lane + i * 32;
          const float v = -distance_bias(hs, float(max(d, 0)));
          ring[d & 127] = v;
          ring[(d & 127) + 128] = v;
        }
        __syncwarp();
      }
      if (k0 + kTcKeys - 1 > pos_q0 + L * kLaneRows) {   // the step touches the diagonal
        const int vis = pos - k0;                      // keys k0 .. k0+vis are visible to this row
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i > vis) r[c][i] = 0xff800000u;   // -inf
      }
      if (first > k0) {                                // keys before this row's first one
        const int lo = first - k0;
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < lo) r[c][i] = 0xff800000u;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          if (MOD) {
            mx4[(i >> 1) & 3] = max3(mx4[(i >> 1) & 3], __uint_as_float(r[c][i]), __uint_as_float(r[c][i + 1]));
          } else {
            mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(r[c][i]));
            mx4[(i & 3) + 1] = fmaxf(mx4[(i & 3) + 1], __uint_as_float(r[c][i + 1]));
          }
        }
      const float m_new = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * sc;
      bool waited = false;
      if (__any_sync(0xffffffffu, m_new > m_used + kTcRescaleStep)) {
        const float m_next = fmaxf(m_used, m_new);
        const float alpha = (m_next == -INFINITY) ? 1.f : tc_ex2(m_used - m_next);
        l *= alpha;
        m_used = m_next;
        if (j > 0) {                                    // O holds steps 0..j-1: bring it to the new reference
          ok = mbar_wait(o_done, (j - 1) & 1, abort_flag);
          ok = __all_sync(0xffffffffu, ok);
          if (!ok) break;
          waited = true;
          tc_fence_after_sync();
#pragma unroll 1
          for (int c = 0; c < VP * 2; ++c) {
            uint32_t o[32];
            tmem_ld_32x32(tmem_o + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x32(tmem_o + c * 32, o);
          }
          tmem_st_wait();
        }
      }
      const float sub = (m_used == -INFINITY) ? 0.f : m_used;
      uint32_t w[kTcKeys / 2];
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      if (MOD) {
        const uint64_t sub2 = pair2(-sub, -sub);
        uint64_t acc[2] = {0, 0};
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            uint32_t x0, x1;
            unpair2(add2(pair2(__uint_as_float(r[c][i]), __uint_as_float(r[c][i + 1])), sub2), x0, x1);
            const float e0 = tc_ex2(__uint_as_float(x0)), e1 = tc_ex2(__uint_as_float(x1));
            acc[(i >> 1) & 1] = add2(acc[(i >> 1) & 1], pair2(e0, e1));
            w[c * 16 + (i >> 1)] = pack_bf16(e0, e1);
          }
        uint32_t lo, hi;
        unpair2(add2(acc[0], acc[1]), lo, hi);
        sum4[0] = __uint_as_float(lo) + __uint_as_float(hi);
      } else
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float p0 = tc_ex2(fmaf(__uint_as_float(r[c][i]), sc, -sub));
          const float p1 = tc_ex2(fmaf(__uint_as_float(r[c][i + 1]), sc, -sub));
          sum4[(i >> 1) & 3] += p0 + p1;
          w[c * 16 + (i >> 1)] = pack_bf16(p0, p1);
        }
      l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      if (j > 0 && !waited) {                           // P V of the previous step still reads sP
        ok = mbar_wait(o_done, (j - 1) & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
      }
#pragma unroll
      for (int c = 0; c < kTcKeys / 8; ++c)             // 16-byte chunks: 8 keys each
        *reinterpret_cast<uint4*>(prow + ((c ^ (row & 7)) << 4)) =
            make_uint4(w[c * 4], w[c * 4 + 1], w[c * 4 + 2], w[c * 4 + 3]);
      fence_proxy_async_smem();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    if (ok && my_steps > 0) {
      ok = mbar_wait(o_done, (my_steps - 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (DIFF) {
      // both lanes arrive at both barriers whatever happened; this lane's P tile is free once its last product is done
      float* mine = reinterpret_cast<float*>(sP + L * kTcPTile);
      const float* other = reinterpret_cast<const float*>(sP + (1 - L) * kTcPTile);
      const float own = l > 0.f ? 1.f / l : 0.f;
      if (ok) mine[row] = own;
      named_bar_sync(1, 256);
      const bool whole = __all_sync(0xffffffffu, ok) && *abort_flag == 0u;
      float v[VP * 32], ssq = 0.f;
      if (whole) {
        tc_fence_after_sync();
        const float theirs = other[row];
        const float f1 = L == 0 ? own : theirs, f2 = (L == 0 ? theirs : own) * p.diff.weight;
        const uint32_t o1 = tmem_base + LANES * 128 + t_lane, o2 = o1 + VP * 64;
#pragma unroll
        for (int c = 0; c < VP; ++c) {                   // this lane's half of the value columns
          uint32_t a[32], b[32];
          tmem_ld_32x32(o1 + (L * VP + c) * 32, a);
          tmem_ld_32x32(o2 + (L * VP + c) * 32, b);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {                 // (columns past the head's width are zero)
            v[c * 32 + i] = __uint_as_float(a[i]) * f1 - __uint_as_float(b[i]) * f2;
            ssq += v[c * 32 + i] * v[c * 32 + i];
          }
        }
        mine[kTcRows + row] = ssq;
      }
      named_bar_sync(1, 256);
      if (whole && lrow < rows) {
        const float inv = p.diff.scale / sqrtf((ssq + other[kTcRows + row]) / float(p.vdim) + p.diff.eps);
        __nv_bfloat16* dst = p.out + (size_t(q0 + lrow) * p.Hq + h) * p.dv + L * VP * 32;
#pragma unroll
        for (int u = 0; u < VP * 4; ++u) {
          if (L * VP * 32 + u * 8 >= p.dv) break;        // dv is a multiple of 8
          uint4 pk;
          pk.x = pack_bf16(v[u * 8] * inv, v[u * 8 + 1] * inv);
          pk.y = pack_bf16(v[u * 8 + 2] * inv, v[u * 8 + 3] * inv);
          pk.z = pack_bf16(v[u * 8 + 4] * inv, v[u * 8 + 5] * inv);
          pk.w = pack_bf16(v[u * 8 + 6] * inv, v[u * 8 + 7] * inv);
          *reinterpret_cast<uint4*>(dst + u * 8) = pk;
        }
      }
    } else if (ok && my_steps > 0) {
      tc_fence_after_sync();
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (p.gate.gate) inv *= head_gate<__nv_bfloat16>(p.gate, size_t(q0 + min(lrow, rows - 1)), h);
      __nv_bfloat16* dst = p.out + (size_t(q0 + min(lrow, rows - 1)) * p.Hq + h) * p.dv;
#pragma unroll 1
      for (int c = 0; c < VP * 2; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_o + c * 32, o);
        tmem_ld_wait();
        if (lrow < rows) {
#pragma unroll
          for (int v = 0; v < 4; ++v) {
            if (c * 32 + v * 8 >= p.dv) break;           // dv is a multiple of 8
            uint4 pk;
            pk.x = pack_bf16(__uint_as_float(o[v * 8]) * inv, __uint_as_float(o[v * 8 + 1]) * inv);
            pk.y = pack_bf16(__uint_as_float(o[v * 8 + 2]) * inv, __uint_as_float(o[v * 8 + 3]) * inv);
            pk.z = pack_bf16(__uint_as_float(o[v * 8 + 4]) * inv, __uint_as_float(o[v * 8 + 5]) * inv);
            pk.w = pack_bf16(__uint_as_float(o[v * 8 + 6]) * inv, __uint_as_float(o[v * 8 + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + v * 8) = pk;
          }
        }
      }
    }
  }

  // ------------------------------------------------------------------ teardown
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, C::kTmemCols);
  }
  if (threadIdx.x == 0 && *abort_flag && p.status) atomicExch(p.status, kStatusMbarTimeout);
  pdl_launch_dependents();
}

template <int LANES, int KP, int VP, bool MOD, bool LAT = false, bool DIFF = false>
static int launch_prefill_tc(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv,
                             TcParams p, int pdl, cudaStream_t st, const CUtensorMap* tkr = nullptr) {
  auto kern = flash_prefill_tc_kernel<LANES, KP, VP, MOD, LAT, DIFF>;
  using C = TcCfg<LANES, KP, VP, MOD, DIFF>;
  constexpr size_t smem = C::kSmem;
  RB_CHECK(set_max_smem(kern, smem));
  if (!p.tiles) p.n_qt = (p.T + kTcRows * LANES - 1) / (kTcRows * LANES);
  return launch(kern, dim3(p.n_qt * p.Hq), dim3(C::kThreads), smem, st, pdl != 0, tq, tk, tv,
                tkr ? *tkr : tk, p);
}

static int prefill_tc_maps(CUtensorMap* tq, CUtensorMap* tk, CUtensorMap* tv, const void* q, const void* k_cache,
                           const void* v_cache, int T, int Hq, int Hkv, int dk, int dv, int num_blocks) {
  int rc = make_tmap_2d_bf16(tq, q, uint64_t(Hq) * dk, uint64_t(T), uint64_t(Hq) * dk * 2, 64, kTcRows);
  if (rc) return rc;
  const uint64_t rows = uint64_t(num_blocks) * Hkv * kTcPage;
  rc = make_tmap_2d_bf16(tk, k_cache, uint64_t(dk), rows, uint64_t(dk) * 2, 64, kTcPage);
  if (rc) return rc;
  return make_tmap_2d_bf16(tv, v_cache, uint64_t(dv), rows, uint64_t(dv) * 2, 64, kTcPage);
}

}  // namespace rb

using namespace rb;

// 1 when the tensor-core kernel covers the shape (head_dim 128; any sliding window).
extern "C" int rmlx_flash_prefill_tc_supported(int HD, int window) {
  (void)window;
  return HD == kTcHd;
}

// q, out: [T, Hq, 128] bf16; caches [num_blocks, Hkv, 16, 128] bf16; block_table: the sequence's
// pages (int32, device); queries sit at positions pos0 .. pos0+T-1 and the cache already holds keys
// 0 .. pos0+T-1. window > 0: sliding-window attention over the last `window` keys. lanes: query tiles per CTA, 1 or 2 (0 = choose; one tile measured at least as
// fast as two at every length tried, so that is the choice). status: optional device int set
// non-zero if a pipeline wait gave up.
extern "C" int rmlx_flash_prefill_tc(const void* q, const void* k_cache, const void* v_cache,
                                     const int* block_table, void* out, int T, int Hq, int Hkv,
                                     int HD, int num_blocks, int pos0, int window, float scale,
                                     int lanes, int* status, int pdl, cudaStream_t st) {
  if (T < 1 || HD != kTcHd || Hkv < 1 || Hq % Hkv || pos0 < 0 || num_blocks < 1) return -2;
  if (lanes == 0) lanes = 1;
  if (lanes != 1 && lanes != 2) return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) |
       reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(out)) & 15)
    return -2;
  CUtensorMap tq, tk, tv;
  const int rc = prefill_tc_maps(&tq, &tk, &tv, q, k_cache, v_cache, T, Hq, Hkv, kTcHd, kTcHd, num_blocks);
  if (rc) return rc;
  TcParams p{};
  p.block_table = block_table;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.pos0 = pos0;
  p.n_qt = 0;
  p.dk = p.dv = kTcHd;
  p.tiles = nullptr; p.max_blocks = 0;
  p.window = window > 0 ? window : 0;
  p.scale_log2 = scale * kLog2e;
  p.status = status;
  return lanes == 2 ? launch_prefill_tc<2, 2, 2, false>(tq, tk, tv, p, pdl, st)
                    : launch_prefill_tc<1, 2, 2, false>(tq, tk, tv, p, pdl, st);
}

// 1 when the form with score modifiers takes these key and value row widths.
extern "C" int rmlx_flash_prefill_scored_supported(int dk, int dv) {
  return dk >= 8 && dv >= 8 && dk % 8 == 0 && dv % 8 == 0 && dk <= 128 && dv <= 128;
}

// Ragged batch with score modifiers. q [T, Hq, dk] and out [T, Hq, dv] bf16, caches [num_blocks, Hkv, 16,
// dk / dv] bf16 already holding the rows' own keys and values; tiles: n_tiles x {first row, rows (1 .. lanes * 128),
// position of the first row, row of block_table [.., max_blocks]} (int32, device), heaviest first.
// gate: bf16 [T, ldg] output gate logits, or null.
extern "C" int rmlx_flash_prefill_scored(const void* q, const void* k_cache, const void* v_cache,
                                         const int* block_table, int max_blocks, const int* tiles, int n_tiles,
                                         void* out, int T, int Hq, int Hkv, int dk, int dv, int num_blocks,
                                         int window, int chunk, float scale, float softcap, const float* temp,
                                         const float* r1, const float* r2, const float* sink, const void* gate,
                                         int ldg, int lanes, int* status, int pdl, cudaStream_t st) {
  if (T < 1 || (lanes != 1 && lanes != 2) || Hkv < 1 || Hq % Hkv || num_blocks < 1 || n_tiles < 1 || !tiles || (r1 && !r2) ||
      !rmlx_flash_prefill_scored_supported(dk, dv))
    return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) |
       reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(out) |
       reinterpret_cast<uintptr_t>(tiles)) & 15)
    return -2;
  CUtensorMap tq, tk, tv;
  const int rc = prefill_tc_maps(&tq, &tk, &tv, q, k_cache, v_cache, T, Hq, Hkv, dk, dv, num_blocks);
  if (rc) return rc;
  TcParams p{};
  p.block_table = block_table; p.max_blocks = max_blocks;
  p.tiles = reinterpret_cast<const int4*>(tiles); p.n_qt = n_tiles;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.pos0 = 0;
  p.dk = dk; p.dv = dv;
  p.window = window > 0 ? window : 0; p.chunk = chunk > 0 ? chunk : 0;
  p.scale_log2 = 1.f;
  p.mod.scale = scale; p.mod.softcap = softcap; p.mod.temp = temp; p.mod.r1 = r1; p.mod.r2 = r2; p.mod.sink = sink;
  p.gate.gate = gate; p.gate.ld = ldg;
  p.status = status;
  // no modifier but the scale: the plain softmax
  const bool plain = softcap <= 0.f && !temp && !r1 && !sink;
  if (plain) p.scale_log2 = scale * kLog2e;
#define RB_FPS(KP_, VP_)                                                             \
  if (plain)                                                                         \
    return lanes == 2 ? launch_prefill_tc<2, KP_, VP_, false>(tq, tk, tv, p, pdl, st)  \
                      : launch_prefill_tc<1, KP_, VP_, false>(tq, tk, tv, p, pdl, st); \
  return lanes == 2 ? launch_prefill_tc<2, KP_, VP_, true>(tq, tk, tv, p, pdl, st)   \
                    : launch_prefill_tc<1, KP_, VP_, true>(tq, tk, tv, p, pdl, st)
  if (dk > 64) {
    if (dv > 64) { RB_FPS(2, 2); }
    RB_FPS(2, 1);
  }
  if (dv > 64) { RB_FPS(1, 2); }
  RB_FPS(1, 1);
#undef RB_FPS
}

// Differential attention over a ragged batch: q [T, Hq, 2, dk], keys [num_blocks, Hkv, 16, 2 dk] = [map 1 | map 2], values
// [num_blocks, Hkv, 16, dv], of which vdim exist (the rest are zero); out [T, Hq, dv] = map_scale * d / rms(d), d = the
// first map's attention - map_weight * the second's. tiles: at most 128 rows each. dk, dv as
// rmlx_flash_prefill_scored_supported.
extern "C" int rmlx_flash_prefill_diff(const void* q, const void* k_cache, const void* v_cache, const int* block_table,
                                       int max_blocks, const int* tiles, int n_tiles, void* out, int T, int Hq, int Hkv, int dk,
                                       int dv, int vdim, int num_blocks, int window, int chunk, float scale, float map_weight,
                                       float map_scale, float map_eps, int* status, int pdl, cudaStream_t st) {
  if (T < 1 || Hkv < 1 || Hq % Hkv || num_blocks < 1 || n_tiles < 1 || !tiles || vdim < 1 || vdim > dv ||
      !rmlx_flash_prefill_scored_supported(dk, dv))
    return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) |
       reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(out) |
       reinterpret_cast<uintptr_t>(tiles)) & 15)
    return -2;
  CUtensorMap tq, tk, tv, tk2;
  int rc = make_tmap_2d_bf16(&tq, q, uint64_t(Hq) * 2 * dk, uint64_t(T), uint64_t(Hq) * 4 * dk, 64, kTcRows);
  if (rc) return rc;
  const uint64_t rows = uint64_t(num_blocks) * Hkv * kTcPage;
  rc = make_tmap_2d_bf16(&tk, k_cache, uint64_t(dk), rows, uint64_t(dk) * 4, 64, kTcPage);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tk2, static_cast<const __nv_bfloat16*>(k_cache) + dk, uint64_t(dk), rows, uint64_t(dk) * 4, 64, kTcPage);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tv, v_cache, uint64_t(dv), rows, uint64_t(dv) * 2, 64, kTcPage);
  if (rc) return rc;
  TcParams p{};
  p.block_table = block_table; p.max_blocks = max_blocks;
  p.tiles = reinterpret_cast<const int4*>(tiles); p.n_qt = n_tiles;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.pos0 = 0;
  p.dk = dk; p.dv = dv; p.vdim = vdim;
  p.window = window > 0 ? window : 0; p.chunk = chunk > 0 ? chunk : 0;
  p.scale_log2 = scale * kLog2e;
  p.diff.weight = map_weight; p.diff.scale = map_scale; p.diff.eps = map_eps;
  p.status = status;
#define RB_FPD(KP_, VP_) return launch_prefill_tc<2, KP_, VP_, false, false, true>(tq, tk, tv, p, pdl, st, &tk2)
  if (dk > 64) { if (dv > 64) RB_FPD(2, 2); RB_FPD(2, 1); }
  if (dv > 64) RB_FPD(1, 2);
  RB_FPD(1, 1);
#undef RB_FPD
}

// 1 when the latent form takes these (eight-padded) widths: unrotated, rotated, value.
extern "C" int rmlx_flash_prefill_latent_supported(int dim, int rot, int dv) {
  return dim >= 8 && dim <= 128 && dim % 8 == 0 && rot >= 8 && rot <= 64 && rot % 8 == 0 && dv >= 8 && dv <= 128 && dv % 8 == 0;
}

// Latent attention over a ragged batch. q [T, H, dim + rot], out [T, H, dv]; kv [ctx_rows, H, dim + dv]: keys and
// values of the contexts, tile i's sequence from row tile_ctx[i] (a multiple of 16) on; cache [num_blocks, 16,
// ldc] with the rotated key part at column c_rot of a row; all bf16. tiles and block_table as above.
extern "C" int rmlx_flash_prefill_latent(const void* q, const void* kv, const void* cache, const int* block_table,
                                         int max_blocks, const int* tiles, const int* tile_ctx, int n_tiles, void* out,
                                         int T, int H, int dim, int rot, int dv, int ctx_rows, int num_blocks, int ldc,
                                         int c_rot, float scale, int lanes, int* status, int pdl, cudaStream_t st) {
  if (T < 1 || H < 1 || (lanes != 1 && lanes != 2) || n_tiles < 1 || !tiles || !tile_ctx || ctx_rows < 1 || num_blocks < 1 ||
      ldc % 8 || c_rot % 8 || c_rot + rot > ldc || !rmlx_flash_prefill_latent_supported(dim, rot, dv))
    return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(cache) |
       reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(tiles)) & 15)
    return -2;
  const int dk = dim + rot, per = dim + dv;
  CUtensorMap tq, tk, tv, tkr;
  int rc = make_tmap_2d_bf16(&tq, q, uint64_t(H) * dk, uint64_t(T), uint64_t(H) * dk * 2, 64, kTcRows);
  if (rc) return rc;
  rc = make_tmap_3d_bf16(&tk, kv, dim, H, ctx_rows, uint64_t(per) * 2, uint64_t(H) * per * 2, 64, 1, kTcKeys);
  if (rc) return rc;
  rc = make_tmap_3d_bf16(&tv, static_cast<const __nv_bfloat16*>(kv) + dim, dv, H, ctx_rows, uint64_t(per) * 2,
                         uint64_t(H) * per * 2, 64, 1, kTcKeys);
  if (rc) return rc;
  rc = make_tmap_2d_bf16(&tkr, cache, uint64_t(c_rot) + rot, uint64_t(num_blocks) * kTcPage, uint64_t(ldc) * 2, 64, kTcPage);
  if (rc) return rc;
  TcParams p{};
  p.block_table = block_table; p.max_blocks = max_blocks;
  p.tiles = reinterpret_cast<const int4*>(tiles); p.n_qt = n_tiles; p.tile_ctx = tile_ctx;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.T = T; p.Hq = H; p.Hkv = H; p.pos0 = 0;
  p.dk = dk; p.dv = dv;
  p.kn = dim > 64 ? 2 : 1; p.q_rot = dim; p.c_rot = c_rot;
  p.scale_log2 = scale * kLog2e;
  p.status = status;
#define RB_FPL(KP_, VP_)                                                                          \
  return lanes == 2 ? launch_prefill_tc<2, KP_, VP_, false, true>(tq, tk, tv, p, pdl, st, &tkr)   \
                    : launch_prefill_tc<1, KP_, VP_, false, true>(tq, tk, tv, p, pdl, st, &tkr)
  if (dim > 64) { if (dv > 64) RB_FPL(3, 2); RB_FPL(3, 1); }
  if (dv > 64) RB_FPL(2, 2);
  RB_FPL(2, 1);
#undef RB_FPL
}
