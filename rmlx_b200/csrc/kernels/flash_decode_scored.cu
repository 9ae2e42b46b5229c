// Paged flash-decode attention with score modifiers (score_mod.cuh): one new query token per row,
// grouped-query heads, different key and value widths, temperature / soft cap / distance bias /
// sink / sliding window / chunked visibility.
//
// Same decomposition as flash_decode.cu: a block owns one (row, kv head, 16-query-head tile, KV
// split); its four warps walk the split's 16-token pages with cp.async rings into swizzled shared
// memory and m16n8k16 tiles (the useful M is 16 rows and the kernel is bound by KV bytes and latency);
// warps merge through shared memory, splits through the last block of a tile. The sink joins the
// denominator once, in the final merge.
//
// Fused form (raw != nullptr): the input is the row's un-normalised fp32 projection [q | k | v]. Every
// block takes the root mean squares of the whole query and key projections itself (a few thousand
// values from L2), normalises its heads' queries, and the block whose split ends the sequence
// normalises and appends the new key and value first: norm, append and attention are one launch.
//
// MAPS 2: differential attention (score_mod.cuh). A tile holds eight query heads: rows 0 - 7 are their first maps'
// queries, rows 8 - 15 their second ones'. A page's keys come as two tiles, one per map; both score products take all
// sixteen rows (each is used for its own half), after which everything up to the merge is as with one map. The merge
// forms the difference of rows r and r + 8, norms it and writes one head.
//
// Rows in shared memory are padded to the class width (64 or 128) with zeros; global memory holds
// dkp / dvp elements per row (multiples of eight), so narrow heads cost no extra bytes.
#include "../common/launch.cuh"
#include "../common/rows.cuh"
#include "../common/score_mod.cuh"

namespace rb {

constexpr int kFsPage = 16;
constexpr int kFsWarps = 4;
constexpr int kFsThreads = kFsWarps * 32;
constexpr int kFsMaxSplits = 64;

__device__ __forceinline__ void fs_cp_async16(void* smem_dst, const void* gsrc) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void fs_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void fs_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void fs_ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void fs_ldm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void fs_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct FsParams {
  const __nv_bfloat16* q;        // plain form: [batch rows, Hq, dkp]
  const float* raw;              // fused form: [batch rows, raw_ld] = [q | k | v], dim / vdim wide heads
  const float* q_w;              // fused form: norm weights [Hq * dim], [Hkv * dim]
  const float* k_w;
  __nv_bfloat16* k_cache;        // [blocks, Hkv, 16, dkp]
  __nv_bfloat16* v_cache;        // [blocks, Hkv, 16, dvp]
  const int* block_table;        // [table rows, max_blocks]
  const int* positions;          // [batch rows] position of the row's token; it sees keys 0 .. position
  const int* rows;               // [B] batch row of each launch row (null: the same)
  const int* table_rows;         // [batch rows] row of the block table (null: the same)
  __nv_bfloat16* out;            // [batch rows, Hq, dvp]
  float* part_o;                 // [B, Hkv*gtiles, S, 16, DV class]
  float* part_ml;                // [B, Hkv*gtiles, S, 16, 2]
  unsigned int* tickets;         // [B * Hkv*gtiles], zero on entry, zero on exit
  int raw_ld, max_blocks, Hq, Hkv, G, gtiles, S, window, chunk, dim, vdim, dkp, dvp;
  int head_norm;                 // fused form: 1: q_w / k_w are [dim], every head is normed on its own; 2: no norm
  // fused form with head_norm: bias of the projection (its layout), rotation of values i and i + rot_dims / 2 by position *
  // inv_freq[i] with cos and sin times `grow`, both before the norm; q_w / k_w may then be null (no weight).
  // neighbours: values 2 i and 2 i + 1 turn together instead
  const float* bias;
  const float* inv_freq;
  int rot_dims, neighbours;
  float grow;
  int gate_col;                  // fused form: gate logits at raw[b][gate_col + head] (< 0: none)
  float eps;
  ScoreMod mod;
  HeadGate gate;                 // plain form
  MapDiff diff;                  // MAPS 2: query heads and key rows are 2 dkp wide, [map 1 | map 2]
};

__device__ __forceinline__ float fs_block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const float t = red[0] + red[1] + red[2] + red[3];
  __syncthreads();
  return t;
}

// One warp copies a page of 16 rows of `chunks` 16-byte pieces into swizzled rows of ROW_BYTES.
template <int ROW_BYTES>
__device__ __forceinline__ void fs_copy_page(char* dst, const char* src, int chunks, int lane) {
  constexpr int FULL = ROW_BYTES / 16;
  if (chunks == FULL) {
#pragma unroll
    for (int u = 0; u < kFsPage * FULL / 32; ++u) {
      const int i = u * 32 + lane, r = i / FULL, c = i % FULL;
      fs_cp_async16(dst + r * ROW_BYTES + ((c ^ (r & 7)) << 4), src + i * 16);
    }
  } else {
    for (int i = lane; i < kFsPage * chunks; i += 32) {
      const int r = i / chunks, c = i - r * chunks;
      fs_cp_async16(dst + r * ROW_BYTES + ((c ^ (r & 7)) << 4), src + i * 16);
    }
  }
}

// The same for rows that hold MAPS keys of `chunks` pieces side by side: a tile of its own for each.
template <int ROW_BYTES, int MAPS>
__device__ __forceinline__ void fs_copy_maps(char* dst, const char* src, int chunks, int lane) {
  if (MAPS == 1) { fs_copy_page<ROW_BYTES>(dst, src, chunks, lane); return; }
  constexpr int FULL = ROW_BYTES / 16;
  if (chunks == FULL) {
#pragma unroll
    for (int u = 0; u < kFsPage * MAPS * FULL / 32; ++u) {
      const int i = u * 32 + lane, r = i / (MAPS * FULL), a = i / FULL % MAPS, c = i % FULL;
      fs_cp_async16(dst + a * (kFsPage * ROW_BYTES) + r * ROW_BYTES + ((c ^ (r & 7)) << 4), src + i * 16);
    }
    return;
  }
  const int per = MAPS * chunks;
  for (int i = lane; i < kFsPage * per; i += 32) {
    const int r = i / per, q = i - r * per, a = q / chunks, c = q - a * chunks;
    fs_cp_async16(dst + a * (kFsPage * ROW_BYTES) + r * ROW_BYTES + ((c ^ (r & 7)) << 4), src + i * 16);
  }
}

// MOD = false: no modifier but the scale.
template <int DK, int DV, int NST, bool MOD, int MAPS>
__global__ void __launch_bounds__(kFsThreads) flash_decode_scored_kernel(FsParams p) {
  constexpr int KS = DK / 16;            // k-steps of the QK^T product
  constexpr int NT = DV / 8;             // n-tiles of the PV product
  constexpr int K_TILE = kFsPage * DK * 2, K_PAGE = MAPS * K_TILE, V_PAGE = kFsPage * DV * 2;
  constexpr int HPT = 16 / MAPS;         // query heads per tile
  constexpr int STAGE = K_PAGE + V_PAGE;
  extern __shared__ __align__(128) char smem[];
  char* wsm = smem + (threadIdx.x >> 5) * (NST * STAGE);   // reused for the merges afterwards
  __shared__ float s_m[kFsWarps][16], s_l[kFsWarps][16];
  __shared__ float s_sink[16], s_gate[16];
  __shared__ float red[kFsWarps];
  __shared__ __align__(16) __nv_bfloat16 sQ[16][DK + 8];
  __shared__ unsigned int s_last;

  const int split = blockIdx.x, yt = blockIdx.y, lb = blockIdx.z;
  const int kvh = yt / p.gtiles, gt = yt % p.gtiles;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t = lane & 3;

  pdl_launch_dependents();
  // narrow heads: shared memory starts at zero, the columns past dkp / dvp are never written again
  if (p.dkp < DK || p.dvp < DV)
    for (int i = lane; i < NST * STAGE / 16; i += 32) reinterpret_cast<uint4*>(wsm)[i] = make_uint4(0u, 0u, 0u, 0u);
  pdl_wait();
  const int b = p.rows ? p.rows[lb] : lb;
  const int len = p.positions[b] + 1;
  const int first = first_key(len - 1, p.window, p.chunk);   // first visible token
  const int pg_begin = first / kFsPage;
  const int pg_end = (len + kFsPage - 1) / kFsPage;
  const int pg_per_split = (pg_end - pg_begin + p.S - 1) / p.S;
  const int pg0 = pg_begin + split * pg_per_split;
  const int pg1 = min(pg0 + pg_per_split, pg_end);
  const int* bt = p.block_table + size_t(p.table_rows ? p.table_rows[b] : b) * p.max_blocks;

  // ---- ask for the first pages before anything else, so that their latency runs beside the query
  // staging. Fused form: the page of the new token waits until the key and value are in it. ----
  const int kch = p.dkp >> 3, vch = p.dvp >> 3;      // 16-byte chunks per row in global memory
  auto issue = [&](int pg, int stage) {
    const int blk = RB_BOUNDS(pg, p.max_blocks) ? bt[pg] : 0;
    const size_t pgi = (size_t(blk) * p.Hkv + kvh) * kFsPage;
    char* kd = wsm + stage * STAGE;
    fs_copy_maps<DK * 2, MAPS>(kd, reinterpret_cast<const char*>(p.k_cache + pgi * (MAPS * p.dkp)), kch, lane);
    fs_copy_page<DV * 2>(kd + K_PAGE, reinterpret_cast<const char*>(p.v_cache + pgi * p.dvp), vch, lane);
  };

  const bool owner = p.raw && pg0 < pg1 && pg1 == pg_end;    // this split ends the sequence
  const int late = owner ? pg_end - 1 : -1;
  __syncwarp();                                              // the warp's zero fill is complete
  int pg = pg0 + warp;
#pragma unroll
  for (int s = 0; s < NST; ++s) {
    if (pg + s * kFsWarps < pg1 && pg + s * kFsWarps != late) issue(pg + s * kFsWarps, s);
    fs_commit();
  }

  // ---- queries of this tile: 16 rows (heads beyond G are zero) ----
  if (p.raw) {
    const float* row = p.raw + size_t(b) * p.raw_ld;
    const int nq = p.Hq * MAPS * p.dim, nk = p.Hkv * MAPS * p.dim;
    if (MAPS > 1 || p.head_norm) {
      // one warp per query head in turn; the owner's last warp also takes the new key's root mean square
      constexpr int PL = DK / 32;
      const int q_heads = min(HPT, p.G - gt * HPT), half = p.rot_dims >> 1;
      // the rotation of this lane's places: own value times cs, partner's (at `other`) times sn
      float cs[PL], sn[PL];
      int other[PL];
#pragma unroll
      for (int i = 0; i < PL; ++i) {
        const int d = i * 32 + lane;
        cs[i] = 1.f; sn[i] = 0.f; other[i] = d;
        if (d < p.rot_dims) {
          const bool low = p.neighbours ? !(d & 1) : d < half;
          float sv, cv;
          rotary_sincos(len - 1, p.inv_freq[p.neighbours ? d >> 1 : low ? d : d - half], sv, cv);
          cs[i] = cv * p.grow;
          sn[i] = (low ? -sv : sv) * p.grow;
          other[i] = p.neighbours ? d ^ 1 : low ? d + half : d - half;
        }
      }
      const bool rot = p.rot_dims > 0;
      auto load_head = [&](int at, bool live, float (&v)[PL], float (&u)[PL]) {
#pragma unroll
        for (int i = 0; i < PL; ++i) v[i] = (live && i * 32 + lane < p.dim) ? __ldcg(row + at + i * 32 + lane) : 0.f;
        if (rot) {
#pragma unroll
          for (int i = 0; i < PL; ++i) u[i] = (live && i * 32 + lane < p.rot_dims) ? __ldcg(row + at + other[i]) : 0.f;
        }
        if (p.bias && live) {
#pragma unroll
          for (int i = 0; i < PL; ++i) {
            if (i * 32 + lane < p.dim) v[i] += p.bias[at + i * 32 + lane];
            if (rot && i * 32 + lane < p.rot_dims) u[i] += p.bias[at + other[i]];
          }
        }
      };
      auto turn = [&](float (&v)[PL], const float (&u)[PL]) {     // returns 1 / rms (1 without a norm)
        if (rot) {
#pragma unroll
          for (int i = 0; i < PL; ++i) v[i] = fmaf(v[i], cs[i], u[i] * sn[i]);
        }
        if (p.head_norm != 1) return 1.f;
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < PL; ++i) ss += v[i] * v[i];
        return 1.f / sqrtf(warp_sum(ss) / float(p.dim) + p.eps);
      };
      float v[4][PL], u[4][PL];
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const int r = warp * 4 + w, hd = r % HPT, a = r / HPT;
        load_head(((kvh * p.G + gt * HPT + hd) * MAPS + a) * p.dim, hd < q_heads, v[w], u[w]);
      }
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float iq = turn(v[w], u[w]);
#pragma unroll
        for (int i = 0; i < PL; ++i) {
          const int d = i * 32 + lane;
          sQ[warp * 4 + w][d] = __float2bfloat16_rn(d < p.dim ? v[w][i] * iq * (p.q_w ? p.q_w[d] : 1.f) : 0.f);
        }
      }
      if (owner && RB_BOUNDS((len - 1) / kFsPage, p.max_blocks)) {
        const size_t slot = (size_t(bt[(len - 1) / kFsPage]) * p.Hkv + kvh) * kFsPage + (len - 1) % kFsPage;
        __nv_bfloat16* kd = p.k_cache + slot * (MAPS * p.dkp);
        __nv_bfloat16* vd = p.v_cache + slot * p.dvp;
        if (warp >= kFsWarps - MAPS) {
          const int a = warp - (kFsWarps - MAPS);
          load_head(nq + (kvh * MAPS + a) * p.dim, true, v[0], u[0]);
          const float ik = turn(v[0], u[0]);
#pragma unroll
          for (int i = 0; i < PL; ++i) {
            const int d = i * 32 + lane;
            if (d < p.dim) kd[a * p.dkp + d] = __float2bfloat16_rn(v[0][i] * ik * (p.k_w ? p.k_w[d] : 1.f));
          }
        }
        for (int d = threadIdx.x; d < p.vdim; d += kFsThreads) {
          const int at = nq + nk + kvh * p.vdim + d;
          vd[d] = __float2bfloat16_rn(__ldcg(row + at) + (p.bias ? p.bias[at] : 0.f));
        }
      }
    } else {
    // this thread's share of the tile's queries, un-normalised but weighted (independent loads)
    constexpr int QPT = 16 * DK / kFsThreads;
    float qv[QPT];
    const int q_rows = min(16, p.G - gt * 16);
#pragma unroll
    for (int u = 0; u < QPT; ++u) {
      const int i = u * kFsThreads + threadIdx.x, r = i / DK, d = i % DK;
      const int src = (kvh * p.G + gt * 16 + r) * p.dim + d;
      qv[u] = (r < q_rows && d < p.dim) ? __ldcg(row + src) * p.q_w[src] : 0.f;
    }
    float sq = 0.f, sk = 0.f;
    if (((nq | nk | p.raw_ld) & 3) == 0) {
      const float4* row4 = reinterpret_cast<const float4*>(row);
      const int n4 = (nq + nk) >> 2, q4 = nq >> 2;
      for (int i0 = threadIdx.x; i0 < n4; i0 += kFsThreads * 8) {
        float4 v[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const int i = i0 + u * kFsThreads;
          v[u] = i < n4 ? __ldcg(row4 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const float s = v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
          if (i0 + u * kFsThreads < q4) sq += s; else sk += s;
        }
      }
    } else {
      for (int i = threadIdx.x; i < nq + nk; i += kFsThreads) {
        const float v = __ldcg(row + i);
        if (i < nq) sq += v * v; else sk += v * v;
      }
    }
    sq = fs_block_sum(sq, red);
    sk = fs_block_sum(sk, red);
    const float iq = 1.f / sqrtf(sq / float(nq) + p.eps), ik = 1.f / sqrtf(sk / float(nk) + p.eps);
#pragma unroll
    for (int u = 0; u < QPT; ++u) {
      const int i = u * kFsThreads + threadIdx.x;
      sQ[i / DK][i % DK] = __float2bfloat16_rn(qv[u] * iq);
    }
    if (owner && RB_BOUNDS((len - 1) / kFsPage, p.max_blocks)) {
      // append the new key and value before this block reads their page
      const size_t slot = (size_t(bt[(len - 1) / kFsPage]) * p.Hkv + kvh) * kFsPage + (len - 1) % kFsPage;
      __nv_bfloat16* kd = p.k_cache + slot * p.dkp;
      __nv_bfloat16* vd = p.v_cache + slot * p.dvp;
      for (int d = threadIdx.x; d < p.dim; d += kFsThreads)
        kd[d] = __float2bfloat16_rn(__ldcg(row + nq + kvh * p.dim + d) * ik * p.k_w[kvh * p.dim + d]);
      for (int d = threadIdx.x; d < p.vdim; d += kFsThreads)
        vd[d] = __float2bfloat16_rn(__ldcg(row + nq + nk + kvh * p.vdim + d));
    }
    }
  } else {
    for (int i = threadIdx.x; i < 16 * (DK / 8); i += kFsThreads) {
      const int r = i / (DK / 8), c = i % (DK / 8), h = gt * HPT + r % HPT;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (h < p.G && c * 8 < p.dkp)
        v = *reinterpret_cast<const uint4*>(p.q + ((size_t(b) * p.Hq + kvh * p.G + h) * MAPS + r / HPT) * p.dkp + c * 8);
      *reinterpret_cast<uint4*>(&sQ[r][c * 8]) = v;
    }
  }
  const float lin = p.mod.scale * kLog2e;
  HeadScore hs0{}, hs1{};
  if (MAPS == 1 && gt * 16 + g < p.G) hs0 = head_score(p.mod, kvh * p.G + gt * 16 + g);
  if (MAPS == 1 && gt * 16 + g + 8 < p.G) hs1 = head_score(p.mod, kvh * p.G + gt * 16 + g + 8);
  if (MAPS > 1 && threadIdx.x < 16) { s_sink[threadIdx.x] = -INFINITY; s_gate[threadIdx.x] = 1.f; }
  if (MAPS == 1 && threadIdx.x < 16) {
    const int h = gt * 16 + threadIdx.x;
    s_sink[threadIdx.x] = (h < p.G && p.mod.sink) ? p.mod.sink[kvh * p.G + h] * kLog2e : -INFINITY;
    float gate = 1.f;
    if (h < p.G) {
      if (!p.raw) gate = head_gate<__nv_bfloat16>(p.gate, b, kvh * p.G + h);
      else if (p.gate_col >= 0) gate = sigmoid_f(__ldcg(p.raw + size_t(b) * p.raw_ld + p.gate_col + kvh * p.G + h));
    }
    s_gate[threadIdx.x] = gate;
  }
  const bool upper = p.G - gt * 16 > 8;      // rows 8 .. 15 of the tile hold heads
  __syncthreads();      // queries staged, the appended key / value written

  uint32_t qa[KS][4];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    const int d = ks * 16 + t * 2;
    qa[ks][0] = *reinterpret_cast<const uint32_t*>(&sQ[g][d]);
    qa[ks][1] = *reinterpret_cast<const uint32_t*>(&sQ[g + 8][d]);
    qa[ks][2] = *reinterpret_cast<const uint32_t*>(&sQ[g][d + 8]);
    qa[ks][3] = *reinterpret_cast<const uint32_t*>(&sQ[g + 8][d + 8]);
  }
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;

  if (owner) {
#pragma unroll
    for (int s = 0; s < NST; ++s)
      if (pg + s * kFsWarps == late) issue(late, s);
    fs_commit();
    fs_wait<0>();
  }
  int stage = 0;
  for (; pg < pg1; pg += kFsWarps) {
    fs_wait<NST - 1>();
    __syncwarp();
    const uint32_t kbase = smem_u32(wsm + stage * STAGE), vbase = kbase + K_PAGE;
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const int mi = lane >> 3, r = lane & 7;
      const int tok = (mi >> 1) * 8 + r, c = 2 * ks + (mi & 1);
      uint32_t kb[4];
      fs_ldm4(kb, kbase + tok * (DK * 2) + ((c ^ (tok & 7)) << 4));
      fs_mma(s0, qa[ks], kb[0], kb[1]);
      fs_mma(s1, qa[ks], kb[2], kb[3]);
    }
    if (MAPS > 1) {                      // rows 8 - 15 against the second map's keys
      float u0[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        const int mi = lane >> 3, r = lane & 7;
        const int tok = (mi >> 1) * 8 + r, c = 2 * ks + (mi & 1);
        uint32_t kb[4];
        fs_ldm4(kb, kbase + (MAPS - 1) * K_TILE + tok * (DK * 2) + ((c ^ (tok & 7)) << 4));
        fs_mma(u0, qa[ks], kb[0], kb[1]);
        fs_mma(u1, qa[ks], kb[2], kb[3]);
      }
      s0[2] = u0[2]; s0[3] = u0[3]; s1[2] = u1[2]; s1[3] = u1[3];
    }
    const int tok0 = pg * kFsPage + t * 2;
    float sv[8] = {s0[0], s0[1], s1[0], s1[1], s0[2], s0[3], s1[2], s1[3]};
    const int tk[4] = {tok0, tok0 + 1, tok0 + 8, tok0 + 9};
    if (MOD) {
      float dist[4], top0 = 0.f, top1 = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        dist[i] = float(len - 1 - tk[i]);
        top0 = fmaxf(top0, fabsf(sv[i]));
        top1 = fmaxf(top1, fabsf(sv[4 + i]));
      }
      const bool near = !__any_sync(0xffffffffu, fmaxf(top0 * fabsf(hs0.inner), top1 * fabsf(hs1.inner)) > kTanhPolyMax);
      scores_base2<4>(sv, hs0, dist, near);
      if (upper) scores_base2<4>(sv + 4, hs1, dist, near);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) sv[i] *= lin;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const bool ok = tk[i] < len && tk[i] >= first;
      sv[i] = ok ? sv[i] : -INFINITY;
      sv[4 + i] = ok ? sv[4 + i] : -INFINITY;
    }
    float mx0 = fmaxf(fmaxf(sv[0], sv[1]), fmaxf(sv[2], sv[3]));
    float mx1 = fmaxf(fmaxf(sv[4], sv[5]), fmaxf(sv[6], sv[7]));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float nm0 = fmaxf(m0, mx0), nm1 = fmaxf(m1, mx1);
    // a page holds at least one visible token, so the new maxima are finite
    const float c0 = ex2_approx(m0 - nm0), c1 = ex2_approx(m1 - nm1);
    m0 = nm0; m1 = nm1;
    float pr[8];
#pragma unroll
    for (int i = 0; i < 4; ++i) { pr[i] = ex2_approx(sv[i] - m0); pr[4 + i] = ex2_approx(sv[4 + i] - m1); }
    l0 = l0 * c0 + (pr[0] + pr[1] + pr[2] + pr[3]);
    l1 = l1 * c1 + (pr[4] + pr[5] + pr[6] + pr[7]);
    uint32_t pa[4] = {pack_bf16(pr[0], pr[1]), pack_bf16(pr[4], pr[5]), pack_bf16(pr[2], pr[3]),
                      pack_bf16(pr[6], pr[7])};
#pragma unroll
    for (int j = 0; j < NT; ++j) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      const int mi = lane >> 3, r = lane & 7;
      const int tok = (mi & 1) * 8 + r, c = j + (mi >> 1);
      uint32_t vb[4];
      fs_ldm4t(vb, vbase + tok * (DV * 2) + ((c ^ (tok & 7)) << 4));
      fs_mma(o[j], pa, vb[0], vb[1]);
      fs_mma(o[j + 1], pa, vb[2], vb[3]);
    }
    __syncwarp();
    if (pg + NST * kFsWarps < pg1) issue(pg + NST * kFsWarps, stage);
    fs_commit();
    stage = (stage + 1 == NST) ? 0 : stage + 1;
  }
  fs_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);

  // ---- merge the four warps of the block ----
  __syncthreads();
  float* so = reinterpret_cast<float*>(smem);  // [warp][16][DV]
  if (t == 0) { s_m[warp][g] = m0; s_m[warp][g + 8] = m1; s_l[warp][g] = l0; s_l[warp][g + 8] = l1; }
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int d = j * 8 + t * 2;
    *reinterpret_cast<float2*>(so + (warp * 16 + g) * DV + d) = make_float2(o[j][0], o[j][1]);
    *reinterpret_cast<float2*>(so + (warp * 16 + g + 8) * DV + d) = make_float2(o[j][2], o[j][3]);
  }
  __syncthreads();
  const size_t tile = (size_t(lb) * p.Hkv * p.gtiles + yt);
  for (int idx = threadIdx.x; idx < 16 * DV; idx += kFsThreads) {
    const int row = idx / DV, d = idx % DV;
    float M = p.S == 1 ? s_sink[row] : -INFINITY;
#pragma unroll
    for (int w = 0; w < kFsWarps; ++w) M = fmaxf(M, s_m[w][row]);
    float L = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < kFsWarps; ++w) {
      const float f = (s_m[w][row] == -INFINITY) ? 0.f : ex2_approx(s_m[w][row] - M);
      L += s_l[w][row] * f;
      acc += so[(w * 16 + row) * DV + d] * f;
    }
    const int h = gt * 16 + row;
    if (p.S == 1) {
      if (s_sink[row] != -INFINITY) L += ex2_approx(s_sink[row] - M);
      if (MAPS > 1) so[row * DV + d] = L > 0.f ? acc / L : 0.f;      // (this thread alone has read the place)
      else if (h < p.G && d < p.dvp)
        p.out[(size_t(b) * p.Hq + size_t(kvh) * p.G + h) * p.dvp + d] = __float2bfloat16_rn(L > 0.f ? acc * s_gate[row] / L : 0.f);
    } else {
      p.part_o[((tile * p.S + split) * 16 + row) * DV + d] = acc;
      if (d == 0) {
        p.part_ml[((tile * p.S + split) * 16 + row) * 2] = M;
        p.part_ml[((tile * p.S + split) * 16 + row) * 2 + 1] = L;
      }
    }
  }
  // MAPS 2: rows r and r + 8 of `val` [16][DV] are a head's two maps
  auto put_difference = [&](const float* val) {
    constexpr int PL = DV / 32;
    for (int r = warp; r < HPT && gt * HPT + r < p.G; r += kFsWarps) {
      float v[PL], ss = 0.f;
#pragma unroll
      for (int i = 0; i < PL; ++i) {
        const int d = i * 32 + lane;
        v[i] = val[r * DV + d] - p.diff.weight * val[(r + HPT) * DV + d];
        if (d < p.vdim) ss += v[i] * v[i];
      }
      const float inv = p.diff.scale / sqrtf(warp_sum(ss) / float(p.vdim) + p.diff.eps);
      __nv_bfloat16* dst = p.out + (size_t(b) * p.Hq + size_t(kvh) * p.G + gt * HPT + r) * p.dvp;
#pragma unroll
      for (int i = 0; i < PL; ++i)
        if (i * 32 + lane < p.dvp) dst[i * 32 + lane] = __float2bfloat16_rn(v[i] * inv);
    }
  };
  if (p.S == 1) {
    if (MAPS > 1) {
      __syncthreads();
      put_difference(so);
    }
    return;
  }

  // ---- last block of this tile merges the splits ----
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = (atomicAdd(p.tickets + tile, 1u) == unsigned(p.S - 1)) ? 1u : 0u;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  float* wgt = reinterpret_cast<float*>(smem);        // [S][16] weights exp2(m_s - M) / L
  float* mls = wgt + kFsMaxSplits * 16;               // [S][16][2] copy of the (max, sum) table
  float* whole = mls + kFsMaxSplits * 32;             // MAPS 2: [16][DV] merged rows
  for (int i = threadIdx.x; i < p.S * 32; i += kFsThreads) mls[i] = p.part_ml[tile * p.S * 32 + i];
  __syncthreads();
  if (threadIdx.x < 16) {
    const int row = threadIdx.x;
    float M = s_sink[row];
    for (int s = 0; s < p.S; ++s) M = fmaxf(M, mls[s * 32 + row * 2]);
    float L = s_sink[row] == -INFINITY ? 0.f : ex2_approx(s_sink[row] - M);
    for (int s = 0; s < p.S; ++s) {
      const float ms = mls[s * 32 + row * 2];
      const float f = (ms == -INFINITY) ? 0.f : ex2_approx(ms - M);
      wgt[s * 16 + row] = f;
      L += mls[s * 32 + row * 2 + 1] * f;
    }
    const float inv = L > 0.f ? s_gate[row] / L : 0.f;
    for (int s = 0; s < p.S; ++s) wgt[s * 16 + row] *= inv;
  }
  __syncthreads();
  const float4* po4 = reinterpret_cast<const float4*>(p.part_o + tile * p.S * 16 * DV);
  constexpr int D4 = DV / 4;
  for (int idx = threadIdx.x; idx < 16 * D4; idx += kFsThreads) {
    const int row = idx / D4, d4 = idx % D4;
    const int h = gt * 16 + row;
    if (MAPS == 1 && (h >= p.G || d4 * 4 >= p.dvp)) continue;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < p.S; s += 16) {
      float4 v[16];
#pragma unroll
      for (int j = 0; j < 16; ++j)
        v[j] = (s + j < p.S) ? po4[(size_t(s + j) * 16 + row) * D4 + d4] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const float w = (s + j < p.S) ? wgt[(s + j) * 16 + row] : 0.f;
        acc.x = fmaf(v[j].x, w, acc.x); acc.y = fmaf(v[j].y, w, acc.y);
        acc.z = fmaf(v[j].z, w, acc.z); acc.w = fmaf(v[j].w, w, acc.w);
      }
    }
    if (MAPS > 1) {
      *reinterpret_cast<float4*>(whole + row * DV + d4 * 4) = acc;
      continue;
    }
    uint2 ov;
    ov.x = pack_bf16(acc.x, acc.y);
    ov.y = pack_bf16(acc.z, acc.w);
    *reinterpret_cast<uint2*>(p.out + (size_t(b) * p.Hq + size_t(kvh) * p.G + h) * p.dvp + d4 * 4) = ov;
  }
  if (MAPS > 1) {
    __syncthreads();
    put_difference(whole);
  }
  if (threadIdx.x == 0) p.tickets[tile] = 0u;
}

__host__ inline int fs_class(int d) { return d <= 64 ? 64 : d <= 128 ? 128 : 0; }

}  // namespace rb

using namespace rb;
RB_BOUNDS_REGISTER("flash_decode_scored.cu")

// 1 when the kernel takes these (eight-padded) key and value widths.
extern "C" int rmlx_flash_decode_scored_supported(int dkp, int dvp) { return fs_class(dkp) && fs_class(dvp); }
// Scratch elements for B launch rows: floats of part_o and part_ml, 32-bit words of tickets.
static long long fs_tiles(int B, int Hq, int Hkv) { return 1LL * B * Hkv * (((Hq / Hkv) + 15) / 16); }
extern "C" long long rmlx_flash_decode_scored_part_o_elems(int B, int Hq, int Hkv, int S, int dvp) {
  return fs_tiles(B, Hq, Hkv) * S * 16 * fs_class(dvp);
}
extern "C" long long rmlx_flash_decode_scored_part_ml_elems(int B, int Hq, int Hkv, int S) {
  return fs_tiles(B, Hq, Hkv) * S * 32;
}
extern "C" long long rmlx_flash_decode_scored_ticket_elems(int B, int Hq, int Hkv) { return fs_tiles(B, Hq, Hkv); }

// q (bf16) or raw (fp32, with q_w, k_w, eps: the fused form), exactly one of them. dkp / dvp: dim /
// vdim rounded up to eight. gate: bf16 [rows, ldg] output gate logits of the plain form, or null; head_norm,
// gate_col (-1: none): the fused form's; with head_norm also bias (fp32, raw's layout, or null) and the rotation of the
// first rot_dims values (inv_freq fp32 [rot_dims / 2]; neighbours: pairs (2 i, 2 i + 1) turn). `tickets` is zero on the
// first call; the kernel leaves it zero. maps 2: differential attention with no modifier but the scale - q [rows, Hq,
// 2 dkp], key rows of 2 dkp values, raw = [q: Hq x 2 x dim | k: Hkv x 2 x dim | v] (head_norm 1 or 2); scratch as for 2 Hq
// query heads.
extern "C" int rmlx_flash_decode_scored(const void* q, const float* raw, int raw_ld, const float* q_w,
                                        const float* k_w, float eps, void* k_cache, void* v_cache,
                                        const int* block_table, const int* positions, const int* rows,
                                        const int* table_rows, void* out, float* part_o, float* part_ml,
                                        unsigned int* tickets, int B, int Hq, int Hkv, int dim, int vdim,
                                        int dkp, int dvp, int max_blocks, int splits, int window, int chunk,
                                        float scale, float softcap, const float* temp, const float* r1,
                                        const float* r2, const float* sink, const void* gate, int ldg,
                                        int head_norm, int gate_col, const float* bias, const float* inv_freq,
                                        int rot_dims, float grow, int neighbours, int maps, float map_weight, float map_scale,
                                        float map_eps, int pdl, cudaStream_t st) {
  if (B < 1 || B > 65535 || Hkv < 1 || Hq % Hkv || splits < 1 || splits > kFsMaxSplits || (!q) == (!raw) ||
      dkp % 8 || dvp % 8 || dim > dkp || vdim > dvp || dim < 1 || vdim < 1 || (r1 && !r2))
    return -2;
  if (maps < 1 || maps > 2 || head_norm < 0 || head_norm > 2) return -2;
  if (maps == 2 && (softcap > 0.f || temp || r1 || sink || gate || gate_col >= 0 || (raw && !head_norm))) return -2;
  if (raw && (((!q_w || !k_w) && !head_norm) || raw_ld < (Hq + Hkv) * maps * dim + Hkv * vdim)) return -2;
  if ((bias || rot_dims) && !(raw && head_norm)) return -2;
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > dim || (rot_dims && !inv_freq)) return -2;
  if (splits > 1 && (!part_o || !part_ml || !tickets)) return -2;
  FsParams p;
  p.q = static_cast<const __nv_bfloat16*>(q); p.raw = raw; p.raw_ld = raw_ld; p.q_w = q_w; p.k_w = k_w; p.eps = eps;
  p.k_cache = static_cast<__nv_bfloat16*>(k_cache); p.v_cache = static_cast<__nv_bfloat16*>(v_cache);
  p.block_table = block_table; p.positions = positions; p.rows = rows; p.table_rows = table_rows;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.part_o = part_o; p.part_ml = part_ml; p.tickets = tickets;
  p.max_blocks = max_blocks; p.Hq = Hq; p.Hkv = Hkv; p.G = Hq / Hkv; p.gtiles = (p.G * maps + 15) / 16;
  p.S = splits; p.window = window; p.chunk = chunk; p.dim = dim; p.vdim = vdim; p.dkp = dkp; p.dvp = dvp;
  p.mod.scale = scale; p.mod.softcap = softcap; p.mod.temp = temp; p.mod.r1 = r1; p.mod.r2 = r2; p.mod.sink = sink;
  p.gate.gate = gate; p.gate.ld = ldg; p.head_norm = head_norm; p.gate_col = gate_col;
  p.bias = bias; p.inv_freq = inv_freq; p.rot_dims = rot_dims; p.grow = grow;
  p.neighbours = neighbours; p.diff.weight = map_weight; p.diff.scale = map_scale; p.diff.eps = map_eps;
  if (raw && gate_col >= 0 && raw_ld < gate_col + Hq) return -2;
  if (p.Hkv * p.gtiles > 65535) return -2;
  const dim3 grid(splits, Hkv * p.gtiles, B);
  const bool plain = softcap <= 0.f && !temp && !r1 && !sink;
  const bool deep = size_t(splits) * Hkv * p.gtiles * B <= size_t(2 * sm_count());
  // staging (>= 4 x 2 x 4 KB) covers the warp merge (4 x 16 x DV floats) and the split tables (12 KB)
#define RB_FS(DK_, DV_, NST_, MAPS_)                                                       \
  {                                                                                        \
    constexpr size_t smem = size_t(kFsWarps) * NST_ * kFsPage * (MAPS_ * DK_ + DV_) * 2;   \
    static_assert(smem >= size_t(kFsWarps) * 16 * DV_ * 4, "warp merge");                  \
    static_assert(smem >= size_t(kFsMaxSplits) * 16 * 3 * 4 + (MAPS_ - 1) * 16 * DV_ * 4, "split tables"); \
    auto kern = plain ? flash_decode_scored_kernel<DK_, DV_, NST_, false, MAPS_>           \
                      : flash_decode_scored_kernel<DK_, DV_, NST_, MAPS_ == 1, MAPS_>;     \
    RB_CHECK(set_max_smem(kern, smem));                                                    \
    return launch(kern, grid, dim3(kFsThreads), smem, st, pdl != 0, p);                    \
  }
#define RB_FSM(DK_, DV_)                          \
  {                                               \
    if (maps == 2 && deep) RB_FS(DK_, DV_, 4, 2)  \
    if (maps == 2) RB_FS(DK_, DV_, 2, 2)          \
    if (deep) RB_FS(DK_, DV_, 4, 1)               \
    RB_FS(DK_, DV_, 2, 1)                         \
  }
  const int ck = fs_class(dkp), cv = fs_class(dvp);
  if (ck == 128 && cv == 128) RB_FSM(128, 128)
  if (ck == 128 && cv == 64) RB_FSM(128, 64)
  if (ck == 64 && cv == 128) RB_FSM(64, 128)
  if (ck == 64 && cv == 64) RB_FSM(64, 64)
#undef RB_FSM
#undef RB_FS
  return -2;
}
