// Paged causal attention for any head sizes, in fp32 or bf16 storage with fp32 arithmetic on the
// CUDA cores: the attention of models run in 32-bit, and of head sizes the tensor-core kernels do
// not take. Rows are single query tokens (a ragged batch of prompt portions and decoded tokens);
// each has a position and a row of the block table.
//
// A block owns one (token, query head); its four warps take 32-key chunks in turn. Lane j scores
// key j (its row read straight from the page), the chunk's softmax update is a warp reduction, and
// the values are accumulated with lanes along the value dimension. The warps merge through shared
// memory at the end.
//
// MAPS 2: differential attention (score_mod.cuh). A query head and a key row hold two maps side by side; both
// are scored against the same values, and their difference is normed here.
#include "../common/launch.cuh"
#include "../common/score_mod.cuh"

namespace rb {

constexpr int kAaWarps = 4;

struct AaParams {
  const void* q;            // [T, Hq, MAPS * dkp]
  const void* k_cache;      // [blocks, Hkv, page, ldk], the first MAPS * dkp values of a row are the key
  const void* v_cache;      // [blocks, Hkv, page, ldv], the first dvp the value (latent rows are both)
  const int* block_table;
  const int* positions;     // [T]
  const int* token_seq;     // [T] row of the block table, or null: token t has row t
  void* out;                // [T, Hq, dvp]
  int Hq, Hkv, dkp, dvp, ldk, ldv, max_blocks, page, window, chunk;
  ScoreMod mod;
  HeadGate gate;
  const int* rows;          // [n] batch rows to run, or null: all
  MapDiff diff;             // MAPS 2
  int vdim;                 // MAPS 2: values of a head that exist
};

__device__ __forceinline__ float aa_dot8(const float* k, const float* q) {
  const float4 a = *reinterpret_cast<const float4*>(k), b = *reinterpret_cast<const float4*>(k + 4);
  float s = a.x * q[0];
  s = fmaf(a.y, q[1], s); s = fmaf(a.z, q[2], s); s = fmaf(a.w, q[3], s);
  s = fmaf(b.x, q[4], s); s = fmaf(b.y, q[5], s); s = fmaf(b.z, q[6], s); s = fmaf(b.w, q[7], s);
  return s;
}
__device__ __forceinline__ float aa_dot8(const __nv_bfloat16* k, const float* q) {
  const uint4 v = *reinterpret_cast<const uint4*>(k);
  float s = bf16lo(v.x) * q[0];
  s = fmaf(bf16hi(v.x), q[1], s); s = fmaf(bf16lo(v.y), q[2], s); s = fmaf(bf16hi(v.y), q[3], s);
  s = fmaf(bf16lo(v.z), q[4], s); s = fmaf(bf16hi(v.z), q[5], s); s = fmaf(bf16lo(v.w), q[6], s);
  s = fmaf(bf16hi(v.w), q[7], s);
  return s;
}
__device__ __forceinline__ float aa_f32(float v) { return v; }
__device__ __forceinline__ float aa_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void aa_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void aa_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// NV: 32-wide slices of the value dimension kept per lane.
template <class T, int NV, int MAPS>
__global__ void __launch_bounds__(kAaWarps * 32) attention_any_kernel(AaParams p) {
  extern __shared__ float smem[];
  const int qw = MAPS * p.dkp;
  float* sq = smem;                                   // the query, fp32
  float* so = smem + qw;                              // [MAPS][warps][dvp]
  __shared__ float s_m[MAPS][kAaWarps], s_l[MAPS][kAaWarps];
  __shared__ float red[kAaWarps];
  pdl_launch_dependents();
  pdl_wait();
  const int t = p.rows ? p.rows[blockIdx.x] : blockIdx.x, h = blockIdx.y, kvh = h / (p.Hq / p.Hkv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[t];
  const int seq = p.token_seq ? p.token_seq[t] : t;
  const int* bt = p.block_table + size_t(seq) * p.max_blocks;
  const T* q = static_cast<const T*>(p.q) + (size_t(t) * p.Hq + h) * qw;
  for (int i = threadIdx.x; i < qw; i += kAaWarps * 32) sq[i] = aa_f32(q[i]);
  __syncthreads();
  // natural units here: the all-32-bit mode uses the full-precision functions
  const float st = p.mod.scale * (p.mod.temp ? p.mod.temp[h] : 1.f);
  const float cap = p.mod.softcap;
  const float r1 = p.mod.r1 ? p.mod.r1[h] : 0.f, r2 = p.mod.r1 ? p.mod.r2[h] : 0.f;
  const int first = first_key(pos, p.window, p.chunk);

  float m[MAPS], l[MAPS], o[MAPS][NV];
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    m[a] = -INFINITY;
    l[a] = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) o[a][i] = 0.f;
  }
  for (int c0 = (first & ~31) + warp * 32; c0 <= pos; c0 += kAaWarps * 32) {
    const int key = c0 + lane;
    const bool ok = key >= first && key <= pos && RB_BOUNDS(key / p.page, p.max_blocks);
    float w[MAPS];
#pragma unroll
    for (int a = 0; a < MAPS; ++a) w[a] = -INFINITY;
    if (ok) {
      const size_t row = (size_t(bt[key / p.page]) * p.Hkv + kvh) * p.page + key % p.page;
      const T* k = static_cast<const T*>(p.k_cache) + row * p.ldk;
#pragma unroll
      for (int a = 0; a < MAPS; ++a) {
        float dot = 0.f;
        for (int d = a * p.dkp; d < (a + 1) * p.dkp; d += 8) dot += aa_dot8(k + d, sq + d);
        float s = dot * st;
        if (cap > 0.f) s = cap * tanhf(s / cap);
        if (p.mod.r1) s -= r1 * log1pf(r2 * float(pos - key));
        w[a] = s;
      }
    }
    bool seen = true;
#pragma unroll
    for (int a = 0; a < MAPS; ++a) {
      const float nm = fmaxf(m[a], warp_max(w[a]));
      seen = nm != -INFINITY;                         // the maps see the same keys
      if (!seen) break;
      const float f = expf(m[a] - nm);                // exp(-inf) = 0
      w[a] = expf(w[a] - nm);
      m[a] = nm;
      l[a] = l[a] * f + warp_sum(w[a]);
#pragma unroll
      for (int i = 0; i < NV; ++i) o[a][i] *= f;
    }
    if (!seen) continue;                              // no visible key in this chunk
    const int n = min(32, pos - c0 + 1);
    for (int j = 0; j < n; ++j) {
      float wj[MAPS], any = 0.f;
#pragma unroll
      for (int a = 0; a < MAPS; ++a) {
        wj[a] = __shfl_sync(0xffffffffu, w[a], j);
        any = fmaxf(any, wj[a]);
      }
      if (any == 0.f) continue;                       // warp-uniform
      const int kj = c0 + j;
      const size_t row = (size_t(bt[kj / p.page]) * p.Hkv + kvh) * p.page + kj % p.page;
      const T* v = static_cast<const T*>(p.v_cache) + row * p.ldv;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i * 32 + lane < p.dvp) {
          const float x = aa_f32(v[i * 32 + lane]);
#pragma unroll
          for (int a = 0; a < MAPS; ++a) o[a][i] = fmaf(wj[a], x, o[a][i]);
        }
    }
  }
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    if (lane == 0) { s_m[a][warp] = m[a]; s_l[a][warp] = l[a]; }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (i * 32 + lane < p.dvp) so[(a * kAaWarps + warp) * p.dvp + i * 32 + lane] = o[a][i];
  }
  __syncthreads();
  // the warps' shares of the result, normalised by the map's sum
  float f[MAPS][kAaWarps];
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    float M = p.mod.sink ? p.mod.sink[h] : -INFINITY;
#pragma unroll
    for (int w = 0; w < kAaWarps; ++w) M = fmaxf(M, s_m[a][w]);
    float L = p.mod.sink ? expf(p.mod.sink[h] - M) : 0.f;
#pragma unroll
    for (int w = 0; w < kAaWarps; ++w) {
      f[a][w] = s_m[a][w] == -INFINITY ? 0.f : expf(s_m[a][w] - M);
      L += s_l[a][w] * f[a][w];
    }
    const float scale = L > 0.f ? head_gate<T>(p.gate, t, h) / L : 0.f;
#pragma unroll
    for (int w = 0; w < kAaWarps; ++w) f[a][w] *= scale;
  }
  T* out = static_cast<T*>(p.out) + (size_t(t) * p.Hq + h) * p.dvp;
  auto value = [&](int a, int i) {
    float acc = 0.f;
#pragma unroll
    for (int w = 0; w < kAaWarps; ++w) acc += so[(a * kAaWarps + w) * p.dvp + i] * f[a][w];
    return acc;
  };
  if (MAPS == 1) {
    for (int i = threadIdx.x; i < p.dvp; i += kAaWarps * 32) aa_put(out + i, value(0, i));
    return;
  }
  float ssq = 0.f;
  for (int i = threadIdx.x; i < p.dvp; i += kAaWarps * 32) {
    const float d = value(0, i) - p.diff.weight * value(MAPS - 1, i);
    so[i] = d;                                        // (only this thread reads place i of any map)
    ssq += i < p.vdim ? d * d : 0.f;
  }
  ssq = warp_sum(ssq);
  if (lane == 0) red[warp] = ssq;
  __syncthreads();
  ssq = 0.f;
#pragma unroll
  for (int w = 0; w < kAaWarps; ++w) ssq += red[w];
  const float inv = p.diff.scale / sqrtf(ssq / float(p.vdim) + p.diff.eps);
  for (int i = threadIdx.x; i < p.dvp; i += kAaWarps * 32) aa_put(out + i, so[i] * inv);
}

template <class T, int NV, int MAPS>
static int launch_any(const AaParams& p, int rows, int pdl, cudaStream_t st) {
  const size_t smem = size_t(MAPS) * (size_t(p.dkp) + size_t(kAaWarps) * p.dvp) * sizeof(float);
  auto kern = attention_any_kernel<T, NV, MAPS>;
  RB_CHECK(set_max_smem(kern, smem));
  return launch(kern, dim3(rows, p.Hq), dim3(kAaWarps * 32), smem, st, pdl != 0, p);
}
template <class T, int MAPS>
static int dispatch_any(const AaParams& p, int rows, int pdl, cudaStream_t st) {
  if (p.dvp <= 64) return launch_any<T, 2, MAPS>(p, rows, pdl, st);
  if (p.dvp <= 128) return launch_any<T, 4, MAPS>(p, rows, pdl, st);
  if (p.dvp <= 256) return launch_any<T, 8, MAPS>(p, rows, pdl, st);
  if (p.dvp <= 1024) return launch_any<T, 32, MAPS>(p, rows, pdl, st);
  return -2;
}

}  // namespace rb

using namespace rb;
RB_BOUNDS_REGISTER("attention_any.cu")

// q [T, Hq, dkp], out [T, Hq, dvp], caches [blocks, Hkv, page, ldk / ldv]: fp32 (f32) or bf16; dkp, dvp, ldk
// and ldv multiples of eight, dvp <= 1024. Token t sits at positions[t] and sees keys 0 .. positions[t]
// (the last `window` of them when window > 0, those of its own
// chunk of `chunk` positions when chunk > 0) of row token_seq[t] of the block table. rows: the n_rows
// batch rows to run (null: all T). gate [T, ldg] in the same type, or null. maps 2: q [T, Hq, 2 dkp], key rows of
// 2 dkp values, heads of vdim values: out = map_scale * d / rms(d), d = the first map's result - map_weight * the
// second's.
extern "C" int rmlx_attention_any(const void* q, const void* k_cache, const void* v_cache,
                                  const int* block_table, const int* positions, const int* token_seq,
                                  const int* rows, int n_rows, void* out, int T, int Hq, int Hkv, int dkp, int dvp,
                                  int ldk, int ldv, int max_blocks, int page, int window, int chunk, float scale, float softcap,
                                  const float* temp, const float* r1, const float* r2, const float* sink,
                                  const void* gate, int ldg, int maps, int vdim, float map_weight, float map_scale,
                                  float map_eps, int f32, int pdl, cudaStream_t st) {
  if (T < 1 || Hkv < 1 || Hq % Hkv || Hq > 65535 || dkp < 8 || dkp % 8 || dvp < 8 || dvp % 8 ||
      dkp > 8192 || maps < 1 || maps > 2 || ldk < maps * dkp || ldk % 8 || ldv < dvp || ldv % 8 || (r1 && !r2) || (rows && n_rows < 1) ||
      (maps == 2 && (vdim < 1 || vdim > dvp)))
    return -2;
  AaParams p;
  p.q = q; p.k_cache = k_cache; p.v_cache = v_cache; p.block_table = block_table;
  p.positions = positions; p.token_seq = token_seq; p.out = out; p.rows = rows;
  p.Hq = Hq; p.Hkv = Hkv; p.dkp = dkp; p.dvp = dvp; p.ldk = ldk; p.ldv = ldv; p.max_blocks = max_blocks; p.page = page;
  p.window = window; p.chunk = chunk;
  p.mod.scale = scale; p.mod.softcap = softcap; p.mod.temp = temp; p.mod.r1 = r1; p.mod.r2 = r2;
  p.mod.sink = sink;
  p.gate.gate = gate; p.gate.ld = ldg;
  const int n = rows ? n_rows : T;
  p.diff.weight = map_weight; p.diff.scale = map_scale; p.diff.eps = map_eps; p.vdim = vdim;
  if (maps == 2) return f32 ? dispatch_any<float, 2>(p, n, pdl, st) : dispatch_any<__nv_bfloat16, 2>(p, n, pdl, st);
  return f32 ? dispatch_any<float, 1>(p, n, pdl, st) : dispatch_any<__nv_bfloat16, 1>(p, n, pdl, st);
}
