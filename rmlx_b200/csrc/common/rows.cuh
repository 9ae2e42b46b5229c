// Pieces of the row-wise kernels (a block or a warp per activation row): conversions, eight-element
// loads and stores, and the block sum. Rows are bf16 (serving) or fp32 (the all-32-bit mode).
#pragma once
#include "ptx.cuh"

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

// Eight elements of which the first n exist (the rest read as zero); `aligned`: all eight, 16-byte aligned.
template <class T>
__device__ __forceinline__ void load8_upto(const T* p, int n, bool aligned, float (&f)[8]) {
  if (aligned) { load8(p, f); return; }
#pragma unroll
  for (int i = 0; i < 8; ++i) f[i] = i < n ? to_f32(p[i]) : 0.f;
}

// sin and cos of pos * freq radians: the product in double, whole turns taken off there, so that a far position costs
// no accuracy (and no branch).
__device__ __forceinline__ void rotary_sincos(int pos, float freq, float& s, float& c) {
  const double turns = double(pos) * double(freq) * 0.15915494309189535;
  sincospif(2.f * float(turns - rint(turns)), &s, &c);
}

// Sum over groups of L consecutive lanes (L a power of two).
template <int L>
__device__ __forceinline__ float group_sum(float v) {
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

}  // namespace rb
