// Device helpers shared by the layer-list kernels.
#pragma once
#include "../common/sm100.cuh"
#include "hybrid.cuh"

namespace oxb {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

template <typename T>
__device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <>
__device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
template <>
__device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 x = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
// The same past L1: rows that are read once, next to vectors that every row reads again
__device__ __forceinline__ void load4_stream(const float* p, float (&v)[4]) {
  const float4 x = __ldcg(reinterpret_cast<const float4*>(p));
  v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
__device__ __forceinline__ void load4_stream(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 x = __ldcg(reinterpret_cast<const uint2*>(p));
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T>
__device__ __forceinline__ void store4(T* p, const float (&v)[4]);
template <>
__device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
  uint2 x;
  x.x = pack_bf16x2(v[0], v[1]);
  x.y = pack_bf16x2(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = x;
}

// Sum over the block; every thread gets it. `scratch` holds 32 floats.
__device__ __forceinline__ float block_sum_all(float v, float* scratch) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  return warp_sum(lane < nw ? scratch[lane] : 0.f);
}
__device__ __forceinline__ float block_max_all(float v, float* scratch) {
  v = warp_max(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  return warp_max(lane < nw ? scratch[lane] : -INFINITY);
}

// sin and cos of position * frequency: the product is formed exactly as a + e (one FMA), the functions are
// taken of a and turned by the small rest e.
__device__ __forceinline__ void rotary_sincos(const RotaryParams& r, int i, int pos, float* sn, float* cs) {
  const float x = static_cast<float>(pos);
  const float a = x * r.freq_hi[i];
  const float e = fmaf(x, r.freq_hi[i], -a) + x * r.freq_lo[i];
  float s, c;
  sincosf(a, &s, &c);
  *sn = r.gain * fmaf(e, fmaf(-0.5f * e, s, c), s);   // second-order turn: e reaches 1/100 at angles of 2^18
  *cs = r.gain * fmaf(-e, fmaf(0.5f * e, c, s), c);
}
__device__ __forceinline__ void rotary_pair(const RotaryParams& r, int i, int* u, int* v) {
  *u = r.interleaved ? 2 * i : i;
  *v = r.interleaved ? 2 * i + 1 : i + (r.dims >> 1);
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// silu of a value that is stored as T: a bf16 result does not need the full-precision exponential and division
template <typename T>
__device__ __forceinline__ float silu_as(float z);
template <>
__device__ __forceinline__ float silu_as<float>(float z) { return silu_f(z); }
template <>
__device__ __forceinline__ float silu_as<__nv_bfloat16>(float z) { return __fdividef(z, 1.f + __expf(-z)); }

}  // namespace oxb
