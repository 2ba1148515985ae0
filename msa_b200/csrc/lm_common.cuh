// Helpers shared by the kernels of the layered decoder designs (lm_*.cu).  These files are compiled without
// --use_fast_math: angles, exponentials and divisions carry the full 32-bit accuracy.
#pragma once

#include "../../include/msa_b200_lm.h"
#include "common.cuh"

namespace msa {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Element of a buffer whose type is known at run time only.
__device__ __forceinline__ float load_any(const void* p, int32_t dtype, long long i) {
  return dtype == MSA_BF16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i])
                           : reinterpret_cast<const float*>(p)[i];
}
__device__ __forceinline__ void store_any(void* p, int32_t dtype, long long i, float v) {
  if (dtype == MSA_BF16) reinterpret_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(v);
  else reinterpret_cast<float*>(p)[i] = v;
}

// Four consecutive elements, 4-element aligned.
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  uint2 r;
  *reinterpret_cast<__nv_bfloat162*>(&r.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&r.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = r;
}

__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over the block; `part` holds one float per warp.  Every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum_f(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  const int n = (blockDim.x + 31) >> 5;
  for (int i = 0; i < n; ++i) t += part[i];
  return t;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// silu in front of a rounding to T.
template <typename T> __device__ __forceinline__ float silu_act(float z) { return silu_f(z); }
template <> __device__ __forceinline__ float silu_act<__nv_bfloat16>(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// Index of the sequence that owns position `i` of a prefix-sum table off[0 .. n].
__device__ __forceinline__ int owner_of(const int32_t* off, int n, int i) {
  int lo = 0, hi = n - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (off[mid] <= i) lo = mid; else hi = mid - 1;
  }
  return lo;
}

#define MSA_LM_DISPATCH(dtype, ...)                                   \
  do {                                                                \
    if ((dtype) == MSA_BF16) { using T = __nv_bfloat16; __VA_ARGS__ } \
    else { using T = float; __VA_ARGS__ }                             \
  } while (0)

}  // namespace msa
