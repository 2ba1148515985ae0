// Short causal convolution over packed tokens: where the inputs before a token come from.
//
// conv_state [slots, 2, taps-1, channels]: the inputs of the taps-1 positions before position p live in half p & 1, so a
// launch may read the old ones in every block while it writes the new ones.
#pragma once
#include "lm_common.cuh"

namespace msa {

template <typename T> struct Raw4;
template <> struct Raw4<float> { using type = float4; };
template <> struct Raw4<__nv_bfloat16> { using type = uint2; };
__device__ __forceinline__ float4 widen(float4 v) { return v; }
__device__ __forceinline__ float4 widen(uint2 r) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// One channel (or four) of the convolved columns, as the tokens of a step see it.
template <typename T>
struct ConvSource {
  const T* proj; long long proj_stride;   // first convolved column of packed row 0
  T* state;
  int channels, taps;
  __device__ __forceinline__ T* half(int slot, int p) const { return state + ((long long)slot * 2 + (p & 1)) * (taps - 1) * channels; }
  // Address of channel c's input `lag` tokens before packed row n (token t of a portion that starts at position p0), null
  // before the sequence's start.
  __device__ __forceinline__ const T* at(long long n, int t, int p0, int slot, int lag, int c) const {
    if (t - lag >= 0) return proj + (n - lag) * proj_stride + c;
    if (p0 + t - lag >= 0) return half(slot, p0) + (long long)(taps - 1 + t - lag) * channels + c;
    return nullptr;
  }
  // The convolution of channel c, weights w [taps, channels].
  __device__ __forceinline__ float value(const float* w, long long n, int t, int p0, int slot, int c) const {
    float acc = 0.f;
    for (int i = 0; i < taps; ++i) {
      const T* x = at(n, t, p0, slot, taps - 1 - i, c);
      if (x) acc = fmaf(w[(long long)i * channels + c], to_f(*x), acc);
    }
    return acc;
  }
};

// Window of TAPS inputs of four channels that slides over consecutive packed rows.
template <typename T, int TAPS>
struct ConvWindow {
  using Raw = typename Raw4<T>::type;
  Raw x[TAPS];
  // Moves to packed row n; `fresh`: the row does not follow the one the window stands on.
  __device__ __forceinline__ void move(const ConvSource<T>& src, long long n, int t, int p0, int slot, int c, bool fresh) {
    if (fresh) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const T* p = src.at(n, t, p0, slot, TAPS - 1 - j, c);
        x[j] = p ? *reinterpret_cast<const Raw*>(p) : Raw{};
      }
    } else {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) x[j] = x[j + 1];
    }
    x[TAPS - 1] = *reinterpret_cast<const Raw*>(src.proj + n * src.proj_stride + c);
  }
  __device__ __forceinline__ float4 value(const float4 (&w)[TAPS]) const {
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float4 f = widen(x[j]);
      y.x = fmaf(w[j].x, f.x, y.x); y.y = fmaf(w[j].y, f.y, y.y); y.z = fmaf(w[j].z, f.z, y.z); y.w = fmaf(w[j].w, f.w, y.w);
    }
    return y;
  }
  // A single-token row leaves its last TAPS-1 inputs for position p + 1.
  __device__ __forceinline__ void leave(const ConvSource<T>& src, int slot, int p, int c) const {
    T* dst = src.half(slot, p + 1) + c;
#pragma unroll
    for (int j = 1; j < TAPS; ++j) *reinterpret_cast<Raw*>(dst + (long long)(j - 1) * src.channels) = x[j];
  }
};

}  // namespace msa
