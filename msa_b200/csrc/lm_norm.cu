// Residual stream (fp32), the norms on either side of a sublayer, the embedding, and the dense feed-forward's gate.
// One launch between two matrix products: branch norm, residual add, next norm, rounding for the next product.
#include "lm_common.cuh"

namespace msa {

struct ResNormParams {
  const float* base; long long base_stride;
  const void* y; int32_t y_dtype; long long y_stride;
  const int32_t* inv; const float* mix; int32_t top;
  const float* w_branch; const float* w_next; float eps;
  const int32_t* rows; int32_t width;
  float* x_out; void* h_out; void* cat_out; long long cat_stride;
};

template <typename TY>
__device__ __forceinline__ float4 branch4(const ResNormParams& p, long long r, int i) {
  const TY* y = reinterpret_cast<const TY*>(p.y);
  if (!p.inv) return load4(y + r * p.y_stride + i);
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int k = 0; k < p.top; ++k) {
    const float w = p.mix[r * p.top + k];
    const float4 v = load4(y + (long long)p.inv[r * p.top + k] * p.y_stride + i);
    a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
  }
  return a;
}
template <typename TY>
__device__ __forceinline__ float branch1(const ResNormParams& p, long long r, int i) {
  const TY* y = reinterpret_cast<const TY*>(p.y);
  if (!p.inv) return to_f(y[r * p.y_stride + i]);
  float a = 0.f;
  for (int k = 0; k < p.top; ++k)
    a = fmaf(p.mix[r * p.top + k], to_f(y[(long long)p.inv[r * p.top + k] * p.y_stride + i]), a);
  return a;
}

// V = 4: every row pointer is 4-element aligned and width % 4 == 0; V = 1: any width.
template <typename T, typename TY, int V>
__global__ void residual_norm_kernel(const ResNormParams p) {
  extern __shared__ float s_row[];   // [width]
  __shared__ float s_part[32];
  const long long r = blockIdx.x;
  const long long rb = p.rows ? p.rows[r] : r;
  const int nt = blockDim.x;
  T* h_out = reinterpret_cast<T*>(p.h_out);
  T* cat = reinterpret_cast<T*>(p.cat_out);
  float scale_b = 1.f;
  if (p.y && p.w_branch) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < p.width; i += nt * V) {
      if constexpr (V == 4) {
        const float4 b = branch4<TY>(p, r, i);
        store4(s_row + i, b);
        ss += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
      } else {
        const float b = branch1<TY>(p, r, i);
        s_row[i] = b;
        ss += b * b;
      }
    }
    scale_b = 1.f / sqrtf(block_sum(ss, s_part) / (float)p.width + p.eps);
  }
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < p.width; i += nt * V) {   // every thread revisits the elements it stored above
    if constexpr (V == 4) {
      float4 x = p.base ? load4(p.base + rb * p.base_stride + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.y) {
        if (p.w_branch) {
          const float4 b = load4(s_row + i), w = load4(p.w_branch + i);
          x.x += b.x * scale_b * w.x; x.y += b.y * scale_b * w.y; x.z += b.z * scale_b * w.z; x.w += b.w * scale_b * w.w;
        } else {
          const float4 b = branch4<TY>(p, r, i);
          x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
        }
      }
      if (p.x_out) store4(p.x_out + r * p.width + i, x);
      if (cat) store4(cat + r * p.cat_stride + i, x);
      store4(s_row + i, x);
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    } else {
      float x = p.base ? p.base[rb * p.base_stride + i] : 0.f;
      if (p.y) x += p.w_branch ? s_row[i] * scale_b * p.w_branch[i] : branch1<TY>(p, r, i);
      if (p.x_out) p.x_out[r * p.width + i] = x;
      if (cat) cat[r * p.cat_stride + i] = from_f<T>(x);
      s_row[i] = x;
      ss += x * x;
    }
  }
  if (!h_out) return;
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)p.width + p.eps);
  for (int i = threadIdx.x * V; i < p.width; i += nt * V) {
    if constexpr (V == 4) {
      const float4 x = load4(s_row + i), w = load4(p.w_next + i);
      store4(h_out + r * p.width + i, make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w));
    } else {
      h_out[r * p.width + i] = from_f<T>(s_row[i] * inv * p.w_next[i]);
    }
  }
}

// The same for rows that a block of width / 4 threads covers in one pass (everything in registers, all loads in flight
// before the first reduction): a decode step has few rows and waits for latency, not for bandwidth.
template <typename T, typename TY>
__global__ void __launch_bounds__(1024) residual_norm_once_kernel(const ResNormParams p) {
  __shared__ float s_part[32];
  const long long r = blockIdx.x;
  const long long rb = p.rows ? p.rows[r] : r;
  const int i = threadIdx.x * 4;
  const bool on = i < p.width;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 x = on && p.base ? load4(p.base + rb * p.base_stride + i) : zero;
  const float4 wb = on && p.w_branch ? load4(p.w_branch + i) : zero;
  const float4 wn = on && p.h_out ? load4(p.w_next + i) : zero;
  float4 b = zero;
  if (p.y && on) {
    const TY* y = reinterpret_cast<const TY*>(p.y);
    if (p.inv) {
      for (int k0 = 0; k0 < p.top; k0 += 4) {
        float4 v[4];
        float w[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const bool in = k0 + k < p.top;
          w[k] = in ? p.mix[r * p.top + k0 + k] : 0.f;
          v[k] = in ? load4(y + (long long)p.inv[r * p.top + k0 + k] * p.y_stride + i) : zero;
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          b.x = fmaf(w[k], v[k].x, b.x); b.y = fmaf(w[k], v[k].y, b.y); b.z = fmaf(w[k], v[k].z, b.z); b.w = fmaf(w[k], v[k].w, b.w);
        }
      }
    } else {
      b = load4(y + r * p.y_stride + i);
    }
  }
  if (p.y && p.w_branch) {
    const float sc = 1.f / sqrtf(block_sum(b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w, s_part) / (float)p.width + p.eps);
    x.x += b.x * sc * wb.x; x.y += b.y * sc * wb.y; x.z += b.z * sc * wb.z; x.w += b.w * sc * wb.w;
  } else {
    x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
  }
  if (on && p.x_out) store4(p.x_out + r * p.width + i, x);
  if (on && p.cat_out) store4(reinterpret_cast<T*>(p.cat_out) + r * p.cat_stride + i, x);
  if (!p.h_out) return;
  const float inv = 1.f / sqrtf(block_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w, s_part) / (float)p.width + p.eps);
  if (on) store4(reinterpret_cast<T*>(p.h_out) + r * p.width + i, make_float4(x.x * inv * wn.x, x.y * inv * wn.y, x.z * inv * wn.z, x.w * inv * wn.w));
}

template <typename T>
__global__ void embed_kernel(const T* __restrict__ table, const int32_t* __restrict__ token, int width, int vocab,
                             const float* __restrict__ w_next, float eps, float* x_out, T* h_out, T* cat0, T* cat1,
                             long long cat_stride, int32_t* status) {
  extern __shared__ float s_row[];
  __shared__ float s_part[32];
  const long long r = blockIdx.x;
  int tok = token[r];
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0 && status) atomicAdd(status + 2, 1);
    tok = 0;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const T raw = table[(long long)tok * width + i];
    const float x = to_f(raw);
    x_out[r * width + i] = x;
    if (cat0) cat0[r * cat_stride + i] = raw;
    if (cat1) cat1[r * cat_stride + i] = raw;
    s_row[i] = x;
    ss += x * x;
  }
  if (!h_out) return;
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)width + eps);
  for (int i = threadIdx.x; i < width; i += blockDim.x) h_out[r * width + i] = from_f<T>(s_row[i] * inv * w_next[i]);
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
lm_silu_mul_kernel(const T* __restrict__ gu, long long stride, int ff, long long n_rows, T* __restrict__ out) {
  const int per_row = ff / V;
  const long long total = n_rows * per_row;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / per_row;
    const int j = (int)(i % per_row) * V;
    if constexpr (V == 4) {
      const float4 g = load4(gu + r * stride + j), u = load4(gu + r * stride + ff + j);
      store4(out + r * ff + j, make_float4(silu_f(g.x) * u.x, silu_f(g.y) * u.y, silu_f(g.z) * u.z, silu_f(g.w) * u.w));
    } else {
      out[r * ff + j] = from_f<T>(silu_f(to_f(gu[r * stride + j])) * to_f(gu[r * stride + ff + j]));
    }
  }
}

inline int row_threads(int width) { return width >= 2048 ? 256 : (width >= 512 ? 128 : 64); }
inline bool vec4_ok(const void* p, int elem) { return p == nullptr || (reinterpret_cast<uintptr_t>(p) % (4 * elem)) == 0; }

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_residual_norm(const float* base, int64_t base_stride, const void* y, int32_t y_dtype,
                                    int64_t y_stride, const int32_t* inv, const float* mix, int32_t top,
                                    const float* w_branch, const float* w_next, float eps, const int32_t* rows,
                                    int32_t n_rows, int32_t width, float* x_out, void* h_out, void* cat_out,
                                    int64_t cat_stride, int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && (!y || dtype_ok(y_dtype)), "residual_norm: bad dtype");
  MSA_REQUIRE(n_rows >= 0 && width > 0 && width <= 12000, "residual_norm: width must be 1..12000");
  MSA_REQUIRE(base || y, "residual_norm: neither base nor branch");
  MSA_REQUIRE(!h_out || w_next, "residual_norm: h_out needs w_next");
  MSA_REQUIRE(!inv || (mix && top > 0 && y), "residual_norm: a mixture needs weights and top > 0");
  if (n_rows == 0) return MSA_OK;
  ResNormParams p{base, base_stride, y, y_dtype, y_stride, inv, mix, top, w_branch, w_next, eps, rows, width, x_out, h_out,
                  cat_out, cat_stride};
  const int e = (int)dtype_size(dtype), ey = (int)dtype_size(y_dtype);
  const bool v4 = width % 4 == 0 && base_stride % 4 == 0 && (!y || y_stride % 4 == 0) && (!cat_out || cat_stride % 4 == 0) &&
                  vec4_ok(base, 4) && vec4_ok(y, ey) && vec4_ok(w_branch, 4) && vec4_ok(w_next, 4) && vec4_ok(x_out, 4) &&
                  vec4_ok(h_out, e) && vec4_ok(cat_out, e);
  const size_t smem = (size_t)width * 4;
  const int threads = row_threads(width);
  cudaStream_t st = (cudaStream_t)stream;
  if (v4 && width <= 4096 && n_rows <= 512) {
    const int once = (width / 4 + 31) / 32 * 32;
    MSA_LM_DISPATCH(dtype, {
      if (y && y_dtype == MSA_BF16) residual_norm_once_kernel<T, __nv_bfloat16><<<n_rows, once, 0, st>>>(p);
      else residual_norm_once_kernel<T, float><<<n_rows, once, 0, st>>>(p);
    });
    MSA_LAUNCH_OK("residual_norm_once_kernel");
    return MSA_OK;
  }
  MSA_LM_DISPATCH(dtype, {
    if (y && y_dtype == MSA_BF16) {
      if (v4) residual_norm_kernel<T, __nv_bfloat16, 4><<<n_rows, threads, smem, st>>>(p);
      else residual_norm_kernel<T, __nv_bfloat16, 1><<<n_rows, threads, smem, st>>>(p);
    } else {
      if (v4) residual_norm_kernel<T, float, 4><<<n_rows, threads, smem, st>>>(p);
      else residual_norm_kernel<T, float, 1><<<n_rows, threads, smem, st>>>(p);
    }
  });
  MSA_LAUNCH_OK("residual_norm_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_embed(const void* table, const int32_t* token, int32_t n_rows, int32_t width, int32_t vocab,
                            const float* w_next, float eps, float* x_out, void* h_out, void* cat0, void* cat1,
                            int64_t cat_stride, int32_t* status, int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && table && token && x_out, "embed: bad arguments");
  MSA_REQUIRE(n_rows >= 0 && width > 0 && width <= 12000 && vocab > 0, "embed: bad sizes");
  MSA_REQUIRE(!h_out || w_next, "embed: h_out needs w_next");
  if (n_rows == 0) return MSA_OK;
  MSA_LM_DISPATCH(dtype, {
    embed_kernel<T><<<n_rows, row_threads(width), (size_t)width * 4, (cudaStream_t)stream>>>(
        (const T*)table, token, width, vocab, w_next, eps, x_out, (T*)h_out, (T*)cat0, (T*)cat1, cat_stride, status);
  });
  MSA_LAUNCH_OK("embed_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_silu_mul(const void* gu, int64_t gu_stride, int32_t n_rows, int32_t ff, void* out, int32_t dtype,
                               void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && gu && out && n_rows >= 0 && ff > 0, "lm_silu_mul: bad arguments");
  if (n_rows == 0) return MSA_OK;
  const int e = (int)dtype_size(dtype);
  const bool v4 = ff % 4 == 0 && gu_stride % 4 == 0 && vec4_ok(gu, e) && vec4_ok(out, e);
  const long long total = (long long)n_rows * (v4 ? ff / 4 : ff);
  const int grid = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  MSA_LM_DISPATCH(dtype, {
    if (v4) lm_silu_mul_kernel<T, 4><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)gu, gu_stride, ff, n_rows, (T*)out);
    else lm_silu_mul_kernel<T, 1><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)gu, gu_stride, ff, n_rows, (T*)out);
  });
  MSA_LAUNCH_OK("lm_silu_mul_kernel");
  return MSA_OK;
}
