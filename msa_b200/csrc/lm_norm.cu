// Residual stream (fp32), the norms on either side of a sublayer, the embedding (with a hashed bigram table), the dense
// feed-forward's gate and the cap of the logits.  One launch between two matrix products: branch norm, residual add, next
// norm (two of them where two branches read the same stream), rounding for the next product.
#include "lm_common.cuh"

namespace msa {

struct ResNormParams {
  const float* base; long long base_stride;
  const void* y; int32_t y_dtype; long long y_stride;
  const int32_t* inv; const float* mix; int32_t top;
  const float* w_branch; const float* w_next; float eps;
  const int32_t* rows; int32_t width;
  float* x_out; void* h_out; void* cat_out; long long cat_stride;
  const float* add;                            // further rows [n, width] that join the stream (null: none)
  const float* w_next2; void* h_out2;          // a second norm of the same stream
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
  T* h_out2 = reinterpret_cast<T*>(p.h_out2);
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
      if (p.add) {
        const float4 b = load4(p.add + r * p.width + i);
        x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
      }
      if (p.x_out) store4(p.x_out + r * p.width + i, x);
      if (cat) store4(cat + r * p.cat_stride + i, x);
      store4(s_row + i, x);
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    } else {
      float x = p.base ? p.base[rb * p.base_stride + i] : 0.f;
      if (p.y) x += p.w_branch ? s_row[i] * scale_b * p.w_branch[i] : branch1<TY>(p, r, i);
      if (p.add) x += p.add[r * p.width + i];
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
      if (h_out2) {
        const float4 w2 = load4(p.w_next2 + i);
        store4(h_out2 + r * p.width + i, make_float4(x.x * inv * w2.x, x.y * inv * w2.y, x.z * inv * w2.z, x.w * inv * w2.w));
      }
    } else {
      h_out[r * p.width + i] = from_f<T>(s_row[i] * inv * p.w_next[i]);
      if (h_out2) h_out2[r * p.width + i] = from_f<T>(s_row[i] * inv * p.w_next2[i]);
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
  const float4 wn2 = on && p.h_out2 ? load4(p.w_next2 + i) : zero;
  const float4 more = on && p.add ? load4(p.add + r * p.width + i) : zero;
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
  x.x += more.x; x.y += more.y; x.z += more.z; x.w += more.w;
  if (on && p.x_out) store4(p.x_out + r * p.width + i, x);
  if (on && p.cat_out) store4(reinterpret_cast<T*>(p.cat_out) + r * p.cat_stride + i, x);
  if (!p.h_out) return;
  const float inv = 1.f / sqrtf(block_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w, s_part) / (float)p.width + p.eps);
  if (on) store4(reinterpret_cast<T*>(p.h_out) + r * p.width + i, make_float4(x.x * inv * wn.x, x.y * inv * wn.y, x.z * inv * wn.z, x.w * inv * wn.w));
  if (on && p.h_out2)
    store4(reinterpret_cast<T*>(p.h_out2) + r * p.width + i, make_float4(x.x * inv * wn2.x, x.y * inv * wn2.y, x.z * inv * wn2.z, x.w * inv * wn2.w));
}

// V = 4: rows and pointers are 4-element aligned; V = 1: any width.
template <typename T, int V>
__global__ void embed_kernel(const msa_lm_embed_args a) {
  extern __shared__ float s_row[];
  __shared__ float s_part[32];
  const long long r = blockIdx.x;
  const int width = a.width;
  int tok = a.token[r];
  if (tok < 0 || tok >= a.vocab) {
    if (threadIdx.x == 0 && a.status) atomicAdd(a.status + 2, 1);
    tok = 0;
  }
  const T* src = reinterpret_cast<const T*>(a.table) + (long long)tok * width;
  const T* pair = nullptr;
  if (a.pair_table) {
    const int s = a.tok_seq[r], t = (int)r - a.cu[s], slot = a.slot[s];
    long long row = a.buckets;
    if (t > 0 || a.start[s] > 0) {
      int prev = t > 0 ? a.token[r - 1] : a.last_token[slot];
      if (prev < 0 || prev >= a.vocab) prev = 0;
      row = ((long long)prev * a.mul_prev + (long long)tok * a.mul_cur) % a.buckets;
      if (row < 0) row += a.buckets;
    }
    pair = reinterpret_cast<const T*>(a.pair_table) + row * width;
    __syncthreads();                             // every thread has read the sequence's previous token
    if (t == 0 && threadIdx.x == 0) a.last_token[slot] = a.token[a.cu[s + 1] - 1];
  }
  T* cat0 = reinterpret_cast<T*>(a.cat0);
  T* cat1 = reinterpret_cast<T*>(a.cat1);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    if constexpr (V == 4) {
      float4 x = load4(src + i);
      if (pair) { const float4 y = load4(pair + i); x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w; }
      store4(a.x_out + r * width + i, x);
      if (a.x_copy) store4(a.x_copy + r * width + i, x);
      if (cat0) store4(cat0 + r * a.cat_stride + i, x);
      if (cat1) store4(cat1 + r * a.cat_stride + i, x);
      store4(s_row + i, x);
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    } else {
      float x = to_f(src[i]);
      if (pair) x += to_f(pair[i]);
      a.x_out[r * width + i] = x;
      if (a.x_copy) a.x_copy[r * width + i] = x;
      if (cat0) cat0[r * a.cat_stride + i] = from_f<T>(x);
      if (cat1) cat1[r * a.cat_stride + i] = from_f<T>(x);
      s_row[i] = x;
      ss += x * x;
    }
  }
  if (!a.h_out) return;
  T* h = reinterpret_cast<T*>(a.h_out);
  T* h2 = reinterpret_cast<T*>(a.h_out2);
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)width + a.eps);
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 x = load4(s_row + i), w = load4(a.w_next + i);
      store4(h + r * width + i, make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w));
      if (h2) {
        const float4 w2 = load4(a.w_next2 + i);
        store4(h2 + r * width + i, make_float4(x.x * inv * w2.x, x.y * inv * w2.y, x.z * inv * w2.z, x.w * inv * w2.w));
      }
    } else {
      h[r * width + i] = from_f<T>(s_row[i] * inv * a.w_next[i]);
      if (h2) h2[r * width + i] = from_f<T>(s_row[i] * inv * a.w_next2[i]);
    }
  }
}

// x = cap * tanh(x / cap), in place.
__global__ void __launch_bounds__(256) softcap_kernel(float* x, long long n, float cap) {
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) x[i] = cap * tanhf(x[i] / cap);
}

// out[r, part * cols + c] = part-th share of tanh(x[r, c]): with two parts the bf16 rounding and what it leaves behind,
// so that a product over both keeps 16 significant bits.
template <typename T>
__global__ void __launch_bounds__(256) tanh_split_kernel(const float* __restrict__ x, int cols, int parts, long long n, T* __restrict__ out) {
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
    const long long r = i / cols;
    const int c = (int)(i - r * cols);
    float v = tanhf(x[i]);
    for (int k = 0; k < parts; ++k) {
      const T part = from_f<T>(v);
      out[(r * parts + k) * cols + c] = part;
      v -= to_f(part);
    }
  }
}

// Row r of h beside row r-1 of its sequence (of the previous step: from `shift`): out[m, r] = h + (before - h) * mu[m].
// The block of a sequence's first row hands the step's last row over to `shift`.
template <typename T, int V>
__global__ void token_shift_kernel(const T* __restrict__ h, const float* __restrict__ mu, int n_mix, int n_tok, int width,
                                   const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ slot,
                                   const int32_t* __restrict__ start, const int32_t* __restrict__ cu, T* shift, T* __restrict__ out) {
  const long long r = blockIdx.x;
  const int s = tok_seq[r], t = (int)r - cu[s];
  T* state = shift + (long long)slot[s] * width;
  const bool from_state = t == 0, none = from_state && start[s] == 0;
  const T* before = from_state ? state : h + (r - 1) * width;
  const T* last = h + (long long)(cu[s + 1] - 1) * width;
  for (int i = (blockIdx.y * blockDim.x + threadIdx.x) * V; i < width; i += gridDim.y * blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 x = load4(h + r * width + i);
      float4 d = none ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(before + i);
      if (from_state) store4(state + i, load4(last + i));
      d.x -= x.x; d.y -= x.y; d.z -= x.z; d.w -= x.w;
      for (int m = 0; m < n_mix; ++m) {
        const float4 w = load4(mu + (long long)m * width + i);
        store4(out + ((long long)m * n_tok + r) * width + i,
               make_float4(fmaf(d.x, w.x, x.x), fmaf(d.y, w.y, x.y), fmaf(d.z, w.z, x.z), fmaf(d.w, w.w, x.w)));
      }
    } else {
      const float x = to_f(h[r * width + i]), d = (none ? 0.f : to_f(before[i])) - x;
      if (from_state) state[i] = last[i];
      for (int m = 0; m < n_mix; ++m) out[((long long)m * n_tok + r) * width + i] = from_f<T>(fmaf(d, mu[(long long)m * width + i], x));
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
lm_silu_mul_kernel(const T* __restrict__ gu, long long stride, int ff, long long n_rows, T* __restrict__ out, long long out_stride) {
  const int per_row = ff / V;
  const long long total = n_rows * per_row;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / per_row;
    const int j = (int)(i % per_row) * V;
    if constexpr (V == 4) {
      const float4 g = load4(gu + r * stride + j), u = load4(gu + r * stride + ff + j);
      store4(out + r * out_stride + j, make_float4(silu_f(g.x) * u.x, silu_f(g.y) * u.y, silu_f(g.z) * u.z, silu_f(g.w) * u.w));
    } else {
      out[r * out_stride + j] = from_f<T>(silu_f(to_f(gu[r * stride + j])) * to_f(gu[r * stride + ff + j]));
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
                                    int64_t cat_stride, const float* add, const float* w_next2, void* h_out2, int32_t dtype,
                                    void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && (!y || dtype_ok(y_dtype)), "residual_norm: bad dtype");
  MSA_REQUIRE(n_rows >= 0 && width > 0 && width <= 12000, "residual_norm: width must be 1..12000");
  MSA_REQUIRE(base || y, "residual_norm: neither base nor branch");
  MSA_REQUIRE(!h_out || w_next, "residual_norm: h_out needs w_next");
  MSA_REQUIRE(!h_out2 || (h_out && w_next2), "residual_norm: h_out2 needs h_out and w_next2");
  MSA_REQUIRE(!inv || (mix && top > 0 && y), "residual_norm: a mixture needs weights and top > 0");
  if (n_rows == 0) return MSA_OK;
  ResNormParams p{base, base_stride, y, y_dtype, y_stride, inv, mix, top, w_branch, w_next, eps, rows, width, x_out, h_out,
                  cat_out, cat_stride, add, w_next2, h_out2};
  const int e = (int)dtype_size(dtype), ey = (int)dtype_size(y_dtype);
  const bool v4 = width % 4 == 0 && base_stride % 4 == 0 && (!y || y_stride % 4 == 0) && (!cat_out || cat_stride % 4 == 0) &&
                  vec4_ok(base, 4) && vec4_ok(y, ey) && vec4_ok(w_branch, 4) && vec4_ok(w_next, 4) && vec4_ok(x_out, 4) &&
                  vec4_ok(h_out, e) && vec4_ok(cat_out, e) && vec4_ok(add, 4) && vec4_ok(w_next2, 4) && vec4_ok(h_out2, e);
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

extern "C" int msa_lm_embed(const msa_lm_embed_args* args, void* stream) {
  MSA_REQUIRE(args, "embed: null arguments");
  const msa_lm_embed_args a = *args;
  MSA_REQUIRE(dtype_ok(a.dtype) && a.table && a.token && a.x_out, "embed: bad arguments");
  MSA_REQUIRE(a.n_rows >= 0 && a.width > 0 && a.width <= 12000 && a.vocab > 0, "embed: bad sizes");
  MSA_REQUIRE((!a.h_out || a.w_next) && (!a.h_out2 || (a.h_out && a.w_next2)), "embed: a norm needs its weight");
  MSA_REQUIRE(!a.pair_table || (a.buckets > 0 && a.last_token && a.tok_seq && a.slot && a.start && a.cu), "embed: a pair table needs the step's tables");
  if (a.n_rows == 0) return MSA_OK;
  const int e = (int)dtype_size(a.dtype);
  const bool v4 = a.width % 4 == 0 && a.cat_stride % 4 == 0 && vec4_ok(a.table, e) && vec4_ok(a.pair_table, e) && vec4_ok(a.x_out, 4) &&
                  vec4_ok(a.x_copy, 4) && vec4_ok(a.h_out, e) && vec4_ok(a.h_out2, e) && vec4_ok(a.cat0, e) && vec4_ok(a.cat1, e) &&
                  vec4_ok(a.w_next, 4) && vec4_ok(a.w_next2, 4);
  const size_t smem = (size_t)a.width * 4;
  MSA_LM_DISPATCH(a.dtype, {
    if (v4) embed_kernel<T, 4><<<a.n_rows, row_threads(a.width), smem, (cudaStream_t)stream>>>(a);
    else embed_kernel<T, 1><<<a.n_rows, row_threads(a.width), smem, (cudaStream_t)stream>>>(a);
  });
  MSA_LAUNCH_OK("embed_kernel");
  return MSA_OK;
}

namespace {
inline int flat_grid(long long n) { return (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16); }
}  // namespace

extern "C" int msa_lm_softcap(float* x, int64_t n, float cap, void* stream) {
  MSA_REQUIRE(x && n >= 0 && cap > 0.f, "softcap: bad arguments");
  if (n == 0) return MSA_OK;
  softcap_kernel<<<flat_grid(n), 256, 0, (cudaStream_t)stream>>>(x, n, cap);
  MSA_LAUNCH_OK("softcap_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_tanh_split(const float* x, int32_t n_rows, int32_t cols, int32_t parts, void* out, int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && x && out && n_rows >= 0 && cols > 0 && parts >= 1, "tanh_split: bad arguments");
  const long long n = (long long)n_rows * cols;
  if (n == 0) return MSA_OK;
  MSA_LM_DISPATCH(dtype, { tanh_split_kernel<T><<<flat_grid(n), 256, 0, (cudaStream_t)stream>>>(x, cols, parts, n, (T*)out); });
  MSA_LAUNCH_OK("tanh_split_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_token_shift(const void* h, const float* mu, int32_t n_mix, int32_t n_tok, int32_t width, const int32_t* tok_seq,
                                  const int32_t* slot, const int32_t* start, const int32_t* cu, void* shift, void* out, int32_t dtype,
                                  void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && h && mu && tok_seq && slot && start && cu && shift && out, "token_shift: null pointer or bad dtype");
  MSA_REQUIRE(n_mix > 0 && n_tok >= 0 && width > 0, "token_shift: bad sizes");
  if (n_tok == 0) return MSA_OK;
  const int e = (int)dtype_size(dtype);
  const bool v4 = width % 4 == 0 && vec4_ok(h, e) && vec4_ok(mu, 4) && vec4_ok(shift, e) && vec4_ok(out, e);
  const int per = v4 ? width / 4 : width, threads = per >= 256 ? 256 : (per + 31) / 32 * 32;
  const dim3 grid((unsigned)n_tok, n_tok <= 256 ? (unsigned)((per + threads - 1) / threads) : 1u);   // few rows: spread the columns
  MSA_LM_DISPATCH(dtype, {
    if (v4) token_shift_kernel<T, 4><<<grid, threads, 0, (cudaStream_t)stream>>>((const T*)h, mu, n_mix, n_tok, width, tok_seq, slot, start, cu, (T*)shift, (T*)out);
    else token_shift_kernel<T, 1><<<grid, threads, 0, (cudaStream_t)stream>>>((const T*)h, mu, n_mix, n_tok, width, tok_seq, slot, start, cu, (T*)shift, (T*)out);
  });
  MSA_LAUNCH_OK("token_shift_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_silu_mul(const void* gu, int64_t gu_stride, int32_t n_rows, int32_t ff, void* out, int64_t out_stride,
                               int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && gu && out && n_rows >= 0 && ff > 0, "lm_silu_mul: bad arguments");
  if (n_rows == 0) return MSA_OK;
  const int e = (int)dtype_size(dtype);
  const bool v4 = ff % 4 == 0 && gu_stride % 4 == 0 && out_stride % 4 == 0 && vec4_ok(gu, e) && vec4_ok(out, e);
  const long long total = (long long)n_rows * (v4 ? ff / 4 : ff);
  const int grid = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  MSA_LM_DISPATCH(dtype, {
    if (v4) lm_silu_mul_kernel<T, 4><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)gu, gu_stride, ff, n_rows, (T*)out, out_stride);
    else lm_silu_mul_kernel<T, 1><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)gu, gu_stride, ff, n_rows, (T*)out, out_stride);
  });
  MSA_LAUNCH_OK("lm_silu_mul_kernel");
  return MSA_OK;
}
