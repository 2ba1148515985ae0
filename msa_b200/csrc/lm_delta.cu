// Gated delta rule: short causal convolution, unit norms, gates, the recurrence in fp32, and the gated output norm.
//
// Per sequence slot a layer keeps the matrix state [heads, dim, vdim] (fp32) and the last taps-1 inputs of the
// convolution.  The convolution inputs are double-buffered by the parity of the sequence's position, so a decode launch
// can read the old ones in every block while it writes the new ones.
//
// One step of a head, with S the state before it, reads S once for both products:
//     c = S^T k,  r = S^T q;   u = beta (v - g c);   S <- g S + k u^T;   o = g r + (q.k) u
#include <type_traits>

#include "lm_common.cuh"
#include "lm_conv.cuh"

namespace msa {

struct DeltaLayout {
  int nqk, nv, chan;   // kv_heads*dim, heads*vdim, 2*nqk + nv
  __host__ __device__ explicit DeltaLayout(const msa_lm_delta_args& a)
      : nqk(a.kv_heads * a.dim), nv(a.heads * a.vdim), chan(2 * a.kv_heads * a.dim + a.heads * a.vdim) {}
};

// Convolution of channel c at token n (row of proj), t tokens into its portion that starts at position p0; then silu.
template <typename T>
__device__ __forceinline__ float conv_silu(const msa_lm_delta_args& a, const T* state_half, int chan, long long n, int t,
                                           int p0, int c) {
  const T* proj = reinterpret_cast<const T*>(a.proj);
  float acc = 0.f;
  for (int i = 0; i < a.taps; ++i) {
    const int lag = a.taps - 1 - i;
    const float w = a.conv_w[(long long)i * chan + c];
    if (t - lag >= 0) acc = fmaf(w, to_f(proj[(n - lag) * a.proj_stride + c]), acc);
    else if (p0 + t - lag >= 0) acc = fmaf(w, to_f(state_half[(long long)(a.taps - 1 + t - lag) * chan + c]), acc);
  }
  return silu_f(acc);
}
template <typename T>
__device__ __forceinline__ const T* conv_half(const msa_lm_delta_args& a, int chan, int slot, int p) {
  return reinterpret_cast<const T*>(a.conv_state) + ((long long)slot * 2 + (p & 1)) * (a.taps - 1) * chan;
}

// ---- prefill: convolution, unit norms, gates ---------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const msa_lm_delta_args a, float* __restrict__ qk, float* __restrict__ v, float* __restrict__ gates) {
  const DeltaLayout L(a);
  const int row = blockIdx.x;                       // counts from the first non-decode token
  const long long n = (long long)a.n_decode + row;
  const int s = a.tok_seq[n], t = (int)(n - a.cu[s]), p0 = a.start[s];
  const T* half = conv_half<T>(a, L.chan, a.slot[s], p0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int hd = warp; hd < 2 * a.kv_heads; hd += 8) {   // heads of q, then of k
    float* dst = qk + (long long)row * 2 * L.nqk + (long long)hd * a.dim;
    float ss = 0.f;
    for (int i = lane; i < a.dim; i += 32) {
      const float x = conv_silu<T>(a, half, L.chan, n, t, p0, hd * a.dim + i);
      dst[i] = x;
      ss += x * x;
    }
    ss = warp_sum_f(ss);
    const float sc = (hd < a.kv_heads ? 1.f / sqrtf((float)a.dim) : 1.f) / sqrtf(ss + 1e-6f);
    for (int i = lane; i < a.dim; i += 32) dst[i] *= sc;
  }
  for (int i = threadIdx.x; i < L.nv; i += blockDim.x)
    v[(long long)row * L.nv + i] = conv_silu<T>(a, half, L.chan, n, t, p0, 2 * L.nqk + i);
  const T* g = reinterpret_cast<const T*>(a.proj) + n * a.proj_stride + 2 * L.nqk + 2 * L.nv;
  for (int h = threadIdx.x; h < a.heads; h += blockDim.x) {
    gates[(long long)row * 2 * a.heads + h] = -expf(a.a_log[h]) * softplus_f(to_f(g[a.heads + h]) + a.dt_bias[h]);
    gates[(long long)row * 2 * a.heads + a.heads + h] = sigmoid_f(to_f(g[h]));
  }
}

// The same with four channels per lane and the convolution's history in registers: a warp walks 8 rows of one unit (a
// head of q or k, or 128 channels of v), so every input is loaded once.
constexpr int kPrepRows = 8;

// SPLIT: q and k leave as pairs of bf16 numbers whose sum they are, [rows, 2 (q, k), 2 (hi, lo), kv_heads, dim], and v in
// bf16.
template <typename T, int TAPS, bool SPLIT>
__global__ void __launch_bounds__(256)
delta_prep_vec_kernel(const msa_lm_delta_args a, void* __restrict__ qk_out, void* __restrict__ v_out, float* __restrict__ gates) {
  using Raw = typename Raw4<T>::type;
  auto raw = [](const T* p) { return *reinterpret_cast<const Raw*>(p); };
  const DeltaLayout L(a);
  const int row0 = blockIdx.x * kPrepRows, n_rows = a.n_tok - a.n_decode;
  const int n_here = min(kPrepRows, n_rows - row0);
  const T* proj = reinterpret_cast<const T*>(a.proj) + ((long long)a.n_decode + row0) * a.proj_stride;   // row 0 of the block
  if (blockIdx.y == 0) {
    for (int i = threadIdx.x; i < n_here * a.heads; i += 256) {
      const int r = i / a.heads, h = i % a.heads;
      const T* g = proj + (long long)r * a.proj_stride + 2 * L.nqk + 2 * L.nv;
      float* dst = gates + (long long)(row0 + r) * 2 * a.heads + h;
      dst[0] = -expf(a.a_log[h]) * softplus_f(to_f(g[a.heads + h]) + a.dt_bias[h]);
      dst[a.heads] = sigmoid_f(to_f(g[h]));
    }
  }
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const bool is_v = unit >= 2 * a.kv_heads;
  const int seg = (unit - 2 * a.kv_heads) * 128;
  if (is_v && seg >= L.nv) return;
  const int c0 = is_v ? seg + lane * 4 : lane * 4;          // within v, or within the head
  const bool on = is_v ? c0 < L.nv : c0 < a.dim;
  const int c = is_v ? 2 * L.nqk + c0 : unit * a.dim + c0;
  const Raw zero{};
  // every input of the block's rows and of the TAPS-1 rows before them, all loads in flight at once
  Raw x[kPrepRows + TAPS - 1];
  const int s0 = a.tok_seq[a.n_decode + row0], first = a.n_decode + row0 - a.cu[s0], p0 = a.start[s0];
  const T* half = conv_half<T>(a, L.chan, a.slot[s0], p0);
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int t = first - (TAPS - 1) + j;                   // token of the portion that the block's first row continues
    x[j] = zero;
    if (on) {
      if (t >= 0) x[j] = raw(proj + (long long)(j - (TAPS - 1)) * a.proj_stride + c);
      else if (p0 + t >= 0) x[j] = raw(half + (long long)(TAPS - 1 + t) * L.chan + c);
    }
  }
#pragma unroll
  for (int r = 0; r < kPrepRows; ++r) x[TAPS - 1 + r] = on && r < n_here ? raw(proj + (long long)r * a.proj_stride + c) : zero;
  float4 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = on ? load4(a.conv_w + (long long)j * L.chan + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float post = unit < a.kv_heads ? 1.f / sqrtf((float)a.dim) : 1.f;
#pragma unroll
  for (int r = 0; r < kPrepRows; ++r) {
    if (r >= n_here) break;
    const long long row = row0 + r, n = a.n_decode + row;
    Raw in[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) in[j] = x[r + j];
    const int s = a.tok_seq[n];
    if (s != s0) {                                          // a row of a later sequence: its own history where that is short
      const int t = (int)(n - a.cu[s]);
      if (t < TAPS - 1) {
        const int q0 = a.start[s];
        const T* h2 = conv_half<T>(a, L.chan, a.slot[s], q0);
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
          const int lag = TAPS - 1 - j;
          if (t - lag < 0) in[j] = on && q0 + t - lag >= 0 ? raw(h2 + (long long)(TAPS - 1 + t - lag) * L.chan + c) : zero;
        }
      }
    }
    float y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float4 f = widen(in[j]);
      y[0] = fmaf(w[j].x, f.x, y[0]); y[1] = fmaf(w[j].y, f.y, y[1]);
      y[2] = fmaf(w[j].z, f.z, y[2]); y[3] = fmaf(w[j].w, f.w, y[3]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = silu_act<T>(y[e]);
    if (is_v) {
      using TV = typename std::conditional<SPLIT, __nv_bfloat16, float>::type;
      if (on) store4(reinterpret_cast<TV*>(v_out) + row * L.nv + c0, make_float4(y[0], y[1], y[2], y[3]));
      continue;
    }
    const float ss = warp_sum_f(on ? y[0] * y[0] + y[1] * y[1] + y[2] * y[2] + y[3] * y[3] : 0.f);
    const float sc = post / sqrtf(ss + 1e-6f);
    if (!on) continue;
    const float4 q = make_float4(y[0] * sc, y[1] * sc, y[2] * sc, y[3] * sc);
    if constexpr (SPLIT) {
      const int is_k = unit >= a.kv_heads;
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(qk_out) + row * 4 * L.nqk + (long long)is_k * 2 * L.nqk +
                           (unit - is_k * a.kv_heads) * a.dim + c0;
      const float4 hi = make_float4(__bfloat162float(__float2bfloat16_rn(q.x)), __bfloat162float(__float2bfloat16_rn(q.y)),
                                    __bfloat162float(__float2bfloat16_rn(q.z)), __bfloat162float(__float2bfloat16_rn(q.w)));
      store4(dst, hi);
      store4(dst + L.nqk, make_float4(q.x - hi.x, q.y - hi.y, q.z - hi.z, q.w - hi.w));
    } else {
      store4(reinterpret_cast<float*>(qk_out) + row * 2 * L.nqk + (long long)unit * a.dim + c0, q);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) delta_conv_store_kernel(const msa_lm_delta_args a) {
  const DeltaLayout L(a);
  const int s = a.n_decode + blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= L.chan) return;
  const int len = a.cu[s + 1] - a.cu[s], p0 = a.start[s], keep = a.taps - 1;
  const T* proj = reinterpret_cast<const T*>(a.proj);
  const T* old = conv_half<T>(a, L.chan, a.slot[s], p0);
  T* dst = reinterpret_cast<T*>(a.conv_state) + ((long long)a.slot[s] * 2 + ((p0 + len) & 1)) * keep * L.chan;
  // ascending: an entry that comes from the old half (possibly the same memory) is read before it is overwritten
  for (int j = 0; j < keep; ++j) {
    const int t = len - keep + j;                   // token of the portion, negative: before it
    T x = from_f<T>(0.f);
    if (t >= 0) x = proj[((long long)a.cu[s] + t) * a.proj_stride + c];
    else if (p0 + t >= 0) x = old[(long long)(keep + t) * L.chan + c];
    dst[(long long)j * L.chan + c] = x;
  }
}

// ---- prefill: the recurrence, token by token ------------------------------------------------------------------------
// 8 lanes share a state column (R rows each, in registers); a warp covers 4 columns, a block of 4 warps 16.  Tokens are
// staged in shared memory 16 at a time.
constexpr int kScTok = 16, kScCols = 16, kScThreads = 128;

template <int R>
__global__ void __launch_bounds__(kScThreads)
delta_scan_kernel(const msa_lm_delta_args a, const float* __restrict__ qk, const float* __restrict__ v,
                  const float* __restrict__ gates, float* __restrict__ o) {
  constexpr int D = 8 * R;
  // dimension d = part * R + r of a token lies at (r / 4) * 32 + part * 4 + r % 4: the eight lanes of a column read
  // 128 consecutive bytes per vector
  __shared__ __align__(16) float s_q[kScTok][D], s_k[kScTok][D];
  __shared__ float s_v[kScTok][kScCols], s_o[kScTok][kScCols], s_g[kScTok], s_b[kScTok], s_qk[kScTok];
  const DeltaLayout L(a);
  const int s = a.n_decode + blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kScCols;
  const int hk = h / (a.heads / a.kv_heads);
  const int len = a.cu[s + 1] - a.cu[s];
  const long long row0 = a.cu[s] - a.n_decode;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int part = lane & 7, cl = warp * 4 + (lane >> 3), col = c0 + cl;
  float* S = a.state + (((long long)a.slot[s] * a.heads + h) * a.dim) * a.vdim;
  float st[R];
  const bool fresh = a.start[s] == 0;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = part * R + r;
    st[r] = (!fresh && d < a.dim && col < a.vdim) ? S[(long long)d * a.vdim + col] : 0.f;
  }
  for (int t0 = 0; t0 < len; t0 += kScTok) {
    const int nt = min(kScTok, len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * D; i += kScThreads) {
      const int t = i / D, d = i % D;
      const float* src = qk + (row0 + t0 + t) * 2 * L.nqk + (long long)hk * a.dim + d;
      const int at = (d % R / 4) * 32 + d / R * 4 + d % 4;
      s_q[t][at] = d < a.dim ? src[0] : 0.f;
      s_k[t][at] = d < a.dim ? src[L.nqk] : 0.f;
    }
    for (int i = threadIdx.x; i < nt * kScCols; i += kScThreads) {
      const int t = i / kScCols, c = i % kScCols;
      s_v[t][c] = c0 + c < a.vdim ? v[(row0 + t0 + t) * L.nv + (long long)h * a.vdim + c0 + c] : 0.f;
    }
    if (threadIdx.x < nt) {
      const float* g = gates + (row0 + t0 + threadIdx.x) * 2 * a.heads + h;
      s_g[threadIdx.x] = expf(g[0]);
      s_b[threadIdx.x] = g[a.heads];
    }
    __syncthreads();
    for (int t = warp; t < nt; t += kScThreads / 32) {
      float d = 0.f;
      for (int i = lane; i < D; i += 32) d = fmaf(s_q[t][i], s_k[t][i], d);
      d = warp_sum_f(d);
      if (lane == 0) s_qk[t] = d;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      float k[R], c = 0.f, r_ = 0.f, c2 = 0.f, r2 = 0.f;
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const float4 kv = load4(&s_k[t][r * 8 + part * 4]), qv = load4(&s_q[t][r * 8 + part * 4]);
        k[r] = kv.x; k[r + 1] = kv.y; k[r + 2] = kv.z; k[r + 3] = kv.w;
        c = fmaf(st[r], kv.x, c); c2 = fmaf(st[r + 1], kv.y, c2); c = fmaf(st[r + 2], kv.z, c); c2 = fmaf(st[r + 3], kv.w, c2);
        r_ = fmaf(st[r], qv.x, r_); r2 = fmaf(st[r + 1], qv.y, r2); r_ = fmaf(st[r + 2], qv.z, r_); r2 = fmaf(st[r + 3], qv.w, r2);
      }
      c += c2;
      r_ += r2;
#pragma unroll
      for (int w = 1; w < 8; w <<= 1) {
        c += __shfl_xor_sync(0xffffffffu, c, w);
        r_ += __shfl_xor_sync(0xffffffffu, r_, w);
      }
      const float g = s_g[t], u = s_b[t] * (s_v[t][cl] - g * c);
#pragma unroll
      for (int r = 0; r < R; ++r) st[r] = fmaf(k[r], u, g * st[r]);
      if (part == 0) s_o[t][cl] = fmaf(g, r_, s_qk[t] * u);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kScCols; i += kScThreads) {
      const int t = i / kScCols, c = i % kScCols;
      if (c0 + c < a.vdim) o[(row0 + t0 + t) * L.nv + (long long)h * a.vdim + c0 + c] = s_o[t][c];
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = part * R + r;
    if (d < a.dim && col < a.vdim) S[(long long)d * a.vdim + col] = st[r];
  }
}

// out = o / rms(o) * w * silu(gate); one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
delta_out_kernel(const msa_lm_delta_args a, const float* __restrict__ o, T* __restrict__ out, long long out_stride, long long n, bool vec) {
  const DeltaLayout L(a);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const unsigned item = blockIdx.x * 8 + warp;
  if (item >= (unsigned)(n * a.heads)) return;
  const long long row = item / (unsigned)a.heads;
  const int h = (int)(item % (unsigned)a.heads);
  const float* src = o + row * L.nv + (long long)h * a.vdim;
  const T* gate = reinterpret_cast<const T*>(a.proj) + (a.n_decode + row) * a.proj_stride + 2 * L.nqk + L.nv + (long long)h * a.vdim;
  float ss = 0.f;
  if (vec) {
    for (int i = lane * 4; i < a.vdim; i += 128) { const float4 x = load4(src + i); ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w; }
    const float inv = 1.f / sqrtf(warp_sum_f(ss) / (float)a.vdim + a.eps);
    for (int i = lane * 4; i < a.vdim; i += 128) {
      const float4 x = load4(src + i), w = load4(a.w_norm + i), z = load4(gate + i);
      store4(out + row * out_stride + (long long)h * a.vdim + i,
             make_float4(x.x * inv * w.x * silu_act<T>(z.x), x.y * inv * w.y * silu_act<T>(z.y), x.z * inv * w.z * silu_act<T>(z.z),
                         x.w * inv * w.w * silu_act<T>(z.w)));
    }
    return;
  }
  for (int i = lane; i < a.vdim; i += 32) ss += src[i] * src[i];
  const float inv = 1.f / sqrtf(warp_sum_f(ss) / (float)a.vdim + a.eps);
  for (int i = lane; i < a.vdim; i += 32)
    out[row * out_stride + (long long)h * a.vdim + i] = from_f<T>(src[i] * inv * a.w_norm[i] * silu_f(to_f(gate[i])));
}

// ---- decode: everything between the projections and the output product -----------------------------------------------
// One block per (sequence, head).  Threads form a grid of row groups x column vectors over the state; the state is read
// (twice, the second time from L1 / L2) and written once.
constexpr int kDdThreads = 256;

// STAGE: the state is copied to shared memory before anything else (cp.async) and read from there both times.
template <typename T, int V, bool STAGE>
__global__ void __launch_bounds__(kDdThreads)
delta_decode_kernel(const msa_lm_delta_args a, T* __restrict__ out, long long out_stride, int groups) {
  extern __shared__ float sm[];
  __shared__ float s_part[32];
  const DeltaLayout L(a);
  const int b = blockIdx.y, h = blockIdx.x, group = a.heads / a.kv_heads, hk = h / group;
  const int dk = a.dim, dv = a.vdim, keep = a.taps - 1;
  float* s_q = sm;                        // [dk]
  float* s_k = s_q + dk;                  // [dk]
  float* s_v = s_k + dk;                  // [dv], then the output row
  float* s_c = sm + (2 * dk + dv + 3) / 4 * 4;   // [groups][dv]
  float* s_r = s_c + groups * dv;         // [groups][dv]
  const int slot = a.slot[b], p = a.pos[b];
  float* S = a.state + (((long long)slot * a.heads + h) * dk) * dv;
  float* s_state = sm + (2 * dk + dv + 3) / 4 * 4 + 2 * groups * dv;   // [dk][dv]
  if constexpr (STAGE) {
    if (p != 0) {
      const uint32_t dst = (uint32_t)__cvta_generic_to_shared(s_state);
      for (int i = threadIdx.x; i < dk * dv / 4; i += kDdThreads)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + i * 16), "l"(S + (long long)i * 4) : "memory");
    } else {
      for (int i = threadIdx.x; i < dk * dv / 4; i += kDdThreads) store4(s_state + i * 4, make_float4(0.f, 0.f, 0.f, 0.f));
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  const T* proj = reinterpret_cast<const T*>(a.proj) + (long long)b * a.proj_stride;
  const float raw_beta = to_f(proj[2 * L.nqk + 2 * L.nv + h]), raw_decay = to_f(proj[2 * L.nqk + 2 * L.nv + a.heads + h]);
  const float a_log = a.a_log[h], dt_bias = a.dt_bias[h];
  const T* gate = proj + 2 * L.nqk + L.nv + (long long)h * dv;
  const float gate0 = threadIdx.x < dv ? to_f(gate[threadIdx.x]) : 0.f, norm0 = threadIdx.x < dv ? a.w_norm[threadIdx.x] : 0.f;
  const T* old = conv_half<T>(a, L.chan, slot, p);
  T* fresh = reinterpret_cast<T*>(a.conv_state) + ((long long)slot * 2 + ((p + 1) & 1)) * keep * L.chan;
  for (int i = threadIdx.x; i < 2 * dk + dv; i += kDdThreads) {
    const int c = i < dk ? hk * dk + i : (i < 2 * dk ? L.nqk + hk * dk + (i - dk) : 2 * L.nqk + h * dv + (i - 2 * dk));
    const bool writer = i >= 2 * dk || h % group == 0;
    const float* w = a.conv_w + c;
    float acc = 0.f;
    for (int j = 0; j < keep; ++j) {
      const T x = p - keep + j >= 0 ? old[(long long)j * L.chan + c] : from_f<T>(0.f);
      acc = fmaf(w[(long long)j * L.chan], to_f(x), acc);
      if (writer && j > 0) fresh[(long long)(j - 1) * L.chan + c] = x;
    }
    const T x = proj[c];
    acc = fmaf(w[(long long)keep * L.chan], to_f(x), acc);
    if (writer && keep > 0) fresh[(long long)(keep - 1) * L.chan + c] = x;
    sm[i] = silu_f(acc);
  }
  __syncthreads();
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int i = threadIdx.x; i < dk; i += kDdThreads) {
    qq += s_q[i] * s_q[i];
    kk += s_k[i] * s_k[i];
    qk += s_q[i] * s_k[i];
  }
  qq = warp_sum_f(qq);
  kk = warp_sum_f(kk);
  qk = warp_sum_f(qk);
  if ((threadIdx.x & 31) == 0) {
    const int w = threadIdx.x >> 5;
    s_part[w] = qq; s_part[8 + w] = kk; s_part[16 + w] = qk;
  }
  if constexpr (STAGE) asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  qq = kk = qk = 0.f;
#pragma unroll
  for (int w = 0; w < kDdThreads / 32; ++w) { qq += s_part[w]; kk += s_part[8 + w]; qk += s_part[16 + w]; }
  const float sq = 1.f / (sqrtf((float)dk) * sqrtf(qq + 1e-6f)), sk = 1.f / sqrtf(kk + 1e-6f);
  qk *= sq * sk;
  const float beta = sigmoid_f(raw_beta);
  const float g = expf(-expf(a_log) * softplus_f(raw_decay + dt_bias));
  const bool zero = p == 0;
  const int cols = dv / V, rg = threadIdx.x / cols, cv = (threadIdx.x % cols) * V;   // groups * cols <= blockDim
  const bool active = rg < groups;
  if constexpr (STAGE) {
    if (active) {
      float4 ac = make_float4(0.f, 0.f, 0.f, 0.f), ar = ac;
#pragma unroll 4
      for (int d = rg; d < dk; d += groups) {
        const float4 x = load4(s_state + d * dv + cv);
        const float kd = s_k[d], qd = s_q[d];
        ac.x = fmaf(x.x, kd, ac.x); ac.y = fmaf(x.y, kd, ac.y); ac.z = fmaf(x.z, kd, ac.z); ac.w = fmaf(x.w, kd, ac.w);
        ar.x = fmaf(x.x, qd, ar.x); ar.y = fmaf(x.y, qd, ar.y); ar.z = fmaf(x.z, qd, ar.z); ar.w = fmaf(x.w, qd, ar.w);
      }
      store4(s_c + rg * dv + cv, ac);
      store4(s_r + rg * dv + cv, ar);
    }
  } else
  // columns are walked in one sweep when they fit the block; otherwise cols > blockDim is split over `cs`
  for (int cs = 0; cs < cols; cs += kDdThreads) {
    const int c = cols > kDdThreads ? (cs + threadIdx.x) * V : cv;
    const int g0 = cols > kDdThreads ? 0 : rg;
    const bool on = cols > kDdThreads ? cs + (int)threadIdx.x < cols : active;
    if (on) {
      float ac[V], ar[V];
#pragma unroll
      for (int e = 0; e < V; ++e) ac[e] = ar[e] = 0.f;
      if (!zero)
#pragma unroll 4
        for (int d = g0; d < dk; d += groups) {
          float x[V];
          if constexpr (V == 4) { const float4 f = load4(S + (long long)d * dv + c); x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w; }
          else x[0] = S[(long long)d * dv + c];
          const float kd = s_k[d], qd = s_q[d];
#pragma unroll
          for (int e = 0; e < V; ++e) { ac[e] = fmaf(x[e], kd, ac[e]); ar[e] = fmaf(x[e], qd, ar[e]); }
        }
#pragma unroll
      for (int e = 0; e < V; ++e) { s_c[g0 * dv + c + e] = ac[e]; s_r[g0 * dv + c + e] = ar[e]; }
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < dv; i += kDdThreads) {
    float c = 0.f, r = 0.f;
    for (int j = 0; j < groups; ++j) { c += s_c[j * dv + i]; r += s_r[j * dv + i]; }
    const float u = beta * (s_v[i] - g * (c * sk)), o = fmaf(g, r * sq, qk * u);
    s_c[i] = u * sk;      // group 0's entry: read by this thread alone
    s_v[i] = o;
    ss += o * o;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)dv + a.eps);   // its barriers publish s_c and s_v
  __syncthreads();
  if constexpr (STAGE) {
    if (active) {
      const float4 u = load4(s_c + cv);
#pragma unroll 4
      for (int d = rg; d < dk; d += groups) {
        const float4 x = load4(s_state + d * dv + cv);
        const float kd = s_k[d];
        store4(S + (long long)d * dv + cv, make_float4(fmaf(kd, u.x, g * x.x), fmaf(kd, u.y, g * x.y), fmaf(kd, u.z, g * x.z), fmaf(kd, u.w, g * x.w)));
      }
    }
  } else
  for (int cs = 0; cs < cols; cs += kDdThreads) {
    const int c = cols > kDdThreads ? (cs + threadIdx.x) * V : cv;
    const int g0 = cols > kDdThreads ? 0 : rg;
    const bool on = cols > kDdThreads ? cs + (int)threadIdx.x < cols : active;
    if (on) {
#pragma unroll 4
      for (int d = g0; d < dk; d += groups) {
        float x[V];
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = 0.f;
        if (!zero) {
          if constexpr (V == 4) { const float4 f = load4(S + (long long)d * dv + c); x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w; }
          else x[0] = S[(long long)d * dv + c];
        }
        const float kd = s_k[d];
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = fmaf(kd, s_c[c + e], g * x[e]);
        if constexpr (V == 4) store4(S + (long long)d * dv + c, make_float4(x[0], x[1], x[2], x[3]));
        else S[(long long)d * dv + c] = x[0];
      }
    }
  }
  for (int i = threadIdx.x; i < dv; i += kDdThreads) {
    const float z = i == (int)threadIdx.x ? gate0 : to_f(gate[i]), w = i == (int)threadIdx.x ? norm0 : a.w_norm[i];
    out[(long long)b * out_stride + (long long)h * dv + i] = from_f<T>(s_v[i] * inv * w * silu_f(z));
  }
}

inline int delta_check(const msa_lm_delta_args* a, const char* what) {
  MSA_REQUIRE(a, "%s: null arguments", what);
  MSA_REQUIRE(dtype_ok(a->dtype) && a->proj && a->conv_w && a->a_log && a->dt_bias && a->w_norm && a->state && a->slot &&
                  a->start && a->cu && a->pos && a->tok_seq, "%s: null pointer or bad dtype", what);
  MSA_REQUIRE(a->taps >= 1 && (a->taps == 1 || a->conv_state), "%s: convolution state missing", what);
  MSA_REQUIRE(a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 && a->dim > 0 && a->vdim > 0,
              "%s: bad head counts or sizes", what);
  MSA_REQUIRE(a->n_decode >= 0 && a->n_decode <= a->n_seq && a->n_tok >= a->n_decode, "%s: bad counts", what);
  return MSA_OK;
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_delta_decode(const msa_lm_delta_args* a, void* out, int64_t out_stride, void* stream) {
  MSA_OK_OR_RETURN(delta_check(a, "delta_decode"));
  MSA_REQUIRE(out, "delta_decode: null output");
  if (a->n_decode == 0) return MSA_OK;
  const int v = a->vdim % 4 == 0 && aligned16(a->state) ? 4 : 1;
  const int cols = a->vdim / v;
  const int groups = cols >= kDdThreads ? 1 : kDdThreads / cols;
  const size_t smem = (size_t)4 * ((2 * a->dim + a->vdim + 3) / 4 * 4 + 2 * groups * a->vdim);
  const bool stage = v == 4 && cols <= kDdThreads && (size_t)a->dim * a->vdim * 4 + smem <= 110 * 1024;
  const dim3 grid((unsigned)a->heads, (unsigned)a->n_decode);
  MSA_LM_DISPATCH(a->dtype, {
    auto launch = [&](auto kernel, DeviceSmem& configured, size_t bytes) -> int {
      MSA_OK_OR_RETURN(ensure_dynamic_smem(kernel, bytes, configured));
      kernel<<<grid, kDdThreads, bytes, (cudaStream_t)stream>>>(*a, (T*)out, out_stride, groups);
      return MSA_OK;
    };
    static DeviceSmem staged, st4, st1;
    if (stage) MSA_OK_OR_RETURN(launch(delta_decode_kernel<T, 4, true>, staged, smem + (size_t)a->dim * a->vdim * 4));
    else if (v == 4) MSA_OK_OR_RETURN(launch(delta_decode_kernel<T, 4, false>, st4, smem));
    else MSA_OK_OR_RETURN(launch(delta_decode_kernel<T, 1, false>, st1, smem));
  });
  MSA_LAUNCH_OK("delta_decode_kernel");
  return MSA_OK;
}

namespace {
bool prep_vec_ok(const msa_lm_delta_args* a, const void* qk, const void* v) {
  const int e4 = 4 * (int)dtype_size(a->dtype);
  return a->taps >= 2 && a->taps <= 4 && a->dim % 4 == 0 && a->dim <= 128 && a->vdim % 4 == 0 && a->proj_stride % 4 == 0 &&
         reinterpret_cast<uintptr_t>(a->proj) % e4 == 0 && reinterpret_cast<uintptr_t>(a->conv_state) % e4 == 0 && aligned16(qk) &&
         aligned16(v) && aligned16(a->conv_w);
}
template <typename T, bool SPLIT>
int launch_prep_vec(const msa_lm_delta_args* a, void* qk, void* v, float* gates, cudaStream_t st) {
  const DeltaLayout L(*a);
  const int units = 2 * a->kv_heads + (L.nv + 127) / 128;
  const dim3 grid((unsigned)((a->n_tok - a->n_decode + kPrepRows - 1) / kPrepRows), (unsigned)((units + 7) / 8));
  if (a->taps == 2) delta_prep_vec_kernel<T, 2, SPLIT><<<grid, 256, 0, st>>>(*a, qk, v, gates);
  else if (a->taps == 3) delta_prep_vec_kernel<T, 3, SPLIT><<<grid, 256, 0, st>>>(*a, qk, v, gates);
  else delta_prep_vec_kernel<T, 4, SPLIT><<<grid, 256, 0, st>>>(*a, qk, v, gates);
  MSA_LAUNCH_OK("delta_prep_vec_kernel");
  return MSA_OK;
}
}  // namespace

extern "C" int msa_lm_delta_prep(const msa_lm_delta_args* a, float* qk, float* v, float* gates, void* stream) {
  MSA_OK_OR_RETURN(delta_check(a, "delta_prep"));
  MSA_REQUIRE(qk && v && gates, "delta_prep: null output");
  const int rows = a->n_tok - a->n_decode;
  if (rows == 0) return MSA_OK;
  if (prep_vec_ok(a, qk, v)) {
    MSA_LM_DISPATCH(a->dtype, { return (launch_prep_vec<T, false>(a, qk, v, gates, (cudaStream_t)stream)); });
  }
  MSA_LM_DISPATCH(a->dtype, { delta_prep_kernel<T><<<rows, 256, 0, (cudaStream_t)stream>>>(*a, qk, v, gates); });
  MSA_LAUNCH_OK("delta_prep_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_delta_prep_split(const msa_lm_delta_args* a, void* qk, void* v, float* gates, void* stream) {
  MSA_OK_OR_RETURN(delta_check(a, "delta_prep_split"));
  MSA_REQUIRE(qk && v && gates && a->dtype == MSA_BF16 && prep_vec_ok(a, qk, v), "delta_prep_split: unsupported sizes or alignment");
  if (a->n_tok == a->n_decode) return MSA_OK;
  return launch_prep_vec<__nv_bfloat16, true>(a, qk, v, gates, (cudaStream_t)stream);
}

extern "C" int msa_lm_delta_conv_store(const msa_lm_delta_args* a, void* stream) {
  MSA_OK_OR_RETURN(delta_check(a, "delta_conv_store"));
  if (a->n_seq == a->n_decode || a->taps == 1) return MSA_OK;
  const DeltaLayout L(*a);
  const dim3 grid((unsigned)((L.chan + 255) / 256), (unsigned)(a->n_seq - a->n_decode));
  MSA_LM_DISPATCH(a->dtype, { delta_conv_store_kernel<T><<<grid, 256, 0, (cudaStream_t)stream>>>(*a); });
  MSA_LAUNCH_OK("delta_conv_store_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_delta_scan(const msa_lm_delta_args* a, const float* qk, const float* v, const float* gates, float* o,
                                 void* stream) {
  MSA_OK_OR_RETURN(delta_check(a, "delta_scan"));
  MSA_REQUIRE(qk && v && gates && o, "delta_scan: null pointer");
  MSA_REQUIRE(a->dim <= 256, "delta_scan: dim must be at most 256");
  if (a->n_seq == a->n_decode) return MSA_OK;
  const dim3 grid((unsigned)((a->vdim + kScCols - 1) / kScCols), (unsigned)a->heads, (unsigned)(a->n_seq - a->n_decode));
  cudaStream_t st = (cudaStream_t)stream;
  if (a->dim <= 32) delta_scan_kernel<4><<<grid, kScThreads, 0, st>>>(*a, qk, v, gates, o);
  else if (a->dim <= 64) delta_scan_kernel<8><<<grid, kScThreads, 0, st>>>(*a, qk, v, gates, o);
  else if (a->dim <= 128) delta_scan_kernel<16><<<grid, kScThreads, 0, st>>>(*a, qk, v, gates, o);
  else delta_scan_kernel<32><<<grid, kScThreads, 0, st>>>(*a, qk, v, gates, o);
  MSA_LAUNCH_OK("delta_scan_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_delta_out(const msa_lm_delta_args* a, const float* o, void* out, int64_t out_stride, void* stream) {
  MSA_OK_OR_RETURN(delta_check(a, "delta_out"));
  MSA_REQUIRE(o && out, "delta_out: null pointer");
  const long long rows = a->n_tok - a->n_decode;
  if (rows == 0) return MSA_OK;
  MSA_REQUIRE(rows * a->heads < (1ll << 31), "delta_out: too many rows");
  const long long blocks = (rows * a->heads + 7) / 8;
  MSA_LM_DISPATCH(a->dtype, {
    const int e4 = 4 * (int)sizeof(T);
    const bool vec = a->vdim % 4 == 0 && a->proj_stride % 4 == 0 && out_stride % 4 == 0 && aligned16(o) && aligned16(a->w_norm) &&
                     reinterpret_cast<uintptr_t>(a->proj) % e4 == 0 && reinterpret_cast<uintptr_t>(out) % e4 == 0 &&
                     (2 * a->kv_heads * a->dim) % 4 == 0;
    delta_out_kernel<T><<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(*a, o, (T*)out, out_stride, rows, vec);
  });
  MSA_LAUNCH_OK("delta_out_kernel");
  return MSA_OK;
}
