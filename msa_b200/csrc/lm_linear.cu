// Recurrences S <- decay S + k v^T per head with the state in fp32: "wkv" (a decay per key channel, read-out before the
// update under a bonus) and "ssd" (one decay per head, keys and queries shared by a group of heads, behind a short
// convolution).  Decode steps, the token-by-token walk for any sizes and types, and what surrounds them; the chunked form
// for prompts is in lm_linear_chunk.cu.
//
// With S the state before a token both read-outs are  o = f (S^T q) + b v:
//     wkv: q = r, f = 1, b = r . (u k);       ssd: q = C, k = B, v = dt x, f = decay, b = C . B.
// So a step reads S once, for the read-out and for the update.
#include "lm_conv.cuh"
#include "lm_linear.cuh"

namespace msa {

// ---- decode -----------------------------------------------------------------------------------------------------------
constexpr int kLinThreads = 256, kLinAhead = 8;

// The pass over one head's state: part[group][dv] = partial sums of S^T q, S <- decay S + k v^T.  A thread owns V columns and
// every groups-th row; the first kLinAhead rows are fetched by `fetch` before q, k and v are known.
template <int V>
struct StatePass {
  float* S;
  int dk, dv, cols, groups, rg, cv;
  bool on, zero;
  float4 x[kLinAhead];
  __device__ __forceinline__ StatePass(float* state, int dk_, int dv_, bool fresh) : S(state), dk(dk_), dv(dv_), zero(fresh) {
    cols = dv / V;
    groups = cols >= kLinThreads ? 1 : kLinThreads / cols;
    rg = threadIdx.x / cols;
    cv = (threadIdx.x - rg * cols) * V;
    on = rg < groups;
  }
  __device__ __forceinline__ float4 get(int d, int c) const {
    if (zero || d >= dk) return make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (V == 4) return load4(S + (long long)d * dv + c);
    else return make_float4(S[(long long)d * dv + c], 0.f, 0.f, 0.f);
  }
  __device__ __forceinline__ void fetch() {
    if (!on) return;
#pragma unroll
    for (int i = 0; i < kLinAhead; ++i) x[i] = get(rg + i * groups, cv);
  }
  // w: decays [dk] (ONE: the same decay w0 for all rows)
  template <bool ONE>
  __device__ __forceinline__ void run(const float* q, const float* k, const float* w, float w0, const float* v, float* part) {
    for (int u = threadIdx.x; u < cols * groups; u += kLinThreads) {       // more than one turn only for dv > kLinThreads * V
      const int g = u / cols, c = (u - g * cols) * V;
      const bool first = u == (int)threadIdx.x;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f), val = acc;
      if constexpr (V == 4) val = load4(v + c); else val.x = v[c];
      for (int d0 = g; d0 < dk; d0 += kLinAhead * groups) {
        if (!(first && d0 == g)) {
#pragma unroll
          for (int i = 0; i < kLinAhead; ++i) x[i] = get(d0 + i * groups, c);
        }
#pragma unroll
        for (int i = 0; i < kLinAhead; ++i) {
          const int d = d0 + i * groups;
          if (d < dk) {
            const float qd = q[d], kd = k[d], wd = ONE ? w0 : w[d];
            acc.x = fmaf(x[i].x, qd, acc.x);
            if constexpr (V == 4) {
              acc.y = fmaf(x[i].y, qd, acc.y); acc.z = fmaf(x[i].z, qd, acc.z); acc.w = fmaf(x[i].w, qd, acc.w);
              store4(S + (long long)d * dv + c, make_float4(fmaf(wd, x[i].x, kd * val.x), fmaf(wd, x[i].y, kd * val.y),
                                                            fmaf(wd, x[i].z, kd * val.z), fmaf(wd, x[i].w, kd * val.w)));
            } else {
              S[(long long)d * dv + c] = fmaf(wd, x[i].x, kd * val.x);
            }
          }
        }
      }
      if constexpr (V == 4) store4(part + g * dv + c, acc); else part[g * dv + c] = acc.x;
    }
  }
  __device__ __forceinline__ float total(const float* part, int c) const {
    float t = 0.f;
    for (int g = 0; g < groups; ++g) t += part[g * dv + c];
    return t;
  }
};
inline int pass_groups(int dv, int v) { return dv / v >= kLinThreads ? 1 : kLinThreads / (dv / v); }

// One block per (head, sequence).
template <typename T, int V>
__global__ void __launch_bounds__(kLinThreads, 4) wkv_decode_kernel(const msa_lm_wkv_args a, T* __restrict__ out, long long out_stride) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float s_part[32];
  const int h = blockIdx.x, b = blockIdx.y, dim = a.dim, pad = (dim + 3) / 4 * 4;
  float *s_r = sm, *s_k = sm + pad, *s_w = sm + 2 * pad, *s_v = sm + 3 * pad, *part = sm + 4 * pad;
  StatePass<V> pass(a.state + ((long long)a.slot[b] * a.heads + h) * dim * dim, dim, dim, a.start[b] == 0);
  pass.fetch();
  const long long row = (long long)b * a.row_stride + h * dim;
  float bonus = 0.f;
  for (int i = threadIdx.x; i < dim; i += kLinThreads) {
    const float r = to_f(reinterpret_cast<const T*>(a.r)[row + i]), k = to_f(reinterpret_cast<const T*>(a.k)[row + i]);
    s_r[i] = r;
    s_k[i] = k;
    s_v[i] = to_f(reinterpret_cast<const T*>(a.v)[row + i]);
    s_w[i] = expf(-expf(a.decay[(long long)b * a.heads * dim + h * dim + i] + a.w0[h * dim + i]));
    bonus = fmaf(r * a.u[h * dim + i], k, bonus);
  }
  bonus = block_sum(bonus, s_part);                        // its barriers publish r, k, v and the decays
  pass.template run<false>(s_r, s_k, s_w, 0.f, s_v, part);
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += kLinThreads) {
    const float o = fmaf(bonus, s_v[i], pass.total(part, i));
    s_r[i] = o;
    ss += o * o;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)dim + a.eps);
  for (int i = threadIdx.x; i < dim; i += kLinThreads)
    out[b * out_stride + h * dim + i] =
        from_f<T>(s_r[i] * inv * a.norm[h * dim + i] * silu_act<T>(to_f(reinterpret_cast<const T*>(a.g)[row + i])));
}

struct SsdLayout {
  int inner, bc, chan;          // heads*vdim, groups*n_state, convolved channels
  __host__ __device__ explicit SsdLayout(const msa_lm_ssd_args& a)
      : inner(a.heads * a.vdim), bc(a.groups * a.n_state), chan(a.heads * a.vdim + 2 * a.groups * a.n_state) {}
};

template <typename T, int V>
__global__ void __launch_bounds__(kLinThreads, 4) ssd_decode_kernel(const msa_lm_ssd_args a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float s_part[32];
  const SsdLayout L(a);
  const int h = blockIdx.x, b = blockIdx.y, ns = a.n_state, vd = a.vdim, per = a.heads / a.groups, gr = h / per;
  const int pn = (ns + 3) / 4 * 4, pv = (vd + 3) / 4 * 4;
  float *s_c = sm, *s_b = sm + pn, *s_x = sm + 2 * pn, *s_v = s_x + pv, *part = s_v + pv;
  const int slot = a.slot[b], pos = a.start[b];
  StatePass<V> pass(a.state + ((long long)slot * a.heads + h) * ns * vd, ns, vd, pos == 0);
  pass.fetch();
  const T* proj = reinterpret_cast<const T*>(a.proj) + (long long)b * a.proj_stride;
  const float dt = softplus_f(to_f(proj[L.inner + L.chan + h]) + a.dt_bias[h]);
  const float decay = expf(-expf(a.a_log[h]) * dt);
  const ConvSource<T> src{reinterpret_cast<const T*>(a.proj) + L.inner, a.proj_stride, reinterpret_cast<T*>(a.conv_state), L.chan, a.taps};
  const bool lead = h % per == 0;                          // the group's first head hands B and C on
  for (int i = threadIdx.x; i < vd + 2 * ns; i += kLinThreads) {
    const int c = i < vd ? h * vd + i : (i < vd + ns ? L.inner + gr * ns + (i - vd) : L.inner + L.bc + gr * ns + (i - vd - ns));
    const float y = silu_act<T>(src.value(a.conv_w, b, 0, pos, slot, c) + a.conv_b[c]);
    const float z = to_f(from_f<T>(y));                    // as the portions see it
    if (i < vd) { s_x[i] = z; s_v[i] = dt * z; }
    else if (i < vd + ns) s_b[i - vd] = z;
    else s_c[i - vd - ns] = z;
    if ((i < vd || lead) && a.taps > 1) {
      T* dst = src.half(slot, pos + 1) + c;
      for (int j = 0; j < a.taps - 1; ++j) {
        const T* x = src.at(b, 0, pos, slot, a.taps - 2 - j, c);
        dst[(long long)j * L.chan] = x ? *x : from_f<T>(0.f);
      }
    }
  }
  __syncthreads();
  float cb = 0.f;
  for (int i = threadIdx.x; i < ns; i += kLinThreads) cb = fmaf(s_c[i], s_b[i], cb);
  cb = block_sum(cb, s_part);
  pass.template run<true>(s_c, s_b, nullptr, decay, s_v, part);
  __syncthreads();
  for (int i = threadIdx.x; i < vd; i += kLinThreads) {
    const float y = fmaf(decay, pass.total(part, i), fmaf(cb, s_v[i], a.d_skip[h] * s_x[i]));
    a.y[(long long)b * L.inner + h * vd + i] = y * silu_act<T>(to_f(proj[h * vd + i]));
  }
}

// ---- portions: convolution, steps ---------------------------------------------------------------------------------------
constexpr int kSpRows = 8;

template <typename T>
__device__ __forceinline__ void ssd_steps(const msa_lm_ssd_args& a, const SsdLayout& L, int row0, int n_here, float* dt) {
  for (int i = threadIdx.x; i < n_here * a.heads; i += blockDim.x) {
    const int r = i / a.heads, h = i - r * a.heads;
    const T raw = reinterpret_cast<const T*>(a.proj)[((long long)a.n_decode + row0 + r) * a.proj_stride + L.inner + L.chan + h];
    dt[(long long)(row0 + r) * a.heads + h] = softplus_f(to_f(raw) + a.dt_bias[h]);
  }
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(256) ssd_prep_vec_kernel(const msa_lm_ssd_args a, T* __restrict__ xbc, float* __restrict__ dt) {
  const SsdLayout L(a);
  const int row0 = blockIdx.x * kSpRows, n_here = min(kSpRows, a.n_tok - a.n_decode - row0);
  if (blockIdx.y == 0) ssd_steps<T>(a, L, row0, n_here, dt);
  const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
  if (c >= L.chan) return;
  const ConvSource<T> src{reinterpret_cast<const T*>(a.proj) + L.inner, a.proj_stride, reinterpret_cast<T*>(a.conv_state), L.chan, TAPS};
  ConvWindow<T, TAPS> win;
  float4 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = load4(a.conv_w + (long long)j * L.chan + c);
  const float4 bias = load4(a.conv_b + c);
#pragma unroll
  for (int r = 0; r < kSpRows; ++r) {
    if (r >= n_here) break;
    const long long n = (long long)a.n_decode + row0 + r;
    const int s = a.tok_seq[n], t = (int)n - a.cu[s];
    win.move(src, n, t, a.start[s], a.slot[s], c, r == 0 || t == 0);
    const float4 y = win.value(w);
    store4(xbc + (long long)(row0 + r) * L.chan + c,
           make_float4(silu_act<T>(y.x + bias.x), silu_act<T>(y.y + bias.y), silu_act<T>(y.z + bias.z), silu_act<T>(y.w + bias.w)));
  }
}
template <typename T>
__global__ void __launch_bounds__(256) ssd_prep_kernel(const msa_lm_ssd_args a, T* __restrict__ xbc, float* __restrict__ dt) {
  const SsdLayout L(a);
  const int row = blockIdx.x;
  ssd_steps<T>(a, L, row, 1, dt);
  const ConvSource<T> src{reinterpret_cast<const T*>(a.proj) + L.inner, a.proj_stride, reinterpret_cast<T*>(a.conv_state), L.chan, a.taps};
  const long long n = (long long)a.n_decode + row;
  const int s = a.tok_seq[n], t = (int)n - a.cu[s];
  for (int c = threadIdx.x; c < L.chan; c += 256)
    xbc[(long long)row * L.chan + c] = from_f<T>(silu_act<T>(src.value(a.conv_w, n, t, a.start[s], a.slot[s], c) + a.conv_b[c]));
}

// ---- portions: token by token -------------------------------------------------------------------------------------------
// 8 lanes share a state column (R rows each, in registers); a warp covers 4 columns, a block of 4 warps 16.  Tokens are
// staged in shared memory 16 at a time.
constexpr int kLsTok = 16, kLsCols = 16, kLsThreads = 128;
template <int R, bool WKV> constexpr size_t scan_smem() {
  return (size_t)4 * kLsTok * ((WKV ? 3 : 2) * 8 * R + 2 * kLsCols + 3);
}

template <typename T, int R>
struct WkvTokens {
  msa_lm_wkv_args a;
  float* o;
  static constexpr bool kChannelDecay = true;
  __device__ int dk() const { return a.dim; }
  __device__ int dv() const { return a.dim; }
  __device__ long long at(long long n, int h, int d) const { return n * a.row_stride + h * a.dim + d; }
  __device__ float q(long long n, int h, int d) const { return to_f(reinterpret_cast<const T*>(a.r)[at(n, h, d)]); }
  __device__ float k(long long n, int h, int d) const { return to_f(reinterpret_cast<const T*>(a.k)[at(n, h, d)]); }
  __device__ float v(long long n, int h, int c) const { return to_f(reinterpret_cast<const T*>(a.v)[at(n, h, c)]); }
  __device__ float w(long long n, int h, int d) const { return expf(-expf(a.decay[n * a.heads * a.dim + h * a.dim + d] + a.w0[h * a.dim + d])); }
  __device__ float own(float q, float k, int h, int d) const { return q * a.u[h * a.dim + d] * k; }     // the term of b
  __device__ float decay(long long, int) const { return 1.f; }
  __device__ float step(long long, int) const { return 1.f; }
  __device__ void put(long long n, int h, int c, float y, float) const { o[(n - a.n_decode) * a.heads * a.dim + h * a.dim + c] = y; }
};
template <typename T, int R>
struct SsdTokens {
  msa_lm_ssd_args a;
  const T* xbc;
  const float* dt;
  static constexpr bool kChannelDecay = false;
  __device__ int dk() const { return a.n_state; }
  __device__ int dv() const { return a.vdim; }
  __device__ const T* row(long long n) const { return xbc + (n - a.n_decode) * SsdLayout(a).chan; }
  __device__ float k(long long n, int h, int d) const { return to_f(row(n)[SsdLayout(a).inner + h / (a.heads / a.groups) * a.n_state + d]); }
  __device__ float q(long long n, int h, int d) const {
    const SsdLayout L(a);
    return to_f(row(n)[L.inner + L.bc + h / (a.heads / a.groups) * a.n_state + d]);
  }
  __device__ float v(long long n, int h, int c) const { return to_f(row(n)[h * a.vdim + c]); }
  __device__ float w(long long, int, int) const { return 1.f; }
  __device__ float own(float q, float k, int, int) const { return q * k; }
  __device__ float step(long long n, int h) const { return dt[(n - a.n_decode) * a.heads + h]; }
  __device__ float decay(long long n, int h) const { return expf(-expf(a.a_log[h]) * step(n, h)); }
  __device__ void put(long long n, int h, int c, float y, float x) const {     // x: the value before its step
    const float z = to_f(reinterpret_cast<const T*>(a.proj)[n * a.proj_stride + h * a.vdim + c]);
    a.y[n * a.heads * a.vdim + h * a.vdim + c] = (y + a.d_skip[h] * x) * silu_act<T>(z);
  }
};

template <int R, typename Tokens>
__global__ void __launch_bounds__(kLsThreads) linear_scan_kernel(const Tokens tk) {
  constexpr int D = 8 * R;
  constexpr bool CD = Tokens::kChannelDecay;
  // dimension d = part * R + r of a token lies at (r / 4) * 32 + part * 4 + r % 4: the eight lanes of a column read
  // 128 consecutive bytes per vector
  extern __shared__ __align__(16) float sm[];
  float* s_q = sm;                               // [tok][D]
  float* s_k = s_q + kLsTok * D;
  float* s_w = s_k + kLsTok * D;                 // channel decays
  float* s_v = s_w + (CD ? kLsTok * D : 0);      // [tok][cols]
  float* s_o = s_v + kLsTok * kLsCols;
  float *s_f = s_o + kLsTok * kLsCols, *s_s = s_f + kLsTok, *s_b = s_s + kLsTok;
  const auto& a = tk.a;
  const int s = a.n_decode + blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kLsCols, dk = tk.dk(), dv = tk.dv();
  const int len = a.cu[s + 1] - a.cu[s];
  const long long n0 = a.cu[s];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int part = lane & 7, cl = warp * 4 + (lane >> 3), col = c0 + cl;
  float* S = a.state + (((long long)a.slot[s] * a.heads + h) * dk) * dv;
  float st[R];
  const bool fresh = a.start[s] == 0;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = part * R + r;
    st[r] = (!fresh && d < dk && col < dv) ? S[(long long)d * dv + col] : 0.f;
  }
  for (int t0 = 0; t0 < len; t0 += kLsTok) {
    const int nt = min(kLsTok, len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * D; i += kLsThreads) {
      const int t = i / D, d = i % D, at = t * D + (d % R / 4) * 32 + d / R * 4 + d % 4;
      const bool on = d < dk;
      s_q[at] = on ? tk.q(n0 + t0 + t, h, d) : 0.f;
      s_k[at] = on ? tk.k(n0 + t0 + t, h, d) : 0.f;
      if constexpr (CD) s_w[at] = on ? tk.w(n0 + t0 + t, h, d) : 0.f;
    }
    for (int i = threadIdx.x; i < nt * kLsCols; i += kLsThreads) {
      const int t = i / kLsCols, c = i % kLsCols;
      s_v[i] = c0 + c < dv ? tk.v(n0 + t0 + t, h, c0 + c) : 0.f;
    }
    if (threadIdx.x < nt) {
      s_f[threadIdx.x] = tk.decay(n0 + t0 + threadIdx.x, h);
      s_s[threadIdx.x] = tk.step(n0 + t0 + threadIdx.x, h);
    }
    __syncthreads();
    for (int t = warp; t < nt; t += kLsThreads / 32) {
      float d = 0.f;
      for (int i = lane; i < D; i += 32) {
        const int e = i % 32, dd = (e / 4) * R + (i / 32) * 4 + e % 4;
        if (dd < dk) d += tk.own(s_q[t * D + i], s_k[t * D + i], h, dd);
      }
      d = warp_sum_f(d);
      if (lane == 0) s_b[t] = d;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float f = s_f[t], v = s_v[t * kLsCols + cl] * s_s[t];
      float y = 0.f, y2 = 0.f;
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const float4 kv = load4(s_k + t * D + r * 8 + part * 4), qv = load4(s_q + t * D + r * 8 + part * 4);
        y = fmaf(st[r], qv.x, y); y2 = fmaf(st[r + 1], qv.y, y2); y = fmaf(st[r + 2], qv.z, y); y2 = fmaf(st[r + 3], qv.w, y2);
        if constexpr (CD) {
          const float4 w = load4(s_w + t * D + r * 8 + part * 4);
          st[r] = fmaf(w.x, st[r], kv.x * v); st[r + 1] = fmaf(w.y, st[r + 1], kv.y * v);
          st[r + 2] = fmaf(w.z, st[r + 2], kv.z * v); st[r + 3] = fmaf(w.w, st[r + 3], kv.w * v);
        } else {
          st[r] = fmaf(f, st[r], kv.x * v); st[r + 1] = fmaf(f, st[r + 1], kv.y * v);
          st[r + 2] = fmaf(f, st[r + 2], kv.z * v); st[r + 3] = fmaf(f, st[r + 3], kv.w * v);
        }
      }
      y += y2;
#pragma unroll
      for (int w = 1; w < 8; w <<= 1) y += __shfl_xor_sync(0xffffffffu, y, w);
      if (part == 0) s_o[t * kLsCols + cl] = fmaf(f, y, s_b[t] * v);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kLsCols; i += kLsThreads) {
      const int t = i / kLsCols, c = i % kLsCols;
      if (c0 + c < dv) tk.put(n0 + t0 + t, h, c0 + c, s_o[i], s_v[i]);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = part * R + r;
    if (d < dk && col < dv) S[(long long)d * dv + col] = st[r];
  }
}

template <template <typename, int> class Tokens, typename T, int R, typename... Args>
int launch_scan_r(dim3 grid, cudaStream_t st, Args... args) {
  using Tk = Tokens<T, R>;
  constexpr size_t smem = scan_smem<R, Tk::kChannelDecay>();
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(linear_scan_kernel<R, Tk>, smem, configured));
  linear_scan_kernel<R, Tk><<<grid, kLsThreads, smem, st>>>(Tk{args...});
  MSA_LAUNCH_OK("linear_scan_kernel");
  return MSA_OK;
}
template <template <typename, int> class Tokens, typename T, typename... Args>
int launch_scan(int dk, int dv, int heads, int seqs, cudaStream_t st, Args... args) {
  const dim3 grid((unsigned)((dv + kLsCols - 1) / kLsCols), (unsigned)heads, (unsigned)seqs);
  if (dk <= 32) return launch_scan_r<Tokens, T, 4>(grid, st, args...);
  if (dk <= 64) return launch_scan_r<Tokens, T, 8>(grid, st, args...);
  if (dk <= 128) return launch_scan_r<Tokens, T, 16>(grid, st, args...);
  return launch_scan_r<Tokens, T, 32>(grid, st, args...);
}

// out = o / rms(o) * w * silu(g); one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) wkv_out_kernel(const msa_lm_wkv_args a, const float* __restrict__ o, T* __restrict__ out,
                                                      long long out_stride, long long items) {
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int lane = threadIdx.x & 31, h = (int)(item % a.heads);
  const long long row = item / a.heads;
  const float* src = o + row * a.heads * a.dim + h * a.dim;
  const T* g = reinterpret_cast<const T*>(a.g) + (a.n_decode + row) * a.row_stride + h * a.dim;
  float ss = 0.f;
  for (int i = lane; i < a.dim; i += 32) ss += src[i] * src[i];
  const float inv = 1.f / sqrtf(warp_sum_f(ss) / (float)a.dim + a.eps);
  for (int i = lane; i < a.dim; i += 32)
    out[row * out_stride + h * a.dim + i] = from_f<T>(src[i] * inv * a.norm[h * a.dim + i] * silu_act<T>(to_f(g[i])));
}

// One block per (row, part).
template <typename T, int V>
__global__ void __launch_bounds__(256) part_norm_kernel(const float* __restrict__ x, long long x_stride, const float* __restrict__ w,
                                                        int size, float eps, T* __restrict__ out, long long out_stride) {
  __shared__ float s_part[32];
  const long long row = blockIdx.x;
  const int c0 = blockIdx.y * size;
  const float* src = x + row * x_stride + c0;
  T* dst = out + row * out_stride + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < size; i += blockDim.x * V) {
    if constexpr (V == 4) { const float4 v = load4(src + i); ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
    else ss += src[i] * src[i];
  }
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)size + eps);
  for (int i = threadIdx.x * V; i < size; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 v = load4(src + i), g = load4(w + c0 + i);
      store4(dst + i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
    } else {
      dst[i] = from_f<T>(src[i] * inv * w[c0 + i]);
    }
  }
}

int wkv_check(const msa_lm_wkv_args* a, const char* what) {
  MSA_REQUIRE(a, "%s: null arguments", what);
  MSA_REQUIRE(dtype_ok(a->dtype) && a->r && a->k && a->v && a->g && a->decay && a->w0 && a->u && a->norm && a->state && a->tok_seq &&
                  a->slot && a->start && a->cu, "%s: null pointer or bad dtype", what);
  MSA_REQUIRE(a->heads > 0 && a->dim > 0 && a->row_stride >= (int64_t)a->heads * a->dim, "%s: bad sizes", what);
  MSA_REQUIRE(a->n_decode >= 0 && a->n_decode <= a->n_seq && a->n_tok >= a->n_decode, "%s: bad counts", what);
  return MSA_OK;
}
int ssd_check(const msa_lm_ssd_args* a, const char* what) {
  MSA_REQUIRE(a, "%s: null arguments", what);
  MSA_REQUIRE(dtype_ok(a->dtype) && a->proj && a->conv_w && a->conv_b && a->dt_bias && a->a_log && a->d_skip && a->state && a->tok_seq &&
                  a->slot && a->start && a->cu && a->y, "%s: null pointer or bad dtype", what);
  MSA_REQUIRE(a->heads > 0 && a->groups > 0 && a->heads % a->groups == 0 && a->vdim > 0 && a->n_state > 0, "%s: bad sizes", what);
  MSA_REQUIRE(a->taps >= 1 && (a->taps == 1 || a->conv_state), "%s: convolution state missing", what);
  MSA_REQUIRE(a->n_decode >= 0 && a->n_decode <= a->n_seq && a->n_tok >= a->n_decode, "%s: bad counts", what);
  return MSA_OK;
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_wkv_decode(const msa_lm_wkv_args* a, void* out, int64_t out_stride, void* stream) {
  MSA_OK_OR_RETURN(wkv_check(a, "wkv_decode"));
  MSA_REQUIRE(out, "wkv_decode: null output");
  if (a->n_decode == 0) return MSA_OK;
  const int v = a->dim % 4 == 0 && aligned16(a->state) ? 4 : 1, pad = (a->dim + 3) / 4 * 4;
  const size_t smem = (size_t)4 * (4 * pad + pass_groups(a->dim, v) * a->dim);
  MSA_REQUIRE(smem <= 48 * 1024, "wkv_decode: head size %d is too large", a->dim);
  const dim3 grid((unsigned)a->heads, (unsigned)a->n_decode);
  MSA_LM_DISPATCH(a->dtype, {
    if (v == 4) wkv_decode_kernel<T, 4><<<grid, kLinThreads, smem, (cudaStream_t)stream>>>(*a, (T*)out, out_stride);
    else wkv_decode_kernel<T, 1><<<grid, kLinThreads, smem, (cudaStream_t)stream>>>(*a, (T*)out, out_stride);
  });
  MSA_LAUNCH_OK("wkv_decode_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_wkv_scan(const msa_lm_wkv_args* a, float* o, void* out, int64_t out_stride, void* stream) {
  MSA_OK_OR_RETURN(wkv_check(a, "wkv_scan"));
  MSA_REQUIRE(out && o, "wkv_scan: null output");
  MSA_REQUIRE(a->dim <= 256, "wkv_scan: dim must be at most 256");
  if (a->n_seq == a->n_decode) return MSA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const long long items = (long long)(a->n_tok - a->n_decode) * a->heads;
  MSA_LM_DISPATCH(a->dtype, {
    MSA_OK_OR_RETURN((launch_scan<WkvTokens, T>(a->dim, a->dim, a->heads, a->n_seq - a->n_decode, st, *a, o)));
    wkv_out_kernel<T><<<(unsigned)((items + 7) / 8), 256, 0, st>>>(*a, o, (T*)out, out_stride, items);
  });
  MSA_LAUNCH_OK("wkv_out_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_ssd_decode(const msa_lm_ssd_args* a, void* stream) {
  MSA_OK_OR_RETURN(ssd_check(a, "ssd_decode"));
  if (a->n_decode == 0) return MSA_OK;
  const int v = a->vdim % 4 == 0 && aligned16(a->state) ? 4 : 1;
  const size_t smem = (size_t)4 * (2 * ((a->n_state + 3) / 4 * 4) + 2 * ((a->vdim + 3) / 4 * 4) + pass_groups(a->vdim, v) * a->vdim);
  MSA_REQUIRE(smem <= 48 * 1024, "ssd_decode: sizes (%d, %d) are too large", a->n_state, a->vdim);
  const dim3 grid((unsigned)a->heads, (unsigned)a->n_decode);
  MSA_LM_DISPATCH(a->dtype, {
    if (v == 4) ssd_decode_kernel<T, 4><<<grid, kLinThreads, smem, (cudaStream_t)stream>>>(*a);
    else ssd_decode_kernel<T, 1><<<grid, kLinThreads, smem, (cudaStream_t)stream>>>(*a);
  });
  MSA_LAUNCH_OK("ssd_decode_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_ssd_prep(const msa_lm_ssd_args* a, void* xbc, float* dt, void* stream) {
  MSA_OK_OR_RETURN(ssd_check(a, "ssd_prep"));
  MSA_REQUIRE(xbc && dt, "ssd_prep: null output");
  const int rows = a->n_tok - a->n_decode;
  if (rows == 0) return MSA_OK;
  const SsdLayout L(*a);
  const int e4 = 4 * (int)dtype_size(a->dtype);
  auto ok4 = [&](const void* q) { return q == nullptr || reinterpret_cast<uintptr_t>(q) % e4 == 0; };
  cudaStream_t st = (cudaStream_t)stream;
  if (a->taps <= 4 && L.inner % 4 == 0 && L.chan % 4 == 0 && a->proj_stride % 4 == 0 && ok4(a->proj) && ok4(a->conv_state) && ok4(xbc) &&
      aligned16(a->conv_w) && aligned16(a->conv_b)) {
    const dim3 grid((unsigned)((rows + kSpRows - 1) / kSpRows), (unsigned)((L.chan + 1023) / 1024));
    MSA_LM_DISPATCH(a->dtype, {
      switch (a->taps) {
        case 1: ssd_prep_vec_kernel<T, 1><<<grid, 256, 0, st>>>(*a, (T*)xbc, dt); break;
        case 2: ssd_prep_vec_kernel<T, 2><<<grid, 256, 0, st>>>(*a, (T*)xbc, dt); break;
        case 3: ssd_prep_vec_kernel<T, 3><<<grid, 256, 0, st>>>(*a, (T*)xbc, dt); break;
        default: ssd_prep_vec_kernel<T, 4><<<grid, 256, 0, st>>>(*a, (T*)xbc, dt);
      }
    });
    MSA_LAUNCH_OK("ssd_prep_vec_kernel");
    return MSA_OK;
  }
  MSA_LM_DISPATCH(a->dtype, { ssd_prep_kernel<T><<<rows, 256, 0, st>>>(*a, (T*)xbc, dt); });
  MSA_LAUNCH_OK("ssd_prep_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_ssd_scan(const msa_lm_ssd_args* a, const void* xbc, const float* dt, void* stream) {
  MSA_OK_OR_RETURN(ssd_check(a, "ssd_scan"));
  MSA_REQUIRE(xbc && dt, "ssd_scan: null pointer");
  MSA_REQUIRE(a->n_state <= 256, "ssd_scan: n_state must be at most 256");
  if (a->n_seq == a->n_decode) return MSA_OK;
  MSA_LM_DISPATCH(a->dtype, {
    return (launch_scan<SsdTokens, T>(a->n_state, a->vdim, a->heads, a->n_seq - a->n_decode, (cudaStream_t)stream, *a, (const T*)xbc, dt));
  });
}

extern "C" int msa_lm_part_norm(const float* x, int64_t x_stride, const float* w, int32_t n_rows, int32_t width, int32_t parts, float eps,
                                void* out, int64_t out_stride, int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && x && w && out && n_rows >= 0 && width > 0 && parts > 0 && width % parts == 0, "part_norm: bad arguments");
  if (n_rows == 0) return MSA_OK;
  MSA_REQUIRE(parts <= 65535, "part_norm: too many parts");
  const int size = width / parts;
  const bool v4 = size % 4 == 0 && x_stride % 4 == 0 && out_stride % 4 == 0 && aligned16(x) && aligned16(w) &&
                  reinterpret_cast<uintptr_t>(out) % (4 * dtype_size(dtype)) == 0;
  const int per = v4 ? size / 4 : size, threads = per >= 256 ? 256 : (per + 31) / 32 * 32;
  const dim3 grid((unsigned)n_rows, (unsigned)parts);
  MSA_LM_DISPATCH(dtype, {
    if (v4) part_norm_kernel<T, 4><<<grid, threads, 0, (cudaStream_t)stream>>>(x, x_stride, w, size, eps, (T*)out, out_stride);
    else part_norm_kernel<T, 1><<<grid, threads, 0, (cudaStream_t)stream>>>(x, x_stride, w, size, eps, (T*)out, out_stride);
  });
  MSA_LAUNCH_OK("part_norm_kernel");
  return MSA_OK;
}
