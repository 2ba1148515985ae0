// Windowed attention over a shared low-rank latent: what happens between the projections and the attention proper
// (norm of the latent, rotation, ring and context upkeep), and the general attention kernel for any sizes and dtypes.
//
// Per sequence slot a layer keeps a ring of the last `ring_rows` rows [latent | rotated shared key part]; position p is
// row p % ring_rows, and ring_rows >= window, so a row is overwritten only when no later query sees it.  A step that
// brings several tokens of a sequence works on a packed context instead: the ring rows its first token still sees, then
// its own rows; the ring takes over the last of them afterwards.
#include "lm_common.cuh"

namespace msa {

struct LatentPrepParams {
  void* proj; long long proj_stride;
  const float* w_norm; float eps; const float* inv_freq;
  int heads, dim, rot, rank;
  const int32_t *pos, *tok_seq, *slot, *start, *cu, *ctx_off, *old_off;
  int n_tok, n_seq, n_decode, window;
  void* ring; long long ring_rows; void* ctx;
};

// Blocks 0 .. n_tok-1: one token each; the blocks after them: one old ring row each.
template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepParams p) {
  __shared__ float s_part[32];
  extern __shared__ float2 s_turn[];       // cosine and sine of the token's angles
  const int width = p.rank + p.rot;
  if ((int)blockIdx.x >= p.n_tok) {
    const int o = (int)blockIdx.x - p.n_tok;
    const int ps = owner_of(p.old_off, p.n_seq - p.n_decode, o), s = ps + p.n_decode;
    const int k = o - p.old_off[ps], start = p.start[s];
    const int first = start - min(start, p.window - 1);
    const T* src = reinterpret_cast<const T*>(p.ring) + ((long long)p.slot[s] * p.ring_rows + (first + k) % p.ring_rows) * width;
    T* dst = reinterpret_cast<T*>(p.ctx) + (long long)(p.ctx_off[ps] + k) * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = src[i];
    return;
  }
  const int n = blockIdx.x, s = p.tok_seq[n], pos = p.pos[n];
  T* row = reinterpret_cast<T*>(p.proj) + (long long)n * p.proj_stride;
  const int hd = p.dim + p.rot, half = p.rot / 2;
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * p.inv_freq[j], &sn, &cs);
    s_turn[j] = make_float2(cs, sn);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.heads * half; i += blockDim.x) {
    const int h = i / half, j = i - h * half;
    T* q = row + h * hd + p.dim + 2 * j;
    const float2 cs = s_turn[j];
    const float u = to_f(q[0]), v = to_f(q[1]);
    q[0] = from_f<T>(u * cs.x - v * cs.y);
    q[1] = from_f<T>(v * cs.x + u * cs.y);
  }
  T* lat = row + p.heads * hd;
  T* dst;
  if (n < p.n_decode) {
    dst = reinterpret_cast<T*>(p.ring) + ((long long)p.slot[s] * p.ring_rows + pos % p.ring_rows) * width;
  } else {
    const int start = p.start[s];
    dst = reinterpret_cast<T*>(p.ctx) + (long long)(p.ctx_off[s - p.n_decode] + min(start, p.window - 1) + (n - p.cu[s])) * width;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.rank; i += blockDim.x) { const float v = to_f(lat[i]); ss += v * v; }
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)p.rank + p.eps);
  for (int i = threadIdx.x; i < p.rank; i += blockDim.x) dst[i] = from_f<T>(to_f(lat[i]) * inv * p.w_norm[i]);
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    const float2 cs = s_turn[j];
    const float u = to_f(lat[p.rank + 2 * j]), v = to_f(lat[p.rank + 2 * j + 1]);
    dst[p.rank + 2 * j] = from_f<T>(u * cs.x - v * cs.y);
    dst[p.rank + 2 * j + 1] = from_f<T>(v * cs.x + u * cs.y);
  }
}

// The same with four elements per access (sizes and strides multiples of 4, rank <= 512): the latent's row is in
// registers before the token's angles are computed, and the heads' rotated parts are turned two pairs at a time.
template <typename T>
__global__ void __launch_bounds__(128) latent_prep_vec_kernel(const LatentPrepParams p) {
  __shared__ float s_part[32];
  extern __shared__ float2 s_turn[];
  const int width = p.rank + p.rot, tid = threadIdx.x;
  if ((int)blockIdx.x >= p.n_tok) {
    const int o = (int)blockIdx.x - p.n_tok;
    const int ps = owner_of(p.old_off, p.n_seq - p.n_decode, o), s = ps + p.n_decode;
    const int k = o - p.old_off[ps], start = p.start[s];
    const int first = start - min(start, p.window - 1);
    const T* src = reinterpret_cast<const T*>(p.ring) + ((long long)p.slot[s] * p.ring_rows + (first + k) % (int)p.ring_rows) * width;
    T* dst = reinterpret_cast<T*>(p.ctx) + (long long)(p.ctx_off[ps] + k) * width;
    for (int i = tid * 4; i < width; i += 512) store4(dst + i, load4(src + i));
    return;
  }
  const int n = blockIdx.x, s = p.tok_seq[n], pos = p.pos[n], half = p.rot / 2, hd = p.dim + p.rot;
  T* row = reinterpret_cast<T*>(p.proj) + (long long)n * p.proj_stride;
  const T* lat = row + p.heads * hd;
  const bool on = tid * 4 < p.rank, turns = tid * 4 < p.rot;
  const float4 c = on ? load4(lat + tid * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 w = on ? load4(p.w_norm + tid * 4) : c;
  float4 kr = turns ? load4(lat + p.rank + tid * 4) : c;
  const int per_head = p.rot / 4, quads = p.heads * per_head;
  constexpr int kAhead = 4;
  float4 q[kAhead];
  int at[kAhead], pair[kAhead];
  const float inv_ph = 1.f / (float)max(per_head, 1);      // (i + 0.5) / per_head rounds down to the head for every i that fits
#pragma unroll
  for (int u = 0; u < kAhead; ++u) {
    const int i = tid + u * 128, h = (int)(((float)i + 0.5f) * inv_ph), j = i - h * per_head;
    at[u] = h * hd + p.dim + j * 4;
    pair[u] = 2 * j;
    if (i < quads) q[u] = load4(row + at[u]);
  }
  T* dst;
  if (n < p.n_decode) {
    dst = reinterpret_cast<T*>(p.ring) + ((long long)p.slot[s] * p.ring_rows + pos % (int)p.ring_rows) * width;
  } else {
    const int start = p.start[s];
    dst = reinterpret_cast<T*>(p.ctx) + (long long)(p.ctx_off[s - p.n_decode] + min(start, p.window - 1) + (n - p.cu[s])) * width;
  }
  for (int j = tid; j < half; j += 128) {
    float sn, cs;
    sincosf((float)pos * p.inv_freq[j], &sn, &cs);
    s_turn[j] = make_float2(cs, sn);
  }
  const float inv = 1.f / sqrtf(block_sum(c.x * c.x + c.y * c.y + c.z * c.z + c.w * c.w, s_part) / (float)p.rank + p.eps);
  if (on) store4(dst + tid * 4, make_float4(c.x * inv * w.x, c.y * inv * w.y, c.z * inv * w.z, c.w * inv * w.w));
  auto turn = [&](float4 x, int pair) {
    const float2 a = s_turn[pair], b = s_turn[pair + 1];
    return make_float4(x.x * a.x - x.y * a.y, x.y * a.x + x.x * a.y, x.z * b.x - x.w * b.y, x.w * b.x + x.z * b.y);
  };
  for (int i = tid * 4; i < p.rot; i += 512) {
    if (i != tid * 4) kr = load4(lat + p.rank + i);
    store4(dst + p.rank + i, turn(kr, i / 2));
  }
#pragma unroll
  for (int u = 0; u < kAhead; ++u) {
    const int i = tid + u * 128;
    if (i < quads) store4(row + at[u], turn(q[u], pair[u]));
  }
  for (int i = tid + kAhead * 128; i < quads; i += 128) {
    const int h = i / per_head, j = i - h * per_head;
    T* x = row + h * hd + p.dim + j * 4;
    store4(x, turn(load4(x), 2 * j));
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
ring_store_kernel(const T* __restrict__ ctx, int width, const int32_t* slot, const int32_t* start, const int32_t* cu,
                  const int32_t* ctx_off, int n_decode, int window, T* ring, long long ring_rows) {
  const int ps = blockIdx.y, s = ps + n_decode;
  const int len = cu[s + 1] - cu[s], p0 = start[s];
  const int keep = (int)min((long long)len, ring_rows);
  for (int k = blockIdx.x; k < keep; k += gridDim.x) {
    const int t = len - keep + k;
    const T* src = ctx + (long long)(ctx_off[ps] + min(p0, window - 1) + t) * width;
    T* dst = ring + ((long long)slot[s] * ring_rows + (p0 + t) % ring_rows) * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = src[i];
  }
}

// General attention: 8 rows per block, a row = (token, head).  A block's rows run over the heads that share a key / value
// head first.  A tile of up to 32 keys and values is staged in shared
// memory as fp32; lane = key for the scores, lane = value column for the output.
constexpr int kGaRows = 8, kGaThreads = 128;

__global__ void __launch_bounds__(kGaThreads) window_attn_kernel(const msa_lm_attn_args a, int heads_per_block, int tile) {
  extern __shared__ float sm[];
  const int dq = a.da + a.db, kstr = dq + 1;
  float* s_q = sm;                         // [8][dq]
  float* s_o = s_q + kGaRows * dq;         // [8][dv]
  float* s_k = s_o + kGaRows * a.dv;       // [tile][dq + 1]
  float* s_v = s_k + tile * kstr;          // [tile][dv]
  const int s = a.seq0 + blockIdx.z, hg = heads_per_block, h0 = blockIdx.y * hg;
  const int len = a.cu[s + 1] - a.cu[s], start = a.start[s];
  const long long n_rows = (long long)len * hg;
  const long long r0 = (long long)blockIdx.x * kGaRows;
  if (r0 >= n_rows) return;
  const int nr = (int)min((long long)kGaRows, n_rows - r0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < nr * dq; i += kGaThreads) {
    const int r = i / dq, c = i % dq;
    const long long rr = r0 + r;
    const long long tok = a.cu[s] + rr / hg;
    const int h = h0 + (int)(rr % hg);
    s_q[r * dq + c] = c < a.da ? load_any(a.qa, a.qa_dtype, (tok - a.cu[a.seq0]) * a.qa_row + h * a.qa_head + c)
                               : load_any(a.qb, a.dtype, (tok - a.cu[a.seq0]) * a.qb_row + h * a.qb_head + (c - a.da));
  }
  for (int i = threadIdx.x; i < kGaRows * a.dv; i += kGaThreads) s_o[i] = 0.f;
  const int t_lo = (int)(r0 / hg), t_hi = (int)((r0 + nr - 1) / hg);
  const int p_lo = start + t_lo, p_hi = start + t_hi;
  const int j0 = max(0, p_lo - a.window + 1);
  const int first = start - min(start, a.window - 1);
  const float m0 = a.sink ? 0.f : -INFINITY, l0 = a.sink ? 1.f : 0.f;     // the sink: one entry with score 0 and no value
  float m[2] = {m0, m0}, l[2] = {l0, l0};
  for (int jt = j0; jt <= p_hi; jt += tile) {
    const int nk = min(tile, p_hi - jt + 1);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * (dq + a.dv); i += kGaThreads) {
      const int k = i / (dq + a.dv), c = i % (dq + a.dv), j = jt + k;
      const long long row = a.ring_rows > 0 ? (long long)a.slot[s] * a.ring_rows + j % a.ring_rows
                                            : (long long)a.ctx_off[s - a.seq0] + (j - first);
      if (c < a.da) s_k[k * kstr + c] = load_any(a.ka, a.dtype, row * a.ka_row + blockIdx.y * a.ka_head + c);
      else if (c < dq) s_k[k * kstr + c] = load_any(a.kb, a.dtype, row * a.kb_row + blockIdx.y * a.kb_head + (c - a.da));
      else s_v[k * a.dv + (c - dq)] = load_any(a.v, a.dtype, row * a.v_row + blockIdx.y * a.v_head + (c - dq));
    }
    __syncthreads();
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int r = warp * 2 + q;
      if (r >= nr) continue;
      const int pos = start + (int)((r0 + r) / hg), j = jt + lane;
      float sc = -INFINITY;
      if (lane < nk && j <= pos && pos - j < a.window) {
        float acc = 0.f;
        for (int c = 0; c < dq; ++c) acc = fmaf(s_q[r * dq + c], s_k[lane * kstr + c], acc);
        sc = acc * a.scale;
      }
      const float mx = fmaxf(m[q], warp_max_f(sc));
      if (mx == -INFINITY) continue;
      const float w = expf(sc - mx), corr = expf(m[q] - mx);
      l[q] = l[q] * corr + warp_sum_f(w);
      m[q] = mx;
      for (int c0 = 0; c0 < a.dv; c0 += 32) {
        const int c = c0 + lane;
        float acc = c < a.dv ? s_o[r * a.dv + c] * corr : 0.f;
        for (int k = 0; k < nk; ++k) {
          const float wk = __shfl_sync(0xffffffffu, w, k);
          if (c < a.dv) acc = fmaf(wk, s_v[k * a.dv + c], acc);
        }
        if (c < a.dv) s_o[r * a.dv + c] = acc;
      }
    }
  }
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const int r = warp * 2 + q;
    if (r >= nr) continue;
    const long long rr = r0 + r;
    const long long tok = a.cu[s] - a.cu[a.seq0] + rr / hg;
    const int h = h0 + (int)(rr % hg);
    const float inv = (a.gate ? sigmoid_f(load_any(a.gate, a.dtype, tok * a.gate_row + h)) : 1.f) / l[q];
    for (int c = lane; c < a.dv; c += 32)
      store_any(a.out, a.out_dtype, tok * a.out_row + h * a.out_head + c, s_o[r * a.dv + c] * inv);
  }
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_latent_prep(void* proj, int64_t proj_stride, const float* w_norm, float eps, const float* inv_freq,
                                  int32_t heads, int32_t dim, int32_t rot, int32_t rank, const int32_t* pos,
                                  const int32_t* tok_seq, const int32_t* slot, const int32_t* start, const int32_t* cu,
                                  const int32_t* ctx_off, const int32_t* old_off, int32_t n_tok, int32_t n_seq,
                                  int32_t n_decode, int32_t n_old, int32_t window, void* ring, int64_t ring_rows, void* ctx,
                                  int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && proj && w_norm && pos && tok_seq && slot && start && cu && ring, "latent_prep: null pointer");
  MSA_REQUIRE(heads > 0 && dim >= 0 && rot >= 0 && rot <= 4096 && rot % 2 == 0 && rank > 0 && window > 0, "latent_prep: bad sizes");
  MSA_REQUIRE(rot == 0 || inv_freq, "latent_prep: inv_freq missing");
  MSA_REQUIRE(ring_rows >= 1 && n_decode >= 0 && n_decode <= n_seq && n_tok >= n_decode && n_old >= 0, "latent_prep: bad counts");
  MSA_REQUIRE(n_seq == n_decode || (ctx && ctx_off && old_off), "latent_prep: portions need a context");
  if (n_tok == 0) return MSA_OK;
  LatentPrepParams p{proj, proj_stride, w_norm, eps, inv_freq, heads, dim, rot, rank, pos, tok_seq, slot, start, cu, ctx_off,
                     old_off, n_tok, n_seq, n_decode, window, ring, ring_rows, ctx};
  const int e4 = 4 * (int)dtype_size(dtype);
  auto ok4 = [&](const void* q) { return q == nullptr || reinterpret_cast<uintptr_t>(q) % e4 == 0; };
  if (dim % 4 == 0 && rot % 4 == 0 && rank % 4 == 0 && rank <= 512 && proj_stride % 4 == 0 && ok4(proj) && ok4(ring) && ok4(ctx) &&
      aligned16(w_norm) && ring_rows < (1ll << 31)) {
    MSA_LM_DISPATCH(dtype, { latent_prep_vec_kernel<T><<<n_tok + n_old, 128, (size_t)rot * 4, (cudaStream_t)stream>>>(p); });
    MSA_LAUNCH_OK("latent_prep_vec_kernel");
    return MSA_OK;
  }
  MSA_LM_DISPATCH(dtype, { latent_prep_kernel<T><<<n_tok + n_old, 128, (size_t)rot * 4, (cudaStream_t)stream>>>(p); });
  MSA_LAUNCH_OK("latent_prep_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_ring_store(const void* ctx, int32_t row_width, const int32_t* slot, const int32_t* start,
                                 const int32_t* cu, const int32_t* ctx_off, int32_t n_seq, int32_t n_decode, int32_t max_len,
                                 int32_t window, void* ring, int64_t ring_rows, int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && ctx && slot && start && cu && ctx_off && ring && row_width > 0 && ring_rows > 0,
              "ring_store: bad arguments");
  if (n_seq <= n_decode || max_len <= 0) return MSA_OK;
  const int64_t rows = max_len < ring_rows ? max_len : ring_rows;
  const dim3 grid((unsigned)(rows < 4096 ? rows : 4096), (unsigned)(n_seq - n_decode));
  MSA_LM_DISPATCH(dtype, {
    ring_store_kernel<T><<<grid, 128, 0, (cudaStream_t)stream>>>((const T*)ctx, row_width, slot, start, cu, ctx_off, n_decode,
                                                                window, (T*)ring, ring_rows);
  });
  MSA_LAUNCH_OK("ring_store_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_window_attn(const msa_lm_attn_args* args, void* stream) {
  MSA_REQUIRE(args, "window_attn: null arguments");
  const msa_lm_attn_args a = *args;
  MSA_REQUIRE(dtype_ok(a.dtype) && dtype_ok(a.qa_dtype) && dtype_ok(a.out_dtype), "window_attn: bad dtype");
  MSA_REQUIRE(a.qa && a.ka && a.v && a.out && a.start && a.cu && (a.db == 0 || (a.qb && a.kb)), "window_attn: null pointer");
  MSA_REQUIRE(a.ring_rows > 0 ? a.slot != nullptr : a.ctx_off != nullptr, "window_attn: no key addressing");
  MSA_REQUIRE(a.heads > 0 && a.da > 0 && a.db >= 0 && a.dv > 0 && a.window > 0, "window_attn: bad sizes");
  if (a.seq1 <= a.seq0 || a.max_len <= 0) return MSA_OK;
  MSA_REQUIRE(a.group > 0 && a.heads % a.group == 0, "window_attn: heads must be a multiple of group");
  const int hg = a.group;
  const int dq = a.da + a.db;
  int tile = 32;
  auto bytes = [&](int t) { return (size_t)4 * ((size_t)kGaRows * (dq + a.dv) + (size_t)t * (dq + 1 + a.dv)); };
  while (tile > 4 && bytes(tile) > 200 * 1024) tile /= 2;
  MSA_REQUIRE(bytes(tile) <= 227 * 1024, "window_attn: head sizes too large (%d, %d)", dq, a.dv);
  static DeviceSmem state;
  MSA_OK_OR_RETURN(ensure_dynamic_smem(window_attn_kernel, bytes(tile), state));
  const dim3 grid((unsigned)(((long long)a.max_len * hg + kGaRows - 1) / kGaRows), (unsigned)(a.heads / hg),
                  (unsigned)(a.seq1 - a.seq0));
  window_attn_kernel<<<grid, kGaThreads, bytes(tile), (cudaStream_t)stream>>>(a, hg, tile);
  MSA_LAUNCH_OK("window_attn_kernel");
  return MSA_OK;
}
