// The recurrences of lm_linear.cu over prompt portions in chunks of 64 tokens, on tensor cores, all chunks at once:
//   1. per chunk, what its tokens add to the state:      dS = sum_i (e^(G_C - G_i) k_i) v_i^T
//   2. along the chunks, elementwise:                    S_(c+1) = e^(G_C) S_c + dS_c
//   3. per chunk, the read-out from S_c and from the chunk's own tokens.
// G is the running sum of the log decays inside the chunk (in units of log 2), per key channel (wkv) or per head (ssd).  A
// difference of two running sums loses what a steep token between the chunk's start and both has cost: wkv's sums restart
// every 16 rows (and no token counts for more than 2^-160, which is zero already), ssd's are 64-bit numbers.
//
// 32-bit operands enter the products as the sum of two bf16 numbers (16 to 17 significant bits), accumulated in fp32; what
// is bf16 by nature (projections, convolved activations) enters as it is.  Decays, sums and the states are plain fp32.
//
// wkv's scores e^(G_(t-1) - G_i) r_t . k_i factor only relative to a reference: a warp takes its 16 rows against every
// earlier block of 16 keys with the decays measured from the start of its rows, where both factors are at most 1.  Inside
// its own block the keys' factor grows, to 2^100 at most; rows that decay further than that are computed pair by pair.
#include "lm_linear.cuh"
#include "mma_helpers.cuh"

namespace msa {

constexpr int kLcRows = 64;
constexpr float kLcSteep = 100.f, kLcGone = -160.f;

__device__ __forceinline__ void lc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lc_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 lc_pair(const unsigned char* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

struct LcChunk { int s, t0, len; long long n0; };    // sequence, first token of the chunk, its tokens, their first packed row
__device__ __forceinline__ LcChunk lc_chunk(const int32_t* chunk_off, const int32_t* cu, int n_decode, int n_seq, int chunk) {
  LcChunk c;
  const int ps = owner_of(chunk_off, n_seq - n_decode, chunk);
  c.s = ps + n_decode;
  c.t0 = (chunk - chunk_off[ps]) * kLcRows;
  c.len = min(kLcRows, cu[c.s + 1] - cu[c.s] - c.t0);
  c.n0 = (long long)cu[c.s] + c.t0;
  return c;
}
// rows of `cols` bf16 (a multiple of 8) to shared memory, padded with zeros to 64 rows of `tile` columns
template <int TILE, int THREADS>
__device__ __forceinline__ void lc_load_rows(uint32_t dst, int pitch, const __nv_bfloat16* src, long long stride, int cols, int len) {
  constexpr int kVecs = TILE / 8;
  for (int i = threadIdx.x; i < kLcRows * kVecs; i += THREADS) {
    const int r = i / kVecs, c = i % kVecs;
    const bool on = r < len && c * 8 < cols;
    cp_async16(dst + r * pitch + c * 16, on ? src + r * stride + c * 8 : src, on ? 16u : 0u);
  }
}
// a [rows, cols] fp32 matrix to a pair of bf16 planes of tile rows x tile columns, zero outside
template <int ROWS, int TILE, int THREADS>
__device__ __forceinline__ void lc_load_split(unsigned char* dst, int pitch, int lo_off, const float* src, int rows, int cols) {
  constexpr int kVecs = TILE / 4;
  constexpr int kAll = ROWS * kVecs / THREADS, kStep = kAll <= 8 ? kAll : (kAll % 8 == 0 ? 8 : 6);
  static_assert(ROWS * kVecs % THREADS == 0 && kAll % kStep == 0, "whole turns");
#pragma unroll 1
  for (int u = 0; u < kAll; u += kStep) {
    float4 x[kStep];
#pragma unroll
    for (int k = 0; k < kStep; ++k) {
      const int i = threadIdx.x + (u + k) * THREADS, r = i / kVecs, c = i % kVecs * 4;
      x[k] = r < rows && c < cols ? load4(src + (long long)r * cols + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int k = 0; k < kStep; ++k) {
      const int i = threadIdx.x + (u + k) * THREADS, r = i / kVecs, c = i % kVecs * 4;
      uint2 hi, lo;
      lc_split2(x[k].x, x[k].y, hi.x, lo.x);
      lc_split2(x[k].z, x[k].w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(dst + r * pitch + c * 2) = hi;
      *reinterpret_cast<uint2*>(dst + lo_off + r * pitch + c * 2) = lo;
    }
  }
}

// ---- step 2 for both ----------------------------------------------------------------------------------------------------
// g: running log2 decays [rows.., stride]; the chunk's total stands in its last row (CHANNEL: the sum of its blocks' last
// rows).  A thread carries four elements.
template <bool CHANNEL, typename G>
__global__ void __launch_bounds__(128) linear_carry_kernel(float* __restrict__ work, const G* __restrict__ g, long long g_stride, int g_row0,
                                                           float* __restrict__ state, const int32_t* slot, const int32_t* start,
                                                           const int32_t* cu, const int32_t* chunk_off, int n_decode, int heads, int dk, int dv) {
  const int e = (blockIdx.x * 128 + threadIdx.x) * 4, h = blockIdx.y, ps = blockIdx.z, s = ps + n_decode;
  if (e >= dk * dv) return;
  const int d = e / dv, len = cu[s + 1] - cu[s], n = (len + kLcRows - 1) / kLcRows;
  const long long step = (long long)heads * dk * dv;
  float* w = work + ((long long)chunk_off[ps] * heads + h) * dk * dv + e;
  float* st = state + ((long long)slot[s] * heads + h) * dk * dv + e;
  const G* gp = g + ((long long)cu[s] - g_row0) * g_stride + (CHANNEL ? h * dk + d : h);
  float4 S = start[s] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(st);
  constexpr int kAhead = 8;
  for (int c0 = 0; c0 < n; c0 += kAhead) {
    float4 x[kAhead];
    float f[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i >= n) break;
      x[i] = load4(w + (c0 + i) * step);
      const int last = min((c0 + i + 1) * kLcRows, len) - 1;
      f[i] = (float)gp[(long long)last * g_stride];
      if constexpr (CHANNEL) {
#pragma unroll
        for (int b = 0; b < kLcRows / 16 - 1; ++b) {
          const int r = (c0 + i) * kLcRows + 16 * b + 15;
          if (r < last) f[i] += gp[(long long)r * g_stride];
        }
      }
    }
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i >= n) break;
      store4(w + (c0 + i) * step, S);
      const float a = exp2f(f[i]);
      S = make_float4(fmaf(a, S.x, x[i].x), fmaf(a, S.y, x[i].y), fmaf(a, S.z, x[i].z), fmaf(a, S.w, x[i].w));
    }
  }
  store4(st, S);
}

// ---- wkv ------------------------------------------------------------------------------------------------------------------
struct WkvChunkParams {
  msa_lm_wkv_args a;
  const int32_t* chunk_off;
  float* work;
  __nv_bfloat16* out; long long out_stride;
};

// Step 1; the decays become running sums, one for every 16 rows, in place.
template <int D>
__global__ void __launch_bounds__(2 * D) wkv_add_kernel(const WkvChunkParams p) {
  constexpr int kP = D * 2 + 16, kThreads = 2 * D;
  extern __shared__ __align__(16) unsigned char sm[];
  unsigned char *s_k = sm, *s_v = sm + 2 * kLcRows * kP;      // decayed keys (hi, lo), values
  float* s_tot = reinterpret_cast<float*>(s_v + kLcRows * kP);   // [D]: the chunk's second half
  const msa_lm_wkv_args& a = p.a;
  const int h = blockIdx.y, dim = a.dim;
  const LcChunk ch = lc_chunk(p.chunk_off, a.cu, a.n_decode, a.n_seq, blockIdx.x);
  const long long row = ch.n0 * a.row_stride + h * dim;
  lc_load_rows<D, kThreads>((uint32_t)__cvta_generic_to_shared(s_v), kP, reinterpret_cast<const __nv_bfloat16*>(a.v) + row, a.row_stride, dim, ch.len);
  cp_async_commit();
  {
    const int d = threadIdx.x % D, part = threadIdx.x / D, r0 = part * 32;
    const bool on = d < dim;
    float* dec = a.decay + ch.n0 * a.heads * dim + h * dim + d;
    const __nv_bfloat16* key = reinterpret_cast<const __nv_bfloat16*>(a.k) + row + d;
    const float w0 = on ? a.w0[h * dim + d] : 0.f;
    float g[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) g[i] = on && r0 + i < ch.len ? dec[(long long)(r0 + i) * a.heads * dim] : -INFINITY;
    __nv_bfloat16 k[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) k[i] = on && r0 + i < ch.len ? key[(long long)(r0 + i) * a.row_stride] : __float2bfloat16_rn(0.f);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      g[i] = fmaxf(kLcGone, -1.4426950408889634f * expf(g[i] + w0));
      sum = i % 16 ? sum + g[i] : g[i];
      if (on && r0 + i < ch.len) dec[(long long)(r0 + i) * a.heads * dim] = sum;
    }
    if (part) {
      sum = 0.f;
#pragma unroll
      for (int i = 0; i < 32; ++i) sum += g[i];
      s_tot[d] = sum;
    }
    __syncthreads();
    float rest = part ? 0.f : s_tot[d];                  // what a key decays by until the chunk's end
#pragma unroll
    for (int i = 31; i >= 0; --i) {
      const int r = r0 + i;
      const float x = __bfloat162float(k[i]) * exp2f(rest);
      rest += g[i];
      const __nv_bfloat16 hi = __float2bfloat16_rn(x);
      *reinterpret_cast<__nv_bfloat16*>(s_k + r * kP + d * 2) = hi;
      *reinterpret_cast<__nv_bfloat16*>(s_k + (kLcRows + r) * kP + d * 2) = __float2bfloat16_rn(x - __bfloat162float(hi));
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  float acc[D / 8][4];
#pragma unroll
  for (int j = 0; j < D / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  // A = keys transposed: stored rows are the reduction index
  const uint32_t a_base = (uint32_t)__cvta_generic_to_shared(s_k) + ((lane & 7) + (lane >> 4) * 8) * kP + (warp * 16 + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t b_base = (uint32_t)__cvta_generic_to_shared(s_v) + ((lane & 7) + ((lane >> 3) & 1) * 8) * kP + (lane >> 4) * 16;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    uint32_t ah[4], al[4];
    ldmatrix_x4_trans(a_base + k * 16 * kP, ah[0], ah[1], ah[2], ah[3]);
    ldmatrix_x4_trans(a_base + (kLcRows + k * 16) * kP, al[0], al[1], al[2], al[3]);
#pragma unroll
    for (int j = 0; j < D / 8; j += 2) {
      uint32_t b[4];
      ldmatrix_x4_trans(b_base + k * 16 * kP + j * 16, b[0], b[1], b[2], b[3]);
      lc_mma(acc[j], al, b[0], b[1]);
      lc_mma(acc[j + 1], al, b[2], b[3]);
      lc_mma(acc[j], ah, b[0], b[1]);
      lc_mma(acc[j + 1], ah, b[2], b[3]);
    }
  }
  float* dst = p.work + ((long long)blockIdx.x * a.heads + h) * dim * dim;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int d = warp * 16 + g + 8 * e;
    if (d >= dim) continue;
#pragma unroll
    for (int j = 0; j < D / 8; ++j)
      if (j * 8 < dim) *reinterpret_cast<float2*>(dst + (long long)d * dim + j * 8 + tq * 2) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
  }
}

// Step 3 with the head norm and the gate.  Four warps, 16 rows each.
template <int D>
__global__ void __launch_bounds__(128) wkv_read_kernel(const WkvChunkParams p) {
  constexpr int kP = D * 2 + 16, kG = D + 8, kTile = kLcRows * kP;
  extern __shared__ __align__(16) unsigned char sm[];
  unsigned char *s_r = sm, *s_k = s_r + kTile, *s_v = s_k + kTile, *s_s = s_v + kTile;      // the state: hi, lo
  float* s_g = reinterpret_cast<float*>(s_s + 2 * D * kP);                                     // [64][kG]
  const msa_lm_wkv_args& a = p.a;
  const int h = blockIdx.y, dim = a.dim;
  const LcChunk ch = lc_chunk(p.chunk_off, a.cu, a.n_decode, a.n_seq, blockIdx.x);
  const long long row = ch.n0 * a.row_stride + h * dim;
  auto sp = [](const void* q) { return (uint32_t)__cvta_generic_to_shared(q); };
  lc_load_rows<D, 128>(sp(s_r), kP, reinterpret_cast<const __nv_bfloat16*>(a.r) + row, a.row_stride, dim, ch.len);
  lc_load_rows<D, 128>(sp(s_k), kP, reinterpret_cast<const __nv_bfloat16*>(a.k) + row, a.row_stride, dim, ch.len);
  lc_load_rows<D, 128>(sp(s_v), kP, reinterpret_cast<const __nv_bfloat16*>(a.v) + row, a.row_stride, dim, ch.len);
  {
    const float* src = a.decay + ch.n0 * a.heads * dim + h * dim;
    for (int i = threadIdx.x; i < kLcRows * (D / 4); i += 128) {       // rows past the end repeat the last one
      const int r = i / (D / 4), c = i % (D / 4) * 4;
      const bool on = c < dim;
      cp_async16(sp(s_g + r * kG + c), on ? src + (long long)min(r, ch.len - 1) * a.heads * dim + c : src, on ? 16u : 0u);
    }
  }
  cp_async_commit();
  lc_load_split<D, D, 128>(s_s, kP, D * kP, p.work + ((long long)blockIdx.x * a.heads + h) * dim * dim, dim, dim);
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3, r0 = warp * 16 + g;
  if (warp * 16 >= ch.len) return;
  bool steep;
  {
    float span = 0.f;
    const float* end = s_g + (warp * 16 + 15) * kG;
    for (int d = lane; d < dim; d += 32) span = fmaxf(span, -end[d]);
    steep = warp_max_f(span) > kLcSteep;
  }
  float o[D / 8][4], s[8][4];
#pragma unroll
  for (int j = 0; j < D / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
  float own[2] = {0.f, 0.f};                           // r . (u k) of rows r0 and r0 + 8
  const uint32_t b_base = sp(s_s) + ((lane & 7) + ((lane >> 3) & 1) * 8) * kP + (lane >> 4) * 16;
  const int n_oct = 2 * warp + (steep ? 0 : 2);
#pragma unroll 1
  for (int kk = 0; kk < D / 16; ++kk) {
    if (kk * 16 >= dim) break;
    uint32_t fh[4], fl[4], th[4], tl[4];               // rows from the chunk's start, from the block's start
    float2 sum[2][4], after[2][4];                     // per block of 16 keys: its decay, that of the blocks up to this warp's
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int c = kk * 16 + tq * 2 + 8 * x;
      float2 run = make_float2(0.f, 0.f);
#pragma unroll
      for (int b = 3; b >= 0; --b) {
        sum[x][b] = b < warp ? *reinterpret_cast<const float2*>(s_g + (16 * b + 15) * kG + c) : make_float2(0.f, 0.f);
        after[x][b] = run;
        run.x += sum[x][b].x;
        run.y += sum[x][b].y;
      }
      const float2 u = c < dim ? *reinterpret_cast<const float2*>(a.u + h * dim + c) : make_float2(0.f, 0.f);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = r0 + 8 * e;
        const float2 r = lc_pair(s_r + t * kP + c * 2), k = lc_pair(s_k + t * kP + c * 2);
        const float2 gt = t & 15 ? *reinterpret_cast<const float2*>(s_g + (t - 1) * kG + c) : make_float2(0.f, 0.f);
        own[e] = fmaf(r.x * u.x, k.x, own[e]);
        own[e] = fmaf(r.y * u.y, k.y, own[e]);
        lc_split2(r.x * exp2f(gt.x + run.x), r.y * exp2f(gt.y + run.y), fh[2 * x + e], fl[2 * x + e]);
        lc_split2(r.x * exp2f(gt.x), r.y * exp2f(gt.y), th[2 * x + e], tl[2 * x + e]);
      }
    }
#pragma unroll
    for (int j = 0; j < D / 8; j += 2) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(b_base + kk * 16 * kP + j * 16, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4_trans(b_base + (D + kk * 16) * kP + j * 16, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        lc_mma(o[j + n], fl, bh[2 * n], bh[2 * n + 1]);
        lc_mma(o[j + n], fh, bl[2 * n], bl[2 * n + 1]);
        lc_mma(o[j + n], fh, bh[2 * n], bh[2 * n + 1]);
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      if (n < n_oct) {
        const int key = n * 8 + g;
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int c = kk * 16 + tq * 2 + 8 * x;
          const float2 k = lc_pair(s_k + key * kP + c * 2), gi = *reinterpret_cast<const float2*>(s_g + key * kG + c);
          const float2 m = sum[x][n / 2], f = after[x][n / 2];
          lc_split2(k.x * exp2f((m.x - gi.x) + f.x), k.y * exp2f((m.y - gi.y) + f.y), bh[x], bl[x]);
        }
        lc_mma(s[n], tl, bh[0], bh[1]);
        lc_mma(s[n], th, bl[0], bl[1]);
        lc_mma(s[n], th, bh[0], bh[1]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    own[e] += __shfl_xor_sync(0xffffffffu, own[e], 1);
    own[e] += __shfl_xor_sync(0xffffffffu, own[e], 2);
  }
#pragma unroll
  for (int n = 0; n < 8; ++n) {                        // this warp's own block: strictly earlier keys, the bonus on the diagonal
    if ((n >> 1) != warp) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = r0 + 8 * (e >> 1), i = n * 8 + tq * 2 + (e & 1);
      float x = s[n][e];
      if (steep && i < t) {
        x = 0.f;
        const float *gt = s_g + (t - 1) * kG, *gi = s_g + i * kG;
        for (int d = 0; d < dim; ++d)
          x = fmaf(__bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(s_r + t * kP + d * 2)) *
                       __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(s_k + i * kP + d * 2)), exp2f(gt[d] - gi[d]), x);
      }
      s[n][e] = i < t ? x : (i == t ? own[e >> 1] : 0.f);
    }
  }
  const uint32_t v_base = sp(s_v) + ((lane & 7) + ((lane >> 3) & 1) * 8) * kP + (lane >> 4) * 16;
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    if (m > warp) break;
    uint32_t ah[4], al[4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 2; ++e) lc_split2(s[2 * m + x][2 * e], s[2 * m + x][2 * e + 1], ah[2 * x + e], al[2 * x + e]);
#pragma unroll
    for (int j = 0; j < D / 8; j += 2) {
      uint32_t b[4];
      ldmatrix_x4_trans(v_base + m * 16 * kP + j * 16, b[0], b[1], b[2], b[3]);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        lc_mma(o[j + n], al, b[2 * n], b[2 * n + 1]);
        lc_mma(o[j + n], ah, b[2 * n], b[2 * n + 1]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < D / 8; ++j) ss += o[j][2 * e] * o[j][2 * e] + o[j][2 * e + 1] * o[j][2 * e + 1];
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    const float inv = 1.f / sqrtf(ss / (float)dim + a.eps);
    const int t = r0 + 8 * e;
    if (t >= ch.len) continue;
    const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(a.g) + row + (long long)t * a.row_stride;
    __nv_bfloat16* dst = p.out + (ch.n0 - a.n_decode + t) * p.out_stride + h * dim;
#pragma unroll
    for (int j = 0; j < D / 8; ++j) {
      if (j * 8 >= dim) break;
      const int c = j * 8 + tq * 2;
      const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + c));
      const float2 w = *reinterpret_cast<const float2*>(a.norm + h * dim + c);
      *reinterpret_cast<__nv_bfloat162*>(dst + c) =
          __floats2bfloat162_rn(o[j][2 * e] * inv * w.x * silu_act<__nv_bfloat16>(z.x), o[j][2 * e + 1] * inv * w.y * silu_act<__nv_bfloat16>(z.y));
    }
  }
}

template <int D>
int launch_wkv_chunk(const WkvChunkParams& p, int n_chunks, cudaStream_t st) {
  constexpr size_t pitch = D * 2 + 16, add = 3 * kLcRows * pitch + 2 * D * 4, read = 3 * kLcRows * pitch + 2 * D * pitch + kLcRows * (D + 8) * 4;
  static_assert(add <= 227 * 1024 && read <= 227 * 1024, "shared memory");
  const msa_lm_wkv_args& a = p.a;
  const dim3 grid((unsigned)n_chunks, (unsigned)a.heads);
  static DeviceSmem s_add{}, s_read{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(wkv_add_kernel<D>, add, s_add));
  MSA_OK_OR_RETURN(ensure_dynamic_smem(wkv_read_kernel<D>, read, s_read));
  wkv_add_kernel<D><<<grid, 2 * D, add, st>>>(p);
  MSA_LAUNCH_OK("wkv_add_kernel");
  const dim3 carry((unsigned)((a.dim * a.dim / 4 + 127) / 128), (unsigned)a.heads, (unsigned)(a.n_seq - a.n_decode));
  linear_carry_kernel<true, float><<<carry, 128, 0, st>>>(p.work, a.decay, (long long)a.heads * a.dim, 0, a.state, a.slot, a.start, a.cu, p.chunk_off,
                                                   a.n_decode, a.heads, a.dim, a.dim);
  MSA_LAUNCH_OK("linear_carry_kernel");
  wkv_read_kernel<D><<<grid, 128, read, st>>>(p);
  MSA_LAUNCH_OK("wkv_read_kernel");
  return MSA_OK;
}

// ---- ssd --------------------------------------------------------------------------------------------------------------------
struct SsdChunkParams {
  msa_lm_ssd_args a;
  const __nv_bfloat16* xbc;      // [rows, inner | groups*n_state | groups*n_state]
  const float* dt;               // [rows, heads]
  const int32_t* chunk_off;
  double* gcum;                  // [rows, heads]
  float* work;                   // [chunks, heads, n_state, vdim]
};

// Step 1; leaves the running sums of the log2 decays in gcum.
template <int N, int V>
__global__ void __launch_bounds__(2 * N) ssd_add_kernel(const SsdChunkParams p) {
  constexpr int kPn = N * 2 + 16, kPv = V * 2 + 16, kThreads = 2 * N;
  extern __shared__ __align__(16) unsigned char sm[];
  unsigned char *s_b = sm, *s_x = s_b + kLcRows * kPn;          // keys; weighted values (hi, lo)
  __shared__ float s_w[kLcRows];
  const msa_lm_ssd_args& a = p.a;
  const int h = blockIdx.y, inner = a.heads * a.vdim, bc = a.groups * a.n_state, chan = inner + 2 * bc, gr = h / (a.heads / a.groups);
  const LcChunk ch = lc_chunk(p.chunk_off, a.cu, a.n_decode, a.n_seq, blockIdx.x);
  const long long row0 = ch.n0 - a.n_decode;
  const __nv_bfloat16* src = p.xbc + row0 * chan;
  lc_load_rows<N, kThreads>((uint32_t)__cvta_generic_to_shared(s_b), kPn, src + inner + gr * a.n_state, chan, a.n_state, ch.len);
  cp_async_commit();
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x, r = 2 * lane;
    const double rate = -1.4426950408889634 * expf(a.a_log[h]);
    const float d0 = r < ch.len ? p.dt[(row0 + r) * a.heads + h] : 0.f, d1 = r + 1 < ch.len ? p.dt[(row0 + r + 1) * a.heads + h] : 0.f;
    double sum = rate * d0 + rate * d1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double x = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += x;
    }
    const double total = __shfl_sync(0xffffffffu, sum, 31), g0 = sum - rate * d1;
    if (r < ch.len) p.gcum[(row0 + r) * a.heads + h] = g0;
    if (r + 1 < ch.len) p.gcum[(row0 + r + 1) * a.heads + h] = sum;
    s_w[r] = d0 * exp2f((float)(total - g0));
    s_w[r + 1] = d1 * exp2f((float)(total - sum));
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kLcRows * (V / 4); i += kThreads) {
    const int r = i / (V / 4), c = i % (V / 4) * 4;
    const float4 x = r < ch.len && c < a.vdim ? load4(src + (long long)r * chan + h * a.vdim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float w = s_w[r];
    uint2 hi, lo;
    lc_split2(w * x.x, w * x.y, hi.x, lo.x);
    lc_split2(w * x.z, w * x.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(s_x + r * kPv + c * 2) = hi;
    *reinterpret_cast<uint2*>(s_x + (kLcRows + r) * kPv + c * 2) = lo;
  }
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  float acc[V / 8][4];
#pragma unroll
  for (int j = 0; j < V / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const uint32_t a_base = (uint32_t)__cvta_generic_to_shared(s_b) + ((lane & 7) + (lane >> 4) * 8) * kPn + (warp * 16 + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t b_base = (uint32_t)__cvta_generic_to_shared(s_x) + ((lane & 7) + ((lane >> 3) & 1) * 8) * kPv + (lane >> 4) * 16;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    uint32_t x[4];
    ldmatrix_x4_trans(a_base + k * 16 * kPn, x[0], x[1], x[2], x[3]);
#pragma unroll
    for (int j = 0; j < V / 8; j += 2) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(b_base + k * 16 * kPv + j * 16, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4_trans(b_base + (kLcRows + k * 16) * kPv + j * 16, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        lc_mma(acc[j + n], x, bl[2 * n], bl[2 * n + 1]);
        lc_mma(acc[j + n], x, bh[2 * n], bh[2 * n + 1]);
      }
    }
  }
  float* dst = p.work + ((long long)blockIdx.x * a.heads + h) * a.n_state * a.vdim;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int d = warp * 16 + g + 8 * e;
    if (d >= a.n_state) continue;
#pragma unroll
    for (int j = 0; j < V / 8; ++j)
      if (j * 8 < a.vdim) *reinterpret_cast<float2*>(dst + (long long)d * a.vdim + j * 8 + tq * 2) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
  }
}

// Step 3 with the skip and the gate.  Eight warps: 16 rows and half of the value columns each.
template <int N, int V>
__global__ void __launch_bounds__(256, 2) ssd_read_kernel(const SsdChunkParams p) {
  constexpr int kPn = N * 2 + 16, kPv = V * 2 + 16, VH = V / 2;
  extern __shared__ __align__(16) unsigned char sm[];
  unsigned char *s_c = sm, *s_b = s_c + kLcRows * kPn, *s_x = s_b + kLcRows * kPn, *s_s = s_x + kLcRows * kPv;
  __shared__ double s_g[kLcRows];
  __shared__ float s_dt[kLcRows];
  const msa_lm_ssd_args& a = p.a;
  const int h = blockIdx.y, inner = a.heads * a.vdim, bc = a.groups * a.n_state, chan = inner + 2 * bc, gr = h / (a.heads / a.groups);
  const LcChunk ch = lc_chunk(p.chunk_off, a.cu, a.n_decode, a.n_seq, blockIdx.x);
  const long long row0 = ch.n0 - a.n_decode;
  const __nv_bfloat16* src = p.xbc + row0 * chan;
  auto sp = [](const void* q) { return (uint32_t)__cvta_generic_to_shared(q); };
  lc_load_rows<N, 256>(sp(s_b), kPn, src + inner + gr * a.n_state, chan, a.n_state, ch.len);
  lc_load_rows<N, 256>(sp(s_c), kPn, src + inner + bc + gr * a.n_state, chan, a.n_state, ch.len);
  lc_load_rows<V, 256>(sp(s_x), kPv, src + h * a.vdim, chan, a.vdim, ch.len);
  cp_async_commit();
  lc_load_split<N, V, 256>(s_s, kPv, N * kPv, p.work + ((long long)blockIdx.x * a.heads + h) * a.n_state * a.vdim, a.n_state, a.vdim);
  if (threadIdx.x < kLcRows) {
    const int r = min((int)threadIdx.x, ch.len - 1);
    s_g[threadIdx.x] = p.gcum[(row0 + r) * a.heads + h];
    s_dt[threadIdx.x] = p.dt[(row0 + r) * a.heads + h];
  }
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5 & 3, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3, r0 = warp * 16 + g;
  const int c0 = (threadIdx.x >> 7) * VH;              // this warp's first column
  if (warp * 16 >= ch.len || c0 >= a.vdim) return;
  float o[VH / 8][4], s[8][4];
#pragma unroll
  for (int j = 0; j < VH / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
  const uint32_t a_base = sp(s_c) + (warp * 16 + (lane & 15)) * kPn + (lane >> 4) * 16;
  const uint32_t k_base = sp(s_b) + ((lane & 7) + ((lane >> 4) << 3)) * kPn + ((lane >> 3) & 1) * 16;
  const uint32_t s_base = sp(s_s) + c0 * 2 + ((lane & 7) + ((lane >> 3) & 1) * 8) * kPv + (lane >> 4) * 16;
#pragma unroll 2
  for (int kk = 0; kk < N / 16; ++kk) {
    uint32_t c[4];
    ldmatrix_x4(a_base + kk * 32, c[0], c[1], c[2], c[3]);
#pragma unroll
    for (int j = 0; j < VH / 8; j += 2) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(s_base + kk * 16 * kPv + j * 16, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4_trans(s_base + (N + kk * 16) * kPv + j * 16, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        lc_mma(o[j + n], c, bl[2 * n], bl[2 * n + 1]);
        lc_mma(o[j + n], c, bh[2 * n], bh[2 * n + 1]);
      }
    }
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      if (n / 2 <= warp) {
        uint32_t b[4];
        ldmatrix_x4(k_base + n * 8 * kPn + kk * 32, b[0], b[1], b[2], b[3]);
        lc_mma(s[n], c, b[0], b[1]);
        lc_mma(s[n + 1], c, b[2], b[3]);
      }
    }
  }
  const double g0 = s_g[r0], g1 = s_g[r0 + 8];
  {
    const float f0 = exp2f((float)g0), f1 = exp2f((float)g1);
#pragma unroll
    for (int j = 0; j < VH / 8; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
  }
  const uint32_t x_base = sp(s_x) + c0 * 2 + ((lane & 7) + ((lane >> 3) & 1) * 8) * kPv + (lane >> 4) * 16;
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    if (m > warp) break;
    uint32_t ah[4], al[4];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int i = (2 * m + x) * 8 + tq * 2;
      const double gx = s_g[i], gy = s_g[i + 1];
      const float2 di = *reinterpret_cast<const float2*>(s_dt + i);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = r0 + 8 * e;
        const double gt = e ? g1 : g0;
        const float p0 = i <= t ? s[2 * m + x][2 * e] * exp2f((float)(gt - gx)) * di.x : 0.f;
        const float p1 = i + 1 <= t ? s[2 * m + x][2 * e + 1] * exp2f((float)(gt - gy)) * di.y : 0.f;
        lc_split2(p0, p1, ah[2 * x + e], al[2 * x + e]);
      }
    }
#pragma unroll
    for (int j = 0; j < VH / 8; j += 2) {
      uint32_t b[4];
      ldmatrix_x4_trans(x_base + m * 16 * kPv + j * 16, b[0], b[1], b[2], b[3]);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        lc_mma(o[j + n], al, b[2 * n], b[2 * n + 1]);
        lc_mma(o[j + n], ah, b[2 * n], b[2 * n + 1]);
      }
    }
  }
  const float skip = a.d_skip[h];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int t = r0 + 8 * e;
    if (t >= ch.len) continue;
    const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(a.proj) + (ch.n0 + t) * a.proj_stride + h * a.vdim;
    float* dst = a.y + (ch.n0 + t) * inner + h * a.vdim;
#pragma unroll
    for (int j = 0; j < VH / 8; ++j) {
      if (c0 + j * 8 >= a.vdim) break;
      const int c = c0 + j * 8 + tq * 2;
      const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + c)), x = lc_pair(s_x + t * kPv + c * 2);
      *reinterpret_cast<float2*>(dst + c) = make_float2(fmaf(skip, x.x, o[j][2 * e]) * silu_act<__nv_bfloat16>(z.x),
                                                        fmaf(skip, x.y, o[j][2 * e + 1]) * silu_act<__nv_bfloat16>(z.y));
    }
  }
}

template <int N, int V>
int launch_ssd_chunk(const SsdChunkParams& p, int n_chunks, cudaStream_t st) {
  constexpr size_t pn = N * 2 + 16, pv = V * 2 + 16, add = kLcRows * pn + 2 * kLcRows * pv, read = 2 * kLcRows * pn + kLcRows * pv + 2 * N * pv;
  static_assert(add <= 227 * 1024 && read <= 227 * 1024, "shared memory");
  const msa_lm_ssd_args& a = p.a;
  const dim3 grid((unsigned)n_chunks, (unsigned)a.heads);
  static DeviceSmem s_add{}, s_read{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(ssd_add_kernel<N, V>, add, s_add));
  MSA_OK_OR_RETURN(ensure_dynamic_smem(ssd_read_kernel<N, V>, read, s_read));
  ssd_add_kernel<N, V><<<grid, 2 * N, add, st>>>(p);
  MSA_LAUNCH_OK("ssd_add_kernel");
  const dim3 carry((unsigned)((a.n_state * a.vdim / 4 + 127) / 128), (unsigned)a.heads, (unsigned)(a.n_seq - a.n_decode));
  linear_carry_kernel<false, double><<<carry, 128, 0, st>>>(p.work, p.gcum, a.heads, a.n_decode, a.state, a.slot, a.start, a.cu, p.chunk_off, a.n_decode,
                                                    a.heads, a.n_state, a.vdim);
  MSA_LAUNCH_OK("linear_carry_kernel");
  ssd_read_kernel<N, V><<<grid, 256, read, st>>>(p);
  MSA_LAUNCH_OK("ssd_read_kernel");
  return MSA_OK;
}
template <int N>
int launch_ssd_chunk_v(const SsdChunkParams& p, int n_chunks, cudaStream_t st) {
  if (p.a.vdim <= 32) return launch_ssd_chunk<N, 32>(p, n_chunks, st);
  return p.a.vdim <= 64 ? launch_ssd_chunk<N, 64>(p, n_chunks, st) : launch_ssd_chunk<N, 128>(p, n_chunks, st);
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_wkv_chunk_supported(int32_t dim) { return dim > 0 && dim % 8 == 0 && dim <= 128; }

extern "C" int msa_lm_wkv_chunk(const msa_lm_wkv_args* a, const int32_t* chunk_off, int32_t n_chunks, float* work, void* out,
                                int64_t out_stride, void* stream) {
  MSA_OK_OR_RETURN(wkv_check(a, "wkv_chunk"));
  MSA_REQUIRE(a->dtype == MSA_BF16 && msa_lm_wkv_chunk_supported(a->dim) && chunk_off && work && out, "wkv_chunk: unsupported sizes or null pointer");
  MSA_REQUIRE(a->row_stride % 8 == 0 && out_stride % 2 == 0 && aligned16(a->r) && aligned16(a->k) && aligned16(a->v) && aligned16(a->g) &&
                  aligned16(a->decay) && aligned16(work) && aligned16(a->state) && aligned16(a->u) && aligned16(a->norm) &&
                  reinterpret_cast<uintptr_t>(out) % 4 == 0, "wkv_chunk: alignment");
  if (a->n_seq == a->n_decode || n_chunks <= 0) return MSA_OK;
  const WkvChunkParams p{*a, chunk_off, work, (__nv_bfloat16*)out, out_stride};
  cudaStream_t st = (cudaStream_t)stream;
  if (a->dim <= 32) return launch_wkv_chunk<32>(p, n_chunks, st);
  if (a->dim <= 64) return launch_wkv_chunk<64>(p, n_chunks, st);
  if (a->dim <= 96) return launch_wkv_chunk<96>(p, n_chunks, st);
  return launch_wkv_chunk<128>(p, n_chunks, st);
}

extern "C" int msa_lm_ssd_chunk_supported(int32_t n_state, int32_t vdim) {
  return n_state > 0 && n_state % 8 == 0 && n_state <= 128 && vdim > 0 && vdim % 8 == 0 && vdim <= 128;
}

extern "C" int msa_lm_ssd_chunk(const msa_lm_ssd_args* a, const void* xbc, const float* dt, const int32_t* chunk_off, int32_t n_chunks,
                                double* gcum, float* work, void* stream) {
  MSA_OK_OR_RETURN(ssd_check(a, "ssd_chunk"));
  MSA_REQUIRE(a->dtype == MSA_BF16 && msa_lm_ssd_chunk_supported(a->n_state, a->vdim) && xbc && dt && chunk_off && gcum && work,
              "ssd_chunk: unsupported sizes or null pointer");
  MSA_REQUIRE(aligned16(xbc) && aligned16(work) && aligned16(a->state) && aligned16(a->y) && a->proj_stride % 2 == 0 &&
                  reinterpret_cast<uintptr_t>(a->proj) % 4 == 0, "ssd_chunk: alignment");
  if (a->n_seq == a->n_decode || n_chunks <= 0) return MSA_OK;
  const SsdChunkParams p{*a, (const __nv_bfloat16*)xbc, dt, chunk_off, gcum, work};
  cudaStream_t st = (cudaStream_t)stream;
  if (a->n_state <= 32) return launch_ssd_chunk_v<32>(p, n_chunks, st);
  return a->n_state <= 64 ? launch_ssd_chunk_v<64>(p, n_chunks, st) : launch_ssd_chunk_v<128>(p, n_chunks, st);
}
