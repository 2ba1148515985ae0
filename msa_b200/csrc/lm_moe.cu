// Mixtures of small experts: top-k routing, grouping of the choices by expert, and the general grouped product
// (any sizes, both dtypes, fp32 accumulation) with the clamped gated activation fused into the first of the two.
#include "lm_common.cuh"

namespace msa {

constexpr int kMoeMaxExperts = 1024;

// One warp per row.  The winners are taken one at a time in descending order; the softmax runs over them alone.
// PER: logits per lane.
template <int PER>
__global__ void __launch_bounds__(256)
moe_topk_kernel(const float* __restrict__ logits, long long stride, const float* __restrict__ bias, int n_rows, int experts,
                int top, int32_t* __restrict__ idx, float* __restrict__ weight) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= n_rows) return;
  float z[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = i * 32 + lane;
    z[i] = e < experts ? logits[(long long)row * stride + e] + (bias ? bias[e] : 0.f) : -INFINITY;
  }
  uint32_t taken = 0;
  float z0 = 0.f, sum = 0.f, mine = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int arg = experts;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (!((taken >> i) & 1u) && i * 32 + lane < experts && (arg == experts || z[i] > best)) { best = z[i]; arg = i * 32 + lane; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
      if (oa < experts && (arg == experts || ob > best || (ob == best && oa < arg))) { best = ob; arg = oa; }
    }
    if (arg >= experts) arg = k;                      // NaN logits: stay in range
    if ((arg & 31) == lane) taken |= 1u << (arg >> 5);
    if (k == 0) z0 = best;
    const float w = expf(best - z0);
    sum += w;
    if (lane == 0) idx[(long long)row * top + k] = arg;
    if (lane == (k & 31)) {
      if (k < 32) mine = w;
      else weight[(long long)row * top + k] = w;      // beyond 32 choices: scaled below
    }
  }
  __syncwarp();
  if (lane < top) weight[(long long)row * top + lane] = mine / sum;
  for (int k = 32 + lane; k < top; k += 32) weight[(long long)row * top + k] /= sum;
}

// One block: histogram, prefix sums, placement, tile list.
__global__ void __launch_bounds__(1024)
moe_sort_kernel(const int32_t* __restrict__ idx, int n, int top, int experts, int tile_rows, int32_t* __restrict__ src,
                int32_t* __restrict__ inv, int32_t* __restrict__ off, int32_t* __restrict__ tiles, int max_tiles) {
  __shared__ int s_cnt[kMoeMaxExperts], s_off[kMoeMaxExperts + 1], s_tile[kMoeMaxExperts + 1];
  for (int e = threadIdx.x; e < experts; e += blockDim.x) s_cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) atomicAdd(&s_cnt[idx[i]], 1);
  __syncthreads();
  if (threadIdx.x < 32) {                               // one warp: prefix sums over the experts
    int o = 0, t = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int c = e < experts ? s_cnt[e] : 0, ct = (c + tile_rows - 1) / tile_rows;
      int so = c, stl = ct;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int x = __shfl_up_sync(0xffffffffu, so, d), y = __shfl_up_sync(0xffffffffu, stl, d);
        if ((int)threadIdx.x >= d) { so += x; stl += y; }
      }
      if (e < experts) { s_off[e] = o + so - c; s_tile[e] = t + stl - ct; }
      o += __shfl_sync(0xffffffffu, so, 31);
      t += __shfl_sync(0xffffffffu, stl, 31);
    }
    if (threadIdx.x == 0) { s_off[experts] = o; s_tile[experts] = t; }
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= experts; e += blockDim.x) off[e] = s_off[e];
  for (int e = threadIdx.x; e < experts; e += blockDim.x)
    for (int t = s_tile[e]; t < s_tile[e + 1] && t < max_tiles; ++t) {
      tiles[2 * t] = e;
      tiles[2 * t + 1] = s_off[e] + (t - s_tile[e]) * tile_rows;
    }
  for (int t = s_tile[experts] + threadIdx.x; t < max_tiles; t += blockDim.x) { tiles[2 * t] = -1; tiles[2 * t + 1] = 0; }
  for (int e = threadIdx.x; e < experts; e += blockDim.x) s_cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = idx[i];
    const int at = s_off[e] + atomicAdd(&s_cnt[e], 1);
    src[at] = i / top;
    inv[i] = at;
  }
}

// The same over many blocks: counts per block of 2,048 choices, then every block places its own from the counts before it.
constexpr int kSortBlock = 2048;

__global__ void __launch_bounds__(256)
moe_count_kernel(const int32_t* __restrict__ idx, int n, int experts, int32_t* __restrict__ cnt) {
  __shared__ int s_cnt[kMoeMaxExperts];
  for (int e = threadIdx.x; e < experts; e += 256) s_cnt[e] = 0;
  __syncthreads();
  const int i1 = min(n, ((int)blockIdx.x + 1) * kSortBlock);
  for (int i = blockIdx.x * kSortBlock + threadIdx.x; i < i1; i += 256) atomicAdd(&s_cnt[idx[i]], 1);
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += 256) cnt[blockIdx.x * experts + e] = s_cnt[e];
}

__global__ void __launch_bounds__(256)
moe_place_kernel(const int32_t* __restrict__ idx, int n, int top, int experts, int tile_rows, const int32_t* __restrict__ cnt,
                 int32_t* __restrict__ src, int32_t* __restrict__ inv, int32_t* __restrict__ off, int32_t* __restrict__ tiles,
                 int max_tiles) {
  __shared__ int s_total[kMoeMaxExperts + 1], s_next[kMoeMaxExperts], s_tile[kMoeMaxExperts + 1];
  for (int e = threadIdx.x; e < experts; e += 256) {
    int total = 0, before = 0;
    for (int b = 0; b < (int)gridDim.x; ++b) {
      const int c = cnt[b * experts + e];
      if (b < (int)blockIdx.x) before += c;
      total += c;
    }
    s_total[e] = total;
    s_next[e] = before;
  }
  __syncthreads();
  if (threadIdx.x < 32) {                               // one warp: prefix sums over the experts
    int o = 0, t = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int c = e < experts ? s_total[e] : 0, ct = (c + tile_rows - 1) / tile_rows;
      int so = c, stl = ct;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int x = __shfl_up_sync(0xffffffffu, so, d), y = __shfl_up_sync(0xffffffffu, stl, d);
        if ((int)threadIdx.x >= d) { so += x; stl += y; }
      }
      if (e < experts) { s_total[e] = o + so - c; s_tile[e] = t + stl - ct; }
      o += __shfl_sync(0xffffffffu, so, 31);
      t += __shfl_sync(0xffffffffu, stl, 31);
    }
    if (threadIdx.x == 0) { s_total[experts] = o; s_tile[experts] = t; }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += 256) s_next[e] += s_total[e];
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e <= experts; e += 256) off[e] = s_total[e];
    for (int e = threadIdx.x; e < experts; e += 256)
      for (int t = s_tile[e]; t < s_tile[e + 1] && t < max_tiles; ++t) {
        tiles[2 * t] = e;
        tiles[2 * t + 1] = s_total[e] + (t - s_tile[e]) * tile_rows;
      }
    for (int t = s_tile[experts] + threadIdx.x; t < max_tiles; t += 256) { tiles[2 * t] = -1; tiles[2 * t + 1] = 0; }
  }
  __syncthreads();
  const int i1 = min(n, ((int)blockIdx.x + 1) * kSortBlock);
  for (int i = blockIdx.x * kSortBlock + threadIdx.x; i < i1; i += 256) {
    const int at = atomicAdd(&s_next[idx[i]], 1);
    src[at] = i / top;
    inv[i] = at;
  }
}

// out[i] = x[src[i]], 16 bytes per lane.
__global__ void __launch_bounds__(256)
gather_rows_kernel(const uint4* __restrict__ x, long long x_vecs, const int32_t* __restrict__ src, int n, int vecs, uint4* __restrict__ out) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= n) return;
  const uint4* from = x + (long long)src[row] * x_vecs;
  uint4* to = out + (long long)row * vecs;
#pragma unroll 4
  for (int c = threadIdx.x & 31; c < vecs; c += 32) to[c] = from[c];
}

__device__ __forceinline__ float clamped_gate(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.f);
}

// 32 rows x 32 columns (act: 32 gate and 32 up columns) per block of 256 threads, K in steps of 32.
constexpr int kMgRows = 32, kMgCols = 32, kMgK = 32;

template <typename T, bool ACT>
__global__ void __launch_bounds__(256)
moe_gemm_kernel(const T* __restrict__ x, long long x_stride, const int32_t* __restrict__ src, const T* __restrict__ w,
                const int32_t* __restrict__ off, const int32_t* __restrict__ tiles, int n_out, int k_dim, float limit,
                void* __restrict__ out, long long out_stride, int32_t out_dtype) {
  __shared__ float s_x[kMgRows][kMgK + 1], s_w[ACT ? 2 : 1][kMgCols][kMgK + 1];
  const int e = tiles[2 * blockIdx.y];
  if (e < 0) return;
  const int i0 = tiles[2 * blockIdx.y + 1], rows = min(kMgRows, off[e + 1] - i0);
  const int n_cols = ACT ? n_out / 2 : n_out, c0 = blockIdx.x * kMgCols;
  const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;   // column, rows ty, ty+8, ...
  const T* we = w + (long long)e * n_out * k_dim;
  float acc[ACT ? 2 : 1][4] = {};
  for (int k0 = 0; k0 < k_dim; k0 += kMgK) {
    for (int i = threadIdx.x; i < kMgRows * kMgK; i += 256) {
      const int r = i / kMgK, k = i % kMgK;
      float v = 0.f;
      if (r < rows && k0 + k < k_dim) v = to_f(x[(long long)(src ? src[i0 + r] : i0 + r) * x_stride + k0 + k]);
      s_x[r][k] = v;
#pragma unroll
      for (int p = 0; p < (ACT ? 2 : 1); ++p)
        s_w[p][r][k] = (c0 + r < n_cols && k0 + k < k_dim) ? to_f(we[((long long)p * n_cols + c0 + r) * k_dim + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kMgK; ++k)
#pragma unroll
      for (int p = 0; p < (ACT ? 2 : 1); ++p) {
        const float b = s_w[p][tx][k];
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[p][q] = fmaf(s_x[ty + 8 * q][k], b, acc[p][q]);
      }
    __syncthreads();
  }
  if (c0 + tx >= n_cols) return;
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const int r = ty + 8 * q;
    if (r >= rows) continue;
    const float v = ACT ? clamped_gate(acc[0][q], acc[ACT ? 1 : 0][q], limit) : acc[0][q];
    store_any(out, out_dtype, (long long)(i0 + r) * out_stride + c0 + tx, v);
  }
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_moe_topk(const float* logits, int64_t stride, const float* bias, int32_t n_rows, int32_t experts,
                               int32_t top, int32_t* idx, float* weight, void* stream) {
  MSA_REQUIRE(logits && idx && weight && n_rows >= 0, "moe_topk: bad arguments");
  MSA_REQUIRE(experts > 0 && experts <= kMoeMaxExperts && top > 0 && top <= experts, "moe_topk: 1 <= top <= experts <= 1024");
  if (n_rows == 0) return MSA_OK;
  const unsigned blocks = (unsigned)((n_rows + 7) / 8);
  cudaStream_t st = (cudaStream_t)stream;
  if (experts <= 32) moe_topk_kernel<1><<<blocks, 256, 0, st>>>(logits, stride, bias, n_rows, experts, top, idx, weight);
  else if (experts <= 64) moe_topk_kernel<2><<<blocks, 256, 0, st>>>(logits, stride, bias, n_rows, experts, top, idx, weight);
  else if (experts <= 128) moe_topk_kernel<4><<<blocks, 256, 0, st>>>(logits, stride, bias, n_rows, experts, top, idx, weight);
  else if (experts <= 256) moe_topk_kernel<8><<<blocks, 256, 0, st>>>(logits, stride, bias, n_rows, experts, top, idx, weight);
  else moe_topk_kernel<32><<<blocks, 256, 0, st>>>(logits, stride, bias, n_rows, experts, top, idx, weight);
  MSA_LAUNCH_OK("moe_topk_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_moe_sort(const int32_t* idx, int32_t n_rows, int32_t top, int32_t experts, int32_t tile_rows,
                               int32_t* src, int32_t* inv, int32_t* off, int32_t* tiles, int32_t max_tiles,
                               int32_t* counts, void* stream) {
  MSA_REQUIRE(idx && src && inv && off && tiles && n_rows >= 0 && top > 0 && tile_rows > 0, "moe_sort: bad arguments");
  MSA_REQUIRE(experts > 0 && experts <= kMoeMaxExperts, "moe_sort: at most 1024 experts");
  const long long n = (long long)n_rows * top;
  MSA_REQUIRE(n < (1ll << 31), "moe_sort: too many rows");
  long long need = n / tile_rows + (n < experts ? n : experts);
  MSA_REQUIRE(max_tiles >= need, "moe_sort: room for %lld tiles needed", need);
  if (counts && n > 2 * kSortBlock) {
    const unsigned blocks = (unsigned)((n + kSortBlock - 1) / kSortBlock);
    moe_count_kernel<<<blocks, 256, 0, (cudaStream_t)stream>>>(idx, (int)n, experts, counts);
    MSA_LAUNCH_OK("moe_count_kernel");
    moe_place_kernel<<<blocks, 256, 0, (cudaStream_t)stream>>>(idx, (int)n, top, experts, tile_rows, counts, src, inv, off, tiles, max_tiles);
    MSA_LAUNCH_OK("moe_place_kernel");
    return MSA_OK;
  }
  moe_sort_kernel<<<1, 1024, 0, (cudaStream_t)stream>>>(idx, (int)n, top, experts, tile_rows, src, inv, off, tiles, max_tiles);
  MSA_LAUNCH_OK("moe_sort_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_moe_gemm(const void* x, int64_t x_stride, const int32_t* src, const void* w, const int32_t* off,
                               const int32_t* tiles, int32_t max_tiles, int32_t n_out, int32_t k, int32_t act, float limit,
                               void* out, int64_t out_stride, int32_t out_dtype, int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && dtype_ok(out_dtype) && x && w && off && tiles && out, "moe_gemm: bad arguments");
  MSA_REQUIRE(n_out > 0 && k > 0 && (!act || n_out % 2 == 0), "moe_gemm: bad sizes");
  if (max_tiles <= 0) return MSA_OK;
  const int cols = act ? n_out / 2 : n_out;
  const dim3 grid((unsigned)((cols + kMgCols - 1) / kMgCols), (unsigned)max_tiles);
  MSA_REQUIRE(max_tiles <= 65535, "moe_gemm: too many tiles");
  MSA_LM_DISPATCH(dtype, {
    if (act) moe_gemm_kernel<T, true><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)x, x_stride, src, (const T*)w, off, tiles, n_out, k, limit, out, out_stride, out_dtype);
    else moe_gemm_kernel<T, false><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)x, x_stride, src, (const T*)w, off, tiles, n_out, k, limit, out, out_stride, out_dtype);
  });
  MSA_LAUNCH_OK("moe_gemm_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_gather_rows(const void* x, int64_t x_stride_bytes, const int32_t* src, int32_t n, int32_t row_bytes, void* out,
                                  void* stream) {
  MSA_REQUIRE(x && src && out && n >= 0 && row_bytes > 0, "gather_rows: bad arguments");
  MSA_REQUIRE(aligned16(x) && aligned16(out) && row_bytes % 16 == 0 && x_stride_bytes % 16 == 0, "gather_rows: 16-byte rows expected");
  if (n == 0) return MSA_OK;
  gather_rows_kernel<<<(unsigned)((n + 7) / 8), 256, 0, (cudaStream_t)stream>>>((const uint4*)x, x_stride_bytes / 16, src, n, row_bytes / 16, (uint4*)out);
  MSA_LAUNCH_OK("gather_rows_kernel");
  return MSA_OK;
}
