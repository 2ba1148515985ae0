// Grouped matrix product of a mixture of experts on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), bf16.
//
// A tile is 128 grouped entries of one expert x 256 output columns (with the gated activation: 128 gate columns and the
// 128 up columns that belong to them, so that the epilogue has both).  Persistent CTAs, one per SM, 192 threads: warps 0-3
// the epilogue (thread = row = TMEM lane), warp 4 the TMA producer, warp 5 the MMA issuer.  Operands go through a ring of
// four 48 KB stages; accumulators are double-buffered in TMEM (2 x 256 columns), so the epilogue of a tile runs under the
// products of the next one.  The rows of the first product are fetched straight from the token rows they belong to
// (TMA gather of four rows per copy; only as many as the tile has); a tail in K, columns past the last one and rows of
// other experts are read as zeros or neighbours and not stored.
#include "lm_common.cuh"
#include "tc_attn_common.cuh"

namespace msa {

constexpr int kMtRows = 128, kMtCols = 256, kMtK = 64, kMtStages = 4;
constexpr int kMtA = kMtRows * 128, kMtB = kMtCols * 128, kMtStage = kMtA + kMtB;
constexpr int kMtThreads = 192;
constexpr size_t kMtSmem = (size_t)kMtStages * kMtStage + 1024;

struct MoeTcParams {
  const int32_t *src, *off, *tiles;
  int max_tiles, n_nt, n_kb, n_out, n_cols;   // n_cols: output columns (n_out / 2 with the activation)
  float limit;
  void* out; long long out_stride;
  int32_t* status;
};

__device__ __forceinline__ void tma_gather4(void* smem_dst, const CUtensorMap* map, int x, int4 rows, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile::gather4.mbarrier::complete_tx::bytes [%0], "
      "[%1, {%3, %4, %5, %6, %7}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(map), "r"(smem_u32(bar)), "r"(x), "r"(rows.x), "r"(rows.y), "r"(rows.z), "r"(rows.w)
      : "memory");
}

template <bool ACT>
__global__ void __launch_bounds__(kMtThreads, 1)
moe_gemm_tc_kernel(const __grid_constant__ CUtensorMap tmap_x, const __grid_constant__ CUtensorMap tmap_w, const MoeTcParams p) {
  extern __shared__ unsigned char smem_dyn[];
  __shared__ uint64_t s_full[kMtStages], s_empty[kMtStages], s_acc_full[2], s_acc_empty[2], s_drain;
  __shared__ uint32_t s_tmem_base;
  __shared__ int s_abort;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  unsigned char* ring = reinterpret_cast<unsigned char*>(((uintptr_t)smem_dyn + 1023) & ~(uintptr_t)1023);
  volatile int* abort_flag = &s_abort;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kMtStages; ++i) { mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&s_acc_full[i], 1); mbar_init(&s_acc_empty[i], 4); }
    mbar_init(&s_drain, 1);
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 5) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem_base)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = s_tmem_base;
  const int n_work = p.max_tiles * p.n_nt;

  if (warp == 4) {
    uint32_t n = 0;
    bool ok = true;
    for (int w = blockIdx.x; w < n_work && ok; w += gridDim.x) {
      const int tile = w / p.n_nt, nt = w % p.n_nt, e = p.tiles[2 * tile];
      if (e < 0) break;                                   // used tiles come first
      const int i0 = p.tiles[2 * tile + 1], rows = min(kMtRows, p.off[e + 1] - i0);
      int4 idx = make_int4(0, 0, 0, 0);                   // lane l: the token rows of entries 4l .. 4l+3
      const int n_quads = (rows + 3) / 4;
      if (p.src && lane < n_quads) {
        idx.x = p.src[i0 + 4 * lane];
        idx.y = 4 * lane + 1 < rows ? p.src[i0 + 4 * lane + 1] : idx.x;
        idx.z = 4 * lane + 2 < rows ? p.src[i0 + 4 * lane + 2] : idx.x;
        idx.w = 4 * lane + 3 < rows ? p.src[i0 + 4 * lane + 3] : idx.x;
      }
      const uint32_t bytes = kMtB + (p.src ? n_quads * 512u : (uint32_t)kMtA);
      const int wrow = e * p.n_out + (ACT ? nt * 128 : nt * 256);
      for (int kb = 0; kb < p.n_kb; ++kb, ++n) {
        const uint32_t st = n % kMtStages, ph = (n / kMtStages) & 1u;
        ok = mbar_wait(&s_empty[st], ph ^ 1u, abort_flag, p.status, 11);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        unsigned char* a = ring + st * kMtStage;
        unsigned char* b = a + kMtA;
        if (lane == 0) {
          mbar_expect_tx(&s_full[st], bytes);
          tma_load_2d(b, &tmap_w, kb * kMtK, wrow, &s_full[st]);
          tma_load_2d(b + kMtB / 2, &tmap_w, kb * kMtK, ACT ? wrow + p.n_cols : wrow + 128, &s_full[st]);
          if (!p.src) tma_load_2d(a, &tmap_x, kb * kMtK, i0, &s_full[st]);
        }
        __syncwarp();
        if (p.src && lane < n_quads) tma_gather4(a + lane * 512, &tmap_x, kb * kMtK, idx, &s_full[st]);
      }
    }
    if (!ok) {
      const unsigned long long w0 = global_ns();
      while (global_ns() - w0 < 1000000ull) {}
    }
  } else if (warp == 5) {
    if (lane == 0) {
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kMtCols >> 3) << 17) | ((uint32_t)(kMtRows >> 4) << 24);
      const uint32_t base = smem_u32(ring);
      uint32_t n = 0, n_acc = 0;
      bool ok = true;
      for (int w = blockIdx.x; w < n_work && ok; w += gridDim.x) {
        if (p.tiles[2 * (w / p.n_nt)] < 0) break;
        const uint32_t ab = n_acc & 1u;
        if (!(ok = mbar_wait(&s_acc_empty[ab], ((n_acc >> 1) & 1u) ^ 1u, abort_flag, p.status, 12))) break;
        tc_fence_after();
        for (int kb = 0; kb < p.n_kb; ++kb, ++n) {
          const uint32_t st = n % kMtStages, ph = (n / kMtStages) & 1u;
          if (!(ok = mbar_wait(&s_full[st], ph, abort_flag, p.status, 13))) break;
          tc_fence_after();
          const uint64_t a = make_smem_desc(base + st * kMtStage), b = make_smem_desc(base + st * kMtStage + kMtA);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            tc_mma_bf16(tmem_base + ab * 256, a + (uint64_t)(2 * k), b + (uint64_t)(2 * k), idesc, (kb > 0 || k > 0) ? 1u : 0u);
          tc_commit(&s_empty[st]);
        }
        if (!ok) break;
        tc_commit(&s_acc_full[ab]);
        ++n_acc;
      }
      tc_commit(&s_drain);
      const unsigned long long w0 = global_ns();
      while (!mbar_try_wait(&s_drain, 0) && global_ns() - w0 < kWaitLimitNs) {}
    }
  } else {
    const uint32_t lane_base = tmem_base + ((uint32_t)(warp * 32) << 16);
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out);
    uint32_t n_acc = 0;
    for (int w = blockIdx.x; w < n_work; w += gridDim.x) {
      const int tile = w / p.n_nt, nt = w % p.n_nt, e = p.tiles[2 * tile];
      if (e < 0) break;
      const int i0 = p.tiles[2 * tile + 1], rows = min(kMtRows, p.off[e + 1] - i0);
      const uint32_t ab = n_acc & 1u;
      bool ok = mbar_wait(&s_acc_full[ab], (n_acc >> 1) & 1u, abort_flag, p.status, 14);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const int r = warp * 32 + lane;
      const bool on = r < rows, warp_on = warp * 32 < rows;
      __nv_bfloat16* dst = out + (long long)(i0 + r) * p.out_stride;
      if (warp_on) {
#pragma unroll
        for (int c = 0; c < (ACT ? 4 : 8); ++c) {
          const int col = nt * (ACT ? 128 : 256) + 32 * c;
          if (col >= p.n_cols) break;
          uint32_t g[32];
          tmem_ld32(lane_base + ab * 256 + 32 * c, g);
          float v[32];
          if constexpr (ACT) {
            uint32_t u[32];
            tmem_ld32(lane_base + ab * 256 + 128 + 32 * c, u);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const float gg = fminf(__uint_as_float(g[i]), p.limit);
              const float uu = fminf(fmaxf(__uint_as_float(u[i]), -p.limit), p.limit);
              v[i] = __fdividef(gg * (uu + 1.f), 1.f + __expf(-1.702f * gg));
            }
          } else {
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(g[i]);
          }
          if (on) {
#pragma unroll
            for (int i = 0; i < 32; i += 8)
              if (col + i < p.n_cols)                       // columns come in eights
                *reinterpret_cast<uint4*>(dst + col + i) = make_uint4(pack2_bf16(v[i], v[i + 1]), pack2_bf16(v[i + 2], v[i + 3]),
                                                                      pack2_bf16(v[i + 4], v[i + 5]), pack2_bf16(v[i + 6], v[i + 7]));
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_acc_empty[ab]);
      ++n_acc;
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 5) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u) : "memory");
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_moe_gemm_tc(const void* x, int64_t x_stride, int32_t x_rows, const int32_t* src, const void* w,
                                  int32_t experts, const int32_t* off, const int32_t* tiles, int32_t max_tiles, int32_t n_out,
                                  int32_t k, int32_t act, float limit, void* out, int64_t out_stride, int32_t* status,
                                  void* stream) {
  MSA_REQUIRE(x && w && off && tiles && out && status && x_rows > 0 && experts > 0, "moe_gemm_tc: bad arguments");
  const int cols = act ? n_out / 2 : n_out;
  MSA_REQUIRE(n_out > 0 && k > 0 && k % 8 == 0 && cols % 8 == 0 && x_stride % 8 == 0 && out_stride % 8 == 0 &&
                  (!act || n_out % 2 == 0) && aligned16(x) && aligned16(w) && aligned16(out),
              "moe_gemm_tc: sizes and strides must be multiples of 8 elements, pointers 16-byte aligned");
  MSA_REQUIRE((long long)experts * n_out < (1ll << 31), "moe_gemm_tc: too many weight rows");
  if (max_tiles <= 0) return MSA_OK;
  CUtensorMap mx, mw;
  MSA_OK_OR_RETURN(make_map(&mx, x, x_rows, k, x_stride, kMtK, src ? 1 : kMtRows));
  MSA_OK_OR_RETURN(make_map(&mw, w, (uint64_t)experts * n_out, k, k, kMtK, 128));
  MoeTcParams p{src, off, tiles, max_tiles, act ? (cols + 127) / 128 : (cols + 255) / 256, (k + kMtK - 1) / kMtK, n_out, cols, limit,
                out, out_stride, status};
  int n_sm = 0;
  MSA_OK_OR_RETURN(device_sm_count(&n_sm));
  const long long work = (long long)max_tiles * p.n_nt;
  MSA_REQUIRE(work < (1ll << 31), "moe_gemm_tc: too many tiles");
  const unsigned grid = (unsigned)(work < n_sm ? work : n_sm);
  if (act) {
    static DeviceSmem s1{};
    MSA_OK_OR_RETURN(ensure_dynamic_smem(moe_gemm_tc_kernel<true>, kMtSmem, s1));
    moe_gemm_tc_kernel<true><<<grid, kMtThreads, kMtSmem, (cudaStream_t)stream>>>(mx, mw, p);
  } else {
    static DeviceSmem s0{};
    MSA_OK_OR_RETURN(ensure_dynamic_smem(moe_gemm_tc_kernel<false>, kMtSmem, s0));
    moe_gemm_tc_kernel<false><<<grid, kMtThreads, kMtSmem, (cudaStream_t)stream>>>(mx, mw, p);
  }
  MSA_LAUNCH_OK("moe_gemm_tc_kernel");
  return MSA_OK;
}
