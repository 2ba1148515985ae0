// Windowed attention of a prompt portion on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), bf16, for heads whose
// plain and rotated query / key parts and values are multiples of 64 wide.
//
// Work item = 256 consecutive query tokens of one head: two tiles of 128 rows that share every key / value tile on its
// way through shared memory.  One persistent CTA per SM, 320 threads: warps 0-3 the softmax of tile 0, 4-7 that of tile 1
// (thread = query row = TMEM lane), warp 8 the TMA producer, warp 9 the MMA issuer.  Per 64-key tile and query tile:
//     S = Q K^T    K-major operands; the key's plain part comes from the expanded keys of the head, its rotated part from
//                  the context row all heads share; fp32 into one of two 64-column TMEM buffers of the tile;
//     softmax      fp32, running maximum advanced only when it moved by more than 2^8; P as bf16 over the consumed columns;
//     O += P V     A = P from TMEM, B = V MN-major; O stays in TMEM.
// While one tile's softmax runs, the tensor pipe works for the other.  A query tile takes part only in the key tiles that
// its window reaches; inside them a 32-key chunk is fully visible, hidden, or cut for a warp.  Rows whose first tiles are
// hidden start from a finite reference maximum, so their exponentials are zero without a special case.
#include "lm_common.cuh"
#include "tc_attn_common.cuh"

namespace msa {

constexpr int kWaRows = 128, kWaTiles = 2, kWaKeys = 64;
constexpr int kWaThreads = 32 * (4 * kWaTiles + 2);
constexpr int kWaQBlk = kWaRows * 128;                    // one 64-column block of a query tile: 16 KB
constexpr int kWaKBlk = kWaKeys * 128;                    // one 64-column block of a key or value tile: 8 KB
constexpr int kWaStage = 32 * 64;                         // per softmax warp: 32 rows x 32 bf16 of output
constexpr uint32_t kWaTmem = 512;
constexpr float kWaRescale = 8.f;

struct WindowAttnTcParams {
  const int32_t *start, *cu, *ctx_off;   // ctx_off counts from seq0
  int seq0, heads, window;
  int q_row0;                            // packed row of the first query row of the map
  int q_head, k_head, v_head;            // column strides of a head
  int group;                             // query heads per key / value head
  int sink;                              // one more entry per softmax, with score 0 and no value
  const __nv_bfloat16* gate; long long gate_row;   // null, or one logit per row and head
  float scale_log2e;
  long long n_sh, n_items;               // sequences * heads; times the row blocks of the longest portion
  __nv_bfloat16* out; long long out_row;
  int32_t* status;
};

// Items are numbered from every portion's last row block to its first: the late ones see the most keys, and the
// fixed-stride walk of the persistent CTAs then ends on short ones.
struct WaItem { int len, r0, h, q_row, k_row, old, n_kt, a[kWaTiles], b[kWaTiles]; bool valid; };
__device__ __forceinline__ WaItem wa_item(const WindowAttnTcParams& p, long long w) {
  WaItem it;
  const int x = (int)(w / p.n_sh);
  const long long sh = w % p.n_sh;
  it.h = (int)(sh % p.heads);
  const int ps = (int)(sh / p.heads), s = p.seq0 + ps;
  const int c0 = p.cu[s];
  it.len = p.cu[s + 1] - c0;
  const int n_mb = (it.len + kWaRows * kWaTiles - 1) / (kWaRows * kWaTiles);
  it.valid = x < n_mb;
  it.r0 = (n_mb - 1 - x) * kWaRows * kWaTiles;
  it.old = min(p.start[s], p.window - 1);
  it.q_row = c0 - p.q_row0 + it.r0;
  const int j_lo = max(0, it.old + it.r0 - p.window + 1);
  it.k_row = p.ctx_off[ps] + j_lo;
  it.n_kt = 0;
#pragma unroll
  for (int q = 0; q < kWaTiles; ++q) {
    const int first = it.r0 + q * kWaRows, last = min(first + kWaRows, it.len) - 1;
    it.a[q] = it.b[q] = 0;
    if (first < it.len) {
      it.a[q] = (max(0, it.old + first - p.window + 1) - j_lo) / kWaKeys;
      it.b[q] = (it.old + last - j_lo) / kWaKeys + 1;
      it.n_kt = max(it.n_kt, it.b[q]);
    }
  }
  it.old -= j_lo;      // from here on: context index of row r relative to the item's first key = old + r
  return it;
}

template <int DB, int RB, int VB>
__global__ void __launch_bounds__(kWaThreads, 1)
window_attn_tc_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                      const __grid_constant__ CUtensorMap tmap_r, const __grid_constant__ CUtensorMap tmap_v,
                      const WindowAttnTcParams p) {
  constexpr int QB = DB + RB;
  constexpr int kStage = (QB + VB) * kWaKBlk;
  constexpr uint32_t kColO = kWaTiles * 2 * kWaKeys;
  static_assert(kColO + kWaTiles * VB * 64 <= kWaTmem, "TMEM columns");
  extern __shared__ unsigned char smem_dyn[];
  __shared__ uint64_t s_q_full, s_q_empty, s_k_full[2], s_k_empty[2], s_v_full[2], s_v_empty[2], s_drain;
  __shared__ uint64_t s_s_full[kWaTiles][2], s_p_full[kWaTiles][2], s_o_full[kWaTiles][2];
  __shared__ uint32_t s_tmem_base;
  __shared__ int s_abort;

  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  unsigned char* tiles = reinterpret_cast<unsigned char*>(((uintptr_t)smem_dyn + 1023) & ~(uintptr_t)1023);
  unsigned char* q_smem = tiles;
  unsigned char* kv_smem = tiles + kWaTiles * QB * kWaQBlk;
  unsigned char* out_stage = kv_smem + 2 * kStage;
  volatile int* abort_flag = &s_abort;

  if (threadIdx.x == 0) {
    mbar_init(&s_q_full, 1); mbar_init(&s_q_empty, 1); mbar_init(&s_drain, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_k_full[i], 1); mbar_init(&s_k_empty[i], 1);
      mbar_init(&s_v_full[i], 1); mbar_init(&s_v_empty[i], 1);
      for (int q = 0; q < kWaTiles; ++q) {
        mbar_init(&s_s_full[q][i], 1);
        mbar_init(&s_p_full[q][i], 4);
        mbar_init(&s_o_full[q][i], 1);
      }
    }
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 4 * kWaTiles + 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem_base)),
                 "r"(kWaTmem) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = s_tmem_base;

  // Every role walks the same items.  n_t counts the CTA's key tiles (stage and phase of the K / V barriers), n_c[q] the
  // tiles query tile q took part in (buffer and phase of its S / P / O barriers), n_it the items (the query buffer).
  if (warp == 4 * kWaTiles) {
    if (lane == 0) {
      uint32_t n_it = 0, n_t = 0;
      bool ok = true;
      for (long long w = blockIdx.x; w < p.n_items && ok; w += gridDim.x) {
        const WaItem it = wa_item(p, w);
        if (!it.valid) continue;
        if (!(ok = mbar_wait(&s_q_empty, (n_it & 1u) ^ 1u, abort_flag, p.status, 1))) break;
        mbar_expect_tx(&s_q_full, kWaTiles * QB * kWaQBlk);
#pragma unroll
        for (int q = 0; q < kWaTiles; ++q)
#pragma unroll
          for (int c = 0; c < QB; ++c)
            tma_load_2d(q_smem + (q * QB + c) * kWaQBlk, &tmap_q, it.h * p.q_head + 64 * c, it.q_row + q * kWaRows, &s_q_full);
        for (int t = 0; t < it.n_kt; ++t, ++n_t) {
          const uint32_t st = n_t & 1u, ph = (n_t >> 1) & 1u;
          unsigned char* ks = kv_smem + st * kStage;
          const int y = it.k_row + t * kWaKeys;
          if (!(ok = mbar_wait(&s_k_empty[st], ph ^ 1u, abort_flag, p.status, 1))) break;
          mbar_expect_tx(&s_k_full[st], QB * kWaKBlk);
#pragma unroll
          for (int c = 0; c < DB; ++c) tma_load_2d(ks + c * kWaKBlk, &tmap_k, it.h / p.group * p.k_head + 64 * c, y, &s_k_full[st]);
#pragma unroll
          for (int c = 0; c < RB; ++c) tma_load_2d(ks + (DB + c) * kWaKBlk, &tmap_r, 64 * c, y, &s_k_full[st]);
          if (!(ok = mbar_wait(&s_v_empty[st], ph ^ 1u, abort_flag, p.status, 1))) break;
          mbar_expect_tx(&s_v_full[st], VB * kWaKBlk);
#pragma unroll
          for (int c = 0; c < VB; ++c)
            tma_load_2d(ks + (QB + c) * kWaKBlk, &tmap_v, it.h / p.group * p.v_head + 64 * c, y, &s_v_full[st]);
        }
        ++n_it;
      }
      if (!ok) {   // gave up: give the copies already issued time to land before shared memory is released
        const unsigned long long w0 = global_ns();
        while (global_ns() - w0 < 1000000ull) {}
      }
    }
  } else if (warp == 4 * kWaTiles + 1) {
    if (lane == 0) {
      const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kWaKeys >> 3) << 17) | ((uint32_t)(kWaRows >> 4) << 24);
      const uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VB * 64 >> 3) << 17) |
                                ((uint32_t)(kWaRows >> 4) << 24);
      const uint32_t qa = smem_u32(q_smem), kva = smem_u32(kv_smem);
      uint32_t n_it = 0, n_t = 0, n_s[kWaTiles] = {}, n_p[kWaTiles] = {};   // n_s / n_p: S and PV tiles issued so far
      bool ok = true;
      auto issue_s = [&](uint32_t g, int q) {       // S of the CTA's key tile g for query tile q
        const uint32_t ka = kva + (g & 1u) * kStage, sb = n_s[q] & 1u;
#pragma unroll
        for (int c = 0; c < QB; ++c) {
          const uint64_t a_desc = make_smem_desc(qa + (q * QB + c) * kWaQBlk), b_desc = make_smem_desc(ka + c * kWaKBlk);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            tc_mma_bf16(tmem_base + (uint32_t)(q * 2 * kWaKeys) + sb * kWaKeys, a_desc + (uint64_t)(2 * k), b_desc + (uint64_t)(2 * k),
                        idesc_s, (c > 0 || k > 0) ? 1u : 0u);
        }
        tc_commit(&s_s_full[q][sb]);
        ++n_s[q];
      };
      auto wait_k = [&](uint32_t g) {
        const bool r = mbar_wait(&s_k_full[g & 1u], (g >> 1) & 1u, abort_flag, p.status, 3);
        tc_fence_after();
        return r;
      };
      for (long long w = blockIdx.x; w < p.n_items && ok; w += gridDim.x) {
        const WaItem it = wa_item(p, w);
        if (!it.valid) continue;
        if (!(ok = mbar_wait(&s_q_full, n_it & 1u, abort_flag, p.status, 2))) break;
        for (int t = 0; t < 2 && t < it.n_kt && ok; ++t) {     // two key tiles of S run ahead of the softmax
          if (!(ok = wait_k(n_t + t))) break;
#pragma unroll
          for (int q = 0; q < kWaTiles; ++q)
            if (t >= it.a[q] && t < it.b[q]) issue_s(n_t + t, q);
          tc_commit(&s_k_empty[(n_t + t) & 1u]);
          if (t + 1 == it.n_kt) tc_commit(&s_q_empty);
        }
        if (!ok) break;
        for (int t = 0; t < it.n_kt; ++t, ++n_t) {
          const uint32_t st = n_t & 1u, ph = (n_t >> 1) & 1u;
          const bool more = t + 2 < it.n_kt;
          if (!(ok = mbar_wait(&s_v_full[st], ph, abort_flag, p.status, 3))) break;
          const uint32_t va = kva + st * kStage + QB * kWaKBlk;
          bool have_k = false;
#pragma unroll
          for (int q = 0; q < kWaTiles; ++q) {
            if (t >= it.a[q] && t < it.b[q]) {
              const uint32_t pb = n_p[q] & 1u;
              if (!(ok = mbar_wait(&s_p_full[q][pb], (n_p[q] >> 1) & 1u, abort_flag, p.status, 4))) break;
              tc_fence_after();
#pragma unroll
              for (int j = 0; j < kWaKeys / 16; ++j)
                tc_mma_bf16_ts(tmem_base + kColO + (uint32_t)(q * VB * 64), tmem_base + (uint32_t)(q * 2 * kWaKeys) + pb * kWaKeys + (uint32_t)(8 * j),
                               make_smem_desc_mn(va + j * 2048, kWaKBlk), idesc_pv, (t > it.a[q] || j > 0) ? 1u : 0u);
              tc_commit(&s_o_full[q][pb]);
              ++n_p[q];
            }
            if (q + 1 == kWaTiles) tc_commit(&s_v_empty[st]);
            if (more && t + 2 >= it.a[q] && t + 2 < it.b[q]) {   // in order behind the PV that read this S buffer
              if (!have_k && !(ok = wait_k(n_t + 2))) break;
              have_k = true;
              issue_s(n_t + 2, q);
            }
          }
          if (!ok) break;
          if (more) {
            if (!have_k && !(ok = wait_k(n_t + 2))) break;
            tc_commit(&s_k_empty[st]);
            if (t + 3 == it.n_kt) tc_commit(&s_q_empty);
          }
        }
        ++n_it;
      }
      tc_commit(&s_drain);
      const unsigned long long w0 = global_ns();
      while (!mbar_try_wait(&s_drain, 0) && global_ns() - w0 < kWaitLimitNs) {}
    }
  } else {
    const int q = warp / 4, wq = warp % 4;
    const uint32_t lane_base = tmem_base + ((uint32_t)(wq * 32) << 16);
    const uint32_t col_s = (uint32_t)(q * 2 * kWaKeys), col_o = kColO + (uint32_t)(q * VB * 64);
    uint32_t n_c = 0;
    bool ok = true;
    for (long long w = blockIdx.x; w < p.n_items && ok; w += gridDim.x) {
      const WaItem it = wa_item(p, w);
      if (!it.valid || it.a[q] == it.b[q]) continue;
      float m_ref = p.sink ? 0.f : -1e30f, l_run = p.sink ? 1.f : 0.f;
      const int row0 = it.r0 + q * kWaRows + wq * 32;          // first row of this warp
      for (int t = it.a[q]; t < it.b[q]; ++t, ++n_c) {
        const uint32_t sb = n_c & 1u;
        ok = mbar_wait(&s_s_full[q][sb], (n_c >> 1) & 1u, abort_flag, p.status, 5);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        const uint32_t s_addr = lane_base + col_s + sb * kWaKeys;
        uint32_t va[32], vb[32];
        tmem_ld32(s_addr, va);
        tmem_ld32(s_addr + 32, vb);
        // Key i of a chunk is visible to lane r iff r + d - window < i <= r + d, d = (index of the warp's first row) -
        // (index of the chunk's first key).
        const int d0 = it.old + row0 - t * kWaKeys;
        tmem_ld_wait();
        int cls[2];
        auto cut = [&](uint32_t (&v)[32], int d, int& c) {
          if (d + 31 < 0 || d - p.window >= 31) { c = 0; return; }
          c = 2;
          if (d >= 31 && d + 31 - p.window < 0) return;
          const int hi = lane + d, lo = lane + d - p.window;
#pragma unroll
          for (int i = 0; i < 32; ++i) if (i > hi || i <= lo) v[i] = 0xff800000u;
        };
        cut(va, d0, cls[0]);
        cut(vb, d0 - 32, cls[1]);
        float mx = -INFINITY, mx2 = -INFINITY;
        if (cls[0]) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            mx = max3(mx, __uint_as_float(va[i]), __uint_as_float(va[i + 1]));
            mx2 = max3(mx2, __uint_as_float(va[i + 2]), __uint_as_float(va[i + 3]));
          }
        }
        if (cls[1]) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            mx = max3(mx, __uint_as_float(vb[i]), __uint_as_float(vb[i + 1]));
            mx2 = max3(mx2, __uint_as_float(vb[i + 2]), __uint_as_float(vb[i + 3]));
          }
        }
        mx = fmaxf(mx, mx2);
        const bool move = (mx - m_ref) * p.scale_log2e > kWaRescale;
        if (__any_sync(0xffffffffu, move)) {
          const float f = move ? exp2f((m_ref - mx) * p.scale_log2e) : 1.f;
          if (t > it.a[q]) {   // wait for the PV in flight, then rescale this warp's rows of O in place
            ok = mbar_wait(&s_o_full[q][(n_c - 1u) & 1u], ((n_c - 1u) >> 1) & 1u, abort_flag, p.status, 6);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
#pragma unroll
            for (int c = 0; c < VB * 4; ++c) {
              uint32_t v[16];
              tmem_ld16(lane_base + col_o + 16 * c, v);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * f);
              tmem_st16(lane_base + col_o + 16 * c, v);
            }
          }
          l_run *= f;
          if (move) m_ref = mx;
        }
        const float neg_m = -m_ref * p.scale_log2e;
        unsigned long long sum_a = 0ull, sum_b = 0ull;
        const unsigned long long scale2 = f32x2(p.scale_log2e, p.scale_log2e), neg_m2 = f32x2(neg_m, neg_m);
        uint32_t pk[16];
        auto exps = [&](const uint32_t (&v)[32], int c) {
          if (c == 0) {
#pragma unroll
            for (int i = 0; i < 16; ++i) pk[i] = 0u;
            return;
          }
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            float x0, x1, x2, x3;
            f32x2_split(fma_f32x2(f32x2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), scale2, neg_m2), x0, x1);
            f32x2_split(fma_f32x2(f32x2(__uint_as_float(v[i + 2]), __uint_as_float(v[i + 3])), scale2, neg_m2), x2, x3);
            const float e0 = ex2_approx(x0), e1 = ex2_approx(x1), e2 = ex2_approx(x2), e3 = ex2_approx(x3);
            sum_a = add_f32x2(sum_a, f32x2(e0, e1));
            sum_b = add_f32x2(sum_b, f32x2(e2, e3));
            pk[i >> 1] = pack2_bf16(e0, e1);
            pk[(i >> 1) + 1] = pack2_bf16(e2, e3);
          }
        };
        exps(va, cls[0]);
        tmem_st16(s_addr, pk);
        exps(vb, cls[1]);
        tmem_st16(s_addr + 16, pk);
        {
          float s0, s1, s2, s3;
          f32x2_split(sum_a, s0, s1);
          f32x2_split(sum_b, s2, s3);
          l_run += (s0 + s1) + (s2 + s3);
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&s_p_full[q][sb]);
      }
      if (!ok) break;
      ok = mbar_wait(&s_o_full[q][(n_c - 1u) & 1u], ((n_c - 1u) >> 1) & 1u, abort_flag, p.status, 6);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      float inv = 1.f / l_run;
      if (p.gate && row0 + lane < it.len)
        inv *= sigmoid_f(__bfloat162float(p.gate[(it.q_row + q * kWaRows + wq * 32 + lane) * p.gate_row + it.h]));
      unsigned char* stg = out_stage + warp * kWaStage;
      __nv_bfloat16* dst0 = p.out + (long long)(it.q_row + q * kWaRows + wq * 32) * p.out_row + (long long)it.h * VB * 64;
#pragma unroll
      for (int c = 0; c < VB * 2; ++c) {
        uint32_t v[32];
        tmem_ld32(lane_base + col_o + 32 * c, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          uint4 o;
          o.x = pack2_bf16(__uint_as_float(v[8 * i]) * inv, __uint_as_float(v[8 * i + 1]) * inv);
          o.y = pack2_bf16(__uint_as_float(v[8 * i + 2]) * inv, __uint_as_float(v[8 * i + 3]) * inv);
          o.z = pack2_bf16(__uint_as_float(v[8 * i + 4]) * inv, __uint_as_float(v[8 * i + 5]) * inv);
          o.w = pack2_bf16(__uint_as_float(v[8 * i + 6]) * inv, __uint_as_float(v[8 * i + 7]) * inv);
          *reinterpret_cast<uint4*>(stg + lane * 64 + ((i ^ ((lane >> 1) & 3)) << 4)) = o;
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int r = (lane >> 2) + 8 * i, piece = lane & 3;
          const uint4 o = *reinterpret_cast<const uint4*>(stg + r * 64 + ((piece ^ ((r >> 1) & 3)) << 4));
          if (row0 + r < it.len) *reinterpret_cast<uint4*>(dst0 + (long long)r * p.out_row + 32 * c + 8 * piece) = o;
        }
        __syncwarp();
      }
      tc_fence_before();
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 4 * kWaTiles + 1)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(kWaTmem) : "memory");
}

template <int DB, int RB, int VB>
int launch_window_attn_tc(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& r, const CUtensorMap& v,
                          const WindowAttnTcParams& p, cudaStream_t stream) {
  constexpr size_t smem = (size_t)kWaTiles * (DB + RB) * kWaQBlk + 2 * (DB + RB + VB) * kWaKBlk + 4 * kWaTiles * kWaStage + 1024;
  static_assert(smem <= 227 * 1024, "shared memory");
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(window_attn_tc_kernel<DB, RB, VB>, smem, configured));
  int n_sm = 0;
  MSA_OK_OR_RETURN(device_sm_count(&n_sm));
  const long long grid = p.n_items < n_sm ? p.n_items : n_sm;
  window_attn_tc_kernel<DB, RB, VB><<<(unsigned)grid, kWaThreads, smem, stream>>>(q, k, r, v, p);
  MSA_LAUNCH_OK("window_attn_tc_kernel");
  return MSA_OK;
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_window_attn_tc_supported(int32_t dim, int32_t rot, int32_t vdim) {
  return (dim == 64 || dim == 128) && (rot == 0 || rot == 64) && (vdim == 64 || vdim == 128);
}

extern "C" int msa_lm_window_attn_tc(const msa_lm_attn_args* args, int32_t n_rows, int32_t n_ctx, int32_t row0, int32_t* status, void* stream) {
  MSA_REQUIRE(args, "window_attn_tc: null arguments");
  const msa_lm_attn_args a = *args;
  const int dim = a.da, rot = a.db, vdim = a.dv;
  MSA_REQUIRE(a.qa && a.ka && a.v && a.start && a.cu && a.ctx_off && a.out && status && a.ring_rows == 0, "window_attn_tc: null pointer");
  MSA_REQUIRE(a.dtype == MSA_BF16 && a.qa_dtype == MSA_BF16 && a.out_dtype == MSA_BF16, "window_attn_tc: bf16 only");
  MSA_REQUIRE(msa_lm_window_attn_tc_supported(dim, rot, vdim), "window_attn_tc: unsupported head sizes (%d, %d, %d)", dim, rot, vdim);
  MSA_REQUIRE(a.heads > 0 && a.window > 0 && a.scale > 0.f && a.group > 0 && a.heads % a.group == 0, "window_attn_tc: bad sizes");
  MSA_REQUIRE(rot == 0 || (a.kb && a.kb_head == 0 && a.qb == (const __nv_bfloat16*)a.qa + dim && a.qb_head == a.qa_head),
              "window_attn_tc: the rotated parts must follow the plain query part and be shared by the keys");
  MSA_REQUIRE(aligned16(a.qa) && aligned16(a.ka) && aligned16(a.v) && aligned16(a.out) && (rot == 0 || aligned16(a.kb)) &&
                  a.qa_row % 8 == 0 && a.ka_row % 8 == 0 && a.v_row % 8 == 0 && a.out_row % 8 == 0 && a.kb_row % 8 == 0 &&
                  a.qa_head % 8 == 0 && a.ka_head % 8 == 0 && a.v_head % 8 == 0 && a.out_head == vdim, "window_attn_tc: rows must be 16-byte aligned");
  if (a.seq1 <= a.seq0 || a.max_len <= 0 || n_rows <= 0) return MSA_OK;
  const int kv_heads = a.heads / a.group;
  CUtensorMap mq, mk, mr, mv;
  MSA_OK_OR_RETURN(make_map(&mq, a.qa, n_rows, (uint64_t)(a.heads - 1) * a.qa_head + dim + rot, a.qa_row, 64, kWaRows));
  MSA_OK_OR_RETURN(make_map(&mk, a.ka, n_ctx, (uint64_t)(kv_heads - 1) * a.ka_head + dim, a.ka_row, 64, kWaKeys));
  MSA_OK_OR_RETURN(make_map(&mv, a.v, n_ctx, (uint64_t)(kv_heads - 1) * a.v_head + vdim, a.v_row, 64, kWaKeys));
  if (rot) MSA_OK_OR_RETURN(make_map(&mr, a.kb, n_ctx, (uint64_t)rot, a.kb_row, 64, kWaKeys));
  else mr = mk;
  WindowAttnTcParams p{};
  p.start = a.start; p.cu = a.cu; p.ctx_off = a.ctx_off;
  p.seq0 = a.seq0; p.heads = a.heads; p.window = a.window; p.q_row0 = row0;
  p.q_head = (int)a.qa_head; p.k_head = (int)a.ka_head; p.v_head = (int)a.v_head;
  p.group = a.group; p.sink = a.sink; p.gate = (const __nv_bfloat16*)a.gate; p.gate_row = a.gate_row;
  p.scale_log2e = a.scale * 1.4426950408889634f;
  p.n_sh = (long long)(a.seq1 - a.seq0) * a.heads;
  p.n_items = p.n_sh * ((a.max_len + kWaRows * kWaTiles - 1) / (kWaRows * kWaTiles));
  p.out = (__nv_bfloat16*)a.out; p.out_row = a.out_row; p.status = status;
  cudaStream_t st = (cudaStream_t)stream;
  const int key = (dim / 64) * 100 + (rot / 64) * 10 + vdim / 64;
  switch (key) {
    case 101: return launch_window_attn_tc<1, 0, 1>(mq, mk, mr, mv, p, st);
    case 102: return launch_window_attn_tc<1, 0, 2>(mq, mk, mr, mv, p, st);
    case 111: return launch_window_attn_tc<1, 1, 1>(mq, mk, mr, mv, p, st);
    case 112: return launch_window_attn_tc<1, 1, 2>(mq, mk, mr, mv, p, st);
    case 201: return launch_window_attn_tc<2, 0, 1>(mq, mk, mr, mv, p, st);
    case 202: return launch_window_attn_tc<2, 0, 2>(mq, mk, mr, mv, p, st);
    case 211: return launch_window_attn_tc<2, 1, 1>(mq, mk, mr, mv, p, st);
    default: return launch_window_attn_tc<2, 1, 2>(mq, mk, mr, mv, p, st);
  }
}
