// Decode attention over the latent ring, bf16: every head's query (key expansion folded in) against the same rows
// [latent | rotated key part]; the values are the latents themselves.  Flash-decode: the visible rows of a sequence are
// split over CTAs, partial results are merged by a second kernel.
//
// One CTA = up to 32 heads x one split, 256 threads; 64-row tiles of the ring are double-buffered, one bulk copy
// per row (rows are read once from HBM for all heads; a warp's worth of instructions per tile).  Scores and output run on mma.sync.m16n8k16.  For the scores the warps split the
// reduction: a warp keeps its slice of the queries in registers for the whole launch, multiplies all 64 rows by it, and
// the slices' partial scores are added up in shared memory, where eight (sixteen) threads per head do the fp32 softmax.
// For the output the warps split the latent columns.
#include "lm_common.cuh"
#include "lm_merge.cuh"
#include "mma_helpers.cuh"
#include "tc_attn_common.cuh"

namespace msa {

constexpr int kLdThreads = 256, kLdKeys = 64, kLdPPitch = 144;   // P rows: 64 bf16 + 16 bytes of padding

struct LatentDecodeParams {
  const __nv_bfloat16* qa; long long qa_row, qa_head;
  const __nv_bfloat16* qb; long long qb_row, qb_head;
  const __nv_bfloat16* ring; long long ring_rows;
  const int32_t *slot, *pos;
  int heads, rank, rot, window, splits;
  float scale_log2e;
  __nv_bfloat16* out;       // [n, heads, rank]
  float *part_o, *part_ml;  // [n, heads, splits, rank], [n, heads, splits, 2]
  int32_t* status;
};

__device__ __forceinline__ void mma_bf16_full(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// MT: 16-head tiles; NT: octets of latent columns per warp; KS: reduction steps of 16 per warp.
__device__ __forceinline__ void bulk_row(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

template <int MT, int NT, int KS>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(const LatentDecodeParams p) {
  constexpr int KQ = 8 / MT, kRows = MT * 16, kPart = 72;            // slices of the reduction; floats per partial row
  constexpr int TPR = kLdThreads / kRows, KPT = kLdKeys / TPR;       // softmax: threads per row, keys per thread
  extern __shared__ __align__(16) unsigned char sm[];
  __shared__ float s_corr[kRows], s_m[kRows], s_l[kRows];
  __shared__ uint64_t s_full[2];
  __shared__ int s_abort;
  const int width = p.rank + p.rot, pitch = width * 2 + 16, vecs = width / 8, steps = width / 16;
  float* s_part = reinterpret_cast<float*>(sm);                      // [KQ][kRows][kPart]
  unsigned char* s_p = sm + KQ * kRows * kPart * 4;                  // [kRows][kLdPPitch]
  unsigned char* s_k = s_p + kRows * kLdPPitch;                      // 2 x [64][pitch]
  const int b = blockIdx.z, h0 = blockIdx.y * kRows, split = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int pos = p.pos[b], lo = max(0, pos - p.window + 1), n_keys = pos - lo + 1;
  int chunk = (n_keys + p.splits - 1) / p.splits;
  chunk = (chunk + kLdKeys - 1) / kLdKeys * kLdKeys;
  const int k0 = split * chunk, k1 = min(n_keys, k0 + chunk);
  const int n_tiles = k1 > k0 ? (k1 - k0 + kLdKeys - 1) / kLdKeys : 0;
  const __nv_bfloat16* ring = p.ring + (long long)p.slot[b] * p.ring_rows * width;

  const int n_ring = (int)p.ring_rows, lo_row = lo % n_ring;
  const uint32_t k_base = (uint32_t)__cvta_generic_to_shared(s_k);
  const uint32_t row_bytes = (uint32_t)width * 2;
  auto load_tile = [&](int t) {             // eight rows per warp; rows past the split's end repeat its first one
    if (threadIdx.x == 0) mbar_expect_tx(&s_full[t & 1], kLdKeys * row_bytes);
    if (lane < kLdKeys / 8) {
      const int r = warp * (kLdKeys / 8) + lane, k = k0 + t * kLdKeys + r;
      int row = lo_row + (k < k1 ? k : k0);                                 // both terms are below the ring's size
      row = row >= n_ring ? row - n_ring : row;
      bulk_row(k_base + ((t & 1) * kLdKeys + r) * pitch, ring + (long long)row * width, row_bytes, &s_full[t & 1]);
    }
  };
  if (threadIdx.x == 0) {
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  if (n_tiles > 0) load_tile(0);
  grid_launch_dependents();
  const int mt = warp % MT, kq = warp / MT, ks0 = kq * KS;
  uint32_t q[KS][4];
#pragma unroll
  for (int i = 0; i < KS; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {                                           // (row g, g + 8) x (columns 2 tq, 2 tq + 8)
      const int h = h0 + mt * 16 + g + 8 * (e & 1), c = (ks0 + i) * 16 + tq * 2 + 8 * (e >> 1);
      uint32_t v = 0u;
      if (h < p.heads && ks0 + i < steps)
        v = c < p.rank ? *reinterpret_cast<const uint32_t*>(p.qa + b * p.qa_row + h * p.qa_head + c)
                       : *reinterpret_cast<const uint32_t*>(p.qb + b * p.qb_row + h * p.qb_head + (c - p.rank));
      q[i][e] = v;
    }
  const uint32_t p_addr = (uint32_t)__cvta_generic_to_shared(s_p) + (lane & 15) * kLdPPitch + (lane >> 4) * 16;
  const uint32_t b_off = ((lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 16 + ks0 * 32;
  const int srow = threadIdx.x / TPR, skey = threadIdx.x % TPR * KPT;       // the scores this thread looks after
  float m_run = -INFINITY, l_run = 0.f;
  float acc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
  for (int t = 0; t < n_tiles; ++t) {
    const bool there = mbar_wait(&s_full[t & 1], (t >> 1) & 1, &s_abort, p.status, 21);
    if (!__syncthreads_and(there)) {       // gave up: the copies in flight land before shared memory is released
      const unsigned long long w0 = global_ns();
      while (global_ns() - w0 < 1000000ull) {}
      return;
    }
    // the tile is there; the other buffer, the scores and P are free
    if (t + 1 < n_tiles) load_tile(t + 1);
    const uint32_t kb = k_base + (t & 1) * kLdKeys * pitch;
    float s[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
    for (int i = 0; i < KS; ++i) {
      if (ks0 + i >= steps) break;
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        uint32_t x[4];
        ldmatrix_x4(kb + b_off + j * 8 * pitch + i * 32, x[0], x[1], x[2], x[3]);
        mma_bf16_full(s[j], q[i], x[0], x[1]);
        mma_bf16_full(s[j + 1], q[i], x[2], x[3]);
      }
    }
    {
      float* dst = s_part + (kq * kRows + mt * 16 + g) * kPart + tq * 2;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        *reinterpret_cast<float2*>(dst + j * 8) = make_float2(s[j][0], s[j][1]);
        *reinterpret_cast<float2*>(dst + 8 * kPart + j * 8) = make_float2(s[j][2], s[j][3]);
      }
    }
    __syncthreads();
    {
      float x[KPT];
#pragma unroll
      for (int i = 0; i < KPT; ++i) x[i] = 0.f;
#pragma unroll
      for (int w = 0; w < KQ; ++w)
#pragma unroll
        for (int i = 0; i < KPT; i += 4) {
          const float4 v = load4(s_part + (w * kRows + srow) * kPart + skey + i);
          x[i] += v.x; x[i + 1] += v.y; x[i + 2] += v.z; x[i + 3] += v.w;
        }
      if (t + 1 == n_tiles) {
        const int valid = k1 - k0 - t * kLdKeys - skey;
#pragma unroll
        for (int i = 0; i < KPT; ++i) x[i] = i < valid ? x[i] : -INFINITY;
      }
      float m = x[0];
#pragma unroll
      for (int i = 1; i < KPT; ++i) m = fmaxf(m, x[i]);
      m = fmaxf(m_run, m * p.scale_log2e);     // the scale is positive
#pragma unroll
      for (int o = 1; o < TPR; o <<= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float corr = ex2_approx(m_run - m);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) { x[i] = ex2_approx(fmaf(x[i], p.scale_log2e, -m)); sum += x[i]; }
      l_run = l_run * corr + sum;          // this thread's keys alone; added up at the end
      m_run = m;
      uint32_t* dst = reinterpret_cast<uint32_t*>(s_p + srow * kLdPPitch + skey * 2);
#pragma unroll
      for (int i = 0; i < KPT; i += 4) *reinterpret_cast<uint2*>(dst + i / 2) = make_uint2(pack_bf16(x[i], x[i + 1]), pack_bf16(x[i + 2], x[i + 3]));
      if (skey == 0) s_corr[srow] = corr;
    }
    __syncthreads();
    float corr[MT][2];
    bool same = true;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) { corr[i][e] = s_corr[i * 16 + g + 8 * e]; same = same && corr[i][e] == 1.f; }
    if (!__all_sync(0xffffffffu, same)) {
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          acc[i][j][0] *= corr[i][0]; acc[i][j][1] *= corr[i][0];
          acc[i][j][2] *= corr[i][1]; acc[i][j][3] *= corr[i][1];
        }
    }
    const uint32_t v_addr = kb + ((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (warp * 8 * NT + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int k = 0; k < kLdKeys; k += 16) {
      uint32_t a[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmatrix_x4(p_addr + i * 16 * kLdPPitch + k * 2, a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t v[4];
        ldmatrix_x4_trans(v_addr + k * pitch + j * 16, v[0], v[1], v[2], v[3]);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16_full(acc[i][j], a[i], v[0], v[1]);
          mma_bf16_full(acc[i][j + 1], a[i], v[2], v[3]);
        }
      }
    }
  }
#pragma unroll
  for (int o = 1; o < TPR; o <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, o);
  if (skey == 0) { s_m[srow] = m_run; s_l[srow] = l_run; }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = i * 16 + g + 8 * e, h = h0 + r;
      if (h >= p.heads) continue;
      const long long row = (long long)b * p.heads + h;
      if (p.splits == 1) {
        const float inv = 1.f / s_l[r];
#pragma unroll
        for (int j = 0; j < NT; ++j)
          *reinterpret_cast<uint32_t*>(p.out + row * p.rank + warp * 8 * NT + j * 8 + tq * 2) =
              pack_bf16(acc[i][j][2 * e] * inv, acc[i][j][2 * e + 1] * inv);
      } else {
        float* o = p.part_o + (row * p.splits + split) * p.rank + warp * 8 * NT + tq * 2;
#pragma unroll
        for (int j = 0; j < NT; ++j) *reinterpret_cast<float2*>(o + j * 8) = make_float2(acc[i][j][2 * e], acc[i][j][2 * e + 1]);
        if (warp == 0 && tq == 0) {
          p.part_ml[(row * p.splits + split) * 2] = s_m[r];
          p.part_ml[(row * p.splits + split) * 2 + 1] = s_l[r];
        }
      }
    }
}

template <int MT, int NT>
int launch_latent_decode(const LatentDecodeParams& p, int n, cudaStream_t stream) {
  constexpr int KQ = 8 / MT, KS = (NT * 4 + 4 + KQ - 1) / KQ;               // up to 64 rotated columns
  const size_t pitch = (size_t)(p.rank + p.rot) * 2 + 16;
  const size_t smem = (size_t)KQ * MT * 16 * 72 * 4 + (size_t)MT * 16 * kLdPPitch + 2 * kLdKeys * pitch;
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(latent_decode_kernel<MT, NT, KS>, smem, configured));
  const dim3 grid((unsigned)p.splits, (unsigned)((p.heads + MT * 16 - 1) / (MT * 16)), (unsigned)n);
  latent_decode_kernel<MT, NT, KS><<<grid, kLdThreads, smem, stream>>>(p);
  MSA_LAUNCH_OK("latent_decode_kernel");
  if (p.splits > 1) {
    const MergeParams m{p.part_o, p.part_ml, p.heads, p.splits, p.rank, 0, nullptr, 0, p.out, (long long)p.heads * p.rank};
    return launch_merge(m, n, stream);
  }
  return MSA_OK;
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_latent_decode_supported(int32_t rank, int32_t rot) {
  return rank >= 128 && rank <= 512 && rank % 128 == 0 && rot % 32 == 0 && rot >= 0 && rot <= 64;
}

extern "C" int msa_lm_latent_decode(const void* qa, int64_t qa_row, int64_t qa_head, const void* qb, int64_t qb_row,
                                    int64_t qb_head, const void* ring, int64_t ring_rows, const int32_t* slot,
                                    const int32_t* pos, int32_t n, int32_t heads, int32_t rank, int32_t rot, int32_t window,
                                    int32_t splits, float scale, void* out, float* part_o, float* part_ml, int32_t* status, void* stream) {
  MSA_REQUIRE(qa && ring && slot && pos && out && status && (rot == 0 || qb), "latent_decode: null pointer");
  MSA_REQUIRE(msa_lm_latent_decode_supported(rank, rot) && heads > 0 && window > 0 && scale > 0.f && ring_rows > 0 && ring_rows < (1ll << 30), "latent_decode: bad sizes");
  MSA_REQUIRE(splits >= 1 && splits <= 64 && (splits == 1 || (part_o && part_ml)), "latent_decode: bad splits");
  MSA_REQUIRE(aligned16(qa) && aligned16(ring) && aligned16(out) && (rot == 0 || aligned16(qb)) && qa_row % 8 == 0 &&
                  qa_head % 8 == 0 && qb_row % 8 == 0 && qb_head % 8 == 0, "latent_decode: rows must be 16-byte aligned");
  if (n <= 0) return MSA_OK;
  LatentDecodeParams p{(const __nv_bfloat16*)qa, qa_row, qa_head, (const __nv_bfloat16*)qb, qb_row, qb_head,
                       (const __nv_bfloat16*)ring, ring_rows, slot, pos, heads, rank, rot, window, splits,
                       scale * 1.4426950408889634f, (__nv_bfloat16*)out, part_o, part_ml, status};
  cudaStream_t st = (cudaStream_t)stream;
  if (heads <= 16) {
    switch (rank) {
      case 128: return launch_latent_decode<1, 2>(p, n, st);
      case 256: return launch_latent_decode<1, 4>(p, n, st);
      case 384: return launch_latent_decode<1, 6>(p, n, st);
      default: return launch_latent_decode<1, 8>(p, n, st);
    }
  }
  switch (rank) {
    case 128: return launch_latent_decode<2, 2>(p, n, st);
    case 256: return launch_latent_decode<2, 4>(p, n, st);
    case 384: return launch_latent_decode<2, 6>(p, n, st);
    default: return launch_latent_decode<2, 8>(p, n, st);
  }
}
