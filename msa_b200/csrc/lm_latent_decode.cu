// Decode attention over the latent ring, bf16: every head's query (key expansion folded in) against the same rows
// [latent | rotated key part]; the values are the latents themselves.  Flash-decode: the visible rows of a sequence are
// split over CTAs, partial results are merged by a second kernel.
//
// One CTA = up to 32 heads x one split, 512 threads.  The queries stay in shared memory; 64-row tiles of the ring are
// double-buffered with cp.async (rows are read once from HBM for all heads, which is what bounds this kernel); scores and
// output on mma.sync.m16n8k16, softmax in fp32.  Warps split the scores over octets of keys and the two 16-head tiles (with
// one head tile: over the two halves of the reduction), and the output over latent columns.
#include "lm_common.cuh"
#include "mma_helpers.cuh"

namespace msa {

constexpr int kLdThreads = 512, kLdKeys = 64, kLdPPitch = 144;   // P rows: 64 bf16 + 16 bytes of padding

struct LatentDecodeParams {
  const __nv_bfloat16* qa; long long qa_row, qa_head;
  const __nv_bfloat16* qb; long long qb_row, qb_head;
  const __nv_bfloat16* ring; long long ring_rows;
  const int32_t *slot, *pos;
  int heads, rank, rot, window, splits;
  float scale_log2e;
  __nv_bfloat16* out;       // [n, heads, rank]
  float *part_o, *part_ml;  // [n, heads, splits, rank], [n, heads, splits, 2]
};

__device__ __forceinline__ void mma_bf16_full(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}

// MT: 16-head tiles; NT: octets of latent columns per warp (rank / 128).
template <int MT, int NT>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(const LatentDecodeParams p) {
  extern __shared__ __align__(16) unsigned char sm[];
  __shared__ float s_max[8][32], s_sum[8][32];
  __shared__ float4 s_half[MT == 1 ? 256 : 1];      // one head tile: scores of the second half of the reduction
  constexpr int kParts = 8;                         // octets of keys of a tile
  const int width = p.rank + p.rot, pitch = width * 2 + 16, vecs = width / 8;
  unsigned char* s_q = sm;                          // [MT*16][pitch]
  unsigned char* s_p = s_q + MT * 16 * pitch;       // [MT*16][kLdPPitch]
  unsigned char* s_k = s_p + MT * 16 * kLdPPitch;   // 2 x [64][pitch]
  const int b = blockIdx.z, h0 = blockIdx.y * MT * 16, split = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.pos[b], lo = max(0, pos - p.window + 1), n_keys = pos - lo + 1;
  int chunk = (n_keys + p.splits - 1) / p.splits;
  chunk = (chunk + kLdKeys - 1) / kLdKeys * kLdKeys;
  const int k0 = split * chunk, k1 = min(n_keys, k0 + chunk);
  const int n_tiles = k1 > k0 ? (k1 - k0 + kLdKeys - 1) / kLdKeys : 0;
  const __nv_bfloat16* ring = p.ring + (long long)p.slot[b] * p.ring_rows * width;

  const int n_ring = (int)p.ring_rows, lo_row = lo % n_ring;
  const uint32_t k_base = (uint32_t)__cvta_generic_to_shared(s_k);
  auto load_tile = [&](int t) {
    const uint32_t dst = k_base + (t & 1) * kLdKeys * pitch;
#pragma unroll 4
    for (int r = threadIdx.x >> 5; r < kLdKeys; r += kLdThreads / 32) {     // a warp per row
      const int k = k0 + t * kLdKeys + r;
      const uint32_t bytes = k < k1 ? 16u : 0u;
      int row = lo_row + k;                                                 // both terms are below the ring's size
      row = k < k1 ? (row >= n_ring ? row - n_ring : row) : 0;
      const __nv_bfloat16* src = ring + (long long)row * width;
      for (int c = threadIdx.x & 31; c < vecs; c += 32) cp_async16(dst + r * pitch + c * 16, src + c * 8, bytes);
    }
    cp_async_commit();
  };
  if (n_tiles > 0) load_tile(0);
  for (int i = threadIdx.x; i < MT * 16 * vecs; i += kLdThreads) {
    const int r = i / vecs, c = (i - r * vecs) * 8, h = h0 + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h < p.heads)
      v = c < p.rank ? *reinterpret_cast<const uint4*>(p.qa + b * p.qa_row + h * p.qa_head + c)
                     : *reinterpret_cast<const uint4*>(p.qb + b * p.qb_row + h * p.qb_head + (c - p.rank));
    *reinterpret_cast<uint4*>(s_q + r * pitch + c * 2) = v;
  }
  const int mt = MT == 2 ? warp & 1 : 0, part = MT == 2 ? warp >> 1 : warp & 7, half = MT == 2 ? 0 : warp >> 3;
  const int steps = width / 32, ks0 = half == 0 ? 0 : steps / 2 * 32, ks1 = MT == 1 && half == 0 ? steps / 2 * 32 : width;
  const int g = lane >> 2, tq = lane & 3;
  const uint32_t q_addr = (uint32_t)__cvta_generic_to_shared(s_q) + (mt * 16 + (lane & 15)) * pitch + (lane >> 4) * 16;
  const uint32_t p_addr = (uint32_t)__cvta_generic_to_shared(s_p) + (lane & 15) * kLdPPitch + (lane >> 4) * 16;
  // scores: keys 8*part .. +7 of the tile, two reduction steps per load
  const int brow = part * 8 + (lane & 7), bcol = (lane >> 3) * 16;
  float acc[MT][NT][4];
  float m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    m_run[i][0] = m_run[i][1] = -INFINITY;
    l_run[i][0] = l_run[i][1] = 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
  }
  for (int t = 0; t < n_tiles; ++t) {
    if (t + 1 < n_tiles) { load_tile(t + 1); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();
    const uint32_t kb = (uint32_t)__cvta_generic_to_shared(s_k + (t & 1) * kLdKeys * pitch);
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};            // two chains, added below
    const uint32_t b_addr = kb + brow * pitch + bcol;
#pragma unroll 3
    for (int k = ks0; k < ks1; k += 32) {
      uint32_t a[4], a2[4], x[4];
      ldmatrix_x4(q_addr + k * 2, a[0], a[1], a[2], a[3]);
      ldmatrix_x4(q_addr + k * 2 + 32, a2[0], a2[1], a2[2], a2[3]);
      ldmatrix_x4(b_addr + k * 2, x[0], x[1], x[2], x[3]);
      mma_bf16_full(s, a, x[0], x[1]);
      mma_bf16_full(s2, a2, x[2], x[3]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] += s2[e];
    if constexpr (MT == 1) {
      if (half == 1) s_half[part * 32 + lane] = make_float4(s[0], s[1], s[2], s[3]);
      __syncthreads();
      if (half == 0) {
        const float4 o = s_half[part * 32 + lane];
        s[0] += o.x; s[1] += o.y; s[2] += o.z; s[3] += o.w;
      }
    }
    // s[0..1]: row g, keys 8*part + 2*tq, +1; s[2..3]: row g+8
    const int valid = k1 - k0 - t * kLdKeys;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = part * 8 + tq * 2 + (e & 1);
      s[e] = key < valid ? s[e] * p.scale_log2e : -INFINITY;
      mx[e >> 1] = fmaxf(mx[e >> 1], s[e]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
    }
    if (half == 0 && tq == 0) { s_max[part][mt * 16 + g] = mx[0]; s_max[part][mt * 16 + g + 8] = mx[1]; }
    __syncthreads();
    // every thread follows the running maximum of all rows it accumulates output for
    float corr[MT][2];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float m = m_run[i][e];
#pragma unroll
        for (int w = 0; w < kParts; ++w) m = fmaxf(m, s_max[w][i * 16 + g + 8 * e]);
        corr[i][e] = exp2f(m_run[i][e] - m);
        m_run[i][e] = m;
      }
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float m = (MT == 1 || mt == 0) ? m_run[0][e] : m_run[MT - 1][e];
      const float x0 = exp2f(s[2 * e] - m), x1 = exp2f(s[2 * e + 1] - m);
      sum[e] = x0 + x1;
      if (half == 0) *reinterpret_cast<uint32_t*>(s_p + (mt * 16 + g + 8 * e) * kLdPPitch + (part * 8 + tq * 2) * 2) = pack_bf16(x0, x1);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
      sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
    }
    if (half == 0 && tq == 0) { s_sum[part][mt * 16 + g] = sum[0]; s_sum[part][mt * 16 + g + 8] = sum[1]; }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float l = l_run[i][e] * corr[i][e];
#pragma unroll
        for (int w = 0; w < kParts; ++w) l += s_sum[w][i * 16 + g + 8 * e];
        l_run[i][e] = l;
      }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        acc[i][j][0] *= corr[i][0]; acc[i][j][1] *= corr[i][0];
        acc[i][j][2] *= corr[i][1]; acc[i][j][3] *= corr[i][1];
      }
    const uint32_t v_last = kb + ((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (warp * 8 * NT + (NT - 1) * 8) * 2;
    const uint32_t v_addr = kb + ((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (warp * 8 * NT + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int k = 0; k < kLdKeys; k += 16) {
      uint32_t a[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmatrix_x4(p_addr + i * 16 * kLdPPitch + k * 2, a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
      for (int j = 0; j + 1 < NT; j += 2) {
        uint32_t v[4];
        ldmatrix_x4_trans(v_addr + k * pitch + j * 16, v[0], v[1], v[2], v[3]);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16_full(acc[i][j], a[i], v[0], v[1]);
          mma_bf16_full(acc[i][j + 1], a[i], v[2], v[3]);
        }
      }
      if constexpr (NT % 2 == 1) {
        uint32_t v[2];
        ldmatrix_x2_trans(v_last + k * pitch, v[0], v[1]);
#pragma unroll
        for (int i = 0; i < MT; ++i) mma_bf16_full(acc[i][NT - 1], a[i], v[0], v[1]);
      }
    }
    __syncthreads();      // the tile's buffer and P are rewritten next
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = h0 + i * 16 + g + 8 * e;
      if (h >= p.heads) continue;
      const long long row = (long long)b * p.heads + h;
      if (p.splits == 1) {
        const float inv = 1.f / l_run[i][e];
#pragma unroll
        for (int j = 0; j < NT; ++j)
          *reinterpret_cast<uint32_t*>(p.out + row * p.rank + warp * 8 * NT + j * 8 + tq * 2) =
              pack_bf16(acc[i][j][2 * e] * inv, acc[i][j][2 * e + 1] * inv);
      } else {
        float* o = p.part_o + (row * p.splits + split) * p.rank + warp * 8 * NT + tq * 2;
#pragma unroll
        for (int j = 0; j < NT; ++j) *reinterpret_cast<float2*>(o + j * 8) = make_float2(acc[i][j][2 * e], acc[i][j][2 * e + 1]);
        if (warp == 0 && tq == 0) {
          p.part_ml[(row * p.splits + split) * 2] = m_run[i][e];
          p.part_ml[(row * p.splits + split) * 2 + 1] = l_run[i][e];
        }
      }
    }
}

__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits, int rank, __nv_bfloat16* __restrict__ out) {
  const long long row = blockIdx.x;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, part_ml[(row * splits + s) * 2]);
  for (int s = 0; s < splits; ++s) l += part_ml[(row * splits + s) * 2 + 1] * exp2f(part_ml[(row * splits + s) * 2] - m);
  const float inv = 1.f / l;
  for (int c = threadIdx.x * 4; c < rank; c += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float w = exp2f(part_ml[(row * splits + s) * 2] - m) * inv;   // an empty split has weight 0 and finite sums
      const float4 v = load4(part_o + (row * splits + s) * rank + c);
      a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
    }
    store4(out + row * rank + c, a);
  }
}

template <int MT, int NT>
int launch_latent_decode(const LatentDecodeParams& p, int n, cudaStream_t stream) {
  const size_t pitch = (size_t)(p.rank + p.rot) * 2 + 16;
  const size_t smem = (size_t)MT * 16 * (pitch + kLdPPitch) + 2 * kLdKeys * pitch;
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(latent_decode_kernel<MT, NT>, smem, configured));
  const dim3 grid((unsigned)p.splits, (unsigned)((p.heads + MT * 16 - 1) / (MT * 16)), (unsigned)n);
  latent_decode_kernel<MT, NT><<<grid, kLdThreads, smem, stream>>>(p);
  MSA_LAUNCH_OK("latent_decode_kernel");
  if (p.splits > 1) {
    latent_merge_kernel<<<(unsigned)(n * p.heads), 128, 0, stream>>>(p.part_o, p.part_ml, p.splits, p.rank, p.out);
    MSA_LAUNCH_OK("latent_merge_kernel");
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
                                    int32_t splits, float scale, void* out, float* part_o, float* part_ml, void* stream) {
  MSA_REQUIRE(qa && ring && slot && pos && out && (rot == 0 || qb), "latent_decode: null pointer");
  MSA_REQUIRE(msa_lm_latent_decode_supported(rank, rot) && heads > 0 && window > 0 && ring_rows > 0 && ring_rows < (1ll << 30), "latent_decode: bad sizes");
  MSA_REQUIRE(splits >= 1 && splits <= 64 && (splits == 1 || (part_o && part_ml)), "latent_decode: bad splits");
  MSA_REQUIRE(aligned16(qa) && aligned16(ring) && aligned16(out) && (rot == 0 || aligned16(qb)) && qa_row % 8 == 0 &&
                  qa_head % 8 == 0 && qb_row % 8 == 0 && qb_head % 8 == 0, "latent_decode: rows must be 16-byte aligned");
  if (n <= 0) return MSA_OK;
  LatentDecodeParams p{(const __nv_bfloat16*)qa, qa_row, qa_head, (const __nv_bfloat16*)qb, qb_row, qb_head,
                       (const __nv_bfloat16*)ring, ring_rows, slot, pos, heads, rank, rot, window, splits,
                       scale * 1.4426950408889634f, (__nv_bfloat16*)out, part_o, part_ml};
  cudaStream_t st = (cudaStream_t)stream;
  if (heads <= 16) {
    switch (rank) {
      case 128: return launch_latent_decode<1, 1>(p, n, st);
      case 256: return launch_latent_decode<1, 2>(p, n, st);
      case 384: return launch_latent_decode<1, 3>(p, n, st);
      default: return launch_latent_decode<1, 4>(p, n, st);
    }
  }
  switch (rank) {
    case 128: return launch_latent_decode<2, 1>(p, n, st);
    case 256: return launch_latent_decode<2, 2>(p, n, st);
    case 384: return launch_latent_decode<2, 3>(p, n, st);
    default: return launch_latent_decode<2, 4>(p, n, st);
  }
}
