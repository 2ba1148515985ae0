// Gated delta rule over prompt portions in chunks of 64 tokens, on tensor cores.
//
// Within a chunk let G_t be the running sum of the log decays, S the state before the chunk, and
//     A_ti = beta_t e^(G_t - G_i) k_t.k_i  (i < t),   T = (I + A)^-1 diag(beta),   M_ti = e^(G_t - G_i) q_t.k_i  (i <= t).
// Unrolling the rule over the chunk gives
//     U = T (V - e^G K S),    O = e^G Q S + M U,    S' = e^(G_C) S + K^T (e^(G_C - G) U),
// so only S passes from chunk to chunk.  delta_chunk_kernel computes T, M and G of every chunk (all chunks at once);
// delta_state_kernel walks the chunks of a (sequence, head, value tile) with S in registers as fp32 accumulators.
//
// 32-bit operands enter the products as the sum of two bf16 numbers (16 to 17 significant bits) and the three products
// that matter are accumulated in fp32: hi*hi + hi*lo + lo*hi.  Decays, the triangular inverse and the state itself are
// plain fp32.  Rows past the end of a portion are zero with beta 0 and decay 1, which leaves the state alone.
#include "lm_common.cuh"
#include "mma_helpers.cuh"

namespace msa {

constexpr int kDcRows = 64, kDcTile = kDcRows * kDcRows;   // a chunk; elements of one T or M plane
constexpr int kDcPitch = 144;                              // smem bytes per row of a 64-column bf16 tile

__device__ __forceinline__ void mma_bf16_acc(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_bf16(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16_rn(x);
  lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct DeltaChunkParams {
  const __nv_bfloat16* qk;      // [rows, 2 (q, k), 2 (hi, lo), kv_heads, dim]
  const __nv_bfloat16* v;       // [rows, heads, vdim]
  const float* gates;           // [rows, 2, heads]
  const int32_t *slot, *start, *cu, *chunk_off;   // chunk_off: prefix sums over the non-decode sequences
  int n_decode, n_seq, heads, kv_heads, dim, vdim, n_chunks;
  __nv_bfloat16* tm;            // [chunks, heads, 2 (T, M), 2 (hi, lo), 64, 64]
  float* gcum;                  // [chunks, heads, 64]
  float* state;
  // output of the state kernel: normalised and gated rows, or raw fp32 rows
  const __nv_bfloat16* gate; long long gate_stride;
  const float* w_norm; float eps;
  __nv_bfloat16* out; long long out_stride;
  float* o;
};

// ---- per chunk: K K^T and Q K^T once per key head, then T, M and G for every head that uses it -----------------------
template <int DK>
__global__ void __launch_bounds__(128) delta_chunk_kernel(const DeltaChunkParams p) {
  constexpr int kPitch = DK * 2 + 16, kKs = DK / 16;
  extern __shared__ __align__(16) unsigned char sm[];
  unsigned char* s_q = sm;                               // hi, lo
  unsigned char* s_k = s_q + 2 * kDcRows * kPitch;       // hi, lo
  // over the operands once they are used up
  float* s_a = reinterpret_cast<float*>(sm);             // [64][68]
  float* s_kk = s_a + kDcRows * 68;                      // [64][65]
  float* s_qk = s_kk + kDcRows * 65;
  __shared__ float s_g[kDcRows], s_b[kDcRows];
  const int chunk = blockIdx.x, hk = blockIdx.y, group = p.heads / p.kv_heads;
  const int ps = owner_of(p.chunk_off, p.n_seq - p.n_decode, chunk), s = ps + p.n_decode;
  const int t0 = (chunk - p.chunk_off[ps]) * kDcRows, len = min(kDcRows, p.cu[s + 1] - p.cu[s] - t0);
  const long long row0 = (long long)p.cu[s] - p.n_decode + t0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int kVecs = DK / 8;
  for (int i = threadIdx.x; i < 4 * kDcRows * kVecs; i += 128) {     // plane = (q / k, hi / lo)
    const int plane = i / (kDcRows * kVecs), r = i / kVecs % kDcRows, c = i % kVecs;
    const bool on = r < len;
    const __nv_bfloat16* src = p.qk + (((row0 + (on ? r : 0)) * 4 + plane) * p.kv_heads + hk) * DK + c * 8;
    cp_async16((uint32_t)__cvta_generic_to_shared(s_q + (plane * kDcRows + r) * kPitch + c * 16), src, on ? 16u : 0u);
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  {
    const uint32_t qa = (uint32_t)__cvta_generic_to_shared(s_q) + (warp * 16 + (lane & 15)) * kPitch + (lane >> 4) * 16;
    const uint32_t ka = qa + 2 * kDcRows * kPitch;
    const uint32_t kb = (uint32_t)__cvta_generic_to_shared(s_k) + ((lane & 7) + ((lane >> 4) << 3)) * kPitch + ((lane >> 3) & 1) * 16;
    constexpr uint32_t kLo = kDcRows * kPitch;
    float kk[8][4], qq[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) kk[j][e] = qq[j][e] = 0.f;
#pragma unroll
    for (int k = 0; k < kKs; ++k) {
      uint32_t ah[4], al[4], qh[4], ql[4];
      ldmatrix_x4(ka + k * 32, ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(ka + kLo + k * 32, al[0], al[1], al[2], al[3]);
      ldmatrix_x4(qa + k * 32, qh[0], qh[1], qh[2], qh[3]);
      ldmatrix_x4(qa + kLo + k * 32, ql[0], ql[1], ql[2], ql[3]);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        if (j * 8 > warp * 16 + 15) break;               // above the diagonal
        uint32_t bh[4], bl[4];
        ldmatrix_x4(kb + j * 8 * kPitch + k * 32, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4(kb + kLo + j * 8 * kPitch + k * 32, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma_bf16_acc(kk[j + n], al, bh[2 * n], bh[2 * n + 1]);
          mma_bf16_acc(kk[j + n], ah, bl[2 * n], bl[2 * n + 1]);
          mma_bf16_acc(kk[j + n], ah, bh[2 * n], bh[2 * n + 1]);
          mma_bf16_acc(qq[j + n], ql, bh[2 * n], bh[2 * n + 1]);
          mma_bf16_acc(qq[j + n], qh, bl[2 * n], bl[2 * n + 1]);
          mma_bf16_acc(qq[j + n], qh, bh[2 * n], bh[2 * n + 1]);
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = warp * 16 + (lane >> 2) + 8 * (e >> 1), c = j * 8 + (lane & 3) * 2 + (e & 1);
        s_kk[r * 65 + c] = kk[j][e];
        s_qk[r * 65 + c] = qq[j][e];
      }
  }
  for (int hg = 0; hg < group; ++hg) {
    const int h = hk * group + hg;
    __syncthreads();
    if (warp == 0) {                                     // running sum of the log decays, two rows per lane
      const float* g = p.gates + row0 * 2 * p.heads + h;
      const int r = 2 * lane;
      const float a = r < len ? g[(long long)r * 2 * p.heads] : 0.f;
      const float b = r + 1 < len ? g[(long long)(r + 1) * 2 * p.heads] : 0.f;
      float sum = a + b;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += x;
      }
      s_g[r] = sum - b;
      s_g[r + 1] = sum;
    } else if (warp <= 2) {
      const int r = threadIdx.x - 32;
      s_b[r] = r < len ? p.gates[(row0 + r) * 2 * p.heads + p.heads + h] : 0.f;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < kDcTile; i += 128) {
      const int t = i >> 6, c = i & 63;
      s_a[t * 68 + c] = c < t ? s_b[t] * expf(s_g[t] - s_g[c]) * s_kk[t * 65 + c] : 0.f;
    }
    __syncthreads();
    const long long tile = ((long long)chunk * p.heads + h) * 4 * kDcTile;
    if (warp < 2) {                                      // column c of (I + A)^-1 by forward substitution, times beta_c
      const int c = threadIdx.x;
      float x[kDcRows];
      const float beta = s_b[c];
#pragma unroll
      for (int t = 0; t < kDcRows; ++t) {
        float acc = t == c ? 1.f : 0.f;
#pragma unroll
        for (int i = 0; i < (t & ~3); i += 4) {
          const float4 a = *reinterpret_cast<const float4*>(s_a + t * 68 + i);
          acc = fmaf(-a.x, x[i], acc); acc = fmaf(-a.y, x[i + 1], acc);
          acc = fmaf(-a.z, x[i + 2], acc); acc = fmaf(-a.w, x[i + 3], acc);
        }
#pragma unroll
        for (int i = t & ~3; i < t; ++i) acc = fmaf(-s_a[t * 68 + i], x[i], acc);
        x[t] = acc;
      }
#pragma unroll
      for (int t = 0; t < kDcRows; ++t) {
        __nv_bfloat16 hi, lo;
        split_bf16(x[t] * beta, hi, lo);
        p.tm[tile + t * kDcRows + c] = hi;
        p.tm[tile + kDcTile + t * kDcRows + c] = lo;
      }
    } else {
      const int tid = threadIdx.x - 64;
      p.gcum[((long long)chunk * p.heads + h) * kDcRows + tid] = s_g[tid];
      for (int i = tid; i < kDcTile; i += 64) {
        const int t = i >> 6, c = i & 63;
        __nv_bfloat16 hi, lo;
        split_bf16(c <= t ? expf(s_g[t] - s_g[c]) * s_qk[t * 65 + c] : 0.f, hi, lo);
        p.tm[tile + 2 * kDcTile + i] = hi;
        p.tm[tile + 3 * kDcTile + i] = lo;
      }
    }
  }
}

// ---- the walk over a sequence's chunks -------------------------------------------------------------------------------
template <int DK, int DVT>
struct DeltaStateSmem {
  static constexpr int kPk = DK * 2 + 16, kPv = DVT * 2 + 16;      // bytes per row
  static constexpr int kQ = 0, kK = kQ + 2 * kDcRows * kPk, kT = kK + 2 * kDcRows * kPk, kM = kT + 2 * kDcRows * kDcPitch,
                       kS = kM + 2 * kDcRows * kDcPitch;
  static constexpr int kU = kS + 2 * (DK > kDcRows ? DK : kDcRows) * kPv;          // S, later the decayed U; then R, later U
  static constexpr int kV = kU + 2 * kDcRows * kPv;
  static constexpr int kTotal = kV + kDcRows * kPv;
};

// 8 * WN warps: warp = (row tile wr, column group wn).  Products with 64 rows and those with the state's rows are dealt so
// that every warp has part of each.
template <int DK, int DVT, int WN, bool FUSE>
__global__ void __launch_bounds__(256 * WN, 1) delta_state_kernel(const DeltaChunkParams p) {
  using L = DeltaStateSmem<DK, DVT>;
  constexpr int kThreads = 256 * WN, kPk = L::kPk, kPv = L::kPv;
  constexpr int NT = DVT / 8 / WN;                 // octets of columns per warp: K S, Q S, M U
  constexpr int N2 = NT / 2;                       // ... T R (twice as many warps per row tile)
  constexpr int N4 = DK == 128 ? NT : NT / 2;      // ... the state
  static_assert(N2 >= 2 && N2 % 2 == 0, "column octets come in pairs");
  extern __shared__ __align__(16) unsigned char sm[];
  __shared__ float s_eg[kDcRows], s_ec[kDcRows], s_ss[WN][kDcRows], s_last;
  const int ps = blockIdx.z, s = ps + p.n_decode, h = blockIdx.y, c0 = blockIdx.x * DVT, hk = h / (p.heads / p.kv_heads);
  const int len = p.cu[s + 1] - p.cu[s], n_chunks = (len + kDcRows - 1) / kDcRows, chunk0 = p.chunk_off[ps];
  const long long row0 = (long long)p.cu[s] - p.n_decode;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3, wr = warp & 7, wn = warp >> 3;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(sm);

  auto load_qk = [&](int ch, bool key) {           // q or k rows of chunk ch, hi and lo
    constexpr int vecs = DK / 8;
    const int n = min(kDcRows, len - ch * kDcRows);
    for (int i = threadIdx.x; i < 2 * kDcRows * vecs; i += kThreads) {
      const int plane = i / (kDcRows * vecs), r = i / vecs % kDcRows, c = i % vecs;
      const bool on = r < n;
      const __nv_bfloat16* src = p.qk + (((row0 + ch * kDcRows + (on ? r : 0)) * 4 + (key ? 2 : 0) + plane) * p.kv_heads + hk) * DK + c * 8;
      cp_async16(base + (key ? L::kK : L::kQ) + (plane * kDcRows + r) * kPk + c * 16, src, on ? 16u : 0u);
    }
  };
  auto load_tm = [&](int ch, bool m) {
    const __nv_bfloat16* src = p.tm + (((long long)(chunk0 + ch) * p.heads + h) * 4 + (m ? 2 : 0)) * kDcTile;
    for (int i = threadIdx.x; i < 2 * kDcRows * 8; i += kThreads)
      cp_async16(base + (m ? L::kM : L::kT) + (i >> 3) * kDcPitch + (i & 7) * 16, src + (long long)i * 8, 16u);
  };
  auto load_v = [&](int ch) {
    constexpr int vecs = DVT / 8;
    const int n = min(kDcRows, len - ch * kDcRows);
    for (int i = threadIdx.x; i < kDcRows * vecs; i += kThreads) {
      const int r = i / vecs, c = i % vecs;
      const bool on = r < n;
      cp_async16(base + L::kV + r * kPv + c * 16,
                 p.v + (row0 + ch * kDcRows + (on ? r : 0)) * p.heads * p.vdim + (long long)h * p.vdim + c0 + c * 8, on ? 16u : 0u);
    }
  };
  if (n_chunks > 0) { load_qk(0, false); load_qk(0, true); load_tm(0, false); load_tm(0, true); load_v(0); }
  cp_async_commit();

  const int sm_tile = DK == 128 ? wr : wr & 3;                                        // this warp's part of the state
  const int sn0 = DK == 128 ? wn * NT : (wn * 2 + (wr >> 2)) * N4;
  float* state = p.state + (((long long)p.slot[s] * p.heads + h) * DK + sm_tile * 16 + g) * p.vdim + c0 + sn0 * 8 + tq * 2;
  float st[N4][4];
  const bool fresh = p.start[s] == 0;
#pragma unroll
  for (int j = 0; j < N4; ++j) {
    float2 a = make_float2(0.f, 0.f), b = a;
    if (!fresh) {
      a = *reinterpret_cast<const float2*>(state + j * 8);
      b = *reinterpret_cast<const float2*>(state + 8ll * p.vdim + j * 8);
    }
    st[j][0] = a.x; st[j][1] = a.y; st[j][2] = b.x; st[j][3] = b.y;
  }
  constexpr int kSLo = DK * kPv, kULo = kDcRows * kPv, kQLo = kDcRows * kPk, kTLo = kDcRows * kDcPitch;
  // a 16 x 8 accumulator tile to a hi / lo pair of bf16 planes
  auto put = [&](int region, int lo_off, int row, int col8, const float (&v)[4], float f0, float f1) {
    uint32_t hi, lo;
    split2(v[0] * f0, v[1] * f0, hi, lo);
    unsigned char* d = sm + region + row * kPv + (col8 * 8 + tq * 2) * 2;
    *reinterpret_cast<uint32_t*>(d) = hi;
    *reinterpret_cast<uint32_t*>(d + lo_off) = lo;
    split2(v[2] * f1, v[3] * f1, hi, lo);
    d += 8 * kPv;
    *reinterpret_cast<uint32_t*>(d) = hi;
    *reinterpret_cast<uint32_t*>(d + lo_off) = lo;
  };
#pragma unroll
  for (int j = 0; j < N4; ++j) put(L::kS, kSLo, sm_tile * 16 + g, sn0 + j, st[j], 1.f, 1.f);

  const uint32_t a_off = (lane & 15), a_col = (lane >> 4) * 16;                         // A operand, rows as stored
  const uint32_t t_row = (lane & 7) + ((lane >> 3) & 1) * 8, t_col = (lane >> 4) * 16;  // B operand by transposition: 16 rows x 16 columns
  // one reduction step of 16: c[0 .. n) += (ah + al) (hi + lo of the B region), without lo * lo
  auto step16 = [&](float (*c)[4], int n, const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t b, int lo_off) {
#pragma unroll
    for (int j = 0; j < n; j += 2) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(b + j * 16, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4_trans(b + lo_off + j * 16, bl[0], bl[1], bl[2], bl[3]);
      mma_bf16_acc(c[j], al, bh[0], bh[1]);
      mma_bf16_acc(c[j + 1], al, bh[2], bh[3]);
      mma_bf16_acc(c[j], ah, bl[0], bl[1]);
      mma_bf16_acc(c[j + 1], ah, bl[2], bl[3]);
      mma_bf16_acc(c[j], ah, bh[0], bh[1]);
      mma_bf16_acc(c[j + 1], ah, bh[2], bh[3]);
    }
  };
  const int r0 = (wr & 3) * 16 + g;
  for (int ch = 0; ch < n_chunks; ++ch) {
    if (threadIdx.x < kDcRows) {
      const float* gc = p.gcum + ((long long)(chunk0 + ch) * p.heads + h) * kDcRows;
      const float gt = gc[threadIdx.x], gl = gc[kDcRows - 1];
      s_eg[threadIdx.x] = expf(gt);
      s_ec[threadIdx.x] = expf(gl - gt);
      if (threadIdx.x == 0) s_last = expf(gl);
    }
    cp_async_wait<0>();
    __syncthreads();
    const bool more = ch + 1 < n_chunks;
    // K S (row tiles 0-3) and Q S (row tiles 4-7)
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    {
      const uint32_t a_base = base + (wr < 4 ? L::kK : L::kQ) + ((wr & 3) * 16 + a_off) * kPk + a_col;
      const uint32_t b_base = base + L::kS + t_row * kPv + wn * NT * 16 + t_col;
#pragma unroll 2
      for (int k = 0; k < DK / 16; ++k) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(a_base + k * 32, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(a_base + kQLo + k * 32, al[0], al[1], al[2], al[3]);
        step16(acc, NT, ah, al, b_base + k * 16 * kPv, kSLo);
      }
    }
    __nv_bfloat162 gate[FUSE ? 2 : 1][FUSE ? NT : 1];
    {
      const float e0 = s_eg[r0], e1 = s_eg[r0 + 8];
      if (wr < 4) {                                 // R = V - e^G K S
        const unsigned char* v0 = sm + L::kV + r0 * kPv + (wn * NT * 8 + tq * 2) * 2;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v0 + j * 16));
          const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v0 + 8 * kPv + j * 16));
          acc[j][0] = fmaf(-e0, acc[j][0], a.x); acc[j][1] = fmaf(-e0, acc[j][1], a.y);
          acc[j][2] = fmaf(-e1, acc[j][2], b.x); acc[j][3] = fmaf(-e1, acc[j][3], b.y);
          put(L::kU, kULo, r0, wn * NT + j, acc[j], 1.f, 1.f);
        }
      } else {
#pragma unroll
        for (int j = 0; j < NT; ++j) { acc[j][0] *= e0; acc[j][1] *= e0; acc[j][2] *= e1; acc[j][3] *= e1; }
        if constexpr (FUSE) {                       // the output's gates, needed at the end of the chunk
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = ch * kDcRows + r0 + 8 * e;
            const __nv_bfloat16* src = p.gate + (row0 + (t < len ? t : 0)) * p.gate_stride + (long long)h * DVT + wn * NT * 8 + tq * 2;
#pragma unroll
            for (int j = 0; j < NT; ++j) gate[e][j] = *reinterpret_cast<const __nv_bfloat162*>(src + j * 8);
          }
        }
      }
    }
    __syncthreads();                                // S, Q and V have been read, R is there
    if (more) { load_qk(ch + 1, false); load_v(ch + 1); }
    // U = T R
    float u[N2][4];
    const int un0 = (wn * 2 + (wr >> 2)) * N2;
#pragma unroll
    for (int j = 0; j < N2; ++j) u[j][0] = u[j][1] = u[j][2] = u[j][3] = 0.f;
    {
      const uint32_t a_base = base + L::kT + ((wr & 3) * 16 + a_off) * kDcPitch + a_col;
      const uint32_t b_base = base + L::kU + t_row * kPv + un0 * 16 + t_col;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (k > (wr & 3)) break;                    // T is lower triangular
        uint32_t ah[4], al[4];
        ldmatrix_x4(a_base + k * 32, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(a_base + kTLo + k * 32, al[0], al[1], al[2], al[3]);
        step16(u, N2, ah, al, b_base + k * 16 * kPv, kULo);
      }
    }
    __syncthreads();                                // R and T have been read
    if (more) load_tm(ch + 1, false);
    {
      const float d0 = s_ec[r0], d1 = s_ec[r0 + 8];
#pragma unroll
      for (int j = 0; j < N2; ++j) {
        put(L::kU, kULo, r0, un0 + j, u[j], 1.f, 1.f);
        put(L::kS, kSLo, r0, un0 + j, u[j], d0, d1);   // decayed to the end of the chunk
      }
    }
    __syncthreads();
    if (wr >= 4) {                                  // O += M U
      const uint32_t a_base = base + L::kM + ((wr & 3) * 16 + a_off) * kDcPitch + a_col;
      const uint32_t b_base = base + L::kU + t_row * kPv + wn * NT * 16 + t_col;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (k > (wr & 3)) break;
        uint32_t ah[4], al[4];
        ldmatrix_x4(a_base + k * 32, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(a_base + kTLo + k * 32, al[0], al[1], al[2], al[3]);
        step16(acc, NT, ah, al, b_base + k * 16 * kPv, kULo);
      }
      if constexpr (FUSE) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float ss = 0.f;
#pragma unroll
          for (int j = 0; j < NT; ++j) ss += acc[j][2 * e] * acc[j][2 * e] + acc[j][2 * e + 1] * acc[j][2 * e + 1];
          ss += __shfl_xor_sync(0xffffffffu, ss, 1);
          ss += __shfl_xor_sync(0xffffffffu, ss, 2);
          if (tq == 0) s_ss[wn][r0 + 8 * e] = ss;
        }
      }
    }
    {                                               // S = e^(G_C) S + K^T (e^(G_C - G) U)
      const float last = s_last;
#pragma unroll
      for (int j = 0; j < N4; ++j) { st[j][0] *= last; st[j][1] *= last; st[j][2] *= last; st[j][3] *= last; }
      // A = K^T: stored rows are the reduction index; the transposed load gives 16 state rows x 16 tokens
      const uint32_t a_base = base + L::kK + ((lane & 7) + (lane >> 4) * 8) * kPk + (sm_tile * 16 + ((lane >> 3) & 1) * 8) * 2;
      const uint32_t b_base = base + L::kS + t_row * kPv + sn0 * 16 + t_col;
#pragma unroll 2
      for (int k = 0; k < 4; ++k) {
        uint32_t ah[4], al[4];
        ldmatrix_x4_trans(a_base + k * 16 * kPk, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4_trans(a_base + kQLo + k * 16 * kPk, al[0], al[1], al[2], al[3]);
        step16(st, N4, ah, al, b_base + k * 16 * kPv, kSLo);
      }
    }
    __syncthreads();                                // K, M, U and the decayed U have been read
    if (more) { load_qk(ch + 1, true); load_tm(ch + 1, true); }
    cp_async_commit();
    if (more) {
#pragma unroll
      for (int j = 0; j < N4; ++j) put(L::kS, kSLo, sm_tile * 16 + g, sn0 + j, st[j], 1.f, 1.f);
    }
    if (wr >= 4) {                                  // rows r0, r0 + 8 of the chunk
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = ch * kDcRows + r0 + 8 * e;
        if (t >= len) continue;
        if constexpr (FUSE) {
          float ss = 0.f;
#pragma unroll
          for (int w = 0; w < WN; ++w) ss += s_ss[w][r0 + 8 * e];
          const float inv = 1.f / sqrtf(ss / (float)DVT + p.eps);
          __nv_bfloat16* out = p.out + (row0 + t) * p.out_stride + (long long)h * DVT + wn * NT * 8 + tq * 2;
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            const float2 z = __bfloat1622float2(gate[e][j]);
            const float2 w = *reinterpret_cast<const float2*>(p.w_norm + (wn * NT + j) * 8 + tq * 2);
            *reinterpret_cast<__nv_bfloat162*>(out + j * 8) =
                __floats2bfloat162_rn(acc[j][2 * e] * inv * w.x * __fdividef(z.x, 1.f + __expf(-z.x)),
                                      acc[j][2 * e + 1] * inv * w.y * __fdividef(z.y, 1.f + __expf(-z.y)));
          }
        } else {
          float* o = p.o + ((row0 + t) * p.heads + h) * p.vdim + c0 + wn * NT * 8 + tq * 2;
#pragma unroll
          for (int j = 0; j < NT; ++j) *reinterpret_cast<float2*>(o + j * 8) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
        }
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int j = 0; j < N4; ++j) {
    *reinterpret_cast<float2*>(state + j * 8) = make_float2(st[j][0], st[j][1]);
    *reinterpret_cast<float2*>(state + 8ll * p.vdim + j * 8) = make_float2(st[j][2], st[j][3]);
  }
}

template <int DK>
int launch_delta_chunk(const DeltaChunkParams& p, cudaStream_t stream) {
  constexpr size_t operands = (size_t)4 * kDcRows * (DK * 2 + 16), square = (size_t)kDcRows * (68 + 65 + 65) * 4;
  constexpr size_t smem = operands > square ? operands : square;
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(delta_chunk_kernel<DK>, smem, configured));
  delta_chunk_kernel<DK><<<dim3((unsigned)p.n_chunks, (unsigned)p.kv_heads), 128, smem, stream>>>(p);
  MSA_LAUNCH_OK("delta_chunk_kernel");
  return MSA_OK;
}
template <int DK, int DVT, bool FUSE>
int launch_delta_state(const DeltaChunkParams& p, cudaStream_t stream) {
  constexpr size_t smem = DeltaStateSmem<DK, DVT>::kTotal;
  constexpr int WN = DVT >= 64 ? 2 : 1;
  static_assert(smem <= 226 * 1024, "shared memory");
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(delta_state_kernel<DK, DVT, WN, FUSE>, smem, configured));
  const dim3 grid((unsigned)(p.vdim / DVT), (unsigned)p.heads, (unsigned)(p.n_seq - p.n_decode));
  delta_state_kernel<DK, DVT, WN, FUSE><<<grid, 256 * WN, smem, stream>>>(p);
  MSA_LAUNCH_OK("delta_state_kernel");
  return MSA_OK;
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_delta_chunk_supported(int32_t dim, int32_t vdim, int32_t taps) {
  return (dim == 64 || dim == 128) && vdim > 0 && vdim % 32 == 0 && taps >= 2 && taps <= 4;
}
extern "C" int64_t msa_lm_delta_chunk_workspace(int32_t n_chunks, int32_t heads) {
  return (int64_t)n_chunks * heads * (4 * kDcTile * 2 + kDcRows * 4);
}

extern "C" int msa_lm_delta_chunk(const msa_lm_delta_args* a, const void* qk, const void* v, const float* gates,
                                  const int32_t* chunk_off, int32_t n_chunks, int32_t tile, void* workspace, float* o,
                                  void* out, int64_t out_stride, void* stream) {
  MSA_REQUIRE(a && qk && v && gates && chunk_off && workspace && out, "delta_chunk: null pointer");
  MSA_REQUIRE(a->dtype == MSA_BF16 && msa_lm_delta_chunk_supported(a->dim, a->vdim, a->taps), "delta_chunk: unsupported sizes");
  MSA_REQUIRE((tile == 32 || tile == 64 || tile == 128) && a->vdim % tile == 0, "delta_chunk: bad value tile");
  MSA_REQUIRE(a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 && a->state && a->slot && a->start && a->cu,
              "delta_chunk: bad arguments");
  MSA_REQUIRE(aligned16(qk) && aligned16(v) && aligned16(workspace) && aligned16(a->state) && aligned16(a->w_norm) &&
                  a->proj_stride % 2 == 0 && out_stride % 2 == 0 && (a->vdim == tile || o), "delta_chunk: alignment");
  if (a->n_seq == a->n_decode || n_chunks <= 0) return MSA_OK;
  DeltaChunkParams p{};
  p.qk = (const __nv_bfloat16*)qk; p.v = (const __nv_bfloat16*)v; p.gates = gates;
  p.slot = a->slot; p.start = a->start; p.cu = a->cu; p.chunk_off = chunk_off;
  p.n_decode = a->n_decode; p.n_seq = a->n_seq; p.heads = a->heads; p.kv_heads = a->kv_heads; p.dim = a->dim; p.vdim = a->vdim;
  p.n_chunks = n_chunks;
  p.tm = (__nv_bfloat16*)workspace;
  p.gcum = (float*)((char*)workspace + (int64_t)n_chunks * a->heads * 4 * kDcTile * 2);
  p.state = a->state;
  p.gate = (const __nv_bfloat16*)a->proj + (int64_t)a->n_decode * a->proj_stride + 2 * a->kv_heads * a->dim + a->heads * a->vdim;
  p.gate_stride = a->proj_stride; p.w_norm = a->w_norm; p.eps = a->eps;
  p.out = (__nv_bfloat16*)out; p.out_stride = out_stride; p.o = o;
  cudaStream_t st = (cudaStream_t)stream;
  const bool fuse = tile == a->vdim;
  if (a->dim == 128) {
    MSA_OK_OR_RETURN(launch_delta_chunk<128>(p, st));
    if (tile == 128) MSA_OK_OR_RETURN((fuse ? launch_delta_state<128, 128, true>(p, st) : launch_delta_state<128, 128, false>(p, st)));
    else if (tile == 64) MSA_OK_OR_RETURN((fuse ? launch_delta_state<128, 64, true>(p, st) : launch_delta_state<128, 64, false>(p, st)));
    else MSA_OK_OR_RETURN((fuse ? launch_delta_state<128, 32, true>(p, st) : launch_delta_state<128, 32, false>(p, st)));
  } else {
    MSA_OK_OR_RETURN(launch_delta_chunk<64>(p, st));
    if (tile == 128) MSA_OK_OR_RETURN((fuse ? launch_delta_state<64, 128, true>(p, st) : launch_delta_state<64, 128, false>(p, st)));
    else if (tile == 64) MSA_OK_OR_RETURN((fuse ? launch_delta_state<64, 64, true>(p, st) : launch_delta_state<64, 64, false>(p, st)));
    else MSA_OK_OR_RETURN((fuse ? launch_delta_state<64, 32, true>(p, st) : launch_delta_state<64, 32, false>(p, st)));
  }
  if (!fuse) return msa_lm_delta_out(a, o, out, out_stride, stream);
  return MSA_OK;
}
