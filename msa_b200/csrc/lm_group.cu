// Grouped-query attention behind a short convolution: what happens between the projections and the attention proper
// (convolution, rotation, ring and context upkeep), and decode attention over the ring.
//
// Per sequence slot a layer keeps a ring of the last `ring_rows` rows [keys | values] (position p in row p % ring_rows) and
// the last taps-1 inputs of the convolutions.  A step that brings several tokens of a sequence works on a packed context:
// the ring rows its first token still sees, then its own rows; the ring takes over the last of them afterwards.
#include "lm_conv.cuh"
#include "lm_merge.cuh"
#include "mma_helpers.cuh"

namespace msa {

constexpr int kGpRows = 8;      // packed rows per block, at most (a step of few rows: one)

struct GroupLayout {
  int nq, nk, nv, chan, width;  // columns of q, k and v, all of them; elements of a ring row
  __host__ __device__ explicit GroupLayout(const msa_lm_group_args& a)
      : nq(a.heads * a.dim), nk(a.kv_heads * a.dim), nv(a.kv_heads * a.vdim), chan(nq + nk + nv),
        width(a.kv_heads * (a.k_pitch + a.v_pitch)) {}
};

// Where channel c goes: dimension i of a head, rotated or not, element `at` of the query row or of the ring row.
struct GroupColumn { int at, i; bool query, turns; };
__device__ __forceinline__ GroupColumn group_column(const msa_lm_group_args& a, const GroupLayout& L, int c) {
  GroupColumn g;
  g.query = c < L.nq;
  if (c < L.nq + L.nk) {
    const int u = g.query ? c : c - L.nq, h = u / a.dim;
    g.i = u - h * a.dim;
    g.turns = g.i < a.rot;
    g.at = h * (g.query ? a.q_pitch : a.k_pitch) + g.i;
  } else {
    const int u = c - L.nq - L.nk, h = u / a.vdim;
    g.i = u - h * a.vdim;
    g.turns = false;
    g.at = a.kv_heads * a.k_pitch + h * a.v_pitch + g.i;
  }
  return g;
}
template <typename T>
__device__ __forceinline__ T* group_row(const msa_lm_group_args& a, const GroupLayout& L, long long n, int s, int t, int p0) {
  if (n < a.n_decode) return reinterpret_cast<T*>(a.ring) + ((long long)a.slot[s] * a.ring_rows + p0 % a.ring_rows) * L.width;
  return reinterpret_cast<T*>(a.ctx) + (long long)(a.ctx_off[s - a.n_decode] + min(p0, a.window - 1) + t) * L.width;
}

// An old ring row that a continued portion still sees goes to the context.
template <typename T, int V>
__device__ __forceinline__ void copy_old_row(const msa_lm_group_args& a, const GroupLayout& L, int o) {
  const int ps = owner_of(a.old_off, a.n_seq - a.n_decode, o), s = ps + a.n_decode;
  const int k = o - a.old_off[ps], start = a.start[s], first = start - min(start, a.window - 1);
  const T* src = reinterpret_cast<const T*>(a.ring) + ((long long)a.slot[s] * a.ring_rows + (first + k) % a.ring_rows) * L.width;
  T* dst = reinterpret_cast<T*>(a.ctx) + (long long)(a.ctx_off[ps] + k) * L.width;
  for (int i = threadIdx.x * V; i < L.width; i += blockDim.x * V) {
    if constexpr (V == 4) store4(dst + i, load4(src + i));
    else dst[i] = src[i];
  }
}

// Any sizes: a block per packed row; a rotated channel computes its partner's convolution as well.
template <typename T>
__global__ void __launch_bounds__(256) group_prep_kernel(const msa_lm_group_args a) {
  extern __shared__ float2 s_turn[];            // cosine and sine of the row's angles
  const GroupLayout L(a);
  if ((int)blockIdx.x >= a.n_tok) { copy_old_row<T, 1>(a, L, (int)blockIdx.x - a.n_tok); return; }
  const long long n = blockIdx.x;
  const int s = a.tok_seq[n], t = (int)n - a.cu[s], p0 = a.start[s], pos = a.pos[n], slot = a.slot[s];
  for (int j = threadIdx.x; j < a.rot / 2; j += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * a.inv_freq[j], &sn, &cs);
    s_turn[j] = make_float2(cs, sn);
  }
  __syncthreads();
  const ConvSource<T> src{reinterpret_cast<const T*>(a.proj), a.proj_stride, reinterpret_cast<T*>(a.conv_state), L.chan, a.taps};
  T* q = reinterpret_cast<T*>(a.q_out) + n * a.heads * a.q_pitch;
  T* row = group_row<T>(a, L, n, s, t, p0);
  for (int c = threadIdx.x; c < L.chan; c += blockDim.x) {
    const GroupColumn g = group_column(a, L, c);
    float y = src.value(a.conv_w, n, t, p0, slot, c);
    if (g.turns) {
      const bool odd = g.i & 1;
      const float z = src.value(a.conv_w, n, t, p0, slot, odd ? c - 1 : c + 1);
      const float2 r = s_turn[g.i >> 1];
      y = odd ? y * r.x + z * r.y : y * r.x - z * r.y;
    }
    (g.query ? q : row)[g.at] = from_f<T>(y);
    if (n < a.n_decode && a.taps > 1) {
      T* dst = src.half(slot, p0 + 1) + c;
      for (int j = 0; j < a.taps - 1; ++j) {
        const T* x = src.at(n, 0, p0, slot, a.taps - 2 - j, c);
        dst[(long long)j * L.chan] = x ? *x : from_f<T>(0.f);
      }
    }
  }
}

// Four channels per thread, up to eight packed rows per block: every input is loaded once.
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) group_prep_vec_kernel(const msa_lm_group_args a, int row_blocks, int rows) {
  extern __shared__ float2 s_turn[];            // [rows][rot / 2]
  const GroupLayout L(a);
  if ((int)blockIdx.x >= row_blocks) {
    if (blockIdx.y == 0) copy_old_row<T, 4>(a, L, (int)blockIdx.x - row_blocks);
    return;
  }
  const int row0 = blockIdx.x * rows, n_here = min(rows, a.n_tok - row0), half = a.rot / 2;
  const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
  const bool on = c < L.chan;
  const ConvSource<T> src{reinterpret_cast<const T*>(a.proj), a.proj_stride, reinterpret_cast<T*>(a.conv_state), L.chan, TAPS};
  ConvWindow<T, TAPS> win;
  float4 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = on ? load4(a.conv_w + (long long)j * L.chan + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  for (int i = threadIdx.x; i < n_here * half; i += 256) {
    const int r = i / half, j = i - r * half;
    float sn, cs;
    sincosf((float)a.pos[row0 + r] * a.inv_freq[j], &sn, &cs);
    s_turn[i] = make_float2(cs, sn);
  }
  __syncthreads();
  if (!on) return;
  const GroupColumn g = group_column(a, L, c);
  const bool turns0 = g.turns, turns1 = g.turns && g.i + 2 < a.rot;
#pragma unroll
  for (int r = 0; r < kGpRows; ++r) {
    if (r >= n_here) break;
    const long long n = row0 + r;
    const int s = a.tok_seq[n], t = (int)n - a.cu[s], p0 = a.start[s], slot = a.slot[s];
    win.move(src, n, t, p0, slot, c, r == 0 || t == 0);
    float4 y = win.value(w);
    const float2* turn = s_turn + r * half + (g.i >> 1);
    if (turns0) { const float2 cs = turn[0]; y = make_float4(y.x * cs.x - y.y * cs.y, y.y * cs.x + y.x * cs.y, y.z, y.w); }
    if (turns1) { const float2 cs = turn[1]; y = make_float4(y.x, y.y, y.z * cs.x - y.w * cs.y, y.w * cs.x + y.z * cs.y); }
    T* dst = g.query ? reinterpret_cast<T*>(a.q_out) + n * a.heads * a.q_pitch : group_row<T>(a, L, n, s, t, p0);
    store4(dst + g.at, y);
    if (n < a.n_decode) win.leave(src, slot, p0, c);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
conv_store_kernel(const T* __restrict__ proj, long long stride, int channels, int taps, T* state, const int32_t* slot,
                  const int32_t* start, const int32_t* cu, int n_decode) {
  const int s = n_decode + blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const int len = cu[s + 1] - cu[s], p0 = start[s], keep = taps - 1;
  const ConvSource<T> src{proj, stride, state, channels, taps};
  T* dst = src.half(slot[s], p0 + len) + c;
  // ascending: an entry that comes from the old half (possibly the same memory) is read before it is overwritten
  for (int j = 0; j < keep; ++j) {
    const T* x = src.at((long long)cu[s] + len - 1, len - 1, p0, slot[s], keep - 1 - j, c);
    dst[(long long)j * channels] = x ? *x : from_f<T>(0.f);
  }
}

// ---- decode -----------------------------------------------------------------------------------------------------------
// A CTA takes one split of a sequence's visible rows for up to 8 (FULL: 16) query heads of a key / value head: the heads are
// rows of the mma tile.  Each of the four warps owns its own stream of 16-key blocks: cp.async into a private 3-stage ring,
// ldmatrix, mma.m16n8k16, online softmax on the accumulator fragments, no CTA-wide barrier inside the loop; the warps'
// partial results are merged through shared memory at the end.
struct GroupDecodeParams {
  const __nv_bfloat16* q; long long q_row;
  const __nv_bfloat16* ring; long long ring_rows;
  const int32_t *slot, *pos;
  int heads, kv_heads, window, splits, sink;
  float scale_log2e;
  const __nv_bfloat16* gate; long long gate_row;
  __nv_bfloat16* out; long long out_row;
  float *part_o, *part_ml;
};

__device__ __forceinline__ void group_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int D, int DV, bool FULL>
__global__ void __launch_bounds__(kMmaWarps * 32, 2) group_decode_kernel(const GroupDecodeParams p) {
  constexpr int kRows = FULL ? 16 : 8, NE = FULL ? 2 : 1;
  constexpr int kPk = D * 2 + 16, kPv = DV * 2 + 16, kStage = kMmaKeys * (kPk + kPv);
  constexpr int kVk = D / 8, kVv = DV / 8;               // 16-byte pieces of a key, of a value
  extern __shared__ __align__(128) unsigned char smem[];
  const int G = p.heads / p.kv_heads, tiles = (G + kRows - 1) / kRows;
  const int split = blockIdx.x, kvh = blockIdx.y / tiles, g0 = blockIdx.y % tiles * kRows, b = blockIdx.z;
  const int n_heads = min(kRows, G - g0), h0 = kvh * G + g0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = lane >> 2, quad = lane & 3;

  const int pos = p.pos[b], lo = max(0, pos - p.window + 1), total = pos - lo + 1;
  int per = (total + p.splits - 1) / p.splits;
  per = (per + kMmaKeys - 1) / kMmaKeys * kMmaKeys;
  const int k0 = split * per, k1 = min(total, k0 + per);
  const int n_blocks = k1 > k0 ? (k1 - k0 + kMmaKeys - 1) / kMmaKeys : 0;
  const int width = p.kv_heads * (D + DV), n_ring = (int)p.ring_rows, lo_row = lo % n_ring;
  const __nv_bfloat16* ring = p.ring + (long long)p.slot[b] * p.ring_rows * width;
  const int k_col = kvh * D, v_col = p.kv_heads * D + kvh * DV;

  uint32_t qa[D / 16][4];
#pragma unroll
  for (int j = 0; j < D / 16; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {                          // rows g, g + 8; columns 2 quad, 2 quad + 8
      const int r = row + 8 * (e & 1);
      qa[j][e] = r < n_heads ? *reinterpret_cast<const uint32_t*>(p.q + b * p.q_row + (long long)(h0 + r) * D + 16 * j + 2 * quad + 8 * (e >> 1)) : 0u;
    }
  grid_launch_dependents();
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem) + warp * kMmaStages * kStage;
  auto issue = [&](int blk, int stage) {
    const uint32_t kdst = base + stage * kStage, vdst = kdst + kMmaKeys * kPk;
    auto source = [&](int r, int col, bool& on) {
      const int k = k0 + blk * kMmaKeys + r;
      on = k < k1;
      int at = lo_row + (on ? k : k0);                     // both terms are below the ring's size
      at = at >= n_ring ? at - n_ring : at;
      return ring + (long long)at * width + col;
    };
#pragma unroll
    for (int c = 0; c < kMmaKeys * kVk / 32; ++c) {
      const int i = lane + 32 * c, r = i / kVk, ch = i % kVk;
      bool on;
      const __nv_bfloat16* src = source(r, k_col + ch * 8, on);
      cp_async16(kdst + r * kPk + ch * 16, src, on ? 16u : 0u);
    }
#pragma unroll
    for (int c = 0; c < kMmaKeys * kVv / 32; ++c) {
      const int i = lane + 32 * c, r = i / kVv, ch = i % kVv;
      bool on;
      const __nv_bfloat16* src = source(r, v_col + ch * 8, on);
      cp_async16(vdst + r * kPv + ch * 16, src, on ? 16u : 0u);
    }
  };
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const int my_n = n_blocks > warp ? (n_blocks - warp + kMmaWarps - 1) / kMmaWarps : 0;
#pragma unroll
  for (int s = 0; s < kMmaStages - 1; ++s) {
    if (s < my_n) issue(warp + s * kMmaWarps, s);
    cp_async_commit();
  }
  for (int it = 0; it < my_n; ++it) {
    cp_async_wait<kMmaStages - 2>();
    __syncwarp();
    const int blk = warp + it * kMmaWarps, stage = it % kMmaStages;
    {  // refill the stage that was consumed in the previous iteration
      const int nxt = it + kMmaStages - 1;
      if (nxt < my_n) issue(warp + nxt * kMmaWarps, nxt % kMmaStages);
      cp_async_commit();
    }
    const uint32_t kbuf = base + stage * kStage, vbuf = kbuf + kMmaKeys * kPk;
    const int mi = lane >> 3, r8 = lane & 7;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};      // 16 keys: two octets
    {
      const uint32_t a = kbuf + ((mi >> 1) * 8 + r8) * kPk + (mi & 1) * 16;
#pragma unroll
      for (int j = 0; j < D / 16; ++j) {
        uint32_t x[4];
        ldmatrix_x4(a + j * 32, x[0], x[1], x[2], x[3]);
        group_mma(s[0], qa[j], x[0], x[1]);
        group_mma(s[1], qa[j], x[2], x[3]);
      }
    }
    const int key = k0 + blk * kMmaKeys + 2 * quad;
    float f[2] = {1.f, 1.f};
    uint32_t pa[4] = {0u, 0u, 0u, 0u};
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      float v00 = key < k1 ? s[0][2 * e] * p.scale_log2e : -INFINITY;
      float v01 = key + 1 < k1 ? s[0][2 * e + 1] * p.scale_log2e : -INFINITY;
      float v10 = key + 8 < k1 ? s[1][2 * e] * p.scale_log2e : -INFINITY;
      float v11 = key + 9 < k1 ? s[1][2 * e + 1] * p.scale_log2e : -INFINITY;
      float mx = fmaxf(fmaxf(v00, v01), fmaxf(v10, v11));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m_run[e], mx);              // finite: every issued block has a valid key
      f[e] = exp2f(m_run[e] - m_new);
      v00 = exp2f(v00 - m_new); v01 = exp2f(v01 - m_new); v10 = exp2f(v10 - m_new); v11 = exp2f(v11 - m_new);
      float sum = (v00 + v01) + (v10 + v11);
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      l_run[e] = l_run[e] * f[e] + sum;
      m_run[e] = m_new;
      pa[e] = pack_bf16(v00, v01);
      pa[2 + e] = pack_bf16(v10, v11);
    }
    const uint32_t a = vbuf + ((mi & 1) * 8 + r8) * kPv + (mi >> 1) * 16;
#pragma unroll
    for (int nb = 0; nb < DV / 8; nb += 2) {
      uint32_t x[4];
      ldmatrix_x4_trans(a + nb * 16, x[0], x[1], x[2], x[3]);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        o[nb + u][0] *= f[0]; o[nb + u][1] *= f[0]; o[nb + u][2] *= f[1]; o[nb + u][3] *= f[1];
        group_mma(o[nb + u], pa, x[2 * u], x[2 * u + 1]);
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();                                           // every ring is idle: shared memory serves the merge
  float* s_o = reinterpret_cast<float*>(smem);               // [warp][kRows][DV]
  float* s_m = s_o + kMmaWarps * kRows * DV;
  float* s_l = s_m + kMmaWarps * kRows;
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int r = warp * kRows + row + 8 * e;
#pragma unroll
    for (int nb = 0; nb < DV / 8; ++nb)
      *reinterpret_cast<float2*>(s_o + r * DV + nb * 8 + 2 * quad) = make_float2(o[nb][2 * e], o[nb][2 * e + 1]);
    if (quad == 0) { s_m[r] = m_run[e]; s_l[r] = l_run[e]; }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n_heads * DV; i += kMmaWarps * 32) {
    const int r = i / DV, d = i % DV, h = h0 + r;
    const bool sink = p.sink && p.splits == 1;
    float m = sink ? 0.f : -INFINITY;
#pragma unroll
    for (int w = 0; w < kMmaWarps; ++w) m = fmaxf(m, s_m[w * kRows + r]);
    float l = sink ? exp2f(-m) : 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < kMmaWarps; ++w) {
      const float mw = s_m[w * kRows + r];
      if (mw > -INFINITY) {
        const float e = exp2f(mw - m);
        l += s_l[w * kRows + r] * e;
        acc += s_o[(w * kRows + r) * DV + d] * e;
      }
    }
    if (p.splits == 1) {
      const float g = p.gate ? sigmoid_f(__bfloat162float(p.gate[b * p.gate_row + h])) : 1.f;
      p.out[b * p.out_row + (long long)h * DV + d] = __float2bfloat16_rn(acc * (g / l));
    } else {
      const long long at = ((long long)b * p.heads + h) * p.splits + split;
      p.part_o[at * DV + d] = acc;
      if (d == 0) { p.part_ml[at * 2] = m; p.part_ml[at * 2 + 1] = l; }
    }
  }
}

template <int D, int DV, bool FULL>
int launch_group_decode(const GroupDecodeParams& p, int n, cudaStream_t stream) {
  constexpr int kRows = FULL ? 16 : 8;
  constexpr size_t ring = (size_t)kMmaWarps * kMmaStages * kMmaKeys * (D * 2 + 16 + DV * 2 + 16);
  constexpr size_t merge = (size_t)kMmaWarps * kRows * (DV + 2) * 4;
  constexpr size_t smem = ring > merge ? ring : merge;
  static DeviceSmem configured{};
  MSA_OK_OR_RETURN(ensure_dynamic_smem(group_decode_kernel<D, DV, FULL>, smem, configured));
  const int G = p.heads / p.kv_heads, tiles = (G + kRows - 1) / kRows;
  group_decode_kernel<D, DV, FULL><<<dim3((unsigned)p.splits, (unsigned)(p.kv_heads * tiles), (unsigned)n), kMmaWarps * 32, smem, stream>>>(p);
  MSA_LAUNCH_OK("group_decode_kernel");
  if (p.splits > 1) {
    const MergeParams m{p.part_o, p.part_ml, p.heads, p.splits, DV, p.sink, p.gate, p.gate_row, p.out, p.out_row};
    return launch_merge(m, n, stream);
  }
  return MSA_OK;
}
template <int D, int DV>
int launch_group_decode_any(const GroupDecodeParams& p, int n, cudaStream_t stream) {
  return p.heads / p.kv_heads > 8 ? launch_group_decode<D, DV, true>(p, n, stream) : launch_group_decode<D, DV, false>(p, n, stream);
}

}  // namespace msa

using namespace msa;

extern "C" int msa_lm_group_prep(const msa_lm_group_args* args, void* stream) {
  MSA_REQUIRE(args, "group_prep: null arguments");
  const msa_lm_group_args a = *args;
  MSA_REQUIRE(dtype_ok(a.dtype) && a.proj && a.conv_w && a.q_out && a.ring && a.pos && a.tok_seq && a.slot && a.start && a.cu,
              "group_prep: null pointer or bad dtype");
  MSA_REQUIRE(a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0 && a.rot >= 0 && a.rot % 2 == 0 &&
                  a.rot <= a.dim && a.rot <= 4096 && a.window > 0 && a.ring_rows > 0, "group_prep: bad sizes");
  MSA_REQUIRE(a.q_pitch >= a.dim && a.k_pitch >= a.dim && a.v_pitch >= a.vdim, "group_prep: a pitch is below its head size");
  MSA_REQUIRE(a.taps >= 1 && (a.taps == 1 || a.conv_state) && (a.rot == 0 || a.inv_freq), "group_prep: convolution state or angles missing");
  MSA_REQUIRE(a.n_decode >= 0 && a.n_decode <= a.n_seq && a.n_tok >= a.n_decode && a.n_old >= 0, "group_prep: bad counts");
  MSA_REQUIRE(a.n_seq == a.n_decode || (a.ctx && a.ctx_off && a.old_off), "group_prep: portions need a context");
  if (a.n_tok == 0) return MSA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const GroupLayout L(a);
  const int e4 = 4 * (int)dtype_size(a.dtype);
  auto ok4 = [&](const void* q) { return q == nullptr || reinterpret_cast<uintptr_t>(q) % e4 == 0; };
  const size_t turn = (size_t)a.rot * 4;         // a row's cosines and sines
  if (a.taps <= 4 && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.proj_stride % 4 == 0 && a.q_pitch % 4 == 0 && a.k_pitch % 4 == 0 &&
      a.v_pitch % 4 == 0 && kGpRows * turn <= 48 * 1024 && ok4(a.proj) && ok4(a.conv_state) && ok4(a.q_out) && ok4(a.ring) && ok4(a.ctx) &&
      aligned16(a.conv_w)) {
    const int rows = a.n_tok <= 256 ? 1 : kGpRows, row_blocks = (a.n_tok + rows - 1) / rows;
    const dim3 grid((unsigned)(row_blocks + a.n_old), (unsigned)((L.chan + 1023) / 1024));
    MSA_LM_DISPATCH(a.dtype, {
      switch (a.taps) {
        case 1: group_prep_vec_kernel<T, 1><<<grid, 256, rows * turn, st>>>(a, row_blocks, rows); break;
        case 2: group_prep_vec_kernel<T, 2><<<grid, 256, rows * turn, st>>>(a, row_blocks, rows); break;
        case 3: group_prep_vec_kernel<T, 3><<<grid, 256, rows * turn, st>>>(a, row_blocks, rows); break;
        default: group_prep_vec_kernel<T, 4><<<grid, 256, rows * turn, st>>>(a, row_blocks, rows);
      }
    });
    MSA_LAUNCH_OK("group_prep_vec_kernel");
    return MSA_OK;
  }
  MSA_LM_DISPATCH(a.dtype, { group_prep_kernel<T><<<a.n_tok + a.n_old, 256, turn, st>>>(a); });
  MSA_LAUNCH_OK("group_prep_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_conv_store(const void* proj, int64_t proj_stride, int32_t channels, int32_t taps, void* conv_state,
                                 const int32_t* slot, const int32_t* start, const int32_t* cu, int32_t n_seq, int32_t n_decode,
                                 int32_t dtype, void* stream) {
  MSA_REQUIRE(dtype_ok(dtype) && proj && slot && start && cu && channels > 0 && taps >= 1 && (taps == 1 || conv_state), "conv_store: bad arguments");
  if (n_seq <= n_decode || taps == 1) return MSA_OK;
  const dim3 grid((unsigned)((channels + 255) / 256), (unsigned)(n_seq - n_decode));
  MSA_LM_DISPATCH(dtype, {
    conv_store_kernel<T><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)proj, proj_stride, channels, taps, (T*)conv_state, slot, start, cu, n_decode);
  });
  MSA_LAUNCH_OK("conv_store_kernel");
  return MSA_OK;
}

extern "C" int msa_lm_group_decode_supported(int32_t dim, int32_t vdim) { return (dim == 64 || dim == 128) && (vdim == 64 || vdim == 128); }

extern "C" int msa_lm_group_decode(const void* q, int64_t q_row, const void* ring, int64_t ring_rows, const int32_t* slot,
                                   const int32_t* pos, int32_t n, int32_t heads, int32_t kv_heads, int32_t dim, int32_t vdim,
                                   int32_t window, int32_t splits, float scale, int32_t sink, const void* gate, int64_t gate_row,
                                   void* out, int64_t out_row, float* part_o, float* part_ml, void* stream) {
  MSA_REQUIRE(q && ring && slot && pos && out, "group_decode: null pointer");
  MSA_REQUIRE(msa_lm_group_decode_supported(dim, vdim) && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && window > 0 &&
                  ring_rows > 0 && ring_rows < (1ll << 30), "group_decode: bad sizes");
  MSA_REQUIRE(splits >= 1 && splits <= 64 && (splits == 1 || (part_o && part_ml)), "group_decode: bad splits");
  MSA_REQUIRE(aligned16(q) && aligned16(ring) && q_row % 8 == 0 && reinterpret_cast<uintptr_t>(out) % 8 == 0 && out_row % 4 == 0 &&
                  (splits == 1 || (aligned16(part_o) && aligned16(part_ml))), "group_decode: alignment");
  if (n <= 0) return MSA_OK;
  const GroupDecodeParams p{(const __nv_bfloat16*)q, q_row, (const __nv_bfloat16*)ring, ring_rows, slot, pos, heads, kv_heads, window, splits,
                            sink, scale * 1.4426950408889634f, (const __nv_bfloat16*)gate, gate_row, (__nv_bfloat16*)out, out_row, part_o, part_ml};
  cudaStream_t st = (cudaStream_t)stream;
  if (dim == 64) return vdim == 64 ? launch_group_decode_any<64, 64>(p, n, st) : launch_group_decode_any<64, 128>(p, n, st);
  return vdim == 64 ? launch_group_decode_any<128, 64>(p, n, st) : launch_group_decode_any<128, 128>(p, n, st);
}
