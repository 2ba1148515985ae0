// Merge of the partial results of a split decode attention: weights e^(m_i - m), a sink, an output gate.
#pragma once
#include "lm_common.cuh"

namespace msa {

struct MergeParams {
  const float *part_o, *part_ml;     // [rows, splits, cols], [rows, splits, 2] (maximum in log2 units, sum)
  int heads, splits, cols;
  int sink;                          // one more entry with score 0 and no value
  const __nv_bfloat16* gate; long long gate_row;   // null, or a logit per (sequence, head)
  __nv_bfloat16* out; long long out_row;           // row stride of a sequence; heads are cols apart
};

// One block per (sequence, head).  Launched early (programmatic dependent launch): waits for the partial results before
// it reads them.
static __global__ void __launch_bounds__(128) merge_partials_kernel(const MergeParams p) {
  const long long row = blockIdx.x;
  const int b = (int)(row / p.heads), h = (int)(row % p.heads);
  const int c = threadIdx.x * 4, splits = p.splits, cols = p.cols;
  const float g = p.gate ? sigmoid_f(__bfloat162float(p.gate[b * p.gate_row + h])) : 1.f;   // older than the partial results
  grid_dependency_wait();
  float m = p.sink ? 0.f : -INFINITY, l = p.sink ? 1.f : 0.f;
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int s0 = 0; s0 < splits; s0 += 8) {               // eight partial results in flight; an empty one has weight 0
    float4 v[8];
    float2 ml[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool on = s0 + i < splits;
      ml[i] = on ? *reinterpret_cast<const float2*>(p.part_ml + (row * splits + s0 + i) * 2) : make_float2(-INFINITY, 0.f);
      v[i] = on && c < cols ? load4(p.part_o + (row * splits + s0 + i) * cols + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float mx = m;
#pragma unroll
    for (int i = 0; i < 8; ++i) mx = fmaxf(mx, ml[i].x);
    const float f = m == -INFINITY ? 0.f : exp2f(m - mx);
    l *= f; a.x *= f; a.y *= f; a.z *= f; a.w *= f;
    m = mx;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float w = ml[i].x == -INFINITY ? 0.f : exp2f(ml[i].x - m);
      l = fmaf(w, ml[i].y, l);
      a.x = fmaf(w, v[i].x, a.x); a.y = fmaf(w, v[i].y, a.y); a.z = fmaf(w, v[i].z, a.z); a.w = fmaf(w, v[i].w, a.w);
    }
  }
  const float inv = g / l;
  if (c < cols) store4(p.out + b * p.out_row + (long long)h * cols + c, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv));
}

inline int launch_merge(const MergeParams& p, int n, cudaStream_t stream) {
  MSA_CUDA_OK(launch_kernel_pdl(merge_partials_kernel, dim3((unsigned)(n * p.heads)), dim3(128), 0, stream, true, p));
  return MSA_OK;
}

}  // namespace msa
