// Shared device code of the dense (bf16 / fp32) operators: output segments and their activations.
#pragma once
#include <cuda_bf16.h>

#include "greta_common.cuh"

namespace greta {

struct Segments {
  greta_out_segment s[GRETA_MAX_SEGMENTS];
  uint32_t n;
};

__device__ __forceinline__ float act_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float act_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float apply_act(int act, float z, float rate = 0.f) {
  switch (act) {
    case GRETA_ACT_GELU_ERF: return 0.5f * z * (1.f + erff(z * 0.70710678118654752f));
    case GRETA_ACT_SIGMOID: return act_sigmoid(z);
    case GRETA_ACT_TANH: return tanhf(z);
    case GRETA_ACT_DELTA_DECAY: return expf(-0.60653065971263342f * act_sigmoid(z));
    case GRETA_ACT_RELU2: return z > 0.f ? z * z : 0.f;
    case GRETA_ACT_SOFTPLUS_DECAY: return expf(-rate * act_softplus(z));
    default: return z;
  }
}
// Segment of a weight row (segments are in row order and cover all rows).
__device__ __forceinline__ int segment_of(const Segments &sg, uint32_t row) {
  int i = 0;
  while (i + 1 < (int)sg.n && row >= sg.s[i + 1].row0) ++i;
  return i;
}
__device__ __forceinline__ void store_out(void *out, int fmt, size_t idx, float v, uint32_t pair_offset = 0) {
  if (fmt == GRETA_OUT_F32) {
    static_cast<float *>(out)[idx] = v;
  } else if (fmt == GRETA_OUT_F16) {
    static_cast<__half *>(out)[idx] = __float2half_rn(v);
  } else {
    const __nv_bfloat16 hi = __float2bfloat16_rn(v);
    static_cast<__nv_bfloat16 *>(out)[idx] = hi;
    if (fmt == GRETA_OUT_BF16_PAIR) static_cast<__nv_bfloat16 *>(out)[idx + pair_offset] = __float2bfloat16_rn(v - __bfloat162float(hi));
  }
}
// old: what is there already, for segments that accumulate.
__device__ __forceinline__ void store_segment(const greta_out_segment &g, uint32_t row, uint32_t m, float z, float old) {
  const uint32_t r = row - g.row0;
  if (g.bias) z += __ldg(g.bias + r);
  z = apply_act(g.act, z, g.rate ? __ldg(g.rate + r) : 0.f);
  const size_t idx = (size_t)m * g.ld + g.col0 + r;
  if (g.accumulate)
    static_cast<float *>(g.out)[idx] = old + z;
  else
    store_out(g.out, g.out_fmt, idx, z, g.pair_offset);
}
__device__ __forceinline__ void store_segment(const greta_out_segment &g, uint32_t row, uint32_t m, float z) {
  store_segment(g, row, m, z, g.accumulate ? static_cast<float *>(g.out)[(size_t)m * g.ld + g.col0 + row - g.row0] : 0.f);
}

__device__ __forceinline__ float block_sum_all(float v, float *sm) {  // every thread receives the total; sm: 32 floats
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) sm[w] = v;
  __syncthreads();
  return warp_sum(l < nw ? sm[l] : 0.f);
}

}  // namespace greta
