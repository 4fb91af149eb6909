// Joining the key splits of an attention: every (token, head) left `splits` partial results (max, sum, unnormalised output) of
// `pstride` floats side by side.
#pragma once
#include <cuda_runtime.h>

namespace kllm {
namespace seq {
namespace {

// Run by one whole warp: weight[s] = exp(m_s - M) / L, so that the joined output is sum_s weight[s] * o_s.  A sink adds
// exp(sink) to L (no key, no value).  Splits that saw no key get weight 0.
__device__ __forceinline__ void split_weights(const float* __restrict__ p, int splits, int pstride, bool has_sink, float sink,
                                              float* weight) {
  const int lane = threadIdx.x & 31;
  float M = has_sink ? sink : -INFINITY;
  for (int s = lane; s < splits; s += 32) M = fmaxf(M, p[s * pstride]);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
  float L = 0.f;
  for (int s = lane; s < splits; s += 32) {
    const float m = p[s * pstride];
    const float w = m > -INFINITY ? expf(m - M) : 0.f;
    weight[s] = w;
    L += w * p[s * pstride + 1];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
  if (has_sink) L += expf(sink - M);
  for (int s = lane; s < splits; s += 32) weight[s] /= L;
}

// sum_s weight[s] * o_s[d]; the first kAhead values of a column are loaded before the weights are needed
constexpr int kMergeAhead = 16;
struct MergeColumn {
  float v[kMergeAhead];
  __device__ __forceinline__ void load(const float* __restrict__ p, int splits, int pstride, int d) {
#pragma unroll
    for (int s = 0; s < kMergeAhead; ++s) v[s] = s < splits ? p[s * pstride + 2 + d] : 0.f;
  }
  __device__ __forceinline__ float join(const float* __restrict__ p, int splits, int pstride, int d, const float* weight) const {
    float o = 0.f;
#pragma unroll
    for (int s = 0; s < kMergeAhead; ++s)
      if (s < splits && weight[s] > 0.f) o = fmaf(weight[s], v[s], o);  // a split without keys is not read into the sum
    for (int s = kMergeAhead; s < splits; ++s)
      if (weight[s] > 0.f) o = fmaf(weight[s], p[s * pstride + 2 + d], o);
    return o;
  }
};

}  // namespace
}  // namespace seq
}  // namespace kllm
