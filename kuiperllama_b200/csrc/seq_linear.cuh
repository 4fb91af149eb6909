// What the kernels of linear attention share: the rotation of its queries and keys, and powers of its decay.
#pragma once
#include <cuda_runtime.h>

#include "seq_engine.h"

namespace kllm {
namespace seq {
namespace {

struct LinearRot {
  RopeArgs rope;   // dims == 0: none
  float k_scale;
};
inline LinearRot linear_rot(const kllm_seq_linear& m) {
  return LinearRot{RopeArgs{m.rope_dims, m.rope_base, m.rope_freq, 1.0f, m.rope_pairing}, m.k_scale == 0.f ? 1.0f : m.k_scale};
}
// cos and sin of pair i at a position
__device__ __forceinline__ void rope_turn(const RopeArgs& r, int i, int pos, float& co, float& si) {
  const float f = r.freq ? r.freq[i] : powf(r.base, -2.0f * static_cast<float>(i) / static_cast<float>(r.dims));
  const float a = static_cast<float>(pos) * f;
  co = cosf(a), si = sinf(a);
}
// decay^n from its logarithm (n >= 0; a decay of 0 has the logarithm -inf)
__device__ __forceinline__ float decay_power(float log_decay, int n) { return n == 0 ? 1.0f : expf(log_decay * static_cast<float>(n)); }

}  // namespace
}  // namespace seq
}  // namespace kllm
