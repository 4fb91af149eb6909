// Residual streams joined by hyper-connections: the step between two sublayers.
//
// The residual of a token is S rows x_1 .. x_S (fp32).  One kernel ends a sublayer and starts the next:
//     x_t <- sum_s mix[s][t] x_s + out_w[t] y        all streams at once from the old ones
//     u   =  sum_s in_w[s] x_s                       what the next sublayer reads (in_w null: the plain sum)
//     out =  N(u; pre)                               in the compute type
// Every stream element is read once and written once: a thread keeps the S old values of its columns in registers, writes the
// new ones, and leaves u in shared memory for the norm.  Bound by the bytes of the streams (prompts) or by one round trip to
// memory (single-token steps).
//
// Until the first sublayer ends, all streams equal the embedding output: that step reads the [T, width] embedding rows
// (src_shared) and is the first to write streams.  The last step of a model gathers the wanted rows and writes no streams.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <cstdint>

#include "seq_engine.h"

namespace kllm {
namespace seq {
namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];
  return t;
}

// V consecutive columns of a row: one 16-byte access, or one float
template <int V> struct Cols;
template <> struct Cols<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
};
template <> struct Cols<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *p = __float2bfloat16_rn(v[0]); }
};

// One CTA per row.  S: streams the kernel is compiled for; n <= S are used (n == S except in the last instantiation, whose
// coefficients are read where they are used instead of being kept in registers).
template <typename AT, int S, int V, bool EXACT>
__global__ void __launch_bounds__(512)
streams_kernel(StreamArgs a) {
  extern __shared__ __align__(16) float us[];  // [width]
  __shared__ float red[33];
  const int W = a.width, n = EXACT ? S : a.streams;
  const size_t row = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  const float* src = a.src + row * W * (a.src_shared ? 1 : n);
  float* dst = a.dst ? a.dst + row * W * n : nullptr;
  const float* y = a.y ? a.y + row * W : nullptr;
  float mix[EXACT ? S : 1][EXACT ? S : 1], ow[EXACT ? S : 1], iw[EXACT ? S : 1];
  if constexpr (EXACT) {
#pragma unroll
    for (int s = 0; s < S; ++s) {
      iw[s] = a.in_w ? __ldg(a.in_w + s) : 1.0f;
      if (y) {
        ow[s] = __ldg(a.out_w + s);
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s][t] = __ldg(a.mix + s * S + t);
      }
    }
  }
  float s1 = 0.f, s2 = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    Cols<V> x[S], u;
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (!EXACT && s >= n) break;
      if (s == 0 || !a.src_shared) x[s].load(src + static_cast<size_t>(s) * W + i);
      else x[s] = x[0];
    }
#pragma unroll
    for (int c = 0; c < V; ++c) u.v[c] = 0.f;
    if (y) {
      Cols<V> yv;
      yv.load(y + i);
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (!EXACT && t >= n) break;
        const float o = EXACT ? ow[t] : __ldg(a.out_w + t);
        const float r = EXACT ? iw[t] : (a.in_w ? __ldg(a.in_w + t) : 1.0f);
        Cols<V> z;
#pragma unroll
        for (int c = 0; c < V; ++c) z.v[c] = o * yv.v[c];
#pragma unroll
        for (int s = 0; s < S; ++s) {
          if (!EXACT && s >= n) break;
          const float m = EXACT ? mix[s][t] : __ldg(a.mix + s * n + t);
#pragma unroll
          for (int c = 0; c < V; ++c) z.v[c] = fmaf(m, x[s].v[c], z.v[c]);
        }
        if (dst) z.store(dst + static_cast<size_t>(t) * W + i);
#pragma unroll
        for (int c = 0; c < V; ++c) u.v[c] = fmaf(r, z.v[c], u.v[c]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (!EXACT && s >= n) break;
        const float r = EXACT ? iw[s] : (a.in_w ? __ldg(a.in_w + s) : 1.0f);
#pragma unroll
        for (int c = 0; c < V; ++c) u.v[c] = fmaf(r, x[s].v[c], u.v[c]);
      }
    }
    u.store(us + i);
    if (a.sum_out) u.store(a.sum_out + static_cast<size_t>(blockIdx.x) * W + i);
#pragma unroll
    for (int c = 0; c < V; ++c) s1 += u.v[c], s2 = fmaf(u.v[c], u.v[c], s2);
  }
  if (!a.out) return;
  const float inv_w = 1.0f / static_cast<float>(W);
  float mean = 0.f, rstd = 1.0f;
  if (a.pre.kind == KLLM_SEQ_NORM_RMS) {
    rstd = 1.0f / sqrtf(block_sum(s2, red) * inv_w + a.eps);
  } else if (a.pre.kind == KLLM_SEQ_NORM_LAYER) {
    mean = block_sum(s1, red) * inv_w;
    float q = 0.f;
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V)  // the thread's own columns
#pragma unroll
      for (int c = 0; c < V; ++c) q += (us[i + c] - mean) * (us[i + c] - mean);
    rstd = 1.0f / sqrtf(block_sum(q, red) * inv_w + a.eps);
  }
  AT* out = static_cast<AT*>(a.out) + static_cast<size_t>(blockIdx.x) * W;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    Cols<V> u, g;
    u.load(us + i);
    if (a.pre.kind != KLLM_SEQ_NORM_NONE) {
      g.load(a.pre.w + i);
#pragma unroll
      for (int c = 0; c < V; ++c) u.v[c] = (u.v[c] - mean) * rstd * g.v[c];
      if (a.pre.b) {
        g.load(a.pre.b + i);
#pragma unroll
        for (int c = 0; c < V; ++c) u.v[c] += g.v[c];
      }
    }
    u.store(out + i);
  }
}

template <typename AT, int S, bool EXACT>
int launch_s(const StreamArgs& a, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(a.width) * sizeof(float);
  if (smem > 48 * 1024) return KLLM_E_UNSUPPORTED;
  const bool vec = a.width % 4 == 0;
  const int per = vec ? (a.width + 3) / 4 : a.width;
  // few rows: as many loads in flight as a row has; many rows: several CTAs per SM, so that one's reduction hides behind the
  // others' loads
  const int threads = std::max(64, std::min(a.T <= 16 ? 512 : 256, (per + 31) / 32 * 32));
  if (vec) streams_kernel<AT, S, 4, EXACT><<<a.T, threads, smem, s>>>(a);
  else streams_kernel<AT, S, 1, EXACT><<<a.T, threads, smem, s>>>(a);
  count_launch();
  return cuda_rc(cudaGetLastError());
}

template <typename AT>
int launch_at(const StreamArgs& a, cudaStream_t s) {
  switch (a.streams) {
    case 1: return launch_s<AT, 1, true>(a, s);
    case 2: return launch_s<AT, 2, true>(a, s);
    case 3: return launch_s<AT, 3, true>(a, s);
    case 4: return launch_s<AT, 4, true>(a, s);
    case 5: return launch_s<AT, 5, true>(a, s);
    case 6: return launch_s<AT, 6, true>(a, s);
    default: return launch_s<AT, kMaxStreams, false>(a, s);
  }
}
}  // namespace

int launch_streams(const StreamArgs& a, cudaStream_t s) {
  if (!a.src || a.T <= 0 || a.width <= 0 || a.streams < 1 || (a.y && (!a.mix || !a.out_w)) || (a.rows && a.dst) ||
      (a.dst && !a.y) || (a.out && a.pre.kind != KLLM_SEQ_NORM_NONE && !a.pre.w))
    return KLLM_E_INVALID;
  if (a.streams > kMaxStreams) return KLLM_E_UNSUPPORTED;
  if (a.dtype == KLLM_SEQ_F32) return launch_at<float>(a, s);
  if (a.dtype == KLLM_SEQ_BF16) return launch_at<__nv_bfloat16>(a, s);
  return KLLM_E_INVALID;
}

}  // namespace seq
}  // namespace kllm
