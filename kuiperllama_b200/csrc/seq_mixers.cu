// Kernels of the mixers that keep something other than per-head keys and values, and of the dense feed-forward:
//
//   attention through a latent   latent_prepare (RMS norms of the two down-projections, rotation of the shared key part,
//                                scatter of [latent | rotated part] into the pages, gates), latent_absorb (a head's plain
//                                query dimensions carried into the latent space, W_uk^T q, and the rotation of its rotated
//                                dimensions), latent_expand (W_uv on the weighted sum of latents).  Between absorb and expand
//                                the paged attention kernel of seq_kernels.cu runs with one key/value "head" of
//                                kv_rank + rot_dim key and kv_rank value dimensions that every query head shares.
//   linear attention             the decayed-state recurrence, chunk by chunk (activated, or rotated as a retention), and its output
//                                norm with the gate; single tokens in one kernel.  bf16 steps with long entries: seq_linear_mma.cu
//   activations                  xIELU and squared ReLU between the two products of a dense feed-forward
//
// Positions and angles, norms, gates, decays and the recurrent state are fp32 in both compute types.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cstdint>

#include "seq_engine.h"
#include "seq_linear.cuh"
#include "seq_merge.cuh"

namespace kllm {
namespace seq {
namespace {

constexpr unsigned kAll = 0xffffffffu;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename AT> __device__ __forceinline__ AT from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(kAll, v, o);
  return v;
}
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];
  return t;
}
__device__ __forceinline__ float sigmoidf(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float siluf(float z) { return z / (1.0f + expf(-z)); }

// V consecutive values of the compute type (16 bytes, or one value), widened to fp32
template <typename AT> struct Wide;
template <> struct Wide<float> {
  static constexpr int N = 4;
  template <int V> __device__ static __forceinline__ void load(const float* __restrict__ p, float* f) {
    if constexpr (V == 4) {
      const float4 v = __ldg(reinterpret_cast<const float4*>(p));
      f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
    } else {
      f[0] = __ldg(p);
    }
  }
};
template <> struct Wide<__nv_bfloat16> {
  static constexpr int N = 8;
  template <int V> __device__ static __forceinline__ void load(const __nv_bfloat16* __restrict__ p, float* f) {
    if constexpr (V == 8) {
      const uint4 v = __ldg(reinterpret_cast<const uint4*>(p));
      const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(u[i] << 16);
        f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
      }
    } else {
      f[0] = to_f(p[0]);
    }
  }
};

// V consecutive fp32 values (16 bytes, or one)
template <int V> __device__ __forceinline__ void get_floats(const float* p, float* f) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
  } else {
    f[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void put_values(float* p, const float* f) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *p = f[0];
}
template <int V> __device__ __forceinline__ void put_values(__nv_bfloat16* p, const float* f) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(f[0]);
  }
}

// frequency of rotated pair j
__device__ __forceinline__ float rope_frequency(const LatentShape& a, int j) {
  if (a.rope_freq) return __ldg(a.rope_freq + j);
  return exp2f(-2.0f * static_cast<float>(j) / static_cast<float>(a.rope_dims) * log2f(a.rope_base));
}

// Rotary position: coordinate i < dims / 2 pairs with i + dims / 2 (or 2i with 2i + 1); angle of pair i = pos * freq[i], or
// pos * base^(-2 i / dims) without a table; coordinates past `dims` pass unchanged.  v: the vector before rotation.
__device__ __forceinline__ float rotated(const LatentShape& a, const float* v, int i, int pos) {
  const int dims = a.rope_dims;
  if (i >= dims) return v[i];
  const int half = dims >> 1;
  const bool pairs = a.rope_pairing == KLLM_SEQ_ROPE_PAIRS;
  const int j = pairs ? i >> 1 : (i < half ? i : i - half);
  float sn, cs;
  sincosf(static_cast<float>(pos) * rope_frequency(a, j), &sn, &cs);
  if (pairs) return (i & 1) == 0 ? v[i] * cs - v[i + 1] * sn : v[i] * cs + v[i - 1] * sn;
  return i < half ? v[i] * cs - v[i + half] * sn : v[i] * cs + v[i - half] * sn;
}

// ---- latent attention: down-projections -> normed query latent, cache row, gates -----------------------------------------
template <typename AT>
__global__ void latent_prepare_kernel(LatentShape a, const float* __restrict__ proj, const float* __restrict__ q_norm_w,
                                      const float* __restrict__ kv_norm_w, float eps, const int32_t* __restrict__ tok_seq,
                                      const int32_t* __restrict__ tok_pos, AT* __restrict__ cq, float* __restrict__ gates,
                                      PagedKV kv, AT* __restrict__ c_rows, float* __restrict__ kr_rows) {
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int stride = latent_proj_rows(a);
  const float* row = proj + static_cast<size_t>(t) * stride;
  const int seq = tok_seq[t], pos = tok_pos[t];
  float ss = 0.f;
  if (a.q_rank > 0) {
    for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) ss += row[i] * row[i];
    const float rq = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(a.q_rank) + eps);
    for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x)
      cq[static_cast<size_t>(t) * a.q_rank + i] = from_f<AT>(row[i] * rq * q_norm_w[i]);
  }
  const float* c = row + latent_query_rows(a);
  ss = 0.f;
  for (int i = threadIdx.x; i < a.kv_rank; i += blockDim.x) ss += c[i] * c[i];
  const float rc = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(a.kv_rank) + eps);
  const int page = kv.table[static_cast<size_t>(seq) * kv.table_stride + pos / kv.page];
  AT* dst = static_cast<AT*>(kv.k) + (static_cast<size_t>(page) * kv.page + pos % kv.page) * kv.k_row;
  for (int i = threadIdx.x; i < a.kv_rank; i += blockDim.x) {
    const AT v = from_f<AT>(c[i] * rc * kv_norm_w[i]);
    dst[i] = v;
    if (c_rows) c_rows[static_cast<size_t>(t) * a.kv_rank + i] = v;
  }
  const float* kr = c + a.kv_rank;
  for (int i = threadIdx.x; i < a.rot_dim; i += blockDim.x) {
    const float v = rotated(a, kr, i, pos);
    dst[a.kv_rank + i] = from_f<AT>(v);
    if (kr_rows) kr_rows[static_cast<size_t>(t) * a.rot_dim + i] = v;
  }
  const float* g = kr + a.rot_dim;
  for (int h = threadIdx.x; a.gate && h < a.heads; h += blockDim.x) gates[static_cast<size_t>(t) * a.heads + h] = sigmoidf(g[h]);
}

// ---- latent attention: queries into the latent space --------------------------------------------------------------------
// One CTA: kAbsTokens tokens of one head.  qa[t, h, r] = sum_d q[t, h, d] * W_uk[h * dim + d, r]: thread r walks the
// rows d of the head's block of W_uk (coalesced over r) with the tokens' queries in shared memory.
constexpr int kAbsTokens = 16;
template <typename AT>
__global__ void latent_absorb_kernel(LatentShape a, const float* __restrict__ q, int q_row, const AT* __restrict__ w_uk,
                                     const int32_t* __restrict__ tok_pos, float* __restrict__ qa, int T) {
  extern __shared__ float qs[];  // [kAbsTokens][dim + rot_dim]
  const int h = blockIdx.y, t0 = blockIdx.x * kAbsTokens;
  const int n = min(kAbsTokens, T - t0);
  const int dq = a.dim + a.rot_dim, dl = a.kv_rank + a.rot_dim;
  for (int i = threadIdx.x; i < n * dq; i += blockDim.x)
    qs[i] = q[static_cast<size_t>(t0 + i / dq) * q_row + h * dq + i % dq];
  __syncthreads();
  const AT* w = w_uk + static_cast<size_t>(h) * a.dim * a.kv_rank;
  // blockIdx.z: a slice of the latent coordinates, so that a step of few tokens still spreads over many SMs
  for (int r = blockIdx.z * blockDim.x + threadIdx.x; r < a.kv_rank; r += gridDim.z * blockDim.x) {
    float acc[kAbsTokens];
#pragma unroll
    for (int j = 0; j < kAbsTokens; ++j) acc[j] = 0.f;
#pragma unroll 8
    for (int d = 0; d < a.dim; ++d) {
      const float wv = to_f(w[static_cast<size_t>(d) * a.kv_rank + r]);
#pragma unroll
      for (int j = 0; j < kAbsTokens; ++j) acc[j] = fmaf(qs[j * dq + d], wv, acc[j]);
    }
#pragma unroll
    for (int j = 0; j < kAbsTokens; ++j)
      if (j < n) qa[(static_cast<size_t>(t0 + j) * a.heads + h) * dl + r] = acc[j];
  }
  if (blockIdx.z != 0) return;
  for (int i = threadIdx.x; i < n * a.rot_dim; i += blockDim.x) {
    const int j = i / a.rot_dim, c = i % a.rot_dim;
    qa[(static_cast<size_t>(t0 + j) * a.heads + h) * dl + a.kv_rank + c] =
        rotated(a, qs + j * dq + a.dim, c, tok_pos[t0 + j]);
  }
}

// The same for steps of at most NT <= 8 tokens: a CTA takes 64 latent coordinates of one head.  A lane owns 16 bytes of a row of
// W_uk, groups of lanes and warps own different rows, and their sums meet at the end; the first rows are fetched before the
// queries have arrived in shared memory.
constexpr int kFewCols = 64, kFewWarps = 8, kFewAhead = 4;
template <typename AT, int NT>
__global__ void __launch_bounds__(kFewWarps * 32)
latent_absorb_few_kernel(LatentShape a, const float* __restrict__ q, int q_row, const AT* __restrict__ w_uk,
                         const int32_t* __restrict__ tok_pos, float* __restrict__ qa, int T) {
  constexpr int V = Wide<AT>::N, LPR = kFewCols / V, RPW = 32 / LPR;  // values per lane, lanes per row, rows per warp
  constexpr int kStep = kFewWarps * RPW;
  extern __shared__ float qs[];                 // [NT][dim + rot_dim]
  __shared__ float red[kFewWarps][NT][kFewCols];
  const int h = blockIdx.x, c0 = blockIdx.y * kFewCols;
  const int dq = a.dim + a.rot_dim, dl = a.kv_rank + a.rot_dim;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int col = c0 + (lane % LPR) * V, d0 = warp * RPW + lane / LPR;
  const bool in = col < a.kv_rank;  // kv_rank is a multiple of V
  const AT* w = w_uk + static_cast<size_t>(h) * a.dim * a.kv_rank + col;
  float wf[kFewAhead][V];
#pragma unroll
  for (int k = 0; k < kFewAhead; ++k)
    if (in && d0 + k * kStep < a.dim) Wide<AT>::template load<V>(w + static_cast<size_t>(d0 + k * kStep) * a.kv_rank, wf[k]);
  for (int i = threadIdx.x; i < T * dq; i += blockDim.x) qs[i] = q[static_cast<size_t>(i / dq) * q_row + h * dq + i % dq];
  __syncthreads();
  float acc[NT][V];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int c = 0; c < V; ++c) acc[t][c] = 0.f;
  if (in) {
    for (int base = 0; base < a.dim; base += kFewAhead * kStep) {
#pragma unroll
      for (int k = 0; k < kFewAhead; ++k) {
        const int d = base + d0 + k * kStep;
        if (base > 0 && d < a.dim) Wide<AT>::template load<V>(w + static_cast<size_t>(d) * a.kv_rank, wf[k]);
      }
#pragma unroll
      for (int k = 0; k < kFewAhead; ++k) {
        const int d = base + d0 + k * kStep;
        if (d >= a.dim) continue;
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          if (t >= T) break;
          const float qv = qs[t * dq + d];
#pragma unroll
          for (int c = 0; c < V; ++c) acc[t][c] = fmaf(qv, wf[k][c], acc[t][c]);
        }
      }
    }
  }
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int c = 0; c < V; ++c) {
      float v = acc[t][c];
#pragma unroll
      for (int o = LPR; o < 32; o <<= 1) v += __shfl_xor_sync(kAll, v, o);
      if (lane < LPR) red[warp][t][lane * V + c] = v;
    }
  __syncthreads();
  for (int i = threadIdx.x; i < T * kFewCols; i += blockDim.x) {
    const int t = i / kFewCols, c = i % kFewCols;
    if (c0 + c >= a.kv_rank) continue;
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < kFewWarps; ++k) v += red[k][t][c];
    qa[(static_cast<size_t>(t) * a.heads + h) * dl + c0 + c] = v;
  }
  if (blockIdx.y != 0) return;
  for (int i = threadIdx.x; i < T * a.rot_dim; i += blockDim.x) {
    const int t = i / a.rot_dim, c = i % a.rot_dim;
    qa[(static_cast<size_t>(t) * a.heads + h) * dl + a.kv_rank + c] = rotated(a, qs + t * dq + a.dim, c, tok_pos[t]);
  }
}

// ---- latent attention with per-head keys and values (prompt steps on the tensor cores) ---------------------------------------
// One CTA per token, a warp per head in turn.  q [heads, dim + rot_dim] fp32 -> the same in the compute type with the rotated part
// rotated; kp [heads * dim] (W_uk c) and kr [rot_dim] (rotated, shared by the heads) -> k [heads, dim + rot_dim];
// vp [heads * vdim] (W_uv c) -> v.  The token's cosines and sines are computed once.  V columns at a time: V == 4 needs sizes
// and row strides that are multiples of 4.
template <typename AT, int V>
__global__ void latent_pack_kernel(LatentShape a, const float* __restrict__ q, int q_row, const float* __restrict__ kp,
                                   int kp_row, const float* __restrict__ kr, const float* __restrict__ vp, int vp_row,
                                   const int32_t* __restrict__ tok_pos, AT* __restrict__ q_out, AT* __restrict__ k_out,
                                   AT* __restrict__ v_out) {
  extern __shared__ float cs[];  // [rope_dims / 2] cosines, then sines
  const int t = blockIdx.x, dq = a.dim + a.rot_dim, half = a.rope_dims >> 1;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float ang = static_cast<float>(tok_pos[t]) * rope_frequency(a, i);
    sincosf(ang, cs + half + i, cs + i);
  }
  __syncthreads();
  const float* kr_t = kr + static_cast<size_t>(t) * a.rot_dim;
  for (int h = warp; h < a.heads; h += nw) {
    const float* qh = q + static_cast<size_t>(t) * q_row + h * dq;
    const float* kh = kp + static_cast<size_t>(t) * kp_row + h * a.dim;
    AT* qo = q_out + (static_cast<size_t>(t) * a.heads + h) * dq;
    AT* ko = k_out + (static_cast<size_t>(t) * a.heads + h) * dq;
    for (int d = lane * V; d < dq; d += 32 * V) {
      float x[V], y[V];
      get_floats<V>(qh + d, x);
      get_floats<V>(d < a.dim ? kh + d : kr_t + d - a.dim, y);
      if (d >= a.dim) {
#pragma unroll
        for (int c = 0; c < V; ++c) {
          const int i = d - a.dim + c;
          if (i < a.rope_dims) {
            const float* r = qh + a.dim;
            if (a.rope_pairing == KLLM_SEQ_ROPE_PAIRS) {
              const float co = cs[i >> 1], si = cs[half + (i >> 1)];
              x[c] = (i & 1) == 0 ? r[i] * co - r[i + 1] * si : r[i] * co + r[i - 1] * si;
            } else {
              const int p = i < half ? i : i - half;
              const float co = cs[p], si = cs[half + p];
              x[c] = i < half ? r[i] * co - r[i + half] * si : r[i] * co + r[i - half] * si;
            }
          }
        }
      }
      put_values<V>(qo + d, x);
      put_values<V>(ko + d, y);
    }
    const float* vh = vp + static_cast<size_t>(t) * vp_row + h * a.vdim;
    AT* vo = v_out + (static_cast<size_t>(t) * a.heads + h) * a.vdim;
    for (int d = lane * V; d < a.vdim; d += 32 * V) {
      float x[V];
      get_floats<V>(vh + d, x);
      put_values<V>(vo + d, x);
    }
  }
}

// ---- latent attention: weighted sums of latents -> per-head values ---------------------------------------------------------
// One CTA: kAbsTokens tokens of one head; a warp per output row of W_uv's head block, dotted with every token's latent sum.
template <typename AT>
__global__ void latent_expand_kernel(LatentShape a, const float* __restrict__ ol, const AT* __restrict__ w_uv,
                                     AT* __restrict__ out, int T) {
  extern __shared__ float ls[];  // [kAbsTokens][kv_rank]
  const int h = blockIdx.y, t0 = blockIdx.x * kAbsTokens;
  const int n = min(kAbsTokens, T - t0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int i = threadIdx.x; i < kAbsTokens * a.kv_rank; i += blockDim.x) {
    const int j = i / a.kv_rank;
    ls[i] = j < n ? ol[(static_cast<size_t>(t0 + j) * a.heads + h) * a.kv_rank + i % a.kv_rank] : 0.f;
  }
  __syncthreads();
  for (int f = warp; f < a.vdim; f += nw) {
    const AT* w = w_uv + (static_cast<size_t>(h) * a.vdim + f) * a.kv_rank;
    float acc[kAbsTokens];
#pragma unroll
    for (int j = 0; j < kAbsTokens; ++j) acc[j] = 0.f;
    for (int r = lane; r < a.kv_rank; r += 32) {
      const float wv = to_f(w[r]);
#pragma unroll
      for (int j = 0; j < kAbsTokens; ++j) acc[j] = fmaf(ls[j * a.kv_rank + r], wv, acc[j]);
    }
#pragma unroll
    for (int j = 0; j < kAbsTokens; ++j) {
      const float v = warp_sum(acc[j]);
      if (lane == 0 && j < n) out[(static_cast<size_t>(t0 + j) * a.heads + h) * a.vdim + f] = from_f<AT>(v);
    }
  }
}

// The same for steps of single tokens, fused with the merge of the key splits: a CTA per (token, head) joins the splits'
// (max, sum, unnormalised latent sums), adds the sink to the denominator, applies the gate, and multiplies by the head's
// block of W_uv -- the merged latent sum never leaves shared memory.
// The grid's y takes slices of kExpandRows value rows of a head; every slice joins the latent sums again (they are few), and
// the first 16 bytes per lane of a warp's rows of W_uv are fetched before the sums are ready.
constexpr int kExpandWarps = 8, kExpandRowsPerWarp = 4, kExpandRows = kExpandWarps * kExpandRowsPerWarp;
template <typename AT, bool VEC>
__global__ void __launch_bounds__(kExpandWarps * 32)
latent_merge_expand_kernel(LatentShape a, int splits, const float* __restrict__ ws, const float* __restrict__ gates,
                           const float* __restrict__ sink, const AT* __restrict__ w_uv, AT* __restrict__ out) {
  extern __shared__ __align__(16) float ls[];  // [kv_rank], then [splits] weights
  float* weight = ls + a.kv_rank;
  constexpr int V = VEC ? Wide<AT>::N : 1;
  const size_t th = blockIdx.x;  // t * heads + h
  const int h = static_cast<int>(th % a.heads);
  const int pstride = a.kv_rank + 2;
  const float* p = ws + th * splits * pstride;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int f0 = blockIdx.y * kExpandRows + warp * kExpandRowsPerWarp;
  const AT* w = w_uv + (static_cast<size_t>(h) * a.vdim + f0) * a.kv_rank;
  float wf[kExpandRowsPerWarp][V];
#pragma unroll
  for (int k = 0; k < kExpandRowsPerWarp; ++k)
    if (f0 + k < a.vdim && lane * V < a.kv_rank) Wide<AT>::template load<V>(w + static_cast<size_t>(k) * a.kv_rank + lane * V, wf[k]);
  MergeColumn col;
  int d = threadIdx.x;
  if (d < a.kv_rank) col.load(p, splits, pstride, d);
  const float g = gates ? gates[th] : 1.0f;
  if (warp == 0) split_weights(p, splits, pstride, sink != nullptr, sink ? sink[h] : 0.f, weight);
  __syncthreads();
  while (d < a.kv_rank) {
    ls[d] = col.join(p, splits, pstride, d, weight) * g;
    d += blockDim.x;
    if (d < a.kv_rank) col.load(p, splits, pstride, d);
  }
  __syncthreads();
  float acc[kExpandRowsPerWarp];
#pragma unroll
  for (int k = 0; k < kExpandRowsPerWarp; ++k) acc[k] = 0.f;
  for (int r = lane * V; r < a.kv_rank; r += 32 * V) {
#pragma unroll
    for (int k = 0; k < kExpandRowsPerWarp; ++k) {
      if (f0 + k >= a.vdim) continue;
      if (r >= 32 * V) Wide<AT>::template load<V>(w + static_cast<size_t>(k) * a.kv_rank + r, wf[k]);
#pragma unroll
      for (int c = 0; c < V; ++c) acc[k] = fmaf(ls[r + c], wf[k][c], acc[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < kExpandRowsPerWarp; ++k) {
    const float v = warp_sum(acc[k]);
    if (lane == 0 && f0 + k < a.vdim) out[th * a.vdim + f0 + k] = from_f<AT>(v);
  }
}

// ---- linear attention ---------------------------------------------------------------------------------------------------------
// Per head, with decay l:  S_t = l S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t.  Columns of S are independent, so one CTA takes
// one entry, one head and kLinCols value columns, and walks the entry's tokens in chunks of kLinChunk.  For a chunk of n
// tokens with the state S before it:
//     o_i = l^(i+1) S^T q_i + sum_(j <= i) l^(i-j) (q_i . k_j) v_j
//     S  <- l^n S + sum_j l^(n-1-j) k_j v_j^T
// Only non-negative powers of l appear.  Everything is fp32; SILU is applied to q, k, v as they are loaded.  The form without
// the activation rotates q and k and scales k: steps of short entries do it on the rows in shared memory (`rot`), steps of long
// ones in place in the projection, before the chunk kernels read them (linear_rotate_kernel).
template <bool SILU> __device__ __forceinline__ float lin_act(float v) { return SILU ? siluf(v) : v; }

// One CTA per token: the angles of its position once, then every q and k head, V pairs at a time.
template <int V>
__global__ void linear_rotate_kernel(int heads, int dim, LinearRot rot, float* __restrict__ proj, int stride,
                                     const int32_t* __restrict__ tok_pos) {
  extern __shared__ __align__(16) float turn[];  // [half] cos, [half] sin
  const int t = blockIdx.x, half = rot.rope.dims / 2;
  float* co = turn;
  float* si = turn + half;
  for (int i = threadIdx.x; i < half; i += blockDim.x) rope_turn(rot.rope, i, tok_pos[t], co[i], si[i]);
  __syncthreads();
  float* row = proj + static_cast<size_t>(t) * stride;
  const bool pairs = rot.rope.pairing == KLLM_SEQ_ROPE_PAIRS;
  const int per = half / V;
  for (int i = threadIdx.x; i < 2 * heads * per; i += blockDim.x) {
    const int u = i / per, p0 = (i % per) * V;
    const float ks = u < heads ? 1.0f : rot.k_scale;
    float* h = row + u * dim;
    if constexpr (V == 4) {  // halves only
      float4 a = *reinterpret_cast<float4*>(h + p0), b = *reinterpret_cast<float4*>(h + half + p0);
      const float4 c = *reinterpret_cast<const float4*>(co + p0), z = *reinterpret_cast<const float4*>(si + p0);
      *reinterpret_cast<float4*>(h + p0) = make_float4((a.x * c.x - b.x * z.x) * ks, (a.y * c.y - b.y * z.y) * ks,
                                                       (a.z * c.z - b.z * z.z) * ks, (a.w * c.w - b.w * z.w) * ks);
      *reinterpret_cast<float4*>(h + half + p0) = make_float4((b.x * c.x + a.x * z.x) * ks, (b.y * c.y + a.y * z.y) * ks,
                                                              (b.z * c.z + a.z * z.z) * ks, (b.w * c.w + a.w * z.w) * ks);
    } else {
      const int d0 = pairs ? 2 * p0 : p0, d1 = pairs ? 2 * p0 + 1 : p0 + half;
      const float a = h[d0], b = h[d1];
      h[d0] = (a * co[p0] - b * si[p0]) * ks;
      h[d1] = (b * co[p0] + a * si[p0]) * ks;
    }
  }
  const int rest = dim - 2 * half;  // coordinates that are not rotated
  if (rest > 0 && rot.k_scale != 1.0f)
    for (int i = threadIdx.x; i < heads * rest; i += blockDim.x) row[(heads + i / rest) * dim + 2 * half + i % rest] *= rot.k_scale;
}
// Fill shared memory from global memory with U loads of a thread in flight before the first is used: the tiles of these
// kernels are small and each CTA waits for them once, so the loop is bound by load latency, not by bandwidth.
template <int U, typename Load, typename Store>
__device__ __forceinline__ void staged_fill(int total, Load load, Store store) {
  for (int i0 = threadIdx.x; i0 < total; i0 += blockDim.x * U) {
    float v[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * blockDim.x;
      v[u] = i < total ? load(i) : 0.f;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * blockDim.x;
      if (i < total) store(i, v[u]);
    }
  }
}

constexpr int kLinChunk = 32;
constexpr int kLinCols = 32;
constexpr int kLinThreads = 128;
constexpr int kLinParallelFrom = 2 * kLinChunk;  // steps whose longest entry has more tokens take the chunk-parallel kernels

template <bool SILU>
__global__ void __launch_bounds__(kLinThreads)
linear_attention_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, LinearRot rot,
                        const float* __restrict__ proj, int stride, float* __restrict__ state, const int32_t* __restrict__ ent_first,
                        const int32_t* __restrict__ ent_count, const int32_t* __restrict__ ent_seq,
                        const int32_t* __restrict__ ent_pos0, float* __restrict__ o) {
  extern __shared__ float sm[];
  const int e = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kLinCols;
  const int count = ent_count[e], first = ent_first[e], seq = ent_seq[e];
  const int cols = min(kLinCols, vdim - c0);
  const int dp = dim + 1;
  float* Qs = sm;                         // [chunk][dp]
  float* Ks = Qs + kLinChunk * dp;        // [chunk][dp]
  float* Vs = Ks + kLinChunk * dp;        // [chunk][kLinCols]
  float* As = Vs + kLinChunk * kLinCols;  // [chunk][chunk + 1]
  float* Ss = As + kLinChunk * (kLinChunk + 1);  // [dim][kLinCols]
  float* pw = Ss + dim * kLinCols;        // [chunk + 1] powers of the decay
  const int tid = threadIdx.x;
  const float lam = decay[h];
  const float llog = logf(lam);
  if (tid <= kLinChunk) pw[tid] = tid == 0 ? 1.0f : expf(llog * static_cast<float>(tid));
  float* sg = state + ((static_cast<size_t>(seq) * heads + h) * dim) * vdim;
  const bool fresh = ent_pos0[e] == 0;
  staged_fill<8>(dim * kLinCols,
                 [&](int i) { return (!fresh && i % kLinCols < cols) ? sg[static_cast<size_t>(i / kLinCols) * vdim + c0 + i % kLinCols] : 0.f; },
                 [&](int i, float v) { Ss[i] = v; });
  const int qn = heads * dim, vn = heads * vdim;
  const bool turned = !SILU && (rot.rope.dims > 0 || rot.k_scale != 1.0f);
  for (int base = 0; base < count; base += kLinChunk) {
    const int n = min(kLinChunk, count - base);
    __syncthreads();  // the previous chunk's tiles are no longer read; Ss / pw are written
    const float* rows = proj + static_cast<size_t>(first + base) * stride;
    staged_fill<8>(n * dim, [&](int i) { return rows[static_cast<size_t>(i / dim) * stride + h * dim + i % dim]; },
                   [&](int i, float v) { Qs[(i / dim) * dp + i % dim] = lin_act<SILU>(v); });
    staged_fill<8>(n * dim, [&](int i) { return rows[static_cast<size_t>(i / dim) * stride + qn + h * dim + i % dim]; },
                   [&](int i, float v) { Ks[(i / dim) * dp + i % dim] = lin_act<SILU>(v); });
    staged_fill<8>(n * kLinCols,
                   [&](int i) { return i % kLinCols < cols ? rows[static_cast<size_t>(i / kLinCols) * stride + 2 * qn + h * vdim + c0 + i % kLinCols] : 0.f; },
                   [&](int i, float v) { Vs[i] = lin_act<SILU>(v); });
    __syncthreads();
    if (turned) {
      const int half = rot.rope.dims / 2, rest = dim - 2 * half;
      const bool pairs = rot.rope.pairing == KLLM_SEQ_ROPE_PAIRS;
      for (int i = tid; i < n * half; i += kLinThreads) {
        const int r = i / half, p = i % half;
        float co, si;
        rope_turn(rot.rope, p, ent_pos0[e] + base + r, co, si);
        const int d0 = r * dp + (pairs ? 2 * p : p), d1 = r * dp + (pairs ? 2 * p + 1 : p + half);
        const float q0 = Qs[d0], q1 = Qs[d1], k0 = Ks[d0], k1 = Ks[d1];
        Qs[d0] = q0 * co - q1 * si, Qs[d1] = q1 * co + q0 * si;
        Ks[d0] = (k0 * co - k1 * si) * rot.k_scale, Ks[d1] = (k1 * co + k0 * si) * rot.k_scale;
      }
      for (int i = tid; i < n * rest; i += kLinThreads) Ks[(i / rest) * dp + 2 * half + i % rest] *= rot.k_scale;
      __syncthreads();
    }
    for (int i = tid; i < n * n; i += kLinThreads) {  // decayed scores inside the chunk
      const int r = i / n, j = i % n;
      float acc = 0.f;
      if (j <= r) {
        for (int d = 0; d < dim; ++d) acc = fmaf(Qs[r * dp + d], Ks[j * dp + d], acc);
        acc *= pw[r - j];
      }
      As[r * (kLinChunk + 1) + j] = acc;
    }
    __syncthreads();
    for (int i = tid; i < n * kLinCols; i += kLinThreads) {  // outputs
      const int r = i / kLinCols, c = i % kLinCols;
      float carry = 0.f;
      for (int d = 0; d < dim; ++d) carry = fmaf(Qs[r * dp + d], Ss[d * kLinCols + c], carry);
      float acc = carry * pw[r + 1];
      for (int j = 0; j <= r; ++j) acc = fmaf(As[r * (kLinChunk + 1) + j], Vs[j * kLinCols + c], acc);
      if (c < cols) o[static_cast<size_t>(first + base + r) * vn + h * vdim + c0 + c] = acc;
    }
    __syncthreads();
    for (int i = tid; i < dim * kLinCols; i += kLinThreads) {  // the state after the chunk
      const int d = i / kLinCols, c = i % kLinCols;
      float acc = Ss[i] * pw[n];
      for (int j = 0; j < n; ++j) acc = fmaf(Ks[j * dp + d] * pw[n - 1 - j], Vs[j * kLinCols + c], acc);
      Ss[i] = acc;
    }
  }
  __syncthreads();
  for (int i = tid; i < dim * kLinCols; i += kLinThreads) {
    const int d = i / kLinCols, c = i % kLinCols;
    if (c < cols) sg[static_cast<size_t>(d) * vdim + c0 + c] = Ss[i];
  }
}

// ---- linear attention over long entries: chunks in parallel ---------------------------------------------------------------
// The recurrence above is sequential only in the state.  For entries of many chunks it is cut into three kernels:
//   linear_chunk_sums_kernel   every chunk on its own: U_c = sum_j l^(n-1-j) k_j v_j^T                       (parallel)
//   linear_scan_kernel         S_before(c) in place of U_c, chunk after chunk: S <- l^n S + U_c; the final state  (per element)
//   linear_chunk_out_kernel    every chunk on its own: o_i = l^(i+1) S_before^T q_i + decayed scores inside the chunk
// Chunk j of entry e lives in slot (first_e + j * chunk) / chunk + e of the scratch buffer [slots][heads][dim][vdim].
__device__ __forceinline__ size_t chunk_slot(int first, int base, int e) { return static_cast<size_t>((first + base) / kLinChunk + e); }

__host__ __device__ inline int lin_dp(int dim) { return ((dim + 3) & ~3) + 4; }  // row stride of Qs / Ks: 16-byte rows, odd in 16-byte units for dim % 8 == 0

// A thread keeps 8 consecutive key coordinates of one value column: two 16-byte broadcast loads and one column load
// feed 8 multiply-adds.
template <bool SILU>
__global__ void __launch_bounds__(kLinThreads)
linear_chunk_sums_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, const float* __restrict__ proj,
                         int stride,
                         const int32_t* __restrict__ ent_first, const int32_t* __restrict__ ent_count,
                         float* __restrict__ sums) {
  extern __shared__ __align__(16) float sm[];
  const int e = blockIdx.z, h = blockIdx.y;
  const int n_slices = (vdim + kLinCols - 1) / kLinCols;
  const int chunk = blockIdx.x / n_slices, c0 = (blockIdx.x % n_slices) * kLinCols;
  const int count = ent_count[e], first = ent_first[e], base = chunk * kLinChunk;
  if (base >= count) return;
  const int n = min(kLinChunk, count - base);
  const int cols = min(kLinCols, vdim - c0);
  const int d8 = (dim + 7) & ~7, dp = lin_dp(dim);
  float* Ks = sm;                       // [chunk][dp], already times l^(n-1-j); zeros from dim to d8
  float* Vs = Ks + kLinChunk * dp;      // [chunk][kLinCols]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float llog = logf(decay[h]);
  const int qn = heads * dim;
  const float* rows = proj + static_cast<size_t>(first + base) * stride;
  staged_fill<8>(n * d8,
                 [&](int i) { return i % d8 < dim ? rows[static_cast<size_t>(i / d8) * stride + qn + h * dim + i % d8] : 0.f; },
                 [&](int i, float v) {
                   const int j = i / d8;
                   const float w = n - 1 - j == 0 ? 1.0f : expf(llog * static_cast<float>(n - 1 - j));
                   Ks[j * dp + i % d8] = lin_act<SILU>(v) * w;
                 });
  staged_fill<8>(n * kLinCols,
                 [&](int i) { return i % kLinCols < cols ? rows[static_cast<size_t>(i / kLinCols) * stride + 2 * qn + h * vdim + c0 + i % kLinCols] : 0.f; },
                 [&](int i, float v) { Vs[i] = lin_act<SILU>(v); });
  __syncthreads();
  float* out = sums + (chunk_slot(first, base, e) * heads + h) * dim * vdim;
  for (int d0 = warp * 8; d0 < d8; d0 += (kLinThreads / 32) * 8) {
    float acc[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) acc[k] = 0.f;
    for (int j = 0; j < n; ++j) {
      const float v = Vs[j * kLinCols + lane];
      const float4 a = *reinterpret_cast<const float4*>(Ks + j * dp + d0);
      const float4 b = *reinterpret_cast<const float4*>(Ks + j * dp + d0 + 4);
      acc[0] = fmaf(a.x, v, acc[0]), acc[1] = fmaf(a.y, v, acc[1]), acc[2] = fmaf(a.z, v, acc[2]), acc[3] = fmaf(a.w, v, acc[3]);
      acc[4] = fmaf(b.x, v, acc[4]), acc[5] = fmaf(b.y, v, acc[5]), acc[6] = fmaf(b.z, v, acc[6]), acc[7] = fmaf(b.w, v, acc[7]);
    }
#pragma unroll
    for (int k = 0; k < 8; ++k)
      if (d0 + k < dim && lane < cols) out[static_cast<size_t>(d0 + k) * vdim + c0 + lane] = acc[k];
  }
}

__global__ void linear_scan_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, float* __restrict__ state,
                                   const int32_t* __restrict__ ent_first, const int32_t* __restrict__ ent_count,
                                   const int32_t* __restrict__ ent_seq, const int32_t* __restrict__ ent_pos0,
                                   float* __restrict__ sums) {
  const int e = blockIdx.z, h = blockIdx.y;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= dim * vdim) return;
  const int count = ent_count[e], first = ent_first[e];
  const float llog = logf(decay[h]);
  const float full = expf(llog * static_cast<float>(kLinChunk));
  float* sg = state + (static_cast<size_t>(ent_seq[e]) * heads + h) * dim * vdim + i;
  float s = ent_pos0[e] == 0 ? 0.f : *sg;
  // the chunk sums are fetched eight chunks ahead: the loads do not depend on one another, only the sums do
  constexpr int U = 8;
  for (int base = 0; base < count; base += U * kLinChunk) {
    float add[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int b = base + u * kLinChunk;
      add[u] = b < count ? sums[(chunk_slot(first, b, e) * heads + h) * dim * vdim + i] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int b = base + u * kLinChunk;
      if (b >= count) break;
      const int n = min(kLinChunk, count - b);
      sums[(chunk_slot(first, b, e) * heads + h) * dim * vdim + i] = s;
      s = fmaf(s, n == kLinChunk ? full : expf(llog * static_cast<float>(n)), add[u]);
    }
  }
  *sg = s;
}

// Each thread keeps kLinChunk / warps rows (warp + warps * k) of one column: a 16-byte broadcast load brings four coordinates
// of a row.  Eight warps per CTA: the shared-memory tiles allow few CTAs per SM, so the warps have to come from the CTA.  Rows and coordinates past the chunk are zero-filled.
constexpr int kLinAs = kLinChunk + 4;

constexpr int kLinOutThreads = 256, kLinOutWarps = kLinOutThreads / 32;
template <bool SILU>
__global__ void __launch_bounds__(kLinOutThreads)
linear_chunk_out_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, const float* __restrict__ proj,
                        int stride,
                        const int32_t* __restrict__ ent_first, const int32_t* __restrict__ ent_count,
                        const float* __restrict__ sums, float* __restrict__ o) {
  extern __shared__ __align__(16) float sm[];
  const int e = blockIdx.z, h = blockIdx.y;
  const int n_slices = (vdim + kLinCols - 1) / kLinCols;
  const int chunk = blockIdx.x / n_slices, c0 = (blockIdx.x % n_slices) * kLinCols;
  const int count = ent_count[e], first = ent_first[e], base = chunk * kLinChunk;
  if (base >= count) return;
  const int n = min(kLinChunk, count - base);
  const int cols = min(kLinCols, vdim - c0);
  const int d4 = (dim + 3) & ~3, dp = lin_dp(dim);
  float* Qs = sm;                          // [chunk][dp]
  float* Ks = Qs + kLinChunk * dp;         // [chunk][dp]
  float* Vs = Ks + kLinChunk * dp;         // [chunk][kLinCols]
  float* As = Vs + kLinChunk * kLinCols;   // [chunk][kLinAs]
  float* Ss = As + kLinChunk * kLinAs;     // [d4][kLinCols]
  float* pw = Ss + d4 * kLinCols;          // [chunk + 1]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float llog = logf(decay[h]);
  if (tid <= kLinChunk) pw[tid] = tid == 0 ? 1.0f : expf(llog * static_cast<float>(tid));
  const float* sb = sums + (chunk_slot(first, base, e) * heads + h) * dim * vdim;
  staged_fill<8>(d4 * kLinCols,
                 [&](int i) { return (i / kLinCols < dim && i % kLinCols < cols) ? sb[static_cast<size_t>(i / kLinCols) * vdim + c0 + i % kLinCols] : 0.f; },
                 [&](int i, float v) { Ss[i] = v; });
  const int qn = heads * dim, vn = heads * vdim;
  const float* rows = proj + static_cast<size_t>(first + base) * stride;
  // the activation of 0 is 0: rows and coordinates past the chunk load as zeros
  staged_fill<8>(kLinChunk * d4,
                 [&](int i) { return (i / d4 < n && i % d4 < dim) ? rows[static_cast<size_t>(i / d4) * stride + h * dim + i % d4] : 0.f; },
                 [&](int i, float v) { Qs[(i / d4) * dp + i % d4] = lin_act<SILU>(v); });
  staged_fill<8>(kLinChunk * d4,
                 [&](int i) { return (i / d4 < n && i % d4 < dim) ? rows[static_cast<size_t>(i / d4) * stride + qn + h * dim + i % d4] : 0.f; },
                 [&](int i, float v) { Ks[(i / d4) * dp + i % d4] = lin_act<SILU>(v); });
  staged_fill<8>(kLinChunk * kLinCols,
                 [&](int i) { return (i / kLinCols < n && i % kLinCols < cols) ? rows[static_cast<size_t>(i / kLinCols) * stride + 2 * qn + h * vdim + c0 + i % kLinCols] : 0.f; },
                 [&](int i, float v) { Vs[i] = lin_act<SILU>(v); });
  __syncthreads();
  constexpr int R = kLinChunk / kLinOutWarps;  // rows per thread
  {  // decayed scores inside the chunk: lane = key j, rows warp + 8 k
    float acc[R];
#pragma unroll
    for (int k = 0; k < R; ++k) acc[k] = 0.f;
    for (int d = 0; d < d4; d += 4) {
      const float4 kv = *reinterpret_cast<const float4*>(Ks + lane * dp + d);
#pragma unroll
      for (int k = 0; k < R; ++k) {
        const float4 qv = *reinterpret_cast<const float4*>(Qs + (warp + kLinOutWarps * k) * dp + d);
        acc[k] = fmaf(qv.x, kv.x, fmaf(qv.y, kv.y, fmaf(qv.z, kv.z, fmaf(qv.w, kv.w, acc[k]))));
      }
    }
#pragma unroll
    for (int k = 0; k < R; ++k) {
      const int r = warp + kLinOutWarps * k;
      As[r * kLinAs + lane] = (lane <= r && r < n) ? acc[k] * pw[r - lane] : 0.f;
    }
  }
  __syncthreads();
  {  // outputs: lane = column, rows warp + 8 k
    float acc[R];
#pragma unroll
    for (int k = 0; k < R; ++k) acc[k] = 0.f;
    for (int d = 0; d < d4; d += 4) {
      const float s0 = Ss[d * kLinCols + lane], s1 = Ss[(d + 1) * kLinCols + lane], s2 = Ss[(d + 2) * kLinCols + lane],
                  s3 = Ss[(d + 3) * kLinCols + lane];
#pragma unroll
      for (int k = 0; k < R; ++k) {
        const float4 qv = *reinterpret_cast<const float4*>(Qs + (warp + kLinOutWarps * k) * dp + d);
        acc[k] = fmaf(qv.x, s0, fmaf(qv.y, s1, fmaf(qv.z, s2, fmaf(qv.w, s3, acc[k]))));
      }
    }
#pragma unroll
    for (int k = 0; k < R; ++k) acc[k] *= pw[min(warp + kLinOutWarps * k + 1, kLinChunk)];
    for (int j = 0; j < kLinChunk; j += 4) {
      const float v0 = Vs[j * kLinCols + lane], v1 = Vs[(j + 1) * kLinCols + lane], v2 = Vs[(j + 2) * kLinCols + lane],
                  v3 = Vs[(j + 3) * kLinCols + lane];
#pragma unroll
      for (int k = 0; k < R; ++k) {
        const float4 av = *reinterpret_cast<const float4*>(As + (warp + kLinOutWarps * k) * kLinAs + j);
        acc[k] = fmaf(av.x, v0, fmaf(av.y, v1, fmaf(av.z, v2, fmaf(av.w, v3, acc[k]))));
      }
    }
#pragma unroll
    for (int k = 0; k < R; ++k) {
      const int r = warp + kLinOutWarps * k;
      if (r < n && lane < cols) o[static_cast<size_t>(first + base + r) * vn + h * vdim + c0 + lane] = acc[k];
    }
  }
}

// One token per entry (decode steps), heads normed one by one: a CTA per (head, token) reads the head's state once, 16 bytes per
// lane, writes it back, and has the head's whole output -- its norm, the gate and the conversion follow in place.  A thread owns
// V columns and every slices-th row; kLinTokenLoads rows of it are in flight before the projections are read.
constexpr int kLinTokenLoads = 8;
template <typename AT, int V>
__global__ void __launch_bounds__(512)
linear_token_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, LinearRot rot, int silu,
                    const float* __restrict__ proj, int stride, int gate_act, float eps, float* __restrict__ state,
                    const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ tok_pos, AT* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33];
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
  const int dp = (dim + 3) & ~3, units = vdim / V, slices = blockDim.x / units;
  float* qs = sm;                         // [dp]
  float* ks = qs + dp;                    // [dp]
  float* vs = ks + dp;                    // [vdim, padded to 4]
  float* part = vs + ((vdim + 3) & ~3);   // [slices][vdim]
  const int pos = tok_pos[t];
  const bool fresh = pos == 0;
  float* S = state + (static_cast<size_t>(tok_seq[t]) * heads + h) * dim * vdim;
  const int c = (tid % units) * V, sl = tid / units;
  const bool works = sl < slices;
  float s[kLinTokenLoads][V];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int u = 0; u < kLinTokenLoads; ++u) {
      const int d = d0 + u * slices;
#pragma unroll
      for (int z = 0; z < V; ++z) s[u][z] = 0.f;
      if (!works || fresh || d >= dim) continue;
      if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(S + static_cast<size_t>(d) * vdim + c);
        s[u][0] = f.x, s[u][1] = f.y, s[u][2] = f.z, s[u][3] = f.w;
      } else {
        s[u][0] = S[static_cast<size_t>(d) * vdim + c];
      }
    }
  };
  fetch(sl);
  const float* row = proj + static_cast<size_t>(t) * stride;
  const float *q = row + h * dim, *k = q + heads * dim, *v = row + 2 * heads * dim + h * vdim;
  const int half = rot.rope.dims / 2;
  const bool pairs = rot.rope.pairing == KLLM_SEQ_ROPE_PAIRS;
  auto act = [&](float x) { return silu ? siluf(x) : x; };
  for (int i = tid; i < half; i += blockDim.x) {
    float co, si;
    rope_turn(rot.rope, i, pos, co, si);
    const int d0 = pairs ? 2 * i : i, d1 = pairs ? 2 * i + 1 : i + half;
    const float q0 = q[d0], q1 = q[d1], k0 = k[d0], k1 = k[d1];
    qs[d0] = q0 * co - q1 * si, qs[d1] = q1 * co + q0 * si;
    ks[d0] = (k0 * co - k1 * si) * rot.k_scale, ks[d1] = (k1 * co + k0 * si) * rot.k_scale;
  }
  for (int d = 2 * half + tid; d < dim; d += blockDim.x) qs[d] = act(q[d]), ks[d] = act(k[d]) * rot.k_scale;
  for (int i = tid; i < vdim; i += blockDim.x) vs[i] = act(v[i]);
  __syncthreads();
  const float lam = decay[h];
  if (works) {
    float acc[V], vc[V];
#pragma unroll
    for (int z = 0; z < V; ++z) acc[z] = 0.f, vc[z] = vs[c + z];
    for (int d0 = sl; d0 < dim; d0 += kLinTokenLoads * slices) {
      if (d0 != sl) fetch(d0);
#pragma unroll
      for (int u = 0; u < kLinTokenLoads; ++u) {
        const int d = d0 + u * slices;
        if (d >= dim) break;
        const float kd = ks[d], qd = qs[d];
#pragma unroll
        for (int z = 0; z < V; ++z) {
          s[u][z] = fmaf(lam, s[u][z], kd * vc[z]);
          acc[z] = fmaf(qd, s[u][z], acc[z]);
        }
        float* dst = S + static_cast<size_t>(d) * vdim + c;
        if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
        else *dst = s[u][0];
      }
    }
#pragma unroll
    for (int z = 0; z < V; ++z) part[sl * vdim + c + z] = acc[z];
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = tid; i < vdim; i += blockDim.x) {
    float o = 0.f;
    for (int p = 0; p < slices; ++p) o += part[p * vdim + i];
    vs[i] = o;
    ss = fmaf(o, o, ss);
  }
  const float rinv = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(vdim) + eps);
  const float* g = row + 2 * heads * dim + heads * vdim + h * vdim;
  for (int i = tid; i < vdim; i += blockDim.x) {
    const float z = g[i];
    const float gate = gate_act == KLLM_SEQ_GATEACT_SILU ? siluf(z) : sigmoidf(z);
    out[(static_cast<size_t>(t) * heads + h) * vdim + i] = from_f<AT>(vs[i] * rinv * gate);
  }
}

__device__ __forceinline__ float lin_gate(int act, float g) { return act == KLLM_SEQ_GATEACT_SILU ? siluf(g) : sigmoidf(g); }

// One CTA per token.  ROW: one norm over the row; HEAD: a warp per head, each by its own root mean square.
template <typename AT, bool HEAD>
__global__ void linear_out_kernel(int heads, int dim, int vdim, const float* __restrict__ o, const float* __restrict__ proj,
                                  int stride, const float* __restrict__ norm_w, int gate_act, float eps, AT* __restrict__ out) {
  __shared__ float red[33];
  const int t = blockIdx.x, vn = heads * vdim;
  const float* row = o + static_cast<size_t>(t) * vn;
  const float* g = proj + static_cast<size_t>(t) * stride + 2 * heads * dim + vn;
  AT* dst = out + static_cast<size_t>(t) * vn;
  if constexpr (HEAD) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int h = warp; h < heads; h += nw) {
      float ss = 0.f;
      for (int d = lane; d < vdim; d += 32) ss = fmaf(row[h * vdim + d], row[h * vdim + d], ss);
      const float rinv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(vdim) + eps);
      for (int d = lane; d < vdim; d += 32) {
        const int i = h * vdim + d;
        dst[i] = from_f<AT>(row[i] * rinv * lin_gate(gate_act, g[i]));
      }
    }
  } else {
    float ss = 0.f;
    for (int i = threadIdx.x; i < vn; i += blockDim.x) ss += row[i] * row[i];
    const float rinv = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(vn) + eps);
    for (int i = threadIdx.x; i < vn; i += blockDim.x) dst[i] = from_f<AT>(row[i] * rinv * norm_w[i] * lin_gate(gate_act, g[i]));
  }
}

// ---- activations ---------------------------------------------------------------------------------------------------------------
template <typename AT>
__global__ void activation_kernel(int act, float a, float b, const float* __restrict__ z, AT* __restrict__ out, size_t n) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = z[i];
  float r;
  if (act == KLLM_SEQ_ACT_XIELU) r = v > 0.f ? a * v * v + 0.5f * v : b * (expm1f(v) - v) + 0.5f * v;
  else r = v > 0.f ? v * v : 0.f;
  out[i] = from_f<AT>(r);
}

__global__ void scale_kernel(float* __restrict__ v, float scale, float cap, size_t n) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float z = v[i] * scale;
  if (cap > 0.f) z = cap * tanhf(z / cap);
  v[i] = z;
}

#define KLLM_SEQ_DISPATCH(dtype, CALL)                         \
  do {                                                         \
    if ((dtype) == KLLM_SEQ_F32) {                             \
      using AT = float;                                        \
      CALL;                                                    \
    } else if ((dtype) == KLLM_SEQ_BF16) {                     \
      using AT = __nv_bfloat16;                                \
      CALL;                                                    \
    } else {                                                   \
      return KLLM_E_INVALID;                                   \
    }                                                          \
  } while (0)

inline int done() {
  count_launch();
  return cuda_rc(cudaGetLastError());
}
}  // namespace

int launch_latent_prepare(int dtype, const LatentShape& a, const float* proj, const float* q_norm_w, const float* kv_norm_w,
                          float eps, const int32_t* tok_seq, const int32_t* tok_pos, void* cq, float* gates,
                          const PagedKV& kv, void* c_rows, float* kr_rows, int T, cudaStream_t s) {
  KLLM_SEQ_DISPATCH(dtype, (latent_prepare_kernel<AT><<<T, 128, 0, s>>>(a, proj, q_norm_w, kv_norm_w, eps, tok_seq, tok_pos,
                                                                       static_cast<AT*>(cq), gates, kv,
                                                                       static_cast<AT*>(c_rows), kr_rows)));
  return done();
}

int launch_latent_pack(int dtype, const LatentShape& a, const float* q, int q_row, const float* kp, int kp_row, const float* kr,
                       const float* vp, int vp_row, const int32_t* tok_pos, void* q_out, void* k_out, void* v_out, int T,
                       cudaStream_t s) {
  const bool vec = ((a.dim | a.rot_dim | a.vdim | q_row | kp_row | vp_row) & 3) == 0 && (reinterpret_cast<uintptr_t>(vp) & 15) == 0;
  const size_t smem = static_cast<size_t>(a.rope_dims) * sizeof(float);
  if (smem > 48 * 1024) return KLLM_E_UNSUPPORTED;
  if (vec)
    KLLM_SEQ_DISPATCH(dtype, (latent_pack_kernel<AT, 4><<<T, 256, smem, s>>>(
                                 a, q, q_row, kp, kp_row, kr, vp, vp_row, tok_pos, static_cast<AT*>(q_out),
                                 static_cast<AT*>(k_out), static_cast<AT*>(v_out))));
  else
    KLLM_SEQ_DISPATCH(dtype, (latent_pack_kernel<AT, 1><<<T, 256, smem, s>>>(
                                 a, q, q_row, kp, kp_row, kr, vp, vp_row, tok_pos, static_cast<AT*>(q_out),
                                 static_cast<AT*>(k_out), static_cast<AT*>(v_out))));
  return done();
}

int launch_latent_absorb(int dtype, const LatentShape& a, const float* q, int q_row, const void* w_uk, const int32_t* tok_pos,
                         float* qa, int T, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(kAbsTokens) * (a.dim + a.rot_dim) * sizeof(float);
  if (smem > 48 * 1024) return KLLM_E_UNSUPPORTED;
  if (T <= 8 && a.kv_rank % 8 == 0 && (reinterpret_cast<uintptr_t>(w_uk) & 15) == 0) {
    const dim3 grid(a.heads, (a.kv_rank + kFewCols - 1) / kFewCols);
    const size_t few = static_cast<size_t>(T) * (a.dim + a.rot_dim) * sizeof(float);
#define KLLM_ABSORB(NT)                                                                                                   \
  KLLM_SEQ_DISPATCH(dtype, (latent_absorb_few_kernel<AT, NT><<<grid, kFewWarps * 32, few, s>>>(a, q, q_row,               \
                                                                                               static_cast<const AT*>(w_uk), \
                                                                                               tok_pos, qa, T)))
    if (T == 1) KLLM_ABSORB(1);
    else if (T == 2) KLLM_ABSORB(2);
    else if (T <= 4) KLLM_ABSORB(4);
    else KLLM_ABSORB(8);
#undef KLLM_ABSORB
    return done();
  }
  // few tokens: 64 latent coordinates per CTA; many tokens: the whole latent (the queries are staged once per CTA)
  const int threads = T <= kAbsTokens ? 64 : (a.kv_rank <= 64 ? 64 : (a.kv_rank <= 128 ? 128 : 256));
  const dim3 grid((T + kAbsTokens - 1) / kAbsTokens, a.heads, (a.kv_rank + threads - 1) / threads);
  KLLM_SEQ_DISPATCH(dtype, (latent_absorb_kernel<AT><<<grid, threads, smem, s>>>(a, q, q_row, static_cast<const AT*>(w_uk), tok_pos,
                                                                                qa, T)));
  return done();
}

int launch_latent_merge_expand(int dtype, const LatentShape& a, int splits, const float* ws, const float* gates,
                               const float* sink, const void* w_uv, void* out, int T, cudaStream_t s) {
  const size_t smem = (static_cast<size_t>(a.kv_rank) + splits) * sizeof(float);
  const dim3 grid(T * a.heads, (a.vdim + kExpandRows - 1) / kExpandRows);
  const bool vec = a.kv_rank % 8 == 0 && (reinterpret_cast<uintptr_t>(w_uv) & 15) == 0;
  if (vec)
    KLLM_SEQ_DISPATCH(dtype, (latent_merge_expand_kernel<AT, true><<<grid, kExpandWarps * 32, smem, s>>>(
                                 a, splits, ws, gates, sink, static_cast<const AT*>(w_uv), static_cast<AT*>(out))));
  else
    KLLM_SEQ_DISPATCH(dtype, (latent_merge_expand_kernel<AT, false><<<grid, kExpandWarps * 32, smem, s>>>(
                                 a, splits, ws, gates, sink, static_cast<const AT*>(w_uv), static_cast<AT*>(out))));
  return done();
}

int launch_latent_expand(int dtype, const LatentShape& a, const float* ol, const void* w_uv, void* out, int T, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(kAbsTokens) * a.kv_rank * sizeof(float);
  if (smem > 48 * 1024) return KLLM_E_UNSUPPORTED;
  const dim3 grid((T + kAbsTokens - 1) / kAbsTokens, a.heads);
  KLLM_SEQ_DISPATCH(dtype, (latent_expand_kernel<AT><<<grid, 256, smem, s>>>(a, ol, static_cast<const AT*>(w_uv),
                                                                            static_cast<AT*>(out), T)));
  return done();
}

size_t linear_attention_scratch_bytes(int heads, int dim, int vdim, int T, int n_entries, int max_count) {
  if (max_count <= kLinParallelFrom) return 0;
  return (static_cast<size_t>(T) / kLinChunk + n_entries + 1) * heads * dim * vdim * sizeof(float);
}

int launch_linear_rotate(const kllm_seq_linear& m, float* proj, int row, const int32_t* tok_pos, int T, cudaStream_t s) {
  const LinearRot rot = linear_rot(m);
  const int half = m.rope_dims / 2;
  const size_t smem = 2 * static_cast<size_t>(half) * sizeof(float);
  const bool vec = m.rope_pairing == KLLM_SEQ_ROPE_HALVES && half % 4 == 0 && m.dim % 4 == 0 && row % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
  if (vec) linear_rotate_kernel<4><<<T, 256, smem, s>>>(m.heads, m.dim, rot, proj, row, tok_pos);
  else linear_rotate_kernel<1><<<T, 256, smem, s>>>(m.heads, m.dim, rot, proj, row, tok_pos);
  return done();
}

template <bool SILU>
static int linear_attention_t(const kllm_seq_linear& m, const float* proj, int row, float* state, int n_entries,
                              const int32_t* ent_first, const int32_t* ent_count, const int32_t* ent_seq,
                              const int32_t* ent_pos0, int max_count, float* scratch, float* o, cudaStream_t s) {
  const int heads = m.heads, dim = m.dim, vdim = m.vdim;
  const float* decay = m.decay;
  if (max_count > kLinParallelFrom && scratch != nullptr) {  // long entries: chunks in parallel
    const size_t smem_out = (2 * static_cast<size_t>(kLinChunk) * lin_dp(dim) + kLinChunk * kLinCols + kLinChunk * kLinAs +
                             static_cast<size_t>((dim + 3) & ~3) * kLinCols + kLinChunk + 4) * sizeof(float);
    static size_t configured_out = 0;
    if (smem_out > 48 * 1024 && smem_out > configured_out) {
      cudaError_t e = cudaFuncSetAttribute(linear_chunk_out_kernel<SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                           static_cast<int>(smem_out));
      if (e == cudaSuccess)
        e = cudaFuncSetAttribute(linear_chunk_sums_kernel<SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 static_cast<int>(smem_out));
      if (e != cudaSuccess) return cuda_rc(e);
      configured_out = smem_out;
    }
    const int n_slices = (vdim + kLinCols - 1) / kLinCols, chunks = (max_count + kLinChunk - 1) / kLinChunk;
    const dim3 grid(chunks * n_slices, heads, n_entries);
    const size_t smem_sums = (static_cast<size_t>(kLinChunk) * lin_dp(dim) + kLinChunk * kLinCols) * sizeof(float);
    linear_chunk_sums_kernel<SILU><<<grid, kLinThreads, smem_sums, s>>>(heads, dim, vdim, decay, proj, row, ent_first, ent_count,
                                                                       scratch);
    count_launch();
    const dim3 sgrid((dim * vdim + 127) / 128, heads, n_entries);
    linear_scan_kernel<<<sgrid, 128, 0, s>>>(heads, dim, vdim, decay, state, ent_first, ent_count, ent_seq, ent_pos0, scratch);
    count_launch();
    linear_chunk_out_kernel<SILU><<<grid, kLinOutThreads, smem_out, s>>>(heads, dim, vdim, decay, proj, row, ent_first, ent_count,
                                                                        scratch, o);
    return done();
  }
  const size_t smem = (2 * static_cast<size_t>(kLinChunk) * (dim + 1) + kLinChunk * kLinCols + kLinChunk * (kLinChunk + 1) +
                       static_cast<size_t>(dim) * kLinCols + kLinChunk + 1) * sizeof(float);
  if (smem > 200 * 1024) return KLLM_E_UNSUPPORTED;
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    const cudaError_t e = cudaFuncSetAttribute(linear_attention_kernel<SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem));
    if (e != cudaSuccess) return cuda_rc(e);
    configured = smem;
  }
  const dim3 grid((vdim + kLinCols - 1) / kLinCols, heads, n_entries);
  linear_attention_kernel<SILU><<<grid, kLinThreads, smem, s>>>(heads, dim, vdim, decay, linear_rot(m), proj, row, state, ent_first,
                                                               ent_count, ent_seq, ent_pos0, o);
  return done();
}

bool linear_attention_rotates(const kllm_seq_linear& m, int max_count) {
  return m.qkv_act == KLLM_SEQ_QKV_PLAIN && max_count > kLinParallelFrom && (m.rope_dims > 0 || (m.k_scale != 0.f && m.k_scale != 1.0f));
}

int launch_linear_attention(const kllm_seq_linear& m, const float* proj, int row, float* state, int n_entries,
                            const int32_t* ent_first, const int32_t* ent_count, const int32_t* ent_seq,
                            const int32_t* ent_pos0, int max_count, float* scratch, float* o, cudaStream_t s) {
  if (m.qkv_act == KLLM_SEQ_QKV_PLAIN)
    return linear_attention_t<false>(m, proj, row, state, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, scratch, o, s);
  return linear_attention_t<true>(m, proj, row, state, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, scratch, o, s);
}

bool linear_token_usable(const kllm_seq_linear& m) {
  const int units = m.vdim % 4 == 0 ? m.vdim / 4 : m.vdim;
  return m.out_norm == KLLM_SEQ_OUTNORM_HEAD && units <= 256;
}

int launch_linear_token(int dtype, const kllm_seq_linear& m, const float* proj, int row, float* state, const int32_t* tok_seq,
                        const int32_t* tok_pos, float eps, void* out, int T, cudaStream_t s) {
  const bool vec = m.vdim % 4 == 0;
  const int units = vec ? m.vdim / 4 : m.vdim;
  int threads = 128;
  while (threads < 512 && (threads < units || threads / units * kLinTokenLoads < m.dim)) threads *= 2;
  const size_t smem = (2 * static_cast<size_t>((m.dim + 3) & ~3) + ((m.vdim + 3) & ~3) + static_cast<size_t>(threads / units) * m.vdim) *
                      sizeof(float);
  if (T > 65535 || smem > 48 * 1024) return KLLM_E_UNSUPPORTED;
  const dim3 grid(m.heads, T);
  const LinearRot rot = linear_rot(m);
  const int silu = m.qkv_act == KLLM_SEQ_QKV_SILU;
  if (vec)
    KLLM_SEQ_DISPATCH(dtype, (linear_token_kernel<AT, 4><<<grid, threads, smem, s>>>(m.heads, m.dim, m.vdim, m.decay, rot, silu, proj, row,
                                                                                    m.gate_act, eps, state, tok_seq, tok_pos,
                                                                                    static_cast<AT*>(out))));
  else
    KLLM_SEQ_DISPATCH(dtype, (linear_token_kernel<AT, 1><<<grid, threads, smem, s>>>(m.heads, m.dim, m.vdim, m.decay, rot, silu, proj, row,
                                                                                    m.gate_act, eps, state, tok_seq, tok_pos,
                                                                                    static_cast<AT*>(out))));
  return done();
}

int launch_linear_out(int dtype, const kllm_seq_linear& m, const float* o, const float* proj, int row, float eps, void* out, int T,
                      cudaStream_t s) {
  if (m.out_norm == KLLM_SEQ_OUTNORM_HEAD) {
    const int threads = T <= 64 ? 512 : 128;
    KLLM_SEQ_DISPATCH(dtype, (linear_out_kernel<AT, true><<<T, threads, 0, s>>>(m.heads, m.dim, m.vdim, o, proj, row, nullptr, m.gate_act,
                                                                               eps, static_cast<AT*>(out))));
    return done();
  }
  KLLM_SEQ_DISPATCH(dtype, (linear_out_kernel<AT, false><<<T, 128, 0, s>>>(m.heads, m.dim, m.vdim, o, proj, row, m.out_norm_w,
                                                                          m.gate_act, eps, static_cast<AT*>(out))));
  return done();
}

int launch_activation(int dtype, int act, float a, float b, const float* z, void* out, size_t n, cudaStream_t s) {
  if (act != KLLM_SEQ_ACT_XIELU && act != KLLM_SEQ_ACT_RELU2) return KLLM_E_UNSUPPORTED;
  const unsigned blocks = static_cast<unsigned>((n + 255) / 256);
  KLLM_SEQ_DISPATCH(dtype, (activation_kernel<AT><<<blocks, 256, 0, s>>>(act, a, b, z, static_cast<AT*>(out), n)));
  return done();
}

int launch_scale(float* v, float scale, float cap, size_t n, cudaStream_t s) {
  scale_kernel<<<static_cast<unsigned>((n + 255) / 256), 256, 0, s>>>(v, scale == 0.f ? 1.0f : scale, cap, n);
  return done();
}

}  // namespace seq
}  // namespace kllm
