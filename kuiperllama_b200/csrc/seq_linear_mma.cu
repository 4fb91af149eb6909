// Linear attention over long entries on the tensor cores (bf16 steps): the recurrence S <- l S + k v^T, o = S^T q of every head,
// chunk by chunk, with fp32 state.
//
//   linear_split_kernel   the step's q, k (activated, or rotated and scaled) and v as TWO bf16 terms each, x = hi + lo, in planes
//                         [T][q | k | k weighted | v]; a weighted key carries the decay from its token to the end of its chunk
//   linear_sums_kernel    every chunk on its own: U_c = sum_j l^(n-1-j) k_j v_j^T                                    (parallel)
//   linear_carry_kernel   S before every chunk, chunk after chunk: S <- l^n S + U_c, left as two bf16 terms; the final state in fp32
//   linear_rows_kernel    every chunk on its own: o_i = l^(i+1) S^T q_i + sum_(j <= i) l^(i-j) (q_i . k_j) v_j; where the heads are
//                         normed one by one the norm, the gate and the conversion follow in the same CTA
//
// Every product is three mma.sync m16n8k16 (hi hi + hi lo + lo hi) into one fp32 accumulator: its operands count to about 2^-16,
// its sums and everything between the products are fp32.  Chunks are kChunk tokens and END with the entry: the first one of an
// entry is the short one, so a weighted key does not depend on how many tokens its chunk has.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <cstdint>
#include <cstdlib>

#include "seq_engine.h"
#include "seq_linear.cuh"
#include "seq_mma.cuh"

namespace kllm {
namespace seq {
namespace {

constexpr int kChunk = 64;
constexpr int kFrom = 64;      // steps whose longest entry has more tokens come here
constexpr int kMaxHead = 128;  // key and value sizes: multiples of 16 up to this
constexpr int kThreads = 256;

// chunk c of entry e: slot in the scratch buffers; rows [base, base + n) of the entry, at places off .. kChunk - 1 of the chunk
struct ChunkAt {
  int base, off, n;
  size_t slot;
};
__device__ __forceinline__ ChunkAt chunk_at(int first, int count, int e, int c) {
  const int chunks = (count + kChunk - 1) / kChunk;
  const int n0 = count - (chunks - 1) * kChunk;  // tokens of the first chunk
  ChunkAt a;
  a.n = c == 0 ? n0 : kChunk;
  a.base = c == 0 ? 0 : n0 + (c - 1) * kChunk;
  a.off = kChunk - a.n;
  a.slot = static_cast<size_t>(first / kChunk + e + c);
  return a;
}

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

struct Planes {  // [T][row] bf16: q | k | k weighted | v
  __nv_bfloat16 *hi, *lo;
  int row;
};
__device__ __forceinline__ void put_split(const Planes& p, size_t at, const float4& v) {
  uint32_t h0, l0, h1, l1;
  split_pack(v.x, v.y, h0, l0);
  split_pack(v.z, v.w, h1, l1);
  *reinterpret_cast<uint2*>(p.hi + at) = make_uint2(h0, h1);
  *reinterpret_cast<uint2*>(p.lo + at) = make_uint2(l0, l1);
}
__device__ __forceinline__ void put_split(const Planes& p, size_t at, float v) {
  const __nv_bfloat16 h = __float2bfloat16_rn(v);
  p.hi[at] = h;
  p.lo[at] = __float2bfloat16_rn(v - __bfloat162float(h));
}
__device__ __forceinline__ float4 times(const float4& a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }

// Grid: (token of the entry, entry).  V: pairs that turn at once (4: halves paired, sizes that allow 16-byte accesses; 1: any).
template <int V, bool SILU>
__global__ void __launch_bounds__(kThreads)
linear_split_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, LinearRot rot, const float* __restrict__ proj,
                    int stride, const int32_t* __restrict__ ent_first, const int32_t* __restrict__ ent_count,
                    const int32_t* __restrict__ ent_pos0, Planes out) {
  extern __shared__ __align__(16) float sm[];  // [half] cos, [half] sin, [heads] weights of this token's keys
  const int e = blockIdx.y, i = blockIdx.x, count = ent_count[e];
  if (i >= count) return;
  const int half = rot.rope.dims / 2, qn = heads * dim;
  float *co = sm, *si = sm + half, *weight = sm + 2 * half;
  for (int p = threadIdx.x; p < half; p += kThreads) rope_turn(rot.rope, p, ent_pos0[e] + i, co[p], si[p]);
  for (int h = threadIdx.x; h < heads; h += kThreads) weight[h] = decay_power(logf(decay[h]), (count - 1 - i) % kChunk);
  __syncthreads();
  const int t = ent_first[e] + i;
  const float* row = proj + static_cast<size_t>(t) * stride;
  const size_t o = static_cast<size_t>(t) * out.row;
  if constexpr (V == 4) {
    const int turn = half / 4, per = turn + (dim - 2 * half) / 4;  // units of a head: pairs of quads, then quads
    for (int u = threadIdx.x; u < 2 * heads * per; u += kThreads) {
      const int g = u / per, p = u % per, h = g < heads ? g : g - heads;  // g: query heads, then key heads
      const float* src = row + g * dim;
      const bool key = g >= heads;
      const float ks = key ? rot.k_scale : 1.0f;
      const int d0 = p < turn ? 4 * p : 2 * half + 4 * (p - turn), d1 = half + 4 * p;
      float4 a = *reinterpret_cast<const float4*>(src + d0);
      const size_t at = o + g * dim, atw = o + 2 * qn + h * dim;
      if (p < turn) {
        const float4 b = *reinterpret_cast<const float4*>(src + d1);
        const float4 c = *reinterpret_cast<const float4*>(co + 4 * p), z = *reinterpret_cast<const float4*>(si + 4 * p);
        const float4 y = make_float4((b.x * c.x + a.x * z.x) * ks, (b.y * c.y + a.y * z.y) * ks, (b.z * c.z + a.z * z.z) * ks,
                                     (b.w * c.w + a.w * z.w) * ks);
        a = make_float4((a.x * c.x - b.x * z.x) * ks, (a.y * c.y - b.y * z.y) * ks, (a.z * c.z - b.z * z.z) * ks,
                        (a.w * c.w - b.w * z.w) * ks);
        put_split(out, at + d1, y);
        if (key) put_split(out, atw + d1, times(y, weight[h]));
      } else if (SILU) {
        a = make_float4(silu(a.x), silu(a.y), silu(a.z), silu(a.w));
      } else {
        a = times(a, ks);
      }
      put_split(out, at + d0, a);
      if (key) put_split(out, atw + d0, times(a, weight[h]));
    }
    for (int c = threadIdx.x * 4; c < heads * vdim; c += kThreads * 4) {
      float4 v = *reinterpret_cast<const float4*>(row + 2 * qn + c);
      if (SILU) v = make_float4(silu(v.x), silu(v.y), silu(v.z), silu(v.w));
      put_split(out, o + 3 * qn + c, v);
    }
  } else {
    const bool pairs = rot.rope.pairing == KLLM_SEQ_ROPE_PAIRS;
    const int per = half + dim - 2 * half;  // pairs, then coordinates that do not turn
    for (int u = threadIdx.x; u < 2 * heads * per; u += kThreads) {
      const int g = u / per, p = u % per, h = g < heads ? g : g - heads;
      const float* src = row + g * dim;
      const bool key = g >= heads;
      const float ks = key ? rot.k_scale : 1.0f;
      const size_t at = o + g * dim, atw = o + 2 * qn + h * dim;
      if (p < half) {
        const int d0 = pairs ? 2 * p : p, d1 = pairs ? 2 * p + 1 : p + half;
        const float a = src[d0], b = src[d1], x = (a * co[p] - b * si[p]) * ks, y = (b * co[p] + a * si[p]) * ks;
        put_split(out, at + d0, x);
        put_split(out, at + d1, y);
        if (key) put_split(out, atw + d0, x * weight[h]), put_split(out, atw + d1, y * weight[h]);
      } else {
        const int d = half + p;
        const float x = SILU ? silu(src[d]) : src[d] * ks;
        put_split(out, at + d, x);
        if (key) put_split(out, atw + d, x * weight[h]);
      }
    }
    for (int c = threadIdx.x; c < heads * vdim; c += kThreads) {
      const float v = row[2 * qn + c];
      put_split(out, o + 3 * qn + c, SILU ? silu(v) : v);
    }
  }
}

// Chunk rows of one head out of the planes into shared memory, both terms: [kChunk][ld] hi, then lo; rows before `off` are zero.
__device__ __forceinline__ void load_rows(uint32_t dst, int ld, const Planes& p, int col, int cols, int t0, int off) {
  const int chunks = cols / 8;
  for (int i = threadIdx.x; i < kChunk * chunks; i += kThreads) {
    const int r = i / chunks, c = (i % chunks) * 8;
    const bool in = r >= off;
    const size_t at = in ? static_cast<size_t>(t0 + r - off) * p.row + col + c : 0;
    cp_async16(dst + (r * ld + c) * 2, p.hi + at, in);
    cp_async16(dst + (kChunk * ld + r * ld + c) * 2, p.lo + at, in);
  }
}

// acc += a b, a and b as two terms each (the product of the two low terms is below what the sum keeps)
__device__ __forceinline__ void mma_split(float (&acc)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1,
                                          uint32_t bl0, uint32_t bl1) {
  mma_bf16(acc, ah, bh0, bh1);
  mma_bf16(acc, ah, bl0, bl1);
  mma_bf16(acc, al, bh0, bh1);
}

// Value columns of a head go to two warps per row tile: pairs of 8-column blocks, the first half (rounded up) and the rest.
__device__ __forceinline__ void column_half(int vdim, int hf, int& first_pair, int& n_pairs) {
  const int pairs = vdim / 16, left = (pairs + 1) / 2;
  first_pair = hf == 0 ? 0 : left;
  n_pairs = hf == 0 ? left : pairs - left;
}
constexpr int kPairs = kMaxHead / 32;

// Grid: (chunk, head, entry).  A warp takes 16 key coordinates and half of the value columns at a time.
__global__ void __launch_bounds__(kThreads)
linear_sums_kernel(int heads, int dim, int vdim, Planes in, const int32_t* __restrict__ ent_first,
                   const int32_t* __restrict__ ent_count, float* __restrict__ sums) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int e = blockIdx.z, h = blockIdx.y, count = ent_count[e], first = ent_first[e];
  if (static_cast<int>(blockIdx.x) * kChunk >= count) return;
  const ChunkAt c = chunk_at(first, count, e, blockIdx.x);
  const int ldk = dim + 8, ldv = vdim + 8;
  const uint32_t k_sm = static_cast<uint32_t>(__cvta_generic_to_shared(raw)), v_sm = k_sm + 2 * kChunk * ldk * 2;
  const int qn = heads * dim;
  load_rows(k_sm, ldk, in, 2 * qn + h * dim, dim, first + c.base, c.off);
  load_rows(v_sm, ldv, in, 3 * qn + h * vdim, vdim, first + c.base, c.off);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3, gq = lane >> 2, t4 = lane & 3;
  float* out = sums + (c.slot * heads + h) * dim * vdim;
  for (int item = warp; item < dim / 8; item += kThreads / 32) {
    const int mt = item >> 1;
    int p0, np;
    column_half(vdim, item & 1, p0, np);
    float acc[kPairs][2][4];
#pragma unroll
    for (int p = 0; p < kPairs; ++p)
#pragma unroll
      for (int z = 0; z < 4; ++z) acc[p][0][z] = acc[p][1][z] = 0.f;
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      uint32_t ah[4], al[4];
      const uint32_t ka = k_sm + ((kk * 16 + (mi >> 1) * 8 + (lane & 7)) * ldk + mt * 16 + (mi & 1) * 8) * 2;
      ldmatrix_x4_trans(ka, ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4_trans(ka + kChunk * ldk * 2, al[0], al[1], al[2], al[3]);
      const uint32_t va = v_sm + ((kk * 16 + (mi & 1) * 8 + (lane & 7)) * ldv + p0 * 16 + (mi >> 1) * 8) * 2;
#pragma unroll
      for (int p = 0; p < kPairs; ++p) {
        if (p >= np) break;
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(va + p * 32, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(va + p * 32 + kChunk * ldv * 2, bl[0], bl[1], bl[2], bl[3]);
        mma_split(acc[p][0], ah, al, bh[0], bh[1], bl[0], bl[1]);
        mma_split(acc[p][1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int p = 0; p < kPairs; ++p) {
      if (p >= np) break;
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        const int col = (p0 + p) * 16 + b * 8 + t4 * 2;
        *reinterpret_cast<float2*>(out + static_cast<size_t>(mt * 16 + gq) * vdim + col) = make_float2(acc[p][b][0], acc[p][b][1]);
        *reinterpret_cast<float2*>(out + static_cast<size_t>(mt * 16 + gq + 8) * vdim + col) = make_float2(acc[p][b][2], acc[p][b][3]);
      }
    }
  }
}

// Grid: (slice of a head's state, head, entry); a thread carries two neighbouring elements through the entry's chunks.
__global__ void linear_carry_kernel(int heads, int size, const float* __restrict__ decay, float* __restrict__ state,
                                    const int32_t* __restrict__ ent_first, const int32_t* __restrict__ ent_count,
                                    const int32_t* __restrict__ ent_seq, const int32_t* __restrict__ ent_pos0,
                                    const float* __restrict__ sums, __nv_bfloat16* __restrict__ before_hi,
                                    __nv_bfloat16* __restrict__ before_lo) {
  const int e = blockIdx.z, h = blockIdx.y, i = (blockIdx.x * blockDim.x + threadIdx.x) * 2;
  if (i >= size) return;
  const int count = ent_count[e], first = ent_first[e], chunks = (count + kChunk - 1) / kChunk;
  const float log_decay = logf(decay[h]), full = decay_power(log_decay, kChunk);
  float2* sg = reinterpret_cast<float2*>(state + (static_cast<size_t>(ent_seq[e]) * heads + h) * size + i);
  float2 s = ent_pos0[e] == 0 ? make_float2(0.f, 0.f) : *sg;
  constexpr int U = 8;  // chunk sums fetched ahead: the loads do not depend on one another, only the sums do
  for (int c0 = 0; c0 < chunks; c0 += U) {
    float2 add[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      add[u] = c0 + u < chunks ? *reinterpret_cast<const float2*>(sums + (chunk_at(first, count, e, c0 + u).slot * heads + h) * size + i)
                               : make_float2(0.f, 0.f);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u >= chunks) break;
      const ChunkAt c = chunk_at(first, count, e, c0 + u);
      uint32_t hi, lo;
      split_pack(s.x, s.y, hi, lo);
      const size_t at = (c.slot * heads + h) * size + i;
      *reinterpret_cast<uint32_t*>(before_hi + at) = hi;
      *reinterpret_cast<uint32_t*>(before_lo + at) = lo;
      const float f = c.n == kChunk ? full : decay_power(log_decay, c.n);
      s.x = fmaf(s.x, f, add[u].x), s.y = fmaf(s.y, f, add[u].y);
    }
  }
  *sg = s;
}

struct RowsOut {
  float* o;               // [T][heads * vdim] fp32, or null: `out` below
  __nv_bfloat16* out;     // [T][heads * vdim]: o / rms(o of the head) * act(gate)
  const float* gate;      // gate rows of the projection
  int gate_stride, gate_act;
  int gate_vec;           // != 0: gate rows can be read 16 bytes at a time
  float eps;
};

// Grid: (chunk, head, entry).  Warp w: rows 16 (w % 4) .. + 15 of the chunk, half w / 4 of the value columns.  Beside the queries
// two tiles of shared memory take turns: keys, the upper and the lower rows of the state, values -- each is on its way while
// the one before it is multiplied, and two CTAs fit an SM.
__global__ void __launch_bounds__(kThreads, 2)
linear_rows_kernel(int heads, int dim, int vdim, const float* __restrict__ decay, Planes in, const int32_t* __restrict__ ent_first,
                   const int32_t* __restrict__ ent_count, const __nv_bfloat16* __restrict__ before_hi,
                   const __nv_bfloat16* __restrict__ before_lo, RowsOut ro) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float pw[kChunk + 1];       // powers of the decay
  __shared__ float square[2][kChunk];    // sums of squares of a row's halves
  const int e = blockIdx.z, h = blockIdx.y, count = ent_count[e], first = ent_first[e];
  if (static_cast<int>(blockIdx.x) * kChunk >= count) return;
  const ChunkAt c = chunk_at(first, count, e, blockIdx.x);
  const int ldq = dim + 8, ldv = vdim + 8, qn = heads * dim;
  const uint32_t q_sm = static_cast<uint32_t>(__cvta_generic_to_shared(raw)), k_sm = q_sm + 2 * kChunk * ldq * 2;
  const uint32_t tile = 2 * kChunk * max(ldq, ldv) * 2, v_sm = k_sm + tile;  // v_sm: the second tile
  const int t0 = first + c.base;
  const int upper = (dim / 16 + 1) / 2 * 16;  // rows of the state in its first part
  auto load_state = [&](uint32_t dst, int d0, int d1) {
    const int chunks = vdim / 8;
    const size_t at0 = (c.slot * heads + h) * dim * vdim;
    for (int i = threadIdx.x; i < (d1 - d0) * chunks; i += kThreads) {
      const int d = i / chunks, col = (i % chunks) * 8;
      const size_t at = at0 + static_cast<size_t>(d0 + d) * vdim + col;
      cp_async16(dst + (d * ldv + col) * 2, before_hi + at, true);
      cp_async16(dst + ((kChunk + d) * ldv + col) * 2, before_lo + at, true);
    }
    cp_async_commit();
  };
  load_rows(q_sm, ldq, in, h * dim, dim, t0, c.off);
  load_rows(k_sm, ldq, in, qn + h * dim, dim, t0, c.off);
  cp_async_commit();
  load_state(v_sm, 0, upper);
  if (threadIdx.x <= kChunk) pw[threadIdx.x] = decay_power(logf(decay[h]), threadIdx.x);

  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3, gq = lane >> 2, t4 = lane & 3;
  const int mt = warp & 3, hf = warp >> 2;
  const int rA = mt * 16 + gq, rB = rA + 8;
  int p0, np;
  column_half(vdim, hf, p0, np);
  const uint32_t qa = q_sm + ((mt * 16 + (lane & 15)) * ldq + (lane >> 4) * 8) * 2;

  cp_async_wait<1>();
  __syncthreads();
  // scores of the rows against the chunk's tokens up to the row tile's last
  float s[kChunk / 8][4];
#pragma unroll
  for (int j = 0; j < kChunk / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
  for (int ks = 0; ks < dim / 16; ++ks) {
    uint32_t ah[4], al[4];
    ldmatrix_x4(qa + ks * 32, ah[0], ah[1], ah[2], ah[3]);
    ldmatrix_x4(qa + ks * 32 + kChunk * ldq * 2, al[0], al[1], al[2], al[3]);
    const uint32_t ka = k_sm + (((mi >> 1) * 8 + (lane & 7)) * ldq + ks * 16 + (mi & 1) * 8) * 2;
#pragma unroll
    for (int p = 0; p < kChunk / 16; ++p) {
      if (p > mt) break;
      uint32_t bh[4], bl[4];
      ldmatrix_x4(ka + p * 16 * ldq * 2, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4(ka + p * 16 * ldq * 2 + kChunk * ldq * 2, bl[0], bl[1], bl[2], bl[3]);
      mma_split(s[2 * p], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(s[2 * p + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    }
  }
#pragma unroll
  for (int j = 0; j < kChunk / 8; ++j)
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      const int r = z < 2 ? rA : rB, key = j * 8 + t4 * 2 + (z & 1);
      s[j][z] = key <= r ? s[j][z] * pw[r - key] : 0.f;
    }
  // the state before the chunk, decayed to each row
  float acc[kPairs][2][4];
#pragma unroll
  for (int p = 0; p < kPairs; ++p)
#pragma unroll
    for (int z = 0; z < 4; ++z) acc[p][0][z] = acc[p][1][z] = 0.f;
  cp_async_wait<0>();
  __syncthreads();  // the upper rows are in; the keys are no longer read
  load_state(k_sm, upper, dim);
  auto times_state = [&](uint32_t part, int ks0, int ks1) {
    for (int ks = ks0; ks < ks1; ++ks) {
      uint32_t ah[4], al[4];
      ldmatrix_x4(qa + ks * 32, ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(qa + ks * 32 + kChunk * ldq * 2, al[0], al[1], al[2], al[3]);
      const uint32_t sa = part + (((ks - ks0) * 16 + (mi & 1) * 8 + (lane & 7)) * ldv + p0 * 16 + (mi >> 1) * 8) * 2;
#pragma unroll
      for (int p = 0; p < kPairs; ++p) {
        if (p >= np) break;
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(sa + p * 32, bh[0], bh[1], bh[2], bh[3]);
        ldmatrix_x4_trans(sa + p * 32 + kChunk * ldv * 2, bl[0], bl[1], bl[2], bl[3]);
        mma_split(acc[p][0], ah, al, bh[0], bh[1], bl[0], bl[1]);
        mma_split(acc[p][1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      }
    }
  };
  times_state(v_sm, 0, upper / 16);
  cp_async_wait<0>();
  __syncthreads();  // the lower rows are in; the upper ones are no longer read
  load_rows(v_sm, ldv, in, 3 * qn + h * vdim, vdim, t0, c.off);
  cp_async_commit();
  times_state(k_sm, upper / 16, dim / 16);
  const float fA = pw[max(0, rA - c.off + 1)], fB = pw[max(0, rB - c.off + 1)];
#pragma unroll
  for (int p = 0; p < kPairs; ++p)
#pragma unroll
    for (int b = 0; b < 2; ++b) acc[p][b][0] *= fA, acc[p][b][1] *= fA, acc[p][b][2] *= fB, acc[p][b][3] *= fB;
  cp_async_wait<0>();
  __syncthreads();  // the values are in; the first tile is free: the head's gate rows come in under the last product
  const bool staged = ro.o == nullptr && ro.gate_vec;
  if (staged) {
    const int quads = vdim / 4;
    for (int i = threadIdx.x; i < kChunk * quads; i += kThreads) {
      const int r = i / quads, col = (i % quads) * 4;
      const bool in = r >= c.off;
      cp_async16(k_sm + (r * ldv + col) * 4, in ? ro.gate + static_cast<size_t>(t0 + r - c.off) * ro.gate_stride + h * vdim + col : ro.gate, in);
    }
    cp_async_commit();
  }
#pragma unroll
  for (int kk = 0; kk < kChunk / 16; ++kk) {
    if (kk > mt) break;
    uint32_t ah[4], al[4];
    split_pack(s[2 * kk][0], s[2 * kk][1], ah[0], al[0]);
    split_pack(s[2 * kk][2], s[2 * kk][3], ah[1], al[1]);
    split_pack(s[2 * kk + 1][0], s[2 * kk + 1][1], ah[2], al[2]);
    split_pack(s[2 * kk + 1][2], s[2 * kk + 1][3], ah[3], al[3]);
    const uint32_t va = v_sm + ((kk * 16 + (mi & 1) * 8 + (lane & 7)) * ldv + p0 * 16 + (mi >> 1) * 8) * 2;
#pragma unroll
    for (int p = 0; p < kPairs; ++p) {
      if (p >= np) break;
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(va + p * 32, bh[0], bh[1], bh[2], bh[3]);
      ldmatrix_x4_trans(va + p * 32 + kChunk * ldv * 2, bl[0], bl[1], bl[2], bl[3]);
      mma_split(acc[p][0], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(acc[p][1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    }
  }
  const int vn = heads * vdim;
  const bool inA = rA >= c.off, inB = rB >= c.off;
  const size_t tA = static_cast<size_t>(t0 + rA - c.off), tB = static_cast<size_t>(t0 + rB - c.off);  // read only when the row exists
  if (ro.o != nullptr) {
#pragma unroll
    for (int p = 0; p < kPairs; ++p) {
      if (p >= np) break;
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        const int col = h * vdim + (p0 + p) * 16 + b * 8 + t4 * 2;
        if (inA) *reinterpret_cast<float2*>(ro.o + tA * vn + col) = make_float2(acc[p][b][0], acc[p][b][1]);
        if (inB) *reinterpret_cast<float2*>(ro.o + tB * vn + col) = make_float2(acc[p][b][2], acc[p][b][3]);
      }
    }
    return;
  }
  float qA = 0.f, qB = 0.f;
#pragma unroll
  for (int p = 0; p < kPairs; ++p)
#pragma unroll
    for (int b = 0; b < 2; ++b) {  // blocks past the columns are zero
      qA = fmaf(acc[p][b][0], acc[p][b][0], fmaf(acc[p][b][1], acc[p][b][1], qA));
      qB = fmaf(acc[p][b][2], acc[p][b][2], fmaf(acc[p][b][3], acc[p][b][3], qB));
    }
  qA = quad_sum(qA), qB = quad_sum(qB);
  if (t4 == 0) square[hf][rA] = qA, square[hf][rB] = qB;
  cp_async_wait<0>();
  __syncthreads();
  const float* gates = reinterpret_cast<const float*>(raw + (k_sm - q_sm));  // [kChunk][ldv] when they are staged
  const float nA = 1.0f / sqrtf((square[0][rA] + square[1][rA]) / static_cast<float>(vdim) + ro.eps);
  const float nB = 1.0f / sqrtf((square[0][rB] + square[1][rB]) / static_cast<float>(vdim) + ro.eps);
  auto gated = [&](float o, float z) { return o * (ro.gate_act == KLLM_SEQ_GATEACT_SILU ? silu(z) : 1.0f / (1.0f + expf(-z))); };
#pragma unroll
  for (int p = 0; p < kPairs; ++p) {
    if (p >= np) break;
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int col = h * vdim + (p0 + p) * 16 + b * 8 + t4 * 2;
#pragma unroll
      for (int z = 0; z < 2; ++z) {
        if (!(z == 0 ? inA : inB)) continue;
        const size_t t = z == 0 ? tA : tB;
        const float n = z == 0 ? nA : nB;
        float2 g;
        if (staged) {
          g = *reinterpret_cast<const float2*>(gates + (z == 0 ? rA : rB) * ldv + col - h * vdim);
        } else {
          const float* src = ro.gate + t * ro.gate_stride + col;
          g = make_float2(src[0], src[1]);
        }
        *reinterpret_cast<__nv_bfloat162*>(ro.out + t * vn + col) =
            __floats2bfloat162_rn(gated(acc[p][b][2 * z] * n, g.x), gated(acc[p][b][2 * z + 1] * n, g.y));
      }
    }
  }
}

size_t slots(int T, int n_entries) { return static_cast<size_t>(T) / kChunk + n_entries + 1; }
size_t plane_elems(const kllm_seq_linear& m, int T) { return static_cast<size_t>(T) * m.heads * (3 * m.dim + m.vdim); }

template <typename Kernel>
int allow_smem(Kernel kernel, size_t smem, size_t* configured) {
  if (smem <= 48 * 1024 || smem <= *configured) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e == cudaSuccess) *configured = smem;
  return cuda_rc(e);
}
int launched() {
  count_launch();
  return cuda_rc(cudaGetLastError());
}

}  // namespace

bool linear_mma_usable(int dtype, const kllm_seq_linear& m, int max_count) {
  static const bool off = [] { const char* e = getenv("KLLM_SEQ_LINEAR_MMA"); return e != nullptr && e[0] == '0'; }();
  return !off && dtype == KLLM_SEQ_BF16 && max_count > kFrom && m.dim % 16 == 0 && m.dim <= kMaxHead && m.vdim % 16 == 0 && m.vdim <= kMaxHead &&
         m.heads <= 65535;
}

size_t linear_mma_scratch_bytes(const kllm_seq_linear& m, int T, int n_entries) {
  // two planes of rows, the chunk sums (fp32), the states before the chunks (two bf16 terms)
  return 2 * plane_elems(m, T) * 2 + slots(T, n_entries) * m.heads * m.dim * m.vdim * 8;
}

int launch_linear_mma(const kllm_seq_linear& m, const float* proj, int row, float* state, int n_entries, const int32_t* ent_first,
                      const int32_t* ent_count, const int32_t* ent_seq, const int32_t* ent_pos0, int max_count, int T, float eps,
                      void* scratch, float* o, void* out, cudaStream_t s) {
  if (n_entries > 65535) return KLLM_E_UNSUPPORTED;
  const int size = m.dim * m.vdim;
  const size_t pe = plane_elems(m, T), se = slots(T, n_entries) * m.heads * size;
  __nv_bfloat16* base = static_cast<__nv_bfloat16*>(scratch);
  const Planes planes{base, base + pe, m.heads * (3 * m.dim + m.vdim)};
  float* sums = reinterpret_cast<float*>(base + 2 * pe);
  __nv_bfloat16* before = reinterpret_cast<__nv_bfloat16*>(sums + se);
  const LinearRot rot = linear_rot(m);
  const int half = m.rope_dims / 2;
  const bool vec = half % 4 == 0 && (half == 0 || m.rope_pairing == KLLM_SEQ_ROPE_HALVES) && row % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
  const size_t smem_split = (2 * static_cast<size_t>(half) + m.heads) * sizeof(float);
  const dim3 tokens(max_count, n_entries);
#define KLLM_LINEAR_SPLIT(V, SILU) \
  linear_split_kernel<V, SILU><<<tokens, kThreads, smem_split, s>>>(m.heads, m.dim, m.vdim, m.decay, rot, proj, row, ent_first, ent_count, ent_pos0, planes)
  if (m.qkv_act == KLLM_SEQ_QKV_SILU) {
    if (vec) KLLM_LINEAR_SPLIT(4, true);
    else KLLM_LINEAR_SPLIT(1, true);
  } else {
    if (vec) KLLM_LINEAR_SPLIT(4, false);
    else KLLM_LINEAR_SPLIT(1, false);
  }
#undef KLLM_LINEAR_SPLIT
  if (int rc = launched()) return rc;
  const size_t rows_k = 2 * static_cast<size_t>(kChunk) * (m.dim + 8) * 2, rows_v = 2 * static_cast<size_t>(kChunk) * (m.vdim + 8) * 2;
  const size_t smem_sums = rows_k + rows_v, smem_rows = rows_k + 2 * std::max(rows_k, rows_v);
  static size_t configured_sums = 0, configured_rows = 0;
  if (int rc = allow_smem(linear_sums_kernel, smem_sums, &configured_sums)) return rc;
  if (int rc = allow_smem(linear_rows_kernel, smem_rows, &configured_rows)) return rc;
  const dim3 grid((max_count + kChunk - 1) / kChunk, m.heads, n_entries);
  linear_sums_kernel<<<grid, kThreads, smem_sums, s>>>(m.heads, m.dim, m.vdim, planes, ent_first, ent_count, sums);
  if (int rc = launched()) return rc;
  const dim3 cgrid((size / 2 + 127) / 128, m.heads, n_entries);
  linear_carry_kernel<<<cgrid, 128, 0, s>>>(m.heads, size, m.decay, state, ent_first, ent_count, ent_seq, ent_pos0, sums, before,
                                            before + se);
  if (int rc = launched()) return rc;
  const float* gate = proj + 2 * m.heads * m.dim + m.heads * m.vdim;
  const RowsOut ro{o, static_cast<__nv_bfloat16*>(out), gate, row, m.gate_act,
                   row % 4 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0, eps};
  linear_rows_kernel<<<grid, kThreads, smem_rows, s>>>(m.heads, m.dim, m.vdim, m.decay, planes, ent_first, ent_count, before, before + se,
                                                       ro);
  return launched();
}

}  // namespace seq
}  // namespace kllm
