// Prompt attention of the sequence-batch engine on the tensor cores (bf16 operands, fp32 accumulation).
//
// Same problem as attention_kernel in seq_kernels.cu -- causal softmax attention of a ragged batch over paged keys and
// values, query heads grouped over key/value heads -- for steps that bring many rows: one CTA takes 64 consecutive rows
// of one entry and one key/value head (row r = token r / rep, query head g * rep + r % rep, so the `rep` query heads of
// a token share every key tile), one warp 16 of them.
//
//   scores    S = Q K^T by mma.sync m16n8k16 (bf16 x bf16 -> fp32); scale, causal mask, running maximum and sum, and
//             the exponentials (ex2.approx on scores in units of log2, relative error about 2^-22) are fp32 in
//             registers (online softmax); only tiles that touch the diagonal are masked
//   weights   the fp32 weights p enter the second product as TWO bf16 terms, p = hi + lo (lo = p - hi rounded), so the
//             product sees them to about 2^-17 instead of 2^-9: the values are bf16 already, the weights are not
//   output    O += (hi + lo) V, fp32 accumulators; V fragments come transposed out of shared memory (ldmatrix.trans)
//   tiles     64 keys x (dim | vdim) bf16 through a two-stage cp.async ring, rows padded by 16 bytes (conflict-free
//             fragment loads); keys past the last visible position are zero-filled
//   sizes     the kernel is compiled for head sizes of 64 and 128; a model's dim / vdim (multiples of 8) run in the
//             next size up with the missing columns zero-filled in shared memory and never stored
//
// With one split the kernel divides by the sum, applies the output gate and writes the compute type; with several it
// leaves (max, sum, unnormalised output) per split for attention_merge_kernel, like the fp32 kernel.
// attention_rows_mma_kernel (second half of this file) serves steps of FEW rows per key head -- single-token steps, short
// portions -- and fp32 queries (an attention through a latent: all query heads share one key row per token): one CTA takes
// at most 16 (token, query head) rows, one split of the keys, and walks tiles of 32 keys.  The queries enter as two bf16
// terms when they are fp32, the weights always do, so both products see their left operand to about 2^-17.
//
// tcgen05 is not used here: at head sizes of 64..128 a 64-row tile is small against TMEM's 128-lane accumulators, and
// the softmax between the two products wants the scores in registers anyway.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cmath>
#include <cstdint>
#include <cstdlib>

#include "seq_engine.h"
#include "seq_mma.cuh"

namespace kllm {
namespace seq {
namespace {

constexpr int kRows = 64, kKeys = 64, kThreads = 128;

__device__ __forceinline__ float exp2_approx(float x) {  // 2^x, relative error about 2^-22; 2^-inf = 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <int DIM, int VDIM>
__global__ void __launch_bounds__(kThreads, (DIM + VDIM <= 128) ? 4 : (DIM > 128 ? 1 : 0))
attention_mma_kernel(AttnShape a, const __nv_bfloat16* __restrict__ q, PagedKV kv, const int32_t* __restrict__ ent_first,
                     const int32_t* __restrict__ ent_count, const int32_t* __restrict__ ent_seq,
                     const int32_t* __restrict__ ent_pos0, int splits, float* __restrict__ ws,
                     const float* __restrict__ gates, __nv_bfloat16* __restrict__ out) {
  constexpr int LDK = DIM + 8, LDV = VDIM + 8;  // bf16 elements per shared-memory row
  constexpr int KS = DIM / 16;                  // k-steps of Q K^T
  constexpr int NB = VDIM / 8;                  // 8-column blocks of the output
  constexpr int KC = DIM / 8, VC = VDIM / 8;    // 16-byte chunks per key / value row
  // grid: x = (entry, key/value head), y = row tile, z = split.  CTAs are handed out in x-fastest order, so the tiles
  // of equal weight (the same rows of every head) start together, heaviest first
  const int e = blockIdx.x / a.kv_heads, g = blockIdx.x % a.kv_heads, split = blockIdx.z;
  const int gv = g / v_share_of(a);  // the value head this key head reads
  const int rep = a.heads / a.kv_heads;
  const int dim = a.dim, vdim = a.vdim;  // <= DIM, VDIM; multiples of 8
  const int count = ent_count[e], first = ent_first[e], seq = ent_seq[e], pos0 = ent_pos0[e];
  const int n_rows = count * rep;
  const int r0 = (gridDim.y - 1 - blockIdx.y) * kRows;  // the tiles with the most keys start first
  if (r0 >= n_rows) return;
  const int rows_here = min(kRows, n_rows - r0);
  const int pmax = pos0 + (r0 + rows_here - 1) / rep;  // last position any row of the tile sees
  const int n_tiles = pmax / kKeys + 1;
  // with a window or chunks no row of the tile sees anything before what its first row sees
  const int tile_first = first_seen(a, pos0 + r0 / rep) / kKeys;
  // tiles before the window that hold kept first positions come ahead of the window's tiles: this CTA's list of tiles
  // is [0, keep_tiles) then [tile_first, n_tiles), cut into `splits` parts
  const int keep_first = a.keep_first;
  const int keep_tiles = min(tile_first, (keep_first + kKeys - 1) / kKeys);
  const int list_n = keep_tiles + n_tiles - tile_first;
  const int per = (list_n + splits - 1) / splits;
  const int tile_lo = split * per, tile_hi = min(list_n, tile_lo + per);
  auto tile_of = [&](int li) { return li < keep_tiles ? li : tile_first + (li - keep_tiles); };
  const float softcap = a.softcap;

  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(sm_raw);  // [2][keys][LDK]
  __nv_bfloat16* Vs = Ks + 2 * kKeys * LDK;                      // [2][keys][LDV]

  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gq = lane >> 2, t4 = lane & 3;
  // the two rows of this thread's accumulator fragments
  const int rA = r0 + warp * 16 + gq, rB = rA + 8;
  const bool exA = rA < n_rows, exB = rB < n_rows;
  const int posA = exA ? pos0 + rA / rep : -1, posB = exB ? pos0 + rB / rep : -1;  // -1: sees nothing
  const size_t thA = exA ? static_cast<size_t>(first + rA / rep) * a.heads + g * rep + rA % rep : 0;
  const size_t thB = exB ? static_cast<size_t>(first + rB / rep) * a.heads + g * rep + rB % rep : 0;
  const int warp_last = __reduce_max_sync(0xffffffffu, max(posA, posB));  // last position any row of the warp sees
  // first position of the warp's rows (rows that do not exist count as -1: their tiles are always masked)
  const int warp_first = __reduce_min_sync(0xffffffffu, min(posA, posB));
  // the first key each of the two rows sees, and the least and greatest of these among the warp's rows
  constexpr int kNone = 0x7fffffff;
  const int loA = exA ? first_seen(a, posA) : kNone, loB = exB ? first_seen(a, posB) : kNone;
  const int warp_lo = __reduce_min_sync(0xffffffffu, min(loA, loB));
  const int warp_lo_last = __reduce_max_sync(0xffffffffu, max(exA ? loA : 0, exB ? loB : 0));
  const float scale2_plain = a.scale * 1.4426950408889634f;  // scores are kept in units of log2: exp(x) = 2^(x log2 e)

  uint32_t qf[KS][4];
  {
    const __nv_bfloat16* qa = q + thA * dim;
    const __nv_bfloat16* qb = q + thB * dim;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const int d = ks * 16 + t4 * 2;
      qf[ks][0] = exA && d < dim ? *reinterpret_cast<const uint32_t*>(qa + d) : 0u;
      qf[ks][1] = exB && d < dim ? *reinterpret_cast<const uint32_t*>(qb + d) : 0u;
      qf[ks][2] = exA && d + 8 < dim ? *reinterpret_cast<const uint32_t*>(qa + d + 8) : 0u;
      qf[ks][3] = exB && d + 8 < dim ? *reinterpret_cast<const uint32_t*>(qb + d + 8) : 0u;
    }
  }
  float o[NB][4];
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.f;
  float mA = -INFINITY, mB = -INFINITY, lA = 0.f, lB = 0.f;

  const __nv_bfloat16* kbase = static_cast<const __nv_bfloat16*>(kv.k);
  const __nv_bfloat16* vbase = static_cast<const __nv_bfloat16*>(kv.v);
  const int32_t* table = kv.table + static_cast<size_t>(seq) * kv.table_stride;
  const uint32_t ks_addr = static_cast<uint32_t>(__cvta_generic_to_shared(Ks));
  const uint32_t vs_addr = static_cast<uint32_t>(__cvta_generic_to_shared(Vs));

  auto load_tile = [&](int tile, int stage) {
    // two threads per key: the page lookup is done once per key and thread
    const int j = tid >> 1, kj = tile * kKeys + j;
    const bool valid = kj <= pmax;
    size_t slot = 0;
    // no page table: the keys and values are the step's own rows, row of position p = first + p - pos0
    if (valid) slot = kv.table ? static_cast<size_t>(table[kj / kv.page]) * kv.page + kj % kv.page
                               : static_cast<size_t>(first + max(kj - pos0, 0));
#pragma unroll
    for (int c = (tid & 1); c < KC + VC; c += 2) {
      if (c < KC) {
        const bool in = valid && c * 8 < dim;
        cp_async16(ks_addr + ((stage * kKeys + j) * LDK + c * 8) * 2,
                   in ? kbase + slot * kv.k_row + g * dim + c * 8 : kbase, in);
      } else {
        const bool in = valid && (c - KC) * 8 < vdim;
        cp_async16(vs_addr + ((stage * kKeys + j) * LDV + (c - KC) * 8) * 2,
                   in ? vbase + slot * kv.v_row + gv * vdim + (c - KC) * 8 : vbase, in);
      }
    }
    cp_async_commit();
  };

  if (tile_lo < tile_hi) load_tile(tile_of(tile_lo), 0);
  for (int li = tile_lo; li < tile_hi; ++li) {
    const int tile = tile_of(li);
    const int stage = (li - tile_lo) & 1;
    if (li + 1 < tile_hi) {
      load_tile(tile_of(li + 1), stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const int k0 = tile * kKeys;
    // otherwise no row of this warp sees a key of the tile (all later, or all before what every row sees)
    if (k0 <= warp_last && (k0 + kKeys > warp_lo || k0 < keep_first)) {
      float s[kKeys / 8][4];
#pragma unroll
      for (int j = 0; j < kKeys / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
      {
        // one ldmatrix.x4 = the key fragments (b0, b1) of two k-steps for 8 keys: lane l addresses key row l % 8 of
        // matrix l / 8 (matrices: dims +0, +8, +16, +24 of the same 8 keys)
        const uint32_t kt = ks_addr + (stage * kKeys * LDK + (lane & 7) * LDK + (lane >> 3) * 8) * 2;
#pragma unroll
        for (int ks = 0; ks < KS; ks += 2)
#pragma unroll
          for (int j = 0; j < kKeys / 8; ++j) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(kt + (j * 8 * LDK + ks * 16) * 2, b0, b1, b2, b3);
            mma_bf16(s[j], qf[ks], b0, b1);
            mma_bf16(s[j], qf[ks + 1], b2, b3);
          }
      }
      if (softcap > 0.f) {  // capped scores, then into units of log2 (the scale2 below is replaced by log2 e)
        const float inv = a.scale / softcap;
#pragma unroll
        for (int j = 0; j < kKeys / 8; ++j)
#pragma unroll
          for (int c = 0; c < 4; ++c) s[j][c] = softcap * tanhf(s[j][c] * inv);
      }
      const float scale2 = softcap > 0.f ? 1.4426950408889634f : scale2_plain;
      float mxA = -INFINITY, mxB = -INFINITY;
      if (k0 + kKeys - 1 <= warp_first && k0 >= warp_lo_last) {  // every row of the warp sees the whole tile
#pragma unroll
        for (int j = 0; j < kKeys / 8; ++j) {
          s[j][0] *= scale2, s[j][1] *= scale2, s[j][2] *= scale2, s[j][3] *= scale2;
          mxA = fmaxf(mxA, fmaxf(s[j][0], s[j][1]));
          mxB = fmaxf(mxB, fmaxf(s[j][2], s[j][3]));
        }
      } else {
#pragma unroll
        for (int j = 0; j < kKeys / 8; ++j) {
          const int kj = k0 + j * 8 + t4 * 2;
          s[j][0] = kj <= posA && (kj >= loA || kj < keep_first) ? s[j][0] * scale2 : -INFINITY;
          s[j][1] = kj + 1 <= posA && (kj + 1 >= loA || kj + 1 < keep_first) ? s[j][1] * scale2 : -INFINITY;
          s[j][2] = kj <= posB && (kj >= loB || kj < keep_first) ? s[j][2] * scale2 : -INFINITY;
          s[j][3] = kj + 1 <= posB && (kj + 1 >= loB || kj + 1 < keep_first) ? s[j][3] * scale2 : -INFINITY;
          mxA = fmaxf(mxA, fmaxf(s[j][0], s[j][1]));
          mxB = fmaxf(mxB, fmaxf(s[j][2], s[j][3]));
        }
      }
      const float nA = fmaxf(mA, quad_max(mxA)), nB = fmaxf(mB, quad_max(mxB));
      // a row that has seen nothing yet keeps max = -inf; subtracting 0 instead keeps 2^(-inf - 0) = 0 free of NaN
      const float subA = nA > -INFINITY ? nA : 0.f, subB = nB > -INFINITY ? nB : 0.f;
      const float alA = exp2_approx(mA - subA), alB = exp2_approx(mB - subB);
      float sumA = 0.f, sumB = 0.f;
#pragma unroll
      for (int j = 0; j < kKeys / 8; ++j) {
        s[j][0] = exp2_approx(s[j][0] - subA);
        s[j][1] = exp2_approx(s[j][1] - subA);
        s[j][2] = exp2_approx(s[j][2] - subB);
        s[j][3] = exp2_approx(s[j][3] - subB);
        sumA += s[j][0] + s[j][1];
        sumB += s[j][2] + s[j][3];
      }
      mA = nA, mB = nB;
      lA = lA * alA + sumA;  // the quad's partial sums are joined at the end (alpha is the same in a quad)
      lB = lB * alB + sumB;
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
        o[nb][0] *= alA, o[nb][1] *= alA;
        o[nb][2] *= alB, o[nb][3] *= alB;
      }
      const uint32_t vt = vs_addr + stage * kKeys * LDV * 2;
      const int mi = lane >> 3;  // which of the four 8x8 matrices this lane addresses
#pragma unroll
      for (int kk = 0; kk < kKeys / 16; ++kk) {
        uint32_t hi[4], lo[4];
        split_pack(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
        split_pack(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
        split_pack(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
        split_pack(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
        const uint32_t row_addr = vt + ((kk * 16 + (mi & 1) * 8 + (lane & 7)) * LDV + (mi >> 1) * 8) * 2;
#pragma unroll
        for (int nb2 = 0; nb2 < NB / 2; ++nb2) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(row_addr + nb2 * 16 * 2, b0, b1, b2, b3);
          mma_bf16(o[2 * nb2], hi, b0, b1);
          mma_bf16(o[2 * nb2], lo, b0, b1);
          mma_bf16(o[2 * nb2 + 1], hi, b2, b3);
          mma_bf16(o[2 * nb2 + 1], lo, b2, b3);
        }
      }
    }
    __syncthreads();  // the stage is loaded again two tiles on
  }
  lA = quad_sum(lA), lB = quad_sum(lB);
  if (splits == 1 && !a.no_merge) {
    if (a.sink != nullptr) {  // exp(sink) joins the denominator; scores are in units of log2
      constexpr float kLog2e = 1.4426950408889634f;
      if (exA) lA = mA > -INFINITY ? lA + exp2_approx(a.sink[thA % a.heads] * kLog2e - mA) : 1.0f;
      if (exB) lB = mB > -INFINITY ? lB + exp2_approx(a.sink[thB % a.heads] * kLog2e - mB) : 1.0f;
    }
    const bool per_element = gates != nullptr && a.gate == KLLM_SEQ_GATE_ELEMENT;
    const float gA = exA && gates && !per_element ? gates[thA] : 1.0f, gB = exB && gates && !per_element ? gates[thB] : 1.0f;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int col = nb * 8 + t4 * 2;
      if (col >= vdim) break;
      float2 eA = make_float2(gA, gA), eB = make_float2(gB, gB);
      if (per_element) {
        if (exA) eA = *reinterpret_cast<const float2*>(gates + thA * vdim + col);
        if (exB) eB = *reinterpret_cast<const float2*>(gates + thB * vdim + col);
      }
      if (exA)
        *reinterpret_cast<__nv_bfloat162*>(out + thA * vdim + col) =
            __floats2bfloat162_rn(o[nb][0] / lA * eA.x, o[nb][1] / lA * eA.y);
      if (exB)
        *reinterpret_cast<__nv_bfloat162*>(out + thB * vdim + col) =
            __floats2bfloat162_rn(o[nb][2] / lB * eB.x, o[nb][3] / lB * eB.y);
    }
    return;
  }
  const int pstride = vdim + 2;
  float* pa = ws + (thA * splits + split) * pstride;
  float* pb = ws + (thB * splits + split) * pstride;
  if (t4 == 0) {
    constexpr float kLn2 = 0.6931471805599453f;  // the merge works with natural logarithms
    if (exA) pa[0] = mA * kLn2, pa[1] = lA;
    if (exB) pb[0] = mB * kLn2, pb[1] = lB;
  }
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) {
    const int col = 2 + nb * 8 + t4 * 2;
    if (col >= pstride) break;
    if (exA) *reinterpret_cast<float2*>(pa + col) = make_float2(o[nb][0], o[nb][1]);
    if (exB) *reinterpret_cast<float2*>(pb + col) = make_float2(o[nb][2], o[nb][3]);
  }
}

template <int DIM, int VDIM>
int launch_mma(const AttnShape& a, const void* q, const float* gates, const PagedKV& kv, int n_entries,
               const int32_t* ent_first, const int32_t* ent_count, const int32_t* ent_seq, const int32_t* ent_pos0,
               int max_count, int splits, float* ws, void* out, cudaStream_t s) {
  constexpr size_t smem = 2 * kKeys * (DIM + 8 + VDIM + 8) * sizeof(__nv_bfloat16);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    const cudaError_t e = cudaFuncSetAttribute(attention_mma_kernel<DIM, VDIM>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return cuda_rc(e);
    configured = true;
  }
  const int rep = a.heads / a.kv_heads;
  const dim3 grid(n_entries * a.kv_heads, (max_count * rep + kRows - 1) / kRows, splits);
  if (grid.y > 65535u) return KLLM_E_UNSUPPORTED;
  attention_mma_kernel<DIM, VDIM><<<grid, kThreads, smem, s>>>(
      a, static_cast<const __nv_bfloat16*>(q), kv, ent_first, ent_count, ent_seq, ent_pos0, splits, ws,
      a.gate ? gates : nullptr, static_cast<__nv_bfloat16*>(out));
  count_launch();
  return cuda_rc(cudaGetLastError());
}

// ---- few rows ---------------------------------------------------------------------------------------------------------------
// Grid: x = 16-row tile, y = (entry, key/value head), z = split.  Four warps.  Scores: a warp takes 8 keys of the tile
// against all 16 rows.  Softmax: a warp takes 4 rows, a lane per key.  Output: the 8-column blocks are dealt out to the
// warps in turn (NBW per warp).  Values that are the head of the key row (SAME) are read from the key tile.
constexpr int kFewRows = 16, kFewKeys = 32, kFewThreads = 128, kFewWarps = 4;

struct FewLayout {  // shared memory, in bytes from its start
  int ldk, ldv, dimp;
  size_t k, v, q_hi, q_lo, s, p_hi, p_lo, stats, total;
};
__host__ __device__ inline FewLayout few_layout(const AttnShape& a, bool same, bool q_f32) {
  FewLayout L;
  L.dimp = (a.dim + 15) & ~15;
  L.ldk = L.dimp + 8, L.ldv = same ? L.ldk : ((a.vdim + 15) & ~15) + 8;
  size_t at = 0;
  L.k = at, at += 2 * static_cast<size_t>(kFewKeys) * L.ldk * 2;
  L.v = same ? L.k : at, at += same ? 0 : 2 * static_cast<size_t>(kFewKeys) * L.ldv * 2;
  L.q_hi = at, at += static_cast<size_t>(kFewRows) * L.ldk * 2;
  L.q_lo = at, at += q_f32 ? static_cast<size_t>(kFewRows) * L.ldk * 2 : 0;
  L.s = at, at += kFewRows * (kFewKeys + 1) * 4;
  at = (at + 15) & ~static_cast<size_t>(15);
  L.p_hi = at, at += kFewRows * (kFewKeys + 8) * 2;
  L.p_lo = at, at += kFewRows * (kFewKeys + 8) * 2;
  L.stats = at, at += 3 * kFewRows * 4;
  L.total = at;
  return L;
}

template <int NBW, bool SAME, bool QF32>
__global__ void __launch_bounds__(kFewThreads)
attention_rows_mma_kernel(AttnShape a, const void* __restrict__ q_, PagedKV kv, const int32_t* __restrict__ ent_first,
                          const int32_t* __restrict__ ent_count, const int32_t* __restrict__ ent_seq,
                          const int32_t* __restrict__ ent_pos0, int splits, float* __restrict__ ws) {
  const int e = blockIdx.y / a.kv_heads, g = blockIdx.y % a.kv_heads, split = blockIdx.z;
  const int gv = g / v_share_of(a);
  const int rep = a.heads / a.kv_heads, dim = a.dim, vdim = a.vdim;
  const int count = ent_count[e], first = ent_first[e], pos0 = ent_pos0[e];
  const int n_rows = count * rep, r0 = blockIdx.x * kFewRows;
  if (r0 >= n_rows) return;
  const int rows_here = min(kFewRows, n_rows - r0);
  const int32_t* table = kv.table + static_cast<size_t>(ent_seq[e]) * kv.table_stride;
  const int pmax = pos0 + (r0 + rows_here - 1) / rep;
  const int n_tiles = pmax / kFewKeys + 1;
  const int keep_first = a.keep_first;
  const int tile_first = first_seen(a, pos0 + r0 / rep) / kFewKeys;
  // this CTA's list of tiles: those with kept first positions ahead of what the rows see, then the others; cut into splits
  const int keep_tiles = min(tile_first, (keep_first + kFewKeys - 1) / kFewKeys);
  const int list_n = keep_tiles + n_tiles - tile_first;
  const int per = (list_n + splits - 1) / splits;
  const int tile_lo = split * per, tile_hi = min(list_n, tile_lo + per);
  auto tile_of = [&](int li) { return li < keep_tiles ? li : tile_first + (li - keep_tiles); };

  extern __shared__ __align__(16) unsigned char few_sm[];
  const FewLayout L = few_layout(a, SAME, QF32);
  const int ldk = L.ldk, ldv = L.ldv;
  __nv_bfloat16* q_hi = reinterpret_cast<__nv_bfloat16*>(few_sm + L.q_hi);
  __nv_bfloat16* q_lo = reinterpret_cast<__nv_bfloat16*>(few_sm + L.q_lo);
  float* Ss = reinterpret_cast<float*>(few_sm + L.s);                          // [rows][keys + 1]
  __nv_bfloat16* p_hi = reinterpret_cast<__nv_bfloat16*>(few_sm + L.p_hi);     // [rows][keys + 8]
  __nv_bfloat16* p_lo = reinterpret_cast<__nv_bfloat16*>(few_sm + L.p_lo);
  float* m_s = reinterpret_cast<float*>(few_sm + L.stats);
  float* l_s = m_s + kFewRows;
  float* al_s = l_s + kFewRows;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t base = static_cast<uint32_t>(__cvta_generic_to_shared(few_sm));
  const uint32_t k_addr = base + static_cast<uint32_t>(L.k), v_addr = base + static_cast<uint32_t>(L.v);

  const __nv_bfloat16* kbase = static_cast<const __nv_bfloat16*>(kv.k) + static_cast<size_t>(g) * dim;
  const __nv_bfloat16* vbase = static_cast<const __nv_bfloat16*>(kv.v) + static_cast<size_t>(gv) * vdim;
  const int kc = L.dimp / 8, vc = SAME ? 0 : (ldv - 8) / 8;
  auto load_tile = [&](int tile, int stage) {  // four threads per key: one page lookup per thread
    const int j = tid >> 2, kj = tile * kFewKeys + j;
    const bool valid = kj <= pmax;
    const size_t slot = valid ? static_cast<size_t>(table[kj / kv.page]) * kv.page + kj % kv.page : 0;
    const __nv_bfloat16 *kr = kbase + slot * kv.k_row, *vr = vbase + slot * kv.v_row;
    const uint32_t kd = k_addr + ((stage * kFewKeys + j) * ldk) * 2, vd = v_addr + ((stage * kFewKeys + j) * ldv) * 2;
    for (int c = tid & 3; c < kc; c += 4) {
      const bool in = valid && c * 8 < dim;
      cp_async16(kd + c * 16, in ? kr + c * 8 : kbase, in);
    }
    for (int c = tid & 3; c < vc; c += 4) {
      const bool in = valid && c * 8 < vdim;
      cp_async16(vd + c * 16, in ? vr + c * 8 : vbase, in);
    }
    cp_async_commit();
  };
  if (tile_lo < tile_hi) load_tile(tile_of(tile_lo), 0);

  // the queries, two neighbouring coordinates at a time (dim is even); rows and coordinates that do not exist are zero
  const int half = L.dimp / 2;
  for (int i = tid; i < kFewRows * half; i += kFewThreads) {
    const int r = i / half, d = (i % half) * 2;
    float x = 0.f, y = 0.f;
    if (r < rows_here && d < dim) {
      const int rr = r0 + r;
      const size_t qi = (static_cast<size_t>(first + rr / rep) * a.heads + g * rep + rr % rep) * dim + d;
      if (QF32) {
        const float2 v = *reinterpret_cast<const float2*>(static_cast<const float*>(q_) + qi);
        x = v.x, y = v.y;
      } else {
        const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(static_cast<const __nv_bfloat16*>(q_) + qi);
        x = __low2float(v), y = __high2float(v);
      }
    }
    uint32_t hi, lo;
    split_pack(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(q_hi + r * ldk + d) = hi;
    if (QF32) *reinterpret_cast<uint32_t*>(q_lo + r * ldk + d) = lo;
  }
  if (tid < kFewRows) m_s[tid] = -INFINITY, l_s[tid] = 0.f;
  float o[NBW][4];
#pragma unroll
  for (int i = 0; i < NBW; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int nb_all = (vdim + 7) / 8;
  const int gq = lane >> 2, t4 = lane & 3;
  // positions of this lane's two rows, and the first key each of them sees
  int row_pos[2], row_lo[2];
#pragma unroll
  for (int z = 0; z < 2; ++z) row_pos[z] = pos0 + (r0 + gq + z * 8) / rep, row_lo[z] = first_seen(a, row_pos[z]);
  // addresses of this lane's rows in the A fragments (16 x 16 tiles: rows lane % 16, columns + 8 for the upper lanes)
  const uint32_t qh_addr = base + static_cast<uint32_t>(L.q_hi) + ((lane & 15) * ldk + (lane >> 4) * 8) * 2;
  const uint32_t ql_addr = base + static_cast<uint32_t>(L.q_lo) + ((lane & 15) * ldk + (lane >> 4) * 8) * 2;
  const uint32_t ph_addr = base + static_cast<uint32_t>(L.p_hi) + ((lane & 15) * (kFewKeys + 8) + (lane >> 4) * 8) * 2;
  const uint32_t pl_addr = base + static_cast<uint32_t>(L.p_lo) + ((lane & 15) * (kFewKeys + 8) + (lane >> 4) * 8) * 2;

  for (int li = tile_lo; li < tile_hi; ++li) {
    const int tile = tile_of(li), stage = (li - tile_lo) & 1, k0 = tile * kFewKeys;
    if (li + 1 < tile_hi) {
      load_tile(tile_of(li + 1), stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    {  // scores of 8 keys: one ldmatrix.x2 brings the key fragments of a k-step (key row lane % 8, coordinates + 8 for lanes 8..15)
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t kt = k_addr + ((stage * kFewKeys + warp * 8 + (lane & 7)) * ldk + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
      for (int ks = 0; ks < L.dimp / 16; ++ks) {
        uint32_t b0, b1, af[4];
        asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(b0), "=r"(b1) : "r"(kt + ks * 32));
        ldmatrix_x4(qh_addr + ks * 32, af[0], af[1], af[2], af[3]);
        mma_bf16(s0, af, b0, b1);
        if (QF32) {
          ldmatrix_x4(ql_addr + ks * 32, af[0], af[1], af[2], af[3]);
          mma_bf16(s1, af, b0, b1);
        }
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int r = gq + (c >> 1) * 8, j = warp * 8 + t4 * 2 + (c & 1), kj = k0 + j;
        float sv = (s0[c] + s1[c]) * a.scale;
        if (a.softcap > 0.f) sv = a.softcap * tanhf(sv / a.softcap);
        const bool visible = r < rows_here && kj <= row_pos[c >> 1] && (kj >= row_lo[c >> 1] || kj < keep_first);
        Ss[r * (kFewKeys + 1) + j] = visible ? sv : -INFINITY;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kFewRows / kFewWarps; ++i) {
      const int r = warp * (kFewRows / kFewWarps) + i;
      const float sv = Ss[r * (kFewKeys + 1) + lane];
      float mx = sv;
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = m_s[r], m_new = fmaxf(m_old, mx);
      float p = 0.f, alpha = 1.0f;
      if (m_new > -INFINITY) p = expf(sv - m_new), alpha = expf(m_old - m_new);
      float sum = p;
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      const __nv_bfloat16 h = __float2bfloat16_rn(p);
      p_hi[r * (kFewKeys + 8) + lane] = h;
      p_lo[r * (kFewKeys + 8) + lane] = __float2bfloat16_rn(p - __bfloat162float(h));
      __syncwarp();  // every lane has read m_s[r]
      if (lane == 0) m_s[r] = m_new, l_s[r] = l_s[r] * alpha + sum, al_s[r] = alpha;
    }
    __syncthreads();
    {
      const float aA = al_s[gq], aB = al_s[gq + 8];
#pragma unroll
      for (int i = 0; i < NBW; ++i) o[i][0] *= aA, o[i][1] *= aA, o[i][2] *= aB, o[i][3] *= aB;
#pragma unroll
      for (int kk = 0; kk < kFewKeys / 16; ++kk) {
        uint32_t ph[4], pl[4];
        ldmatrix_x4(ph_addr + kk * 32, ph[0], ph[1], ph[2], ph[3]);
        ldmatrix_x4(pl_addr + kk * 32, pl[0], pl[1], pl[2], pl[3]);
        const uint32_t vt = v_addr + ((stage * kFewKeys + kk * 16 + (lane & 15)) * ldv) * 2;
#pragma unroll
        for (int i = 0; i < NBW; ++i) {
          const int nb = warp + i * kFewWarps;
          if (nb < nb_all) {  // the same for the whole warp
            uint32_t b0, b1;
            asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(b0), "=r"(b1) : "r"(vt + nb * 16));
            mma_bf16(o[i], ph, b0, b1);
            mma_bf16(o[i], pl, b0, b1);
          }
        }
      }
    }
    __syncthreads();  // the stage is loaded again, the scores are written again
  }
  if (tile_lo >= tile_hi) __syncthreads();  // an empty split still writes its (empty) statistics
  const int pstride = vdim + 2;
#pragma unroll
  for (int z = 0; z < 2; ++z) {
    const int r = gq + z * 8;
    if (r >= rows_here) continue;
    const int rr = r0 + r;
    float* p = ws + ((static_cast<size_t>(first + rr / rep) * a.heads + g * rep + rr % rep) * splits + split) * pstride;
    if (warp == 0 && t4 == 0) p[0] = m_s[r], p[1] = l_s[r];
#pragma unroll
    for (int i = 0; i < NBW; ++i) {
      const int col = (warp + i * kFewWarps) * 8 + t4 * 2;
      if (col < vdim) *reinterpret_cast<float2*>(p + 2 + col) = make_float2(o[i][z * 2], o[i][z * 2 + 1]);
    }
  }
}

template <int NBW, bool SAME, bool QF32>
int launch_few(const AttnShape& a, const void* q, const PagedKV& kv, int n_entries, const int32_t* ent_first,
               const int32_t* ent_count, const int32_t* ent_seq, const int32_t* ent_pos0, int max_count, int splits, float* ws,
               cudaStream_t s) {
  const size_t smem = few_layout(a, SAME, QF32).total;
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    const cudaError_t e = cudaFuncSetAttribute(attention_rows_mma_kernel<NBW, SAME, QF32>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return cuda_rc(e);
    configured = smem;
  }
  const dim3 grid((max_count * (a.heads / a.kv_heads) + kFewRows - 1) / kFewRows, n_entries * a.kv_heads, splits);
  if (grid.y > 65535u) return KLLM_E_UNSUPPORTED;
  attention_rows_mma_kernel<NBW, SAME, QF32><<<grid, kFewThreads, smem, s>>>(a, q, kv, ent_first, ent_count, ent_seq, ent_pos0,
                                                                            splits, ws);
  count_launch();
  return cuda_rc(cudaGetLastError());
}

inline bool values_in_keys(const AttnShape& a, const PagedKV& kv) {
  return kv.v == kv.k && kv.v_row == kv.k_row && a.kv_heads == 1 && a.vdim <= a.dim;
}

}  // namespace

bool attention_rows_mma_usable(int dtype, const AttnShape& a, const PagedKV& kv, int n_entries) {
  static const bool off = [] { const char* e = getenv("KLLM_SEQ_ROWS_MMA"); return e != nullptr && e[0] == '0'; }();
  if (off || dtype != KLLM_SEQ_BF16 || a.kv_heads <= 0 || a.heads % a.kv_heads || kv.table == nullptr) return false;
  // 16-byte chunks of every key and value row
  if (a.dim % 8 || a.vdim % 8 || kv.k_row % 8 || kv.v_row % 8 || a.vdim > 512) return false;
  if (static_cast<long long>(n_entries) * a.kv_heads > 65535) return false;
  return few_layout(a, values_in_keys(a, kv), a.q_f32 != 0).total <= 200 * 1024;
}

int launch_attention_rows_mma(const AttnShape& a, const void* q, const PagedKV& kv, int n_entries, const int32_t* ent_first,
                              const int32_t* ent_count, const int32_t* ent_seq, const int32_t* ent_pos0, int max_count,
                              int splits, float* ws, cudaStream_t s) {
  const bool same = values_in_keys(a, kv);
#define KLLM_FEW(N)                                                                                                              \
  if (a.vdim <= N * kFewWarps * 8) {                                                                                              \
    if (same)                                                                                                                     \
      return a.q_f32 ? launch_few<N, true, true>(a, q, kv, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, splits, ws, s)   \
                     : launch_few<N, true, false>(a, q, kv, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, splits, ws, s); \
    return a.q_f32 ? launch_few<N, false, true>(a, q, kv, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, splits, ws, s)    \
                   : launch_few<N, false, false>(a, q, kv, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, splits, ws, s);  \
  }
  KLLM_FEW(2)
  KLLM_FEW(4)
  KLLM_FEW(8)
  KLLM_FEW(16)
#undef KLLM_FEW
  return KLLM_E_UNSUPPORTED;
}

bool attention_mma_usable(int dtype, const AttnShape& a, int max_count) {
  if (dtype != KLLM_SEQ_BF16 || a.kv_heads <= 0 || a.heads % a.kv_heads) return false;
  // fp32 queries / outputs are the split-key kernel's
  if (a.q_f32 || a.out_f32) return false;
  const bool dims = a.dim % 8 == 0 && a.dim <= 256 && a.vdim % 8 == 0 && a.vdim <= 128;
  // steps of single tokens keep the split-key kernel (and stay capturable: no attribute call on their path)
  return dims && max_count >= 2 && max_count * (a.heads / a.kv_heads) >= 16;
}

int launch_attention_mma(const AttnShape& a, const void* q, const float* gates, const PagedKV& kv, int n_entries,
                         const int32_t* ent_first, const int32_t* ent_count, const int32_t* ent_seq,
                         const int32_t* ent_pos0, int max_count, int splits, float* ws, void* out, cudaStream_t s) {
#define KLLM_MMA(D, V)                                                                                             \
  if (a.dim <= D && a.vdim <= V)                                                                                   \
    return launch_mma<D, V>(a, q, gates, kv, n_entries, ent_first, ent_count, ent_seq, ent_pos0, max_count, splits, ws, \
                            out, s)
  KLLM_MMA(64, 64);
  KLLM_MMA(64, 128);
  KLLM_MMA(128, 64);
  KLLM_MMA(128, 128);
  KLLM_MMA(256, 128);
#undef KLLM_MMA
  return KLLM_E_UNSUPPORTED;
}

}  // namespace seq
}  // namespace kllm
