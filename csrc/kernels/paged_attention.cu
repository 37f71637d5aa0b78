// Paged KV cache: append and single-token (decode) attention through a block table (page size 16 by default).
//
// Decode attention is bandwidth-bound (every cached key and value is read once per step), so the kernel is built
// around memory access and parallelism: one CTA per (sequence, KV head, 256-token slice of the context) serves all
// query heads of that group (split-KV, so a batch of 32 sequences still fills 148 SMs); K and V rows are fetched
// coalesced into a padded shared tile, the group's heads are the rows of mma.sync tensor-core tiles for both
// Q K^T and P V, and a second kernel merges the slices' (max, sum, output) triples.
//
// The reference's PagedCache is block-table bookkeeping without tensor storage and its KVCache::append drops
// the new entries (crates/nn/src/kv_cache.rs:172-216,382-432); this is the storage and the kernel they lack.
#include "paged_attention.h"

#include <float.h>

#include "rb_common.cuh"

namespace rb {

__global__ void __launch_bounds__(128)
kv_append_kernel(const __nv_bfloat16* __restrict__ k_new, long long ld_k, const __nv_bfloat16* __restrict__ v_new,
                 long long ld_v, __nv_bfloat16* __restrict__ k_cache, __nv_bfloat16* __restrict__ v_cache,
                 const long long* __restrict__ slots, long long tokens, int row_elems, long long num_slots RB_BOUNDS_PARAM) {
  const int chunks = row_elems / 8;
  const long long total = tokens * chunks;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
    const long long t = i / chunks;
    const int c = static_cast<int>(i - t * chunks) * 8;
    const long long slot = slots[t];
    if (slot >= num_slots && c == 0) RB_BOUNDS_HIT(103);           // a negative slot means "skip this token"
    if (slot < 0 || slot >= num_slots) continue;
    *reinterpret_cast<uint4*>(k_cache + slot * row_elems + c) = *reinterpret_cast<const uint4*>(k_new + t * ld_k + c);
    *reinterpret_cast<uint4*>(v_cache + slot * row_elems + c) = *reinterpret_cast<const uint4*>(v_new + t * ld_v + c);
  }
}

constexpr int kMaxGroup = 16;    // query heads per KV head served by one CTA pass (the M of the mma tile)
constexpr int kPaWarps = 4;
constexpr int kSplitTokens = 256;          // cached tokens per CTA (split-KV): 2 passes of 32 tokens per warp

__device__ __forceinline__ void pa_ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void pa_ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void pa_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16-byte asynchronous global -> shared copy; bytes == 0 writes zeros and reads nothing
__device__ __forceinline__ void pa_cp_async16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void pa_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void pa_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ uint32_t pa_pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

template <int N>
struct PaInt { static constexpr int value = N; };
__device__ __forceinline__ float pa_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

// Split-KV decode attention.  One CTA = (sequence, KV head, 256-token slice of the context); the slices of a sequence
// run on different SMs and a second kernel merges their (max, sum, accumulator) triples.  Inside a CTA a warp takes
// 32 tokens at a time.  Their K rows and V rows are fetched with fully coalesced 16-byte asynchronous copies (cp.async,
// 16 lanes per 256-byte row) into two padded shared tiles per warp; the K tile of the next pass is requested as soon
// as the scores of this pass are computed and the V tile as soon as P V is done, so every warp always has a tile in
// flight while it computes.  The query heads of the group
// form the 16 rows of an m16n8k16 tensor-core tile (rows beyond the group are zero): S = Q K^T is 4 n-tiles x D/16
// k-steps of mma.sync, the softmax runs on the accumulator fragments, and O += P V reuses those fragments as the A
// operand against ldmatrix.trans-fed V.  One query token per sequence gives M <= 16, far below the 64-row minimum
// of a tcgen05 tile, which is why this kernel is on the warp-level tensor path; it is bound by the K / V reads.
//
// DK / DV are the key / value head sizes rounded up to a compiled size; columns beyond the real sizes are zero-filled in
// shared memory and never leave it.  RULE adds a score cap, a linear and a logarithmic distance bias, chunked or windowed visibility, a
// sink and output gates (see RbPagedRowsArgs).  A window's slices cover the kept first tokens and then the window.
struct PaRule {
  float softcap;
  const float* slopes;
  int chunk;
  const __nv_bfloat16* gate;
  const float* head_gate;
  long long ld_g;
  int window, keep, sink;
  const float* log_amount;
  const float* log_rate;
  float out_scale;
};
// cap * tanh(s / cap) as cap * (1 - 2 / (1 + e^(2 s / cap))): two special-function instructions, absolute error about
// 1e-7 * cap (tanh.approx would be off by 5e-4 of the score)
__device__ __forceinline__ float pa_softcap(float s, float cap, float two_over_cap) {
  return fmaf(-2.f * cap, __fdividef(1.f, 1.f + __expf(s * two_over_cap)), cap);
}
// The visible tokens of a sequence, numbered without gaps: number v is token v below `kept`, else token v + gap.
struct PaVisible {
  int kept, gap, count;
};
__device__ __forceinline__ PaVisible pa_visible(int ctx, const PaRule& r) {
  if (r.window > 0) {
    const int kept = min(r.keep, ctx), lo = max(kept, ctx - r.window);
    return {kept, lo - kept, ctx - (lo - kept)};
  }
  const int lo = r.chunk > 0 ? (ctx - 1) / r.chunk * r.chunk : 0;
  return {0, lo, ctx - lo};
}
__device__ __forceinline__ float pa_gate(const PaRule& r, long long row, int head, long long col) {
  if (r.gate) return pa_sigmoid(__bfloat162float(r.gate[row * r.ld_g + col]));
  return r.head_gate ? pa_sigmoid(r.head_gate[row * r.ld_g + head]) : 1.f;
}

template <int DK, int DV, bool RULE>
__global__ void __launch_bounds__(kPaWarps * 32, 3)
paged_decode_split_kernel(const __nv_bfloat16* __restrict__ q, long long ld_q, const __nv_bfloat16* __restrict__ k_cache,
                          const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ block_tables, int max_blocks,
                          const int* __restrict__ context_lens, int heads, int kv_heads, int dk_real, int dv_real,
                          int block_size, long long num_blocks, float scale, int g0, int gcount, float* __restrict__ partial,
                          int nsplit, __nv_bfloat16* __restrict__ direct_out, long long ld_o, const PaRule rule
                          RB_BOUNDS_PARAM) {
  constexpr int LPK = DK / 8, LPV = DV / 8;  // 16-byte pieces per K / V row = copies per lane for a 32-row tile
  constexpr int KROW = DK + 8, VROW = DV + 8;  // padded rows (elements): ldmatrix rows 272 (144) bytes apart hit distinct banks
  constexpr int NT = DV / 8;                 // n-tiles of the output accumulator
  constexpr int kKTile = 32 * KROW, kVTile = 32 * VROW;   // one tile of one warp
  const int dk = RULE ? dk_real : DK, dv = RULE ? dv_real : DV;
  extern __shared__ __align__(16) uint8_t big[];   // [warp][K tile, V tile] bf16, then q_sh; later the warp merge area
  __nv_bfloat16* q_sh = reinterpret_cast<__nv_bfloat16*>(big) + kPaWarps * (kKTile + kVTile);
  __shared__ float m_sh[kPaWarps][kMaxGroup], l_sh[kPaWarps][kMaxGroup];
  const int b = blockIdx.x, hk = blockIdx.y, sp = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gq = lane >> 2, tq = lane & 3;   // fragment coordinates: row (and row + 8), column pair
  const int group = heads / kv_heads;
  const int ctx = context_lens[b];
  const PaVisible vis = RULE ? pa_visible(ctx, rule) : PaVisible{0, 0, ctx};
  const int t_begin = sp * kSplitTokens;
  if (t_begin >= vis.count) return;
  const int t_end = min(vis.count, t_begin + kSplitTokens);
  const int h_base = hk * group + g0;        // first query head of this pass
  const uint32_t kt_u32 = smem_u32(reinterpret_cast<__nv_bfloat16*>(big) + warp * (kKTile + kVTile));
  const uint32_t vt_u32 = kt_u32 + kKTile * 2;
  const uint32_t q_u32 = smem_u32(q_sh);
  float slope0 = 0.f, slope1 = 0.f, two_over_cap = 0.f;
  float amount0 = 0.f, amount1 = 0.f, rate0 = 0.f, rate1 = 0.f;
  if (RULE) {
    if (rule.log_rate) {
      if (gq < gcount) { amount0 = rule.log_amount[h_base + gq]; rate0 = rule.log_rate[h_base + gq]; }
      if (gq + 8 < gcount) { amount1 = rule.log_amount[h_base + gq + 8]; rate1 = rule.log_rate[h_base + gq + 8]; }
    }
    if (rule.slopes) {
      if (gq < gcount) slope0 = rule.slopes[h_base + gq];
      if (gq + 8 < gcount) slope1 = rule.slopes[h_base + gq + 8];
    }
    if (rule.softcap > 0.f) two_over_cap = 2.f / rule.softcap;
  }

  // the group's query rows as bf16 [16][D] (rows >= gcount are zero)
  for (int i = threadIdx.x; i < kMaxGroup * LPK; i += blockDim.x) {
    const int g = i / LPK, c = (i - g * LPK) * 8;
    uint4 u = make_uint4(0u, 0u, 0u, 0u);
    if (g < gcount && c < dk) {
      const __nv_bfloat16* src = q + static_cast<long long>(b) * ld_q + static_cast<long long>(h_base + g) * dk + c;
      uint32_t w[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) w[j] = *reinterpret_cast<const uint32_t*>(src + 2 * j);   // rows are 4-byte aligned at least
      u = make_uint4(w[0], w[1], w[2], w[3]);
    }
    *reinterpret_cast<uint4*>(q_sh + g * KROW + c) = u;
  }
  __syncthreads();

  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;      // rows gq and gq + 8
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;

  int slot = -1;                             // cache slot of token `first + lane` of the located tile (-1: past the end)
  int n_next = 0;
  // cache slots of the 32 tokens that start at `first` (the host bounds num_blocks * block_size below 2^31)
  auto locate = [&](int first) {
    const int num = first + lane;
    slot = -1;
    if (num < t_end) {
      const int tok = RULE && num >= vis.kept ? num + vis.gap : num;
      const int blk_idx = tok / block_size;
      int blk = blk_idx < max_blocks ? block_tables[static_cast<long long>(b) * max_blocks + blk_idx] : -1;
      if (blk < 0 || blk >= num_blocks) {                            // corrupt tables read block 0 instead of faulting
        RB_BOUNDS_HIT(104);
        blk = 0;
      }
      slot = blk * block_size + (tok - blk_idx * block_size);
    }
    n_next = min(32, t_end - first);
  };
  // one tile = one asynchronous 16-byte copy per lane and piece, one commit group; rows past the context and columns past
  // the real head size are zero-filled
  auto request = [&](const __nv_bfloat16* cache, uint32_t tile_u32, auto pieces, int dim) {
    constexpr int LP = decltype(pieces)::value;
#pragma unroll
    for (int i = 0; i < LP; ++i) {
      const int idx = i * 32 + lane;
      const int r = idx / LP, c = (idx - r * LP) * 8;
      const int s_r = __shfl_sync(0xffffffffu, slot, r);
      const bool ok = s_r >= 0 && c < dim;
      pa_cp_async16(tile_u32 + (r * (LP * 8 + 8) + c) * 2,
                    ok ? cache + (static_cast<long long>(s_r) * kv_heads + hk) * dim + c : cache, ok ? 16 : 0);
    }
    pa_cp_commit();
  };
  const PaInt<LPK> pk{};
  const PaInt<LPV> pv{};
  int base = t_begin + warp * 32;
  if (base < t_end) {
    locate(base);
    request(k_cache, kt_u32, pk, dk);
    request(v_cache, vt_u32, pv, dv);
  }
  for (; base < t_end; base += kPaWarps * 32) {
    const int n_tok = n_next;
    const bool more = base + kPaWarps * 32 < t_end;
    pa_cp_wait<1>();                                                 // this pass's K tile has landed (V may be in flight)
    __syncwarp();
    // ---- S[16 heads, 32 tokens] = Q K^T
    float s[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
    for (int k0 = 0; k0 < DK; k0 += 16) {
      uint32_t a[4];
      // A fragment: matrices (rows 0-7, k0), (rows 8-15, k0), (rows 0-7, k0 + 8), (rows 8-15, k0 + 8)
      pa_ldsm_x4(q_u32 + ((lane & 15) * KROW + k0 + (lane >> 4) * 8) * 2, a);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t bfr[4];
        // B fragments of two n-tiles: (tokens 16np..+7, k0), (same tokens, k0 + 8), (tokens 16np + 8.., k0), (.., k0 + 8)
        pa_ldsm_x4(kt_u32 + ((np * 16 + (lane & 7) + ((lane >> 4) << 3)) * KROW + k0 + ((lane >> 3) & 1) * 8) * 2, bfr);
        pa_mma(s[2 * np], a, bfr[0], bfr[1]);
        pa_mma(s[2 * np + 1], a, bfr[2], bfr[3]);
      }
    }
    __syncwarp();                                                    // every lane has read its K fragments
    if (more) {                                                      // the next pass's K tile flies under softmax and P V
      locate(base + kPaWarps * 32);
      request(k_cache, kt_u32, pk, dk);
    }
    // ---- online softmax over the 32 tokens; this thread holds 8 of them for rows gq and gq + 8
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const bool ok = n * 8 + 2 * tq + j < n_tok;
        float v0 = s[n][j] * scale, v1 = s[n][2 + j] * scale;
        if (RULE) {
          if (rule.softcap > 0.f) {
            v0 = pa_softcap(v0, rule.softcap, two_over_cap);
            v1 = pa_softcap(v1, rule.softcap, two_over_cap);
          }
          const int num = base + n * 8 + 2 * tq + j;
          const float dist = static_cast<float>(ctx - 1 - (num < vis.kept ? num : num + vis.gap));
          v0 = fmaf(-slope0, dist, v0);
          v1 = fmaf(-slope1, dist, v1);
          if (rule.log_rate) {                       // distances behind the last token are masked below
            v0 = fmaf(-amount0, __logf(fmaf(rate0, fmaxf(dist, 0.f), 1.f)), v0);
            v1 = fmaf(-amount1, __logf(fmaf(rate1, fmaxf(dist, 0.f), 1.f)), v1);
          }
        }
        s[n][j] = ok ? v0 : -INFINITY;
        s[n][2 + j] = ok ? v1 : -INFINITY;
        mx0 = fmaxf(mx0, s[n][j]);
        mx1 = fmaxf(mx1, s[n][2 + j]);
      }
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);          // finite: token 0 of the pass is always valid
    const float al0 = (m0 == -INFINITY) ? 0.f : __expf(m0 - mn0);
    const float al1 = (m1 == -INFINITY) ? 0.f : __expf(m1 - mn1);
    float sum0 = 0.f, sum1 = 0.f;
    uint32_t pfr[2][4];                                              // P as the A operand of the two 16-token k-steps
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const float p0 = __expf(s[n][0] - mn0), p1 = __expf(s[n][1] - mn0);
      const float p2 = __expf(s[n][2] - mn1), p3 = __expf(s[n][3] - mn1);
      sum0 += p0 + p1;
      sum1 += p2 + p3;
      pfr[n >> 1][(n & 1) * 2 + 0] = pa_pack_bf16(p0, p1);          // rows gq
      pfr[n >> 1][(n & 1) * 2 + 1] = pa_pack_bf16(p2, p3);          // rows gq + 8
    }
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
    l0 = l0 * al0 + sum0;
    l1 = l1 * al1 + sum1;
    m0 = mn0;
    m1 = mn1;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      acc[n][0] *= al0; acc[n][1] *= al0; acc[n][2] *= al1; acc[n][3] *= al1;
    }
    // ---- O[16, DV] += P[16, 32] V[32, DV]
    if (more) pa_cp_wait<1>(); else pa_cp_wait<0>();                 // this pass's V tile has landed
    __syncwarp();
#pragma unroll
    for (int ks = 0; ks < 2; ++ks) {
#pragma unroll
      for (int n2 = 0; n2 < NT / 2; ++n2) {
        uint32_t bfr[4];
        // transposed 8x8 blocks: (tokens 16ks..+7, dims 16n2), (tokens +8, same dims), (tokens.., dims + 8), (+8, + 8)
        pa_ldsm_x4_t(vt_u32 + ((ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VROW + n2 * 16 + (lane >> 4) * 8) * 2, bfr);
        pa_mma(acc[2 * n2], pfr[ks], bfr[0], bfr[1]);
        pa_mma(acc[2 * n2 + 1], pfr[ks], bfr[2], bfr[3]);
      }
    }
    __syncwarp();                                                    // every lane has read its V fragments
    if (more) request(v_cache, vt_u32, pv, dv);
  }

  // ---- merge the warps, write this slice's (max, sum, accumulator) per head
  __syncthreads();                            // every warp is done with its tile: the buffer becomes the merge area
  float (*acc_sh)[kMaxGroup][DV] = reinterpret_cast<float (*)[kMaxGroup][DV]>(big);
  if (tq == 0) {
    m_sh[warp][gq] = m0; l_sh[warp][gq] = l0;
    m_sh[warp][gq + 8] = m1; l_sh[warp][gq + 8] = l1;
  }
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    *reinterpret_cast<float2*>(&acc_sh[warp][gq][n * 8 + 2 * tq]) = make_float2(acc[n][0], acc[n][1]);
    *reinterpret_cast<float2*>(&acc_sh[warp][gq + 8][n * 8 + 2 * tq]) = make_float2(acc[n][2], acc[n][3]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < gcount * dv; i += blockDim.x) {
    const int g = i / dv, d = i - g * dv;
    float mx = -INFINITY;
#pragma unroll
    for (int w = 0; w < kPaWarps; ++w) mx = fmaxf(mx, m_sh[w][g]);
    float num = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < kPaWarps; ++w) {
      const float sc = (m_sh[w][g] == -INFINITY) ? 0.f : __expf(m_sh[w][g] - mx);
      num += acc_sh[w][g][d] * sc;
      den += l_sh[w][g] * sc;
    }
    if (direct_out) {                        // a single slice: this is the result
      const long long col = static_cast<long long>(h_base + g) * dv + d;
      if (RULE && rule.sink) {               // a score 0 without a value
        const float top = fmaxf(mx, 0.f), sc = __expf(mx - top);
        num *= sc;
        den = fmaf(den, sc, __expf(-top));
      }
      float o = num / den;
      if (RULE) o *= pa_gate(rule, b, h_base + g, col) * rule.out_scale;
      direct_out[b * ld_o + col] = __float2bfloat16(o);
      continue;
    }
    float* pp = partial + ((static_cast<long long>(b) * heads + h_base + g) * nsplit + sp) * (dv + 2);
    pp[2 + d] = num;
    if (d == 0) { pp[0] = mx; pp[1] = den; }
  }
}

// out[b, h, :] = merge over the slices that hold tokens of sequence b (times sigmoid(gate)); one thread per value column
__global__ void __launch_bounds__(128)
paged_decode_merge_kernel(const float* __restrict__ partial, const int* __restrict__ context_lens, int heads, int dv,
                          int nsplit, __nv_bfloat16* __restrict__ out, long long ld_o, const PaRule rule) {
  const int b = blockIdx.x, h = blockIdx.y, d = threadIdx.x;
  if (d >= dv) return;
  const int ctx = context_lens[b];
  const int n = min(nsplit, (pa_visible(ctx, rule).count + kSplitTokens - 1) / kSplitTokens);
  const float* base = partial + (static_cast<long long>(b) * heads + h) * nsplit * (dv + 2);
  float mx = -INFINITY;
  for (int s = 0; s < n; ++s) mx = fmaxf(mx, base[s * (dv + 2)]);
  if (rule.sink) mx = fmaxf(mx, 0.f);
  float num = 0.f, den = rule.sink ? __expf(-mx) : 0.f;      // a sink is a score 0 without a value
  for (int s = 0; s < n; ++s) {
    const float ms = base[s * (dv + 2)];
    const float sc = (ms == -INFINITY) ? 0.f : __expf(ms - mx);
    num += base[s * (dv + 2) + 2 + d] * sc;
    den += base[s * (dv + 2) + 1] * sc;
  }
  const long long col = static_cast<long long>(h) * dv + d;
  float o = den > 0.f ? num / den : 0.f;
  o *= pa_gate(rule, b, h, col) * rule.out_scale;
  out[static_cast<long long>(b) * ld_o + col] = __float2bfloat16(o);
}

// ---- any rows, any head sizes, bf16 or fp32 ------------------------------------------------------------------------
__device__ __forceinline__ float pr_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float pr_get(const float* p) { return *p; }
__device__ __forceinline__ void pr_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void pr_put(float* p, float v) { *p = v; }

constexpr int kPrMaxV = 16;                // value columns per lane; heads with more than 512 take several CTAs

// One warp per (row, query head): lanes are keys for the scores, value columns for the weighted sum.
template <typename T>
__global__ void __launch_bounds__(128)
paged_rows_kernel(const RbPagedRowsArgs a RB_BOUNDS_PARAM) {
  extern __shared__ float pr_q[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long item = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + warp;
  if (item >= static_cast<long long>(a.rows) * a.heads) return;
  const int r = static_cast<int>(item / a.heads), h = static_cast<int>(item - static_cast<long long>(r) * a.heads);
  const int hk = h / (a.heads / a.kv_heads);
  float* q = pr_q + warp * a.dk;
  const T* qg = reinterpret_cast<const T*>(a.q) + r * a.ld_q + static_cast<long long>(h) * a.dk;
  for (int c = lane; c < a.dk; c += 32) q[c] = pr_get(qg + c);
  __syncwarp();
  const long long ld_kc = a.ld_kc ? a.ld_kc : static_cast<long long>(a.kv_heads) * a.dk;
  const long long ld_vc = a.ld_vc ? a.ld_vc : static_cast<long long>(a.kv_heads) * a.dv;
  const int v0 = blockIdx.y * 32 * kPrMaxV;                            // first value column of this CTA
  const long long pos = a.row_pos[r];
  const int* table = a.block_tables + static_cast<long long>(a.row_seq[r]) * a.max_blocks;
  // visible keys are numbered without gaps: number v is key v below `kept`, else key v + gap
  const long long kept = a.window > 0 ? (a.keep_first < pos + 1 ? a.keep_first : pos + 1) : 0;
  long long gap = a.chunk > 0 ? pos / a.chunk * a.chunk : a.window > 0 ? pos + 1 - a.window - kept : 0;
  if (gap < 0) gap = 0;
  const long long count = pos + 1 - gap;
  const float slope = a.slopes ? a.slopes[h] : 0.f;
  const float amount = a.log_rate ? a.log_amount[h] : 0.f, log_rate = a.log_rate ? a.log_rate[h] : 0.f;
  const T* K = reinterpret_cast<const T*>(a.k_cache);
  const T* V = reinterpret_cast<const T*>(a.v_cache);
  float acc[kPrMaxV];
#pragma unroll
  for (int i = 0; i < kPrMaxV; ++i) acc[i] = 0.f;
  float m = a.sink ? 0.f : -INFINITY, l = a.sink ? 1.f : 0.f;        // a sink is a score 0 met before all keys
  for (long long j0 = 0; j0 < count; j0 += 32) {
    const long long num = j0 + lane;
    const long long j = num < kept ? num : num + gap;
    long long slot = 0;
    float s = -INFINITY;
    if (num < count) {
      const long long bi = j / a.block_size;
      int blk = bi < a.max_blocks ? table[bi] : -1;
      if (blk < 0 || blk >= a.num_blocks) {                          // corrupt tables read block 0 instead of faulting
        RB_BOUNDS_HIT(104);
        blk = 0;
      }
      slot = static_cast<long long>(blk) * a.block_size + (j - bi * a.block_size);
      const T* k = K + slot * ld_kc + static_cast<long long>(hk) * a.dk;
      float d = 0.f;
      for (int c = 0; c < a.dk; ++c) d = fmaf(q[c], pr_get(k + c), d);
      s = d * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      s -= slope * static_cast<float>(pos - j);
      if (a.log_rate) s -= amount * log1pf(log_rate * static_cast<float>(pos - j));
    }
    const float mn = fmaxf(m, warp_max(s));                          // finite: key j0 is always visible
    const float al = m == -INFINITY ? 0.f : expf(m - mn);
    const float p = num < count ? expf(s - mn) : 0.f;
    l = l * al + warp_sum(p);
    m = mn;
#pragma unroll
    for (int i = 0; i < kPrMaxV; ++i) acc[i] *= al;
    const int n = static_cast<int>(count - j0 < 32 ? count - j0 : 32);
    for (int jj = 0; jj < n; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const long long sj = __shfl_sync(0xffffffffu, slot, jj);
      const T* vals = V + sj * ld_vc + static_cast<long long>(hk) * a.dv + v0;
#pragma unroll
      for (int i = 0; i < kPrMaxV; ++i) {
        const int c = i * 32 + lane;
        if (v0 + c < a.dv) acc[i] = fmaf(pj, pr_get(vals + c), acc[i]);
      }
    }
  }
  T* o = reinterpret_cast<T*>(a.out) + r * a.ld_o + static_cast<long long>(h) * a.dv;
  const T* g = a.gate ? reinterpret_cast<const T*>(a.gate) + r * a.ld_g + static_cast<long long>(h) * a.dv : nullptr;
  const float inv = a.out_scale * (a.head_gate ? 1.f / (l * (1.f + expf(-a.head_gate[r * a.ld_g + h]))) : 1.f / l);
#pragma unroll
  for (int i = 0; i < kPrMaxV; ++i) {
    const int c = v0 + i * 32 + lane;
    if (c < a.dv) pr_put(o + c, acc[i] * inv * (g ? 1.f / (1.f + expf(-pr_get(g + c))) : 1.f));
  }
}

}  // namespace rb

RB_API int rb_paged_attention_rows(const RbPagedRowsArgs* args, void* stream_v) {
  const RbPagedRowsArgs& a = *args;
  if (a.rows <= 0) return 0;
  if (!a.q || !a.out || !a.k_cache || !a.v_cache || !a.block_tables || !a.row_seq || !a.row_pos || a.heads <= 0 ||
      a.kv_heads <= 0 || a.heads % a.kv_heads || a.dk <= 0 || a.dv <= 0 || a.dk > 2048 || !a.log_amount != !a.log_rate ||
      a.block_size <= 0 || a.max_blocks <= 0)
    return -1;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_v);
  const long long items = static_cast<long long>(a.rows) * a.heads;
  const dim3 grid(static_cast<unsigned int>((items + 3) / 4), (a.dv + 32 * rb::kPrMaxV - 1) / (32 * rb::kPrMaxV));
  const size_t smem = sizeof(float) * 4 * a.dk;
  if (a.f32) rb::paged_rows_kernel<float><<<grid, 128, smem, stream>>>(a RB_BOUNDS_ARG);
  else rb::paged_rows_kernel<__nv_bfloat16><<<grid, 128, smem, stream>>>(a RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

RB_API int rb_kv_append(const void* k_new, long long ld_k, const void* v_new, long long ld_v, void* k_cache, void* v_cache,
                        const long long* slot_mapping, long long tokens, int kv_heads, int head_dim, long long num_slots,
                        void* stream_v) {
  if (tokens <= 0) return 0;
  const int row = kv_heads * head_dim;
  if (row <= 0 || (row % 8) || (ld_k % 8) || (ld_v % 8)) return -1;
  if ((reinterpret_cast<uintptr_t>(k_new) | reinterpret_cast<uintptr_t>(v_new) | reinterpret_cast<uintptr_t>(k_cache) |
       reinterpret_cast<uintptr_t>(v_cache)) & 15)
    return -2;
  const long long total = tokens * (row / 8);
  long long blocks = (total + 127) / 128;
  if (blocks > 148 * 16) blocks = 148 * 16;
  rb::kv_append_kernel<<<static_cast<int>(blocks), 128, 0, reinterpret_cast<cudaStream_t>(stream_v)>>>(
      reinterpret_cast<const __nv_bfloat16*>(k_new), ld_k, reinterpret_cast<const __nv_bfloat16*>(v_new), ld_v,
      reinterpret_cast<__nv_bfloat16*>(k_cache), reinterpret_cast<__nv_bfloat16*>(v_cache), slot_mapping, tokens, row,
      num_slots RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

RB_API long long rb_paged_attention_scratch_floats(int batch, int heads, int head_dim, int max_blocks, int block_size) {
  const long long nsplit = (static_cast<long long>(max_blocks) * block_size + rb::kSplitTokens - 1) / rb::kSplitTokens;
  return static_cast<long long>(batch) * heads * nsplit * (head_dim + 2);
}

namespace {
template <int DK, int DV, bool RULE>
int pd_launch(const RbPagedDecodeArgs& a, cudaStream_t stream) {
  const int group = a.heads / a.kv_heads;
  long long span = static_cast<long long>(a.max_blocks) * a.block_size;      // most keys a row can see
  if (a.chunk > 0 && a.chunk < span) span = a.chunk;
  if (a.window > 0 && static_cast<long long>(a.window) + a.keep_first < span) span = a.window + a.keep_first;
  const int nsplit = static_cast<int>((span + rb::kSplitTokens - 1) / rb::kSplitTokens);
  // dynamic shared memory: per warp a K and a V tile of 32 padded rows, plus the 16 padded query rows
  const int smem = (rb::kPaWarps * 32 * (DK + 8 + DV + 8) + rb::kMaxGroup * (DK + 8)) * 2;
  auto kern = rb::paged_decode_split_kernel<DK, DV, RULE>;
  static bool attr_set[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -3;
  if (!attr_set[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr_set[dev] = true;
  }
  auto O = reinterpret_cast<__nv_bfloat16*>(a.out);
  const rb::PaRule rule = {a.softcap, a.slopes, a.chunk, reinterpret_cast<const __nv_bfloat16*>(a.gate), a.head_gate, a.ld_g,
                           a.window, a.keep_first, a.sink, a.log_amount, a.log_rate, a.out_scale};
  const dim3 grid(a.batch, a.kv_heads, nsplit);
  for (int g0 = 0; g0 < group; g0 += rb::kMaxGroup)       // groups wider than 16 heads take several passes
    kern<<<grid, rb::kPaWarps * 32, smem, stream>>>(
        reinterpret_cast<const __nv_bfloat16*>(a.q), a.ld_q, reinterpret_cast<const __nv_bfloat16*>(a.k_cache),
        reinterpret_cast<const __nv_bfloat16*>(a.v_cache), a.block_tables, a.max_blocks, a.context_lens, a.heads, a.kv_heads,
        a.dk, a.dv, a.block_size, a.num_blocks, a.scale, g0, group - g0 < rb::kMaxGroup ? group - g0 : rb::kMaxGroup,
        a.scratch, nsplit, nsplit == 1 ? O : nullptr, a.ld_o, rule RB_BOUNDS_ARG);
  if (nsplit > 1)
    rb::paged_decode_merge_kernel<<<dim3(a.batch, a.heads), 128, 0, stream>>>(a.scratch, a.context_lens, a.heads, a.dv, nsplit,
                                                                              O, a.ld_o, rule);
  return static_cast<int>(cudaGetLastError());
}

template <int DK>
int pd_by_dv(const RbPagedDecodeArgs& a, cudaStream_t s) {
  if (a.dv <= 64) return pd_launch<DK, 64, true>(a, s);
  if (a.dv <= 96) return pd_launch<DK, 96, true>(a, s);
  return pd_launch<DK, 128, true>(a, s);
}
}  // namespace

RB_API int rb_paged_attention_decode_rule(const RbPagedDecodeArgs* args, void* stream_v) {
  const RbPagedDecodeArgs& a = *args;
  if (a.batch <= 0) return 0;
  if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dk <= 0 || a.dv <= 0 || a.dk > 128 || a.dv > 128 ||
      ((a.dk | a.dv) & 7) || a.block_size <= 0 || a.max_blocks <= 0 || !a.scratch || !a.log_amount != !a.log_rate || (a.ld_q & 1) ||
      a.num_blocks * a.block_size >= (1ll << 31))
    return -1;
  if ((reinterpret_cast<uintptr_t>(a.k_cache) | reinterpret_cast<uintptr_t>(a.v_cache)) & 15) return -2;
  if (reinterpret_cast<uintptr_t>(a.q) & 3) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  if (a.dk <= 64) return pd_by_dv<64>(a, s);
  if (a.dk <= 96) return pd_by_dv<96>(a, s);
  return pd_by_dv<128>(a, s);
}

RB_API int rb_paged_attention_decode(const void* q, long long ld_q, void* out, long long ld_o, const void* k_cache,
                                     const void* v_cache, const int* block_tables, int max_blocks, const int* context_lens,
                                     int batch, int heads, int kv_heads, int head_dim, int block_size, long long num_blocks,
                                     float scale, float* scratch, void* stream_v) {
  if (batch <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || (head_dim != 64 && head_dim != 128) || block_size <= 0 ||
      max_blocks <= 0 || !scratch || num_blocks * block_size >= (1ll << 31))
    return -1;
  if ((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) return -2;
  RbPagedDecodeArgs a = {};
  a.q = q; a.ld_q = ld_q; a.out = out; a.ld_o = ld_o; a.k_cache = k_cache; a.v_cache = v_cache;
  a.block_tables = block_tables; a.max_blocks = max_blocks; a.context_lens = context_lens; a.batch = batch;
  a.heads = heads; a.kv_heads = kv_heads; a.dk = a.dv = head_dim; a.block_size = block_size; a.num_blocks = num_blocks;
  a.scale = scale; a.scratch = scratch; a.out_scale = 1.f;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_v);
  return head_dim == 128 ? pd_launch<128, 128, false>(a, stream) : pd_launch<64, 64, false>(a, stream);
}
