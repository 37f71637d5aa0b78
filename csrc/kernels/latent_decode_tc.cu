// Latent attention, decoding, on the 5th-generation tensor cores (rb_latent_decode for the sizes below; latent_attention.cu has the
// interface and the form for all others).
//
// One CTA = (16 or 32 heads, slice of the context, sequence).  Tiles of 64 cached tokens; the M of the products are cached rows, then
// columns of the cached vectors, the N are heads:
//     S^T [tokens, heads]  = C [tokens, rank + rot] Q^T        A: cached rows as they lie, K-major
//     O^T [rank, heads]   += C^T [rank, tokens] P^T            A: the same bytes, MN-major
// so a tile's shared memory is filled once by TMA, page by page, and no thread ever touches it.  S^T and O^T live in TMEM.
// Products this narrow cost the same whatever their N and whether M is 64 or 128.  So a product of the scores takes two blocks of 64
// columns at once: its A has the tokens' first block in rows 0 - 63 and their second block in rows 64 - 127 (the order in which they lie
// in shared memory anyway), its B both blocks of the queries; the two diagonal quarters of the result, added, are the scores.
// The columns come in pieces of 128 through a ring that holds 2.5 tiles of the widest vectors; a piece is released as soon as its product
// with P is done, and whichever of the next scores and the next sum is ready first is issued first.
// Softmax (warps 0-3): warps 2 and 3 hand their quarter of the scores over, a thread of warps 0 and 1 has a token.  A head's maximum over
// the tokens comes by a transposing butterfly in either warp and one exchange between them; sums are kept per thread until the end.  O is
// rescaled only when a maximum has grown by more than 2^8, by all four warps.
// Warps 4-7 issue the copies (a page each), warp 8 the products.
#include "latent_attention.h"

#include "rb_common.cuh"
#include "latent_common.cuh"

namespace rb {

constexpr int kLtThreads = 288, kLtTile = 64, kLtCopyWarps = 4;
constexpr int kLtAtom = kLtTile * 128;               // 64 columns of a tile
constexpr int kLtPiece = 2 * kLtAtom;

struct LtParams {
  __nv_bfloat16* out;
  const int* block_tables;
  const int* context_lens;
  float* scratch;
  long long ld_o, num_blocks;
  int max_blocks, heads, rank, block_size, splits;
  float scale;
};

__device__ __forceinline__ float lt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void lt_sync_four() { asm volatile("bar.sync 1, 128;" ::: "memory"); }     // warps 0-3
__device__ __forceinline__ void lt_sync_two() { asm volatile("bar.sync 2, 64;" ::: "memory"); }       // warps 0, 1

template <int N>
__device__ __forceinline__ void lt_ld(uint32_t taddr, uint32_t (&r)[N]) {
  if constexpr (N == 32) tmem_ld_32x32(taddr, r);
  else tmem_ld_32x16(taddr, r);
}
template <int N>
__device__ __forceinline__ void lt_st(uint32_t taddr, const uint32_t (&r)[N]) {
#pragma unroll
  for (int c = 0; c < N; c += 16) {
    uint32_t h[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) h[i] = r[c + i];
    tmem_st_32x16(taddr + c, h);
  }
}
// Over the 32 lanes: lane l ends up with the reduction of v[l % N].
template <int N, bool MAX>
__device__ __forceinline__ float lt_reduce(const float (&v)[N]) {
  const int lane = threadIdx.x & 31;
  float a[N];
#pragma unroll
  for (int i = 0; i < N; ++i) a[i] = v[i];
#pragma unroll
  for (int n = N / 2; n >= 1; n >>= 1) {
    const bool up = lane & n;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float send = up ? a[i] : a[i + n], keep = up ? a[i + n] : a[i];
      const float got = __shfl_xor_sync(0xffffffffu, send, n);
      a[i] = MAX ? fmaxf(keep, got) : keep + got;
    }
  }
  if (N == 16) {
    const float got = __shfl_xor_sync(0xffffffffu, a[0], 16);
    a[0] = MAX ? fmaxf(a[0], got) : a[0] + got;
  }
  return a[0];
}

template <int N, int RP>
struct LtSmem {
  static constexpr int kSlots = N == 16 ? 11 : 10;
  static constexpr int kRing = 0;
  static constexpr int kRot = kRing + kSlots * kLtPiece;              // rotated parts of two tiles
  static constexpr int kQ = kRot + 2 * kLtAtom;                       // 2 RP + 1 pieces of 64 columns, N rows
  static constexpr int kP = kQ + (2 * RP + 1) * N * 128;              // N rows of 64 tokens
  static constexpr int kHand = kP + N * 128;                          // [N][64] scores that warps 2 and 3 hand over
  static constexpr int kRed = kHand + N * 64 * 4;                     // [2][2][N] maxima of warps 0 and 1, [N] maxima, [N] factors, a flag
  static constexpr int kBar = kRed + 6 * N * 4 + 16;
  static constexpr int kNumBars = 2 * kSlots + 9;                     // q, full / empty per slot, rot full[2] / empty[2], s[2], p, o
  static constexpr int kTotal = kBar + kNumBars * 8 + 16;
};

template <int N, int RP>
__global__ void __launch_bounds__(kLtThreads, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmCr,
                        const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQr, const LtParams p,
                        unsigned int* status RB_BOUNDS_PARAM) {
  using L = LtSmem<N, RP>;
  extern __shared__ __align__(1024) uint8_t lt_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sbase = smem_u32(smem);
  const uint32_t sRing = sbase + L::kRing, sRot = sbase + L::kRot, sQ = sbase + L::kQ, sP = sbase + L::kP;
  float* hand = reinterpret_cast<float*>(smem + L::kHand);
  float* red = reinterpret_cast<float*>(smem + L::kRed);
  float* m_sh = red + 4 * N;
  float* f_sh = red + 5 * N;
  volatile int* any_sh = reinterpret_cast<volatile int*>(red + 6 * N);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kBar);
  const uint32_t bar_q = smem_u32(bars);
  const uint32_t bar_full = bar_q + 8, bar_empty = bar_full + 8 * L::kSlots;
  const uint32_t bar_rfull = bar_empty + 8 * L::kSlots, bar_rempty = bar_rfull + 16;
  const uint32_t bar_s = bar_rempty + 16, bar_p = bar_s + 16, bar_o = bar_p + 8;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + L::kNumBars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int h0 = blockIdx.x * N, sp = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ctx = p.context_lens[b];
  const int chunk = latent_chunk(ctx, p.splits);
  const int t_begin = sp * chunk;
  if (t_begin >= ctx) return;
  const int t_end = min(ctx, t_begin + chunk);
  const int tiles = (t_end - t_begin + kLtTile - 1) / kLtTile;
  const int nheads = min(N, p.heads - h0);
  constexpr int kO = 4 * N;                            // TMEM: both score accumulators (2 N columns each), then RP pieces of O^T
  constexpr uint32_t kTmemCols = kO + RP * N <= 128 ? 128 : 256;

  // copies: first cache row of page `k` of tile j (-1: past the end)
  auto page_row = [&](int j, int k) {
    const int tok = t_begin + j * kLtTile + k * p.block_size;
    if (j >= tiles || k * p.block_size >= kLtTile || tok >= t_end) return -1;
    const int bi = tok / p.block_size;
    int blk = bi < p.max_blocks ? p.block_tables[static_cast<long long>(b) * p.max_blocks + bi] : -1;
    if (blk < 0 || blk >= p.num_blocks) {              // corrupt tables read block 0 instead of faulting
      RB_BOUNDS_HIT(104);
      blk = 0;
    }
    return blk * p.block_size;
  };
  const int k0 = warp - 4, k1 = k0 + kLtCopyWarps;     // pages of a tile that a copying warp takes (eight with pages of 8 tokens)
  int row0 = -1, row1 = -1;
  if (warp >= 4 && warp < 8) { row0 = page_row(0, k0); row1 = page_row(0, k1); }

  if (threadIdx.x == 0) {
    mbar_init(bar_q, 1);
    for (int s = 0; s < L::kSlots; ++s) {
      mbar_init(bar_full + 8 * s, kLtCopyWarps);
      mbar_init(bar_empty + 8 * s, 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(bar_rfull + 8 * s, kLtCopyWarps);
      mbar_init(bar_rempty + 8 * s, 1);
      mbar_init(bar_s + 8 * s, 1);
    }
    mbar_init(bar_p, 4);
    mbar_init(bar_o, 1);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmC);
    tma_prefetch_desc(&tmCr);
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmQr);
  }
  if (warp == 8) {
    tmem_alloc(smem_u32(tmem_ptr), kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_ptr;

  if (warp == 8) {
    // ---------------------------------------------------------------- products: one elected lane
    if (elect_one()) {
      mbar_arrive_expect_tx(bar_q, (2 * RP + 1) * N * 128);
#pragma unroll
      for (int i = 0; i < 2 * RP; ++i) tma_load_4d(sQ + i * N * 128, &tmQ, i * 64, h0, b, 0, bar_q);
      tma_load_4d(sQ + 2 * RP * N * 128, &tmQr, 0, h0, b, 0, bar_q);
      constexpr uint32_t idesc_s = umma_idesc_bf16(128, 2 * N, 0, 0);
      constexpr uint32_t idesc_r = umma_idesc_bf16(128, N, 0, 0);
      constexpr uint32_t idesc_o = umma_idesc_bf16(128, N, 1, 0);
      // descriptors of the first piece; an offset of o bytes is o / 16 in the address field
      constexpr uint64_t kPiece = kLtPiece / 16, kAtom = kLtAtom / 16, kRows = 2048 / 16, kHeads = N * 128 / 16;
      const uint64_t dC = umma_smem_desc_sw128(sRing, 16, 1024), dCt = umma_smem_desc_sw128(sRing, kLtAtom, 1024);
      const uint64_t dR = umma_smem_desc_sw128(sRot, 16, 1024), dQ = umma_smem_desc_sw128(sQ, 16, 1024), dP = umma_smem_desc_sw128(sP, 16, 1024);
      int sj = 0, ss = 0, sphase = 0;                  // next scores: tile, slot and phase of its next piece
      int si = 0;                                      // that piece (RP: the rotated part)
      int os = 0;                                      // slot of the first piece of the next sum
      bool ok = mbar_wait(bar_q, 0, abort_flag, status, 63);
      // Scores as far as their operands are there, `all`: until tile sj is through (a tile has to come).
      auto scores = [&](bool all) {
        const uint32_t d = tmem + (sj & 1) * 2 * N;
        while (si < RP) {
          if (all ? !mbar_wait(bar_full + 8 * ss, sphase, abort_flag, status, 64) : !mbar_test(bar_full + 8 * ss, sphase)) return !all;
          tc_fence_after();
          const uint64_t da = dC + ss * kPiece, dq = dQ + 2 * si * kHeads;
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) umma_bf16_ss(d, da + ks * 2, dq + ks * 2, idesc_s, (si | ks) != 0);
          ++si;
          if (++ss == L::kSlots) { ss = 0; sphase ^= 1; }
        }
        if (all ? !mbar_wait(bar_rfull + 8 * (sj & 1), (sj >> 1) & 1, abort_flag, status, 68)
                : !mbar_test(bar_rfull + 8 * (sj & 1), (sj >> 1) & 1))
          return !all;
        tc_fence_after();
        // rows 64 - 127 of this A are whatever lies behind: they end up where nobody looks
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) umma_bf16_ss(d, dR + (sj & 1) * kAtom + ks * 2, dQ + 2 * RP * kHeads + ks * 2, idesc_r, 1u);
        umma_commit(bar_rempty + 8 * (sj & 1));
        umma_commit(bar_s + 8 * (sj & 1));
        ++sj;
        si = 0;
        return true;
      };
      for (int oj = 0; oj < tiles && ok; ++oj) {
        if (sj <= oj) ok = scores(true);
        // S^T of tile oj + 1 goes where that of oj - 1 was, read when P of oj - 1 came
        while (ok && sj == oj + 1 && sj < tiles && !mbar_test(bar_p, oj & 1)) {
          const int before = si;
          ok = scores(false);
          if (sj == oj + 1 && si == before) break;     // the operand is not there yet: P is more likely to come first
        }
        if (!ok || !mbar_wait(bar_p, oj & 1, abort_flag, status, 69)) break;
        tc_fence_after();
#pragma unroll
        for (int ks = 0; ks < kLtTile / 16; ++ks) {
          int s = os;
#pragma unroll
          for (int i = 0; i < RP; ++i) {
            umma_bf16_ss(tmem + kO + i * N, dCt + s * kPiece + ks * kRows, dP + ks * 2, idesc_o, (oj | ks) != 0);
            s = s + 1 == L::kSlots ? 0 : s + 1;
          }
        }
#pragma unroll
        for (int i = 0; i < RP; ++i) {
          umma_commit(bar_empty + 8 * os);
          os = os + 1 == L::kSlots ? 0 : os + 1;
        }
        umma_commit(bar_o);
      }
    }
    __syncwarp();
  } else if (warp >= 4) {
    // ---------------------------------------------------------------- copies
    const uint32_t page = p.block_size * 128, to0 = k0 * page, to1 = k1 * page;
    int s = 0, phase = 1;
    bool ok = true;
    for (int j = 0; j < tiles && ok; ++j) {
      const int next0 = page_row(j + 1, k0), next1 = page_row(j + 1, k1);
      const uint32_t bytes = ((row0 >= 0) + (row1 >= 0)) * page;
      for (int i = 0; i < RP; ++i) {
        ok = mbar_wait(bar_empty + 8 * s, phase, abort_flag, status, 61);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (elect_one()) {
          const uint32_t dst = sRing + s * kLtPiece, bar = bar_full + 8 * s;
          mbar_arrive_expect_tx(bar, 2 * bytes);
          if (row0 >= 0) {
            tma_load_4d(dst + to0, &tmC, i * 128, row0, 0, 0, bar);
            tma_load_4d(dst + kLtAtom + to0, &tmC, i * 128 + 64, row0, 0, 0, bar);
          }
          if (row1 >= 0) {
            tma_load_4d(dst + to1, &tmC, i * 128, row1, 0, 0, bar);
            tma_load_4d(dst + kLtAtom + to1, &tmC, i * 128 + 64, row1, 0, 0, bar);
          }
        }
        __syncwarp();
        if (++s == L::kSlots) { s = 0; phase ^= 1; }
      }
      if (!ok) break;
      ok = mbar_wait(bar_rempty + 8 * (j & 1), ((j >> 1) & 1) ^ 1, abort_flag, status, 62);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (elect_one()) {
        const uint32_t dst = sRot + (j & 1) * kLtAtom, bar = bar_rfull + 8 * (j & 1);
        mbar_arrive_expect_tx(bar, bytes);
        if (row0 >= 0) tma_load_4d(dst + to0, &tmCr, 0, row0, 0, 0, bar);
        if (row1 >= 0) tma_load_4d(dst + to1, &tmCr, 0, row1, 0, 0, bar);
      }
      __syncwarp();
      row0 = next0;
      row1 = next1;
    }
  } else {
    // ------------------------------------------------------------------ softmax.  After a wait that gave up the loop runs on without
    // waiting, so that the warps keep meeting at the named barriers.
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
    const float sl2 = p.scale * 1.4426950408889634f;
    const bool owner = warp < 2;                       // has a token per thread
    const int tok = (warp & 1) * 32 + lane;
    float m_run = -INFINITY;                           // owners: of head lane % N, the same in both warps
    float l_part[N];                                   // owners: of this thread's tokens
#pragma unroll
    for (int h = 0; h < N; ++h) l_part[h] = 0.f;
    bool ok = true;
    for (int j = 0; j < tiles; ++j) {
      if (ok) ok = mbar_wait(bar_s + 8 * (j & 1), (j >> 1) & 1, abort_flag, status, 65);
      __syncwarp();
      tc_fence_after();
      uint32_t raw[N];
      lt_ld<N>(tmem + (j & 1) * 2 * N + (owner ? 0 : N) + lane_off, raw);
      tmem_ld_wait();
      if (!owner) {
#pragma unroll
        for (int h = 0; h < N; ++h) hand[h * kLtTile + tok] = __uint_as_float(raw[h]);
      }
      lt_sync_four();                                  // both halves of the scores are there
      float x[N];
      const bool live = tok < t_end - t_begin - j * kLtTile;
      if (owner) {
#pragma unroll
        for (int h = 0; h < N; ++h) x[h] = live ? (__uint_as_float(raw[h]) + hand[h * kLtTile + tok]) * sl2 : -INFINITY;
        float mx = lt_reduce<N, true>(x);
        float* r = red + (j & 1) * 2 * N;
        if (lane < N) r[warp * N + lane] = mx;
        lt_sync_two();
        mx = fmaxf(r[lane % N], r[N + lane % N]);
        const bool grow = mx > m_run + 8.f;            // also when there is no maximum yet
        const float m_new = grow ? mx : m_run;
        const float factor = grow ? lt_ex2(m_run - m_new) : 1.f;
        m_run = m_new;
        const bool any = __any_sync(0xffffffffu, grow);
        if (warp == 0) {
          if (lane < N) { m_sh[lane] = m_new; f_sh[lane] = factor; }
          if (lane == 0) *any_sh = any;
        }
      }
      lt_sync_four();                                  // maxima and factors are there
      const bool any = *any_sh;
      if (j > 0) {                                     // O holds tiles 0 .. j - 1, and P is free again
        if (ok) ok = mbar_wait(bar_o, (j - 1) & 1, abort_flag, status, 66);
        __syncwarp();
        tc_fence_after();
        if (any) {
#pragma unroll 1
          for (int i = 0; i < RP; ++i) {
            uint32_t o[N];
            lt_ld<N>(tmem + kO + i * N + lane_off, o);
            tmem_ld_wait();
#pragma unroll
            for (int h = 0; h < N; h += 4) {
              const float4 f = *reinterpret_cast<const float4*>(f_sh + h);
              o[h] = __float_as_uint(__uint_as_float(o[h]) * f.x);
              o[h + 1] = __float_as_uint(__uint_as_float(o[h + 1]) * f.y);
              o[h + 2] = __float_as_uint(__uint_as_float(o[h + 2]) * f.z);
              o[h + 3] = __float_as_uint(__uint_as_float(o[h + 3]) * f.w);
            }
            lt_st<N>(tmem + kO + i * N + lane_off, o);
          }
          tmem_st_wait();
#pragma unroll
          for (int h = 0; h < N; ++h) l_part[h] *= f_sh[h];
        }
      }
      if (owner) {
        // P^T as the B operand: rows are heads, 64 tokens per swizzled 128-byte row
        uint8_t* prow = smem + L::kP + (tok & 7) * 2;
        const int piece = tok >> 3;
#pragma unroll
        for (int h = 0; h < N; h += 4) {
          const float4 m4 = *reinterpret_cast<const float4*>(m_sh + h);
          const float ms[4] = {m4.x, m4.y, m4.z, m4.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float e = lt_ex2(x[h + i] - ms[i]);
            l_part[h + i] += e;
            *reinterpret_cast<__nv_bfloat16*>(prow + (h + i) * 128 + ((piece ^ ((h + i) & 7)) << 4)) = __float2bfloat16(e);
          }
        }
        if (!live) {                                   // rows without a token hold what was there before: 0 times that must be 0
          for (int i = 0; i < RP; ++i) {
            uint4* z = reinterpret_cast<uint4*>(smem + L::kRing + (j * RP + i) % L::kSlots * kLtPiece + tok * 128);
#pragma unroll
            for (int c = 0; c < 8; ++c) {
              z[c] = make_uint4(0u, 0u, 0u, 0u);
              z[kLtAtom / 16 + c] = make_uint4(0u, 0u, 0u, 0u);
            }
          }
        }
        fence_proxy_async_smem();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_p);
    }
    // ---- sums over the tokens, then this slice's (maximum, sum, O) per head, or the result when there is one slice only
    if (ok) ok = mbar_wait(bar_o, (tiles - 1) & 1, abort_flag, status, 67);     // also: nobody reads the last factors any more
    __syncwarp();
    tc_fence_after();
    if (owner) {
      const float part = lt_reduce<N, false>(l_part);
      lt_sync_two();                                   // nobody reads the last maxima any more
      if (lane < N) red[warp * N + lane] = part;
      lt_sync_two();
      const float sum = red[lane % N] + red[N + lane % N];
      if (warp == 0 && lane < N) {
        f_sh[lane] = 1.f / sum;
        if (p.splits > 1 && lane < nheads) {
          float* pp = p.scratch + ((static_cast<long long>(b) * p.heads + h0 + lane) * p.splits + sp) * (p.rank + 2);
          pp[0] = m_run;
          pp[1] = sum;
        }
      }
    }
    lt_sync_four();
#pragma unroll 1
    for (int i = 0; i < RP; ++i) {
      uint32_t o[N];
      __syncwarp();
      lt_ld<N>(tmem + kO + i * N + lane_off, o);
      tmem_ld_wait();
      const int col = i * 128 + warp * 32 + lane;
      if (col < p.rank && p.splits > 1) {
        float* pp = p.scratch + ((static_cast<long long>(b) * p.heads + h0) * p.splits + sp) * (p.rank + 2) + 2 + col;
#pragma unroll
        for (int h = 0; h < N; ++h)
          if (h < nheads) pp[static_cast<long long>(h) * p.splits * (p.rank + 2)] = __uint_as_float(o[h]);
      } else if (col < p.rank) {
        __nv_bfloat16* op = p.out + b * p.ld_o + static_cast<long long>(h0) * p.rank + col;
#pragma unroll
        for (int h = 0; h < N; ++h)
          if (h < nheads) op[static_cast<long long>(h) * p.rank] = __float2bfloat16(__uint_as_float(o[h]) * f_sh[h]);
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    if (*abort_flag) {
      // a wait gave up: let copies and products in flight land before the accumulators are released
      const unsigned long long t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
    tc_fence_after();
    tmem_dealloc(tmem, kTmemCols);
  }
}

template <int N, int RP>
int lt_launch(const RbLatentDecodeArgs& a, int splits, const CUtensorMap* const (&tm)[4], cudaStream_t s) {
  auto kern = latent_decode_tc_kernel<N, RP>;
  constexpr int smem = LtSmem<N, RP>::kTotal + 1024;
  static_assert(smem <= 232448, "shared memory of one CTA");
  static bool cfg[64] = {};
  bool& done = cfg[rbhost::device_slot()];
  if (!done) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    done = true;
  }
  const LtParams p = {reinterpret_cast<__nv_bfloat16*>(a.out), a.block_tables, a.context_lens, a.scratch, a.ld_o, a.num_blocks, a.max_blocks,
                      a.heads, a.rank, a.block_size, splits, a.scale};
  kern<<<dim3((a.heads + N - 1) / N, splits, a.batch), kLtThreads, smem, s>>>(*tm[0], *tm[1], *tm[2], *tm[3], p, rbhost::status_ptr()
                                                                             RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

// -9: not a problem for this kernel
int latent_decode_tc(const RbLatentDecodeArgs& a, int splits, cudaStream_t s) {
  const int bs = a.block_size, W = a.rank + a.rot;
  if (a.rot < 8 || a.rot > 64 || a.rank > 512 || (bs != 8 && bs != 16 && bs != 32 && bs != 64) || (a.ld_q & 7) ||
      ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.cache)) & 15) || a.num_blocks * bs >= (1ll << 24))
    return -9;
  const int n = a.heads > 16 ? 32 : 16, rp = (a.rank + 127) / 128;
  const uint64_t rows = static_cast<uint64_t>(a.num_blocks) * bs;
  auto cache_map = [&](int first, int cols, int* err) {
    const uint64_t dims[4] = {static_cast<uint64_t>(cols), rows, 1, 1};
    const uint64_t str[3] = {static_cast<uint64_t>(W) * 2, rows * W * 2, rows * W * 2};
    const uint32_t box[4] = {64, static_cast<uint32_t>(bs), 1, 1};
    return rbhost::get_tmap_4d(reinterpret_cast<const __nv_bfloat16*>(a.cache) + first, 2, dims, str, box, 1, err);
  };
  auto query_map = [&](int first, int cols, int* err) {
    const uint64_t dims[4] = {static_cast<uint64_t>(cols), static_cast<uint64_t>(a.heads), static_cast<uint64_t>(a.batch), 1};
    const uint64_t str[3] = {static_cast<uint64_t>(W) * 2, static_cast<uint64_t>(a.ld_q) * 2, static_cast<uint64_t>(a.ld_q) * 2 * a.batch};
    const uint32_t box[4] = {64, static_cast<uint32_t>(n), 1, 1};
    return rbhost::get_tmap_4d(reinterpret_cast<const __nv_bfloat16*>(a.q) + first, 2, dims, str, box, 1, err);
  };
  int err = 0;
  const CUtensorMap* tm[4] = {cache_map(0, a.rank, &err), cache_map(a.rank, a.rot, &err), query_map(0, a.rank, &err), query_map(a.rank, a.rot, &err)};
  for (const CUtensorMap* m : tm)
    if (!m) return err ? err : -5;
  if (n == 32) {
    if (rp == 1) return lt_launch<32, 1>(a, splits, tm, s);
    if (rp == 2) return lt_launch<32, 2>(a, splits, tm, s);
    if (rp == 3) return lt_launch<32, 3>(a, splits, tm, s);
    return lt_launch<32, 4>(a, splits, tm, s);
  }
  if (rp == 1) return lt_launch<16, 1>(a, splits, tm, s);
  if (rp == 2) return lt_launch<16, 2>(a, splits, tm, s);
  if (rp == 3) return lt_launch<16, 3>(a, splits, tm, s);
  return lt_launch<16, 4>(a, splits, tm, s);
}

}  // namespace rb
