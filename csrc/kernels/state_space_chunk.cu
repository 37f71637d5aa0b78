// Mamba-2 state-space recurrence over prompts (or the one with a fixed decay per head), chunked: 128 tokens at a time become matrix products on the 5th-generation tensor
// cores.
//
// With c_t the running sum of the logarithms of the decays inside a chunk and S0 the state in front of it,
//   y_t = exp(c_t) C_t S0 + sum_{s <= t} exp(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//   S   = exp(c_end) S0 + sum_s B_s (exp(c_end - c_s) dt_s x_s)^T
// One CTA owns 64 value columns of one head over a span of chunks.  Its roles:
//   warp 0   TMA: B, C and x of a chunk, two buffers each, refilled as soon as their own last reader is done
//   warp 1   issues the MMAs:  dS = B^T xs,  Y2 = C S0,  G = C B^T (of the next chunk),  Y1 = M x   (accumulators in TMEM, all
//            512 columns)
//   warp 2   step sizes, running log decays and the factors made of them, one chunk ahead
//   group 1  (warps 4-7)    M = G times decays and step sizes below the diagonal, plus D on it, bf16 in TMEM over G itself: the A
//            operand of Y1
//   groups 2, 3 (warps 8-15) xs = x scaled by what it adds to the state, as soon as the chunk before has read its own; then
//   group 2  S = exp(c_end) S + dS, one state row per thread
//   group 3  y = exp(c_t) Y2 + Y1
// The chain from chunk to chunk is xs -> dS; the state's update, its copy, M and y run beside the next chunk's products.
// The state stays in fp32 registers; its bf16 copy in shared memory is the operand of the read-out only.  xs is split into two bf16
// numbers (about 16 bits), decays and step sizes are fp32, so the state itself is good to fp32-like accuracy.
//
// Decays inside M: for 32 x 32 blocks below the diagonal exp(c_t - c_s) = exp(c_t - c_e) exp(c_e - c_s) with e the block's last
// token; both factors are at most 1, and only diagonal blocks need an exponential per element.
//
// A long segment is cut into spans that run side by side: a first pass (STATE_ONLY) computes what every span but the last adds to
// the state (from zero) and its total decay, and each span of the second pass starts from the combination of those before it.
// Rows behind the segment's end are other sequences' rows: their step size counts as zero, and nothing of them is stored.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

constexpr int kScChunk = 128;
constexpr int kScCols = 64;
constexpr int kScThreads = 512;
constexpr float kScLog2e = 1.4426950408889634f;

struct ScSmem {
  static constexpr int kAtom = kScChunk * 128;                       // 128 rows of 64 bf16, 128-byte swizzle
  static constexpr int kC = 0;
  static constexpr int kB = kC + 2 * kAtom;
  static constexpr int kX = kB + 2 * kAtom;
  static constexpr int kStage = kX + kAtom;
  static constexpr int kXs = 2 * kStage;                             // scaled x: high half, low half
  static constexpr int kS = kXs + 2 * kAtom;                         // bf16 copy of the state [128 rows][64]
  static constexpr int kTab = kS + kAtom;                            // two buffers of fp32 [4][128]
  static constexpr int kBar = kTab + 2 * 4 * kScChunk * 4;
  static constexpr int kNumBars = 6 + 6 + 2 + 2 + 7;
  static constexpr int kTotal = kBar + kNumBars * 8 + 16;
};
static_assert(ScSmem::kTotal + 1024 <= 227 * 1024, "shared memory of a CTA");

// columns of TMEM
constexpr int kTmG = 0, kTmY1 = 256, kTmY2 = 320, kTmS = 384;       // two buffers of G (M over it) and of dS

__device__ __forceinline__ float sc_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// v = hi + lo with both halves bf16
__device__ __forceinline__ void sc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - h.x, b - h.y);
}
// 16-byte piece `piece` of row `row` of a 128-byte swizzled tile
__device__ __forceinline__ int sc_piece(int row, int piece) { return row * 128 + ((piece ^ (row & 7)) << 4); }

template <bool STATE_ONLY>
__global__ void __launch_bounds__(kScThreads, 1)
state_space_chunk_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmB,
                         const __grid_constant__ CUtensorMap tmX, const RbStateSpaceArgs a, float* __restrict__ span_state,
                         float* __restrict__ span_decay, int span, unsigned int* status) {
  using L = ScSmem;
  extern __shared__ __align__(1024) uint8_t sc_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(sc_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t base = smem_u32(smem);
  const uint32_t b0 = base + L::kBar;
  const uint32_t bar_bfull = b0, bar_cfull = b0 + 16, bar_xfull = b0 + 32, bar_bempty = b0 + 48, bar_cempty = b0 + 64,
                 bar_xempty = b0 + 80, bar_g = b0 + 96, bar_tab = b0 + 112;                    // [2] each
  const uint32_t bar_m = b0 + 128, bar_y = b0 + 136, bar_yfree = b0 + 144, bar_xs = b0 + 152, bar_ds = b0 + 160, bar_s0 = b0 + 168,
                 bar_y2 = b0 + 176;
  uint32_t* tmem_ptr_smem = reinterpret_cast<uint32_t*>(smem + L::kBar + L::kNumBars * 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr_smem + 1);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ptiles = (a.p + kScCols - 1) / kScCols;
  const int h = blockIdx.x / ptiles, c0 = (blockIdx.x - h * ptiles) * kScCols;
  const int tile = blockIdx.y;
  const RcSegment seg = rc_segment(a.segments, a.tiles[2 * tile], a.num_slots);
  const int off = a.tiles[2 * tile + 1];
  const int end = min(seg.len, off + span);
  if (off >= seg.len) return;
  if (STATE_ONLY && end == seg.len) return;        // nobody starts from what the last span adds
  const int chunks = (end - off + kScChunk - 1) / kScChunk;
  const int g = h / (a.heads / a.groups);
  const int atoms = a.n > 64 ? 2 : 1;

  if (tid == 0) {
    for (int s = 0; s < 2; ++s) {
      mbar_init(bar_bfull + 8 * s, 1);
      mbar_init(bar_cfull + 8 * s, 1);
      mbar_init(bar_xfull + 8 * s, 1);
      mbar_init(bar_bempty + 8 * s, 1);
      mbar_init(bar_cempty + 8 * s, 1);
      mbar_init(bar_xempty + 8 * s, 1);
      mbar_init(bar_g + 8 * s, 1);
      mbar_init(bar_tab + 8 * s, 1);
    }
    mbar_init(bar_m, 4);
    mbar_init(bar_y, 1);
    mbar_init(bar_yfree, 4);
    mbar_init(bar_xs, 8);
    mbar_init(bar_y2, 1);
    mbar_init(bar_ds, 1);
    mbar_init(bar_s0, 4);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmC);
    tma_prefetch_desc(&tmB);
    tma_prefetch_desc(&tmX);
  }
  if (atoms == 1) {                                // the state has 128 rows in TMEM: columns 64 .. 127 of B are zero
    for (int i = tid; i < 2 * L::kAtom / 16; i += kScThreads) {
      const int s = i / (L::kAtom / 16);
      *reinterpret_cast<uint4*>(smem + s * L::kStage + L::kB + L::kAtom + (i - s * (L::kAtom / 16)) * 16) = make_uint4(0u, 0u, 0u, 0u);
    }
    fence_proxy_async_smem();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_ptr_smem), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_ptr_smem;

  // xs of chunk i: half of a token's columns per thread of groups 2 and 3.  Gives exp(c_end) to group 2 and the row's exp(c_t) to
  // group 3 (the tables are free once Y1 is done); false: a wait gave up.
  auto scale_x = [&](int i, float& e) -> bool {
    const float* tab = reinterpret_cast<const float*>(smem + L::kTab + (i & 1) * 4 * kScChunk * 4);
    const uint8_t* x = smem + (i & 1) * L::kStage + L::kX;
    if (!mbar_wait(bar_tab + 8 * (i & 1), (i >> 1) & 1, abort_flag, status, 71)) return false;
    if (!mbar_wait(bar_xfull + 8 * (i & 1), (i >> 1) & 1, abort_flag, status, 72)) return false;
    const int row = (warp & 3) * 32 + lane, q0 = warp < 12 ? 0 : kScCols / 16;
    const float w = tab[3 * kScChunk + row];
    e = sc_ex2(tab[warp < 12 ? kScChunk - 1 : row]);
#pragma unroll
    for (int q = 0; q < kScCols / 16; ++q) {
      float v[8];
      RcVec<__nv_bfloat16, 8>::load(reinterpret_cast<const __nv_bfloat16*>(x + sc_piece(row, q0 + q)), v);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) sc_split(w * v[2 * k], w * v[2 * k + 1], hi[k], lo[k]);
      *reinterpret_cast<uint4*>(smem + L::kXs + sc_piece(row, q0 + q)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(smem + L::kXs + L::kAtom + sc_piece(row, q0 + q)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    fence_proxy_async_smem();
    __syncwarp();
    if (lane == 0) mbar_arrive(bar_xs);
    return true;
  };

  if (warp == 0) {
    if (lane == 0) {
      // ------------------------------------------------------------------ TMA
      for (int i = 0; i < chunks; ++i) {
        const int s = i & 1, row = seg.first + off + i * kScChunk;
        const uint32_t st = base + s * L::kStage, par = ((i >> 1) & 1) ^ 1;
        if (!mbar_wait(bar_bempty + 8 * s, par, abort_flag, status, 61)) break;
        mbar_arrive_expect_tx(bar_bfull + 8 * s, L::kAtom * atoms);
        for (int k = 0; k < atoms; ++k) tma_load_4d(st + L::kB + k * L::kAtom, &tmB, k * 64, g, row, 0, bar_bfull + 8 * s);
        if (!STATE_ONLY) {
          if (!mbar_wait(bar_cempty + 8 * s, par, abort_flag, status, 78)) break;
          mbar_arrive_expect_tx(bar_cfull + 8 * s, L::kAtom * atoms);
          for (int k = 0; k < atoms; ++k) tma_load_4d(st + L::kC + k * L::kAtom, &tmC, k * 64, g, row, 0, bar_cfull + 8 * s);
        }
        if (!mbar_wait(bar_xempty + 8 * s, par, abort_flag, status, 79)) break;
        mbar_arrive_expect_tx(bar_xfull + 8 * s, L::kAtom);
        tma_load_4d(st + L::kX, &tmX, c0, h, row, 0, bar_xfull + 8 * s);
      }
    }
  } else if (warp == 1) {
    // -------------------------------------------------------------------- MMA: the whole warp walks, one elected lane issues
    constexpr uint32_t idesc_g = umma_idesc_bf16(128, 128, 0, 0);
    constexpr uint32_t idesc_y = umma_idesc_bf16(128, kScCols, 0, 1);         // A K-major (C) or in TMEM (M), B MN-major
    constexpr uint32_t idesc_s = umma_idesc_bf16(128, kScCols, 1, 1);         // A = B^T: MN-major
    // descriptors of the first stage and the first 16 of the contraction; an offset of o bytes is o / 16 in the address field
    constexpr uint64_t kStage = L::kStage / 16, kAtom = L::kAtom / 16, kRows = 2048 / 16;
    const uint64_t dC = umma_smem_desc_sw128(base + L::kC, 16, 1024), dB = umma_smem_desc_sw128(base + L::kB, 16, 1024);
    const uint64_t dBt = umma_smem_desc_sw128(base + L::kB, L::kAtom, 1024), dX = umma_smem_desc_sw128(base + L::kX, L::kAtom, 1024);
    const uint64_t dXs = umma_smem_desc_sw128(base + L::kXs, L::kAtom, 1024), dS0 = umma_smem_desc_sw128(base + L::kS, L::kAtom, 1024);
    const int n = a.n;
    auto issue_g = [&](int i) -> bool {
      if (!mbar_wait(bar_bfull + 8 * (i & 1), (i >> 1) & 1, abort_flag, status, 62)) return false;
      if (STATE_ONLY) return true;
      if (!mbar_wait(bar_cfull + 8 * (i & 1), (i >> 1) & 1, abort_flag, status, 80)) return false;
      tc_fence_after();
      if (elect_one()) {
        const uint64_t st = (i & 1) * kStage;
        const uint32_t d = tmem + kTmG + (i & 1) * 128;
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (k * 16 >= n) break;                  // the rest of the columns is zero
          const uint64_t o = st + (k >> 2) * kAtom + (k & 3) * 2;
          umma_bf16_ss(d, dC + o, dB + o, idesc_g, k != 0 ? 1u : 0u);
        }
        umma_commit(bar_g + 8 * (i & 1));
      }
      __syncwarp();
      return true;
    };
    bool ok = issue_g(0);
    for (int i = 0; i < chunks && ok; ++i) {
      const uint64_t st = (i & 1) * kStage;
      if (!mbar_wait(bar_xs, i & 1, abort_flag, status, 63)) break;
      tc_fence_after();
      if (elect_one()) {
        const uint32_t d = tmem + kTmS + (i & 1) * 64;
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int k = 0; k < kScChunk / 16; ++k)
            umma_bf16_ss(d, dBt + st + k * kRows, dXs + half * kAtom + k * kRows, idesc_s, (half | k) != 0 ? 1u : 0u);
        umma_commit(bar_ds);
        umma_commit(bar_bempty + 8 * (i & 1));
      }
      __syncwarp();
      if (!STATE_ONLY) {
        if (!mbar_wait(bar_s0, i & 1, abort_flag, status, 64)) break;
        if (!mbar_wait(bar_yfree, (i & 1) ^ 1, abort_flag, status, 65)) break;
        tc_fence_after();
        if (elect_one()) {
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            if (k * 16 >= n) break;
            umma_bf16_ss(tmem + kTmY2, dC + st + (k >> 2) * kAtom + (k & 3) * 2, dS0 + k * kRows, idesc_y, k != 0 ? 1u : 0u);
          }
          umma_commit(bar_y2);
          umma_commit(bar_cempty + 8 * (i & 1));
        }
        __syncwarp();
      }
      if (i + 1 < chunks && !issue_g(i + 1)) break;         // behind Y1 of the chunk before, which read its buffer
      if (!STATE_ONLY) {
        if (!mbar_wait(bar_m, i & 1, abort_flag, status, 66)) break;
        tc_fence_after();
      }
      if (elect_one()) {
        if (!STATE_ONLY) {
          const uint32_t m = tmem + kTmG + (i & 1) * 128;
#pragma unroll
          for (int k = 0; k < kScChunk / 16; ++k)
            umma_bf16_ts(tmem + kTmY1, m + k * 8, dX + st + k * kRows, idesc_y, k != 0 ? 1u : 0u);
          umma_commit(bar_y);
        }
        umma_commit(bar_xempty + 8 * (i & 1));
      }
      __syncwarp();
    }
  } else if (warp == 2) {
    // -------------------------------------------------------------------- factors of a chunk, four tokens per lane
    const bool fixed = a.decay != nullptr;         // steps of 1
    const float rate2 = fixed ? -log2f(a.decay[h]) : expf(a.a_log[h]) * kScLog2e, dt_bias = fixed ? 0.f : a.dt_bias[h];
    float raw[4] = {0.f, 0.f, 0.f, 0.f}, total = 0.f;
    auto fetch = [&](int i) {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int t = off + i * kScChunk + 4 * lane + k;
        if (t < end && !fixed) raw[k] = a.dt_raw[static_cast<long long>(seg.first + t) * a.ld_dt + h];
      }
    };
    fetch(0);
    for (int i = 0; i < chunks; ++i) {
      float d[4], c[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        d[k] = off + i * kScChunk + 4 * lane + k < end ? (fixed ? 1.f : rc_softplus(raw[k] + dt_bias)) : 0.f;
        c[k] = (k ? c[k ? k - 1 : 0] : 0.f) - rate2 * d[k];
      }
      if (i + 1 < chunks) fetch(i + 1);
      float run = c[3];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += u;
      }
      const float before = run - c[3];
      const float c_end = __shfl_sync(0xffffffffu, run, 31), c_blk = __shfl_sync(0xffffffffu, run, lane | 7);
      total += c_end;
      if (!mbar_wait(bar_xempty + 8 * (i & 1), ((i >> 1) & 1) ^ 1, abort_flag, status, 67)) break;
      float4* tab = reinterpret_cast<float4*>(smem + L::kTab + (i & 1) * 4 * kScChunk * 4) + lane;
      float v[4][4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        v[0][k] = before + c[k];
        v[1][k] = d[k];
        v[2][k] = d[k] * sc_ex2(c_blk - v[0][k]);  // towards the end of the token's block of 32
        v[3][k] = d[k] * sc_ex2(c_end - v[0][k]);  // towards the end of the chunk
      }
#pragma unroll
      for (int q = 0; q < 4; ++q) tab[q * 32] = make_float4(v[q][0], v[q][1], v[q][2], v[q][3]);
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_tab + 8 * (i & 1));
    }
    if (STATE_ONLY && lane == 0 && c0 == 0) span_decay[static_cast<long long>(tile) * a.heads + h] = total;
  } else if (warp >= 4 && warp < 8) {
    if (!STATE_ONLY) {
      // ------------------------------------------------------------------ M, one row per thread
      const int wq = warp & 3, row = wq * 32 + lane;
      const uint32_t lane_off = static_cast<uint32_t>(wq * 32) << 16;
      const float dskip = a.D ? a.D[h] : 0.f;
      const uint32_t zero[16] = {0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u, 0u};
      for (int i = 0; i < chunks; ++i) {
        const float* tab = reinterpret_cast<const float*>(smem + L::kTab + (i & 1) * 4 * kScChunk * 4);
        if (!mbar_wait(bar_tab + 8 * (i & 1), (i >> 1) & 1, abort_flag, status, 68)) break;
        if (!mbar_wait(bar_g + 8 * (i & 1), (i >> 1) & 1, abort_flag, status, 69)) break;
        tc_fence_after();
        const uint32_t tm = tmem + kTmG + (i & 1) * 128 + lane_off;            // block b's M (16 columns) never reaches past block b
        const float ct = tab[row];
        for (int b = 0; b <= wq; ++b) {
          uint32_t r[32];
          tmem_ld_32x32(tm + b * 32, r);
          tmem_ld_wait();
          uint32_t packed[16];
          if (b < wq) {
            const float e = sc_ex2(ct - tab[b * 32 + 31]);
            const float4* f = reinterpret_cast<const float4*>(tab + 2 * kScChunk + b * 32);
#pragma unroll
            for (int q = 0; q < 8; ++q) {
              const float4 u = f[q];
              packed[2 * q] = pack_bf16x2(__uint_as_float(r[4 * q]) * e * u.x, __uint_as_float(r[4 * q + 1]) * e * u.y);
              packed[2 * q + 1] = pack_bf16x2(__uint_as_float(r[4 * q + 2]) * e * u.z, __uint_as_float(r[4 * q + 3]) * e * u.w);
            }
          } else {
            const float4* cs = reinterpret_cast<const float4*>(tab + b * 32);
            const float4* ds = reinterpret_cast<const float4*>(tab + kScChunk + b * 32);
#pragma unroll
            for (int q = 0; q < 8; ++q) {
              const float4 c = cs[q], d = ds[q];
              const float m0 = 4 * q <= lane ? fmaf(__uint_as_float(r[4 * q]) * d.x, sc_ex2(ct - c.x), 4 * q == lane ? dskip : 0.f) : 0.f;
              const float m1 = 4 * q + 1 <= lane ? fmaf(__uint_as_float(r[4 * q + 1]) * d.y, sc_ex2(ct - c.y), 4 * q + 1 == lane ? dskip : 0.f) : 0.f;
              const float m2 = 4 * q + 2 <= lane ? fmaf(__uint_as_float(r[4 * q + 2]) * d.z, sc_ex2(ct - c.z), 4 * q + 2 == lane ? dskip : 0.f) : 0.f;
              const float m3 = 4 * q + 3 <= lane ? fmaf(__uint_as_float(r[4 * q + 3]) * d.w, sc_ex2(ct - c.w), 4 * q + 3 == lane ? dskip : 0.f) : 0.f;
              packed[2 * q] = pack_bf16x2(m0, m1);
              packed[2 * q + 1] = pack_bf16x2(m2, m3);
            }
          }
          tmem_st_32x16(tm + b * 16, packed);
        }
        for (int b = wq + 1; b < 4; ++b) tmem_st_32x16(tm + b * 16, zero);     // above the diagonal
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar_m);
      }
    }
  } else if (warp >= 8 && warp < 12) {
    // -------------------------------------------------------------------- xs and the state
    const int row = (warp & 3) * 32 + lane;
    const uint32_t ts = tmem + kTmS + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    const long long state_n = static_cast<long long>(a.n) * a.p;
    const long long at = static_cast<long long>(row) * a.p + c0;
    float* slot = a.state + (static_cast<long long>(seg.slot) * a.heads + h) * state_n;
    const bool live = row < a.n;
    const int cols = min(kScCols, a.p - c0);       // multiple of 8
    float S[kScCols];
#pragma unroll
    for (int j = 0; j < kScCols; j += 4) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!STATE_ONLY && seg.start > 0 && live && j < cols) v = *reinterpret_cast<const float4*>(slot + at + j);
      S[j] = v.x; S[j + 1] = v.y; S[j + 2] = v.z; S[j + 3] = v.w;
    }
    if (!STATE_ONLY) {
      for (int t = tile - off / span; t < tile; ++t) {               // spans of this segment in front of this one
        const float d = sc_ex2(span_decay[static_cast<long long>(t) * a.heads + h]);
        const float* add = span_state + (static_cast<long long>(t) * a.heads + h) * state_n + at;
#pragma unroll
        for (int j = 0; j < kScCols; j += 4) {
          if (!live || j >= cols) continue;
          const float4 v = *reinterpret_cast<const float4*>(add + j);
          S[j] = fmaf(S[j], d, v.x); S[j + 1] = fmaf(S[j + 1], d, v.y);
          S[j + 2] = fmaf(S[j + 2], d, v.z); S[j + 3] = fmaf(S[j + 3], d, v.w);
        }
      }
    }
    auto publish = [&]() {                         // bf16 copy of the state for the read-out
#pragma unroll
      for (int q = 0; q < kScCols / 8; ++q)
        *reinterpret_cast<uint4*>(smem + L::kS + sc_piece(row, q)) =
            make_uint4(pack_bf16x2(S[8 * q], S[8 * q + 1]), pack_bf16x2(S[8 * q + 2], S[8 * q + 3]),
                       pack_bf16x2(S[8 * q + 4], S[8 * q + 5]), pack_bf16x2(S[8 * q + 6], S[8 * q + 7]));
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_s0);
    };
    float e_end = 1.f, e_next = 1.f;
    bool ok = scale_x(0, e_end);
    if (!STATE_ONLY) publish();
    for (int i = 0; i < chunks && ok; ++i) {
      ok = mbar_wait(bar_ds, i & 1, abort_flag, status, 73);
      if (!ok) break;
      if (i + 1 < chunks && !(ok = scale_x(i + 1, e_next))) break;
      tc_fence_after();
#pragma unroll
      for (int q = 0; q < kScCols / 32; ++q) {
        uint32_t r[32];
        tmem_ld_32x32(ts + (i & 1) * 64 + q * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) S[q * 32 + j] = fmaf(S[q * 32 + j], e_end, __uint_as_float(r[j]));
      }
      tc_fence_before();
      e_end = e_next;
      if (!STATE_ONLY && i + 1 < chunks) {
        ok = mbar_wait(bar_y2, i & 1, abort_flag, status, 77);       // the copy has been read
        if (!ok) break;
        publish();
      }
    }
    if (ok && live && (STATE_ONLY || end == seg.len)) {
      float* dst = STATE_ONLY ? span_state + (static_cast<long long>(tile) * a.heads + h) * state_n : slot;
#pragma unroll
      for (int j = 0; j < kScCols; j += 4)
        if (j < cols) *reinterpret_cast<float4*>(dst + at + j) = make_float4(S[j], S[j + 1], S[j + 2], S[j + 3]);
    }
  } else if (warp >= 12) {
    // -------------------------------------------------------------------- xs and y, one row per thread
    const int row = (warp & 3) * 32 + lane;
    const uint32_t ty = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    const int cols = min(kScCols, a.p - c0);
    float e = 1.f, e_next = 1.f;
    bool ok = scale_x(0, e);
    for (int i = 0; i < chunks && ok; ++i) {
      if (i + 1 < chunks) {
        ok = mbar_wait(bar_ds, i & 1, abort_flag, status, 74) && scale_x(i + 1, e_next);
        if (!ok) break;
      }
      if (!STATE_ONLY) {
        if (!mbar_wait(bar_y, i & 1, abort_flag, status, 76)) break;
        tc_fence_after();
        uint32_t packed[kScCols / 2];
#pragma unroll
        for (int q = 0; q < kScCols / 32; ++q) {
          uint32_t y1[32], y2[32];
          tmem_ld_32x32(ty + kTmY1 + q * 32, y1);
          tmem_ld_32x32(ty + kTmY2 + q * 32, y2);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j)
            packed[q * 16 + j] = pack_bf16x2(fmaf(e, __uint_as_float(y2[2 * j]), __uint_as_float(y1[2 * j])),
                                             fmaf(e, __uint_as_float(y2[2 * j + 1]), __uint_as_float(y1[2 * j + 1])));
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar_yfree);
        e = e_next;
        const int t = off + i * kScChunk + row;
        if (t < end) {
          __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.y) + static_cast<long long>(seg.first + t) * a.ld_y +
                               static_cast<long long>(h) * a.p + c0;
#pragma unroll
          for (int q = 0; q < kScCols / 8; ++q)
            if (q * 8 < cols)
              *reinterpret_cast<uint4*>(out + q * 8) = make_uint4(packed[4 * q], packed[4 * q + 1], packed[4 * q + 2], packed[4 * q + 3]);
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    if (*abort_flag) {
      // a wait gave up: let copies and MMAs in flight land before the accumulators are released
      const unsigned long long t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace rb

namespace {
// [rows, heads, size] part of a packed row-major matrix, 64 columns of 128 rows of one head at a time
const CUtensorMap* sc_map(const void* base, int size, int heads, long long rows, long long ld, int* err) {
  const uint64_t dims[4] = {(uint64_t)size, (uint64_t)heads, (uint64_t)rows, 1};
  const uint64_t str[3] = {(uint64_t)size * 2, (uint64_t)ld * 2, (uint64_t)(rows * ld) * 2};
  const uint32_t box[4] = {64, 1, (uint32_t)rb::kScChunk, 1};
  return rbhost::get_tmap_4d(base, 2, dims, str, box, 1, err);
}
}  // namespace

RB_API int rb_state_space_chunked(const RbStateSpaceArgs* args, float* span_state, float* span_decay, int span, void* stream_v) {
  const RbStateSpaceArgs& a = *args;
  if (a.num_tiles <= 0) return 0;
  if (!a.xbc || (!a.decay && (!a.dt_raw || !a.dt_bias || !a.a_log)) || !a.state || !a.y || !a.segments || !a.tiles || a.f32 || a.heads <= 0 ||
      a.groups <= 0 || a.heads % a.groups || a.p <= 0 || a.n <= 0 || a.num_slots <= 0 || a.num_tiles > 65535 || a.rows <= 0 ||
      span <= 0 || span % rb::kScChunk || (span_state != nullptr) != (span_decay != nullptr))
    return -1;
  if (a.n > 128 || ((a.n | a.p) & 7) || ((a.ld_xbc | a.ld_y) & 7)) return -9;
  if ((reinterpret_cast<uintptr_t>(a.xbc) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.state) |
       reinterpret_cast<uintptr_t>(span_state)) & 15)
    return -9;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.xbc);
  const __nv_bfloat16* b = x + static_cast<long long>(a.heads) * a.p;
  const __nv_bfloat16* c = b + static_cast<long long>(a.groups) * a.n;
  int err = 0;
  const CUtensorMap* tx = sc_map(x, a.p, a.heads, a.rows, a.ld_xbc, &err);
  const CUtensorMap* tb = sc_map(b, a.n, a.groups, a.rows, a.ld_xbc, &err);
  const CUtensorMap* tc = sc_map(c, a.n, a.groups, a.rows, a.ld_xbc, &err);
  if (!tx || !tb || !tc) return err ? err : -5;
  auto first = rb::state_space_chunk_kernel<true>;
  auto second = rb::state_space_chunk_kernel<false>;
  const int smem = rb::ScSmem::kTotal + 1024;
  static bool cfg_dev[64] = {false};
  bool& cfg = cfg_dev[rbhost::device_slot()];
  if (!cfg) {
    cudaError_t e = cudaFuncSetAttribute(first, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(second, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  const dim3 grid(a.heads * ((a.p + rb::kScCols - 1) / rb::kScCols), a.num_tiles);
  if (span_state) first<<<grid, rb::kScThreads, smem, s>>>(*tc, *tb, *tx, a, span_state, span_decay, span, rbhost::status_ptr());
  second<<<grid, rb::kScThreads, smem, s>>>(*tc, *tb, *tx, a, span_state, span_decay, span, rbhost::status_ptr());
  return static_cast<int>(cudaGetLastError());
}
