// Flash attention forward, two query tiles per CTA in ping-pong on the 5th-generation tensor cores.
//
// One CTA owns 256 queries of one (batch, head): tile A (rows 0-127) and tile B (rows 128-255).  TMEM (all 512
// columns of the SM) holds S_A, S_B (128 fp32 columns each) and the output accumulators O_A, O_B (head-dim columns
// each).  Per 128-key block j the single MMA-issuing thread runs, in this order,
//     PV(j, A)   O_A += P_A V_j      A operand P read from TMEM (TS form), V_j read MN-major from shared memory
//     QK(j+1, A) S_A  = Q_A K_j+1^T
//     PV(j, B), QK(j+1, B)
// so while softmax warp group A turns S_A into P_A the tensor cores work for tile B and the other way round.
// Softmax (warps 0-3 for A, 4-7 for B, one query row per thread): S is read from TMEM once into registers (the
// producer warp group hands most of its registers to the softmax groups with setmaxnreg), the probabilities are written back as packed bf16 over the first 64 columns of the same S buffer, O stays in TMEM and
// is only rescaled when the running row maximum moved by more than 2^8 (the stale maximum keeps the exponentials
// bounded by 256, exact after the final division by the row sum).  A share of the exponentials can be computed with a
// polynomial on the FMA pipe (template parameter; off by default, see rb_attention_fwd_tc2).  Warp 8 is the TMA producer (Q once, K / V through a ring of stages), warp 9 issues MMAs.
//
// The RULE form serves inference of decoders with their own score rule: separate key / value head sizes (columns beyond the
// real sizes are zero-filled by TMA), capped scores, a linear or (LOG) a logarithmic distance bias, chunked or windowed visibility (key blocks before a
// tile's first visible key are skipped, so the two tiles may start at different blocks), first keys that a window keeps (their
// blocks are walked before the window's), a sink in the softmax and a sigmoid output gate per value column or per head.
// With DR > 0 queries and keys have a second part whose keys all heads share (rotary positions of latent attention): it is one more
// 64-column piece of the Q and K tiles, loaded from its own array.
//
// Same semantics as the other forward kernels (causal alignment to the end of the keys, GQA, log-sum-exp output).
// Replaces the reference's materialised-score attention (crates/nn/src/attention.rs:640-836).
#include "attention.h"

#include "rb_common.cuh"

namespace rb {

constexpr int kF2Threads = 384;          // warps 0-7 softmax, 8 TMA, 9 MMA, 10-11 only give their registers away
constexpr int kF2Tile = 128;
constexpr float kF2Log2e = 1.4426950408889634f;
constexpr float kF2RescaleThreshold = 8.f;   // log2 units

struct F2Params {
  __nv_bfloat16* out;
  float* lse;
  long long o_bs, o_rs, o_hs;
  int seq_q, seq_k, heads, kv_heads, causal;
  float scale;
  const int* kv_lens;       // optional [batch]: number of real keys
  // RULE kernels only
  int dk, dv;               // real head sizes
  float softcap;            // 0: none
  const float* slopes;      // [heads] or NULL
  int chunk;                // 0: none; key 0 starts a chunk
  const __nv_bfloat16* gate;   // [seq_q, heads * dv] or NULL
  const float* head_gate;      // [seq_q, heads] or NULL
  long long ld_gate;
  int window, keep, sink;
  int dr;                   // DR > 0: real size of the second part
  const float* log_amount;  // LOG: [heads] each
  const float* log_rate;
  float out_scale;
};

__device__ __forceinline__ float f2_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float f2_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two fp32 lanes per instruction (sm_100 packed arithmetic)
__device__ __forceinline__ uint64_t f2_pack(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void f2_unpack(uint64_t v, uint32_t& lo, uint32_t& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=r"(lo), "=r"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t f2_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t f2_add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t f2_mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// Capped scores of one thread's row, in place and in log2 units: r <- cap2 * tanh(c * r) + slope2 * i + bias0 (i: column).
// For |c r| < sqrt(2) tanh(x) = x P(x^2), P the degree-6 Chebyshev interpolant of tanh(sqrt(y)) / sqrt(y) on [0, 2]
// (largest error 2.0e-6), on packed pairs: no special-function instruction.  Where a warp meets a larger argument it
// starts over from the raw scores with f2_cap_scores_wide.
struct F2Cap {
  uint64_t c, k[7];                                  // c and cap2 * coefficients, each in both halves
  __device__ __forceinline__ void init(float c1, float cap2) {
    const float k1[7] = {0.999997556f, -0.333212644f, 0.132326901f, -0.0506877862f, 0.0164362881f, -0.00365187856f, 0.00038573076f};
    c = f2_pack(c1, c1);
#pragma unroll
    for (int i = 0; i < 7; ++i) k[i] = f2_pack(cap2 * k1[i], cap2 * k1[i]);
  }
};
// Returns the bits of all x^2 combined: the top exponent bit (30) says that one of them is >= 2.
__device__ __forceinline__ uint32_t f2_cap_scores(uint32_t (&r)[128], const F2Cap& f, float slope2, float bias0) {
  const uint64_t two_slope = f2_pack(2.f * slope2, 2.f * slope2);
  uint32_t any = 0u;
#pragma unroll
  for (int g = 0; g < 4; ++g) {
    uint64_t b = f2_pack(fmaf(slope2, static_cast<float>(g * 32), bias0), fmaf(slope2, static_cast<float>(g * 32 + 1), bias0));
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      uint32_t& r0 = r[g * 32 + 2 * i];
      uint32_t& r1 = r[g * 32 + 2 * i + 1];
      const uint64_t x = f2_mul2(f2_pack(__uint_as_float(r0), __uint_as_float(r1)), f.c);
      const uint64_t y = f2_mul2(x, x);
      uint32_t lo, hi;
      f2_unpack(y, lo, hi);
      any |= lo | hi;
      uint64_t p = f2_fma2(y, f.k[6], f.k[5]);
#pragma unroll
      for (int q = 4; q >= 0; --q) p = f2_fma2(p, y, f.k[q]);
      p = f2_fma2(x, p, b);
      b = f2_add2(b, two_slope);
      f2_unpack(p, r0, r1);
    }
  }
  return any;
}
// The same for arguments of any size: tanh(x) = 1 - 2 / (1 + e^(2x)).
__device__ __forceinline__ void f2_cap_scores_wide(uint32_t (&r)[128], float c, float cap2, float slope2, float bias0) {
#pragma unroll
  for (int i = 0; i < 128; ++i) {
    const float e = f2_ex2(__uint_as_float(r[i]) * (2.f * kF2Log2e) * c);
    r[i] = __float_as_uint(fmaf(-2.f * cap2, f2_rcp(1.f + e), cap2 + fmaf(slope2, static_cast<float>(i), bias0)));
  }
}
// r <- mul * r - amount * log2(1 + rate * (dist0 - i)) for the columns i of one thread's row (scores in log2 units; distances below 0 are
// masked afterwards).  With u = i - 63.5 the logarithm is log2(a) + log2(e) ln(1 - x), a = 1 + rate (dist0 - 63.5), x = rate u / a: where
// |x| <= 1/8 for all columns (`far`, which the warp's first row decides for all) five terms of ln's series (largest error 8e-7) on packed
// pairs do, otherwise one logarithm per score.
__device__ __forceinline__ float f2_lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void f2_log_bias(uint32_t (&r)[128], float mul, float amount, float rate, float dist0, bool far) {
  if (!far) {
#pragma unroll
    for (int i = 0; i < 128; ++i) {
      const float t = f2_lg2(fmaf(rate, fmaxf(dist0 - static_cast<float>(i), 0.f), 1.f));
      r[i] = __float_as_uint(fmaf(-amount, t, mul * __uint_as_float(r[i])));
    }
    return;
  }
  const float a = fmaf(rate, dist0 - 63.5f, 1.f), rho = rate * f2_rcp(a), base = -amount * f2_lg2(a), top = amount * kF2Log2e;
  const uint64_t m = f2_pack(mul, mul), b = f2_pack(base, base), step = f2_pack(2.f * rho, 2.f * rho);
  const uint64_t k1 = f2_pack(top, top), k2 = f2_pack(top / 2.f, top / 2.f), k3 = f2_pack(top / 3.f, top / 3.f), k4 = f2_pack(top / 4.f, top / 4.f),
                 k5 = f2_pack(top / 5.f, top / 5.f);
#pragma unroll
  for (int g = 0; g < 4; ++g) {
    uint64_t x = f2_pack(rho * (g * 32 - 63.5f), rho * (g * 32 - 62.5f));
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      uint32_t& r0 = r[g * 32 + 2 * i];
      uint32_t& r1 = r[g * 32 + 2 * i + 1];
      uint64_t p = f2_fma2(x, k5, k4);
      p = f2_fma2(p, x, k3);
      p = f2_fma2(p, x, k2);
      p = f2_fma2(p, x, k1);
      p = f2_fma2(p, x, b);
      p = f2_fma2(f2_pack(__uint_as_float(r0), __uint_as_float(r1)), m, p);
      x = f2_add2(x, step);
      f2_unpack(p, r0, r1);
    }
  }
}
// 2^x on the FMA / integer pipes: round-to-nearest split x = n + f, |f| <= 0.5, degree-4 polynomial for 2^f
// (relative error about 4e-5, well below bf16 rounding), exponent added to the bit pattern.  x must be >= -126.
__device__ __forceinline__ float f2_ex2_poly(float x) {
  x = fmaxf(x, -125.f);
  const float magic = 12582912.f;                     // 1.5 * 2^23: the sum's low mantissa bits hold round(x)
  const float t = x + magic;
  const float n = t - magic;
  const float f = x - n;
  float p = fmaf(f, 0.0096181291f, 0.0555041087f);
  p = fmaf(p, f, 0.2402265070f);
  p = fmaf(p, f, 0.6931471806f);
  p = fmaf(p, f, 1.0f);
  return __int_as_float(__float_as_int(p) + (__float_as_int(t) << 23));
}

// Register reallocation between warp groups (four consecutive warps, all of which must execute the instruction): the
// producer group shrinks to a few registers per thread and the softmax groups grow, so that a whole row of 128 scores
// fits in registers.
// (setmaxnreg_inc / setmaxnreg_dec: rb_common.cuh)

__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]),
      "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]),
      "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_ld_32x32_ptr(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}

// D: columns of Q and K tiles, both parts
template <int D, int DV>
struct F2Smem {
  static constexpr int kStages = D == 64 && DV == 64 ? 4 : D >= 128 && DV == 128 ? 2 : D == 192 ? 2 : 3;     // of K
  static constexpr int kVStages = D == 192 && DV == 128 ? 1 : kStages;
  static constexpr int kHalf = kF2Tile * 128;                 // one 64-column swizzle atom: 128 rows x 128 B
  static constexpr int kTileBytes = (D / 64) * kHalf;         // a 128-row tile of Q or K
  static constexpr int kVTileBytes = (DV / 64) * kHalf;       // a 128-row tile of V
  static constexpr int kQ = 0;                                // two tiles
  static constexpr int kK = kQ + 2 * kTileBytes;
  static constexpr int kV = kK + kStages * kTileBytes;
  static constexpr int kBar = kV + kVStages * kVTileBytes;
  static constexpr int kNumBars = 2 + 2 * (kStages + kVStages) + 6;   // q[2], full and empty per K and V stage, s_full[2], p_full[2], o_ready[2]
  static constexpr int kTotal = kBar + kNumBars * 8 + 16;
};

template <int D, int DV, int kPolyEvery, bool RULE, int DR = 0, bool LOG = false>
__global__ void __launch_bounds__(kF2Threads, 1)
attn_fwd2_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                 const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmQr,
                 const __grid_constant__ CUtensorMap tmKr, F2Params p, unsigned int* status) {
  using L = F2Smem<D + DR, DV>;
  constexpr int kStages = L::kStages, kVStages = L::kVStages;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sbase = smem_u32(smem);
  const uint32_t sQ = sbase + L::kQ, sK = sbase + L::kK, sV = sbase + L::kV;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kBar);
  const uint32_t b0 = smem_u32(bars);
  const uint32_t bar_q = b0;                                   // [2]
  const uint32_t bar_kfull = b0 + 16;                          // [kStages]
  const uint32_t bar_kempty = bar_kfull + 8 * kStages;
  const uint32_t bar_vfull = bar_kempty + 8 * kStages;         // [kVStages]
  const uint32_t bar_vempty = bar_vfull + 8 * kVStages;
  const uint32_t bar_sfull = bar_vempty + 8 * kVStages;        // [2]
  const uint32_t bar_pfull = bar_sfull + 16;                   // [2]
  const uint32_t bar_oready = bar_pfull + 16;                  // [2]
  uint32_t* tmem_ptr_smem = reinterpret_cast<uint32_t*>(bars + L::kNumBars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr_smem + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int m_blk = gridDim.x - 1 - blockIdx.x;                // long causal rows first
  const int h = blockIdx.y, b = blockIdx.z;
  const int hk = h / (p.heads / p.kv_heads);
  const int q0 = m_blk * 2 * kF2Tile;
  const int shift = p.seq_k - p.seq_q;
  // keys at positions >= kv_len are padding: never visible, and key blocks that hold only padding are skipped
  const int kv_len = p.kv_lens ? max(0, min(p.seq_k, p.kv_lens[b])) : p.seq_k;
  const int n_all = (kv_len + kF2Tile - 1) / kF2Tile;
  // key blocks seen by tile A and by tile B (0: the tile starts beyond the last query)
  auto blocks_of = [&](int qt) {
    int n = qt < p.seq_q ? n_all : 0;
    if (n > 0 && p.causal) {
      const int lim = (qt + kF2Tile - 1 + shift) / kF2Tile + 1;
      if (lim < n) n = lim;
    }
    return n;
  };
  int n_a = blocks_of(q0), n_b = blocks_of(q0 + kF2Tile);
  // first key block of each tile: the one that holds the first key its first row sees.  Tile A starts first, and tile B
  // starts no later than one block after tile A's last.
  auto first_of = [&](int t) {
    const int pos = q0 + t * kF2Tile + shift;
    if (RULE && p.chunk > 0) return pos / p.chunk * p.chunk / kF2Tile;
    if (RULE && p.window > 0) return max(0, pos - p.window + 1) / kF2Tile;
    return 0;
  };
  int f_a = first_of(0), f_b = first_of(1);
  // Kept first keys: both tiles walk their blocks (kept_blocks of them) before those of tile A's window, and the counters below
  // number the blocks in that order; block_at gives the key block.
  int kept_blocks = 0, skipped = 0;
  if (RULE && p.window > 0 && p.keep > 0 && n_a > 0) {
    kept_blocks = (p.keep + kF2Tile - 1) / kF2Tile;
    skipped = max(0, f_a - kept_blocks);
    n_a -= skipped;
    n_b = max(0, n_b - skipped);
    f_a = f_b = 0;
  }
  auto block_at = [&](int j) { return RULE && j >= kept_blocks ? j + skipped : j; };
  auto n_of = [&](int t) { return t == 0 ? n_a : n_b; };
  const int n_max = n_a > n_b ? n_a : n_b;
  auto f_of = [&](int t) { return t == 0 ? f_a : f_b; };
  const int f_min = n_a > 0 ? f_a : f_b;
  constexpr uint32_t kTmemCols = 512;

  if (threadIdx.x == 0) {
    for (int t = 0; t < 2; ++t) {
      mbar_init(bar_q + 8 * t, 1);
      mbar_init(bar_sfull + 8 * t, 1);
      mbar_init(bar_pfull + 8 * t, 4);
      mbar_init(bar_oready + 8 * t, 1);
    }
    for (int s = 0; s < kStages; ++s) {
      mbar_init(bar_kfull + 8 * s, 1);
      mbar_init(bar_kempty + 8 * s, 1);
    }
    for (int s = 0; s < kVStages; ++s) {
      mbar_init(bar_vfull + 8 * s, 1);
      mbar_init(bar_vempty + 8 * s, 1);
    }
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 9) {
    tmem_alloc(smem_u32(tmem_ptr_smem), kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr_smem;

  if (warp >= 8) {
  setmaxnreg_dec<56>();
  if (warp == 8) {
    if (elect_one()) {
      // ---------------------------------------------------------------- TMA producer
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        if (n_of(t) == 0) continue;
        mbar_arrive_expect_tx(bar_q + 8 * t, L::kTileBytes);
#pragma unroll
        for (int hf = 0; hf < D / 64; ++hf)
          tma_load_4d(sQ + t * L::kTileBytes + hf * L::kHalf, &tmQ, hf * 64, h, q0 + t * kF2Tile, b, bar_q + 8 * t);
        if (DR > 0)
          tma_load_4d(sQ + t * L::kTileBytes + (D / 64) * L::kHalf, &tmQr, 0, h, q0 + t * kF2Tile, b, bar_q + 8 * t);
      }
      for (int j = f_min; j < n_max; ++j) {
        const int s = (j - f_min) % kStages, use = (j - f_min) / kStages;
        if (!mbar_wait(bar_kempty + 8 * s, (use & 1) ^ 1, abort_flag, status, 41)) break;
        mbar_arrive_expect_tx(bar_kfull + 8 * s, L::kTileBytes);
#pragma unroll
        for (int hf = 0; hf < D / 64; ++hf)
          tma_load_4d(sK + s * L::kTileBytes + hf * L::kHalf, &tmK, hf * 64, hk, block_at(j) * kF2Tile, b, bar_kfull + 8 * s);
        if (DR > 0)
          tma_load_4d(sK + s * L::kTileBytes + (D / 64) * L::kHalf, &tmKr, 0, 0, block_at(j) * kF2Tile, b, bar_kfull + 8 * s);
        const int v = (j - f_min) % kVStages, vuse = (j - f_min) / kVStages;
        if (!mbar_wait(bar_vempty + 8 * v, (vuse & 1) ^ 1, abort_flag, status, 49)) break;
        mbar_arrive_expect_tx(bar_vfull + 8 * v, L::kVTileBytes);
#pragma unroll
        for (int hf = 0; hf < DV / 64; ++hf)
          tma_load_4d(sV + v * L::kVTileBytes + hf * L::kHalf, &tmV, hf * 64, hk, block_at(j) * kF2Tile, b, bar_vfull + 8 * v);
      }
    }
  } else if (warp == 9) {
    // elect_one, not lane 0: the compiler then knows that one lane runs this and keeps the descriptors in uniform registers
    if (elect_one()) {
      // ---------------------------------------------------------------- MMA issuer
      // descriptors of the first tile and stage; an offset of o bytes is o / 16 in the address field
      const uint64_t dQ = umma_smem_desc_sw128(sQ, 16, 1024), dK = umma_smem_desc_sw128(sK, 16, 1024), dV = umma_smem_desc_sw128(sV, L::kHalf, 1024);
      constexpr uint32_t idesc_qk = umma_idesc_bf16(128, 128, 0, 0);
      constexpr uint32_t idesc_pv = umma_idesc_bf16(128, DV, 0, 1);        // A = P (TMEM, K-major), B = V MN-major
      auto issue_qk = [&](int j, int t) -> bool {
        const int s = (j - f_min) % kStages;
        if (!mbar_wait(bar_kfull + 8 * s, ((j - f_min) / kStages) & 1, abort_flag, status, 42)) return false;
        tc_fence_after();
        uint64_t q = dQ + t * (L::kTileBytes / 16), k = dK + s * (L::kTileBytes / 16);
        asm volatile("" : "+l"(q), "+l"(k));                  // keeps the sums below from being formed ahead of the loop and spilled
#pragma unroll
        for (int ks = 0; ks < (D + DR) / 16; ++ks) {
          if (RULE && ks < D / 16 && ks * 16 >= p.dk) continue;            // the rest of the columns is zero
          if (DR > 0 && ks >= D / 16 && (ks - D / 16) * 16 >= p.dr) continue;
          const uint64_t off = (ks >> 2) * (L::kHalf / 16) + (ks & 3) * 2;
          umma_bf16_ss(tmem_base + t * 128, q + off, k + off, idesc_qk, ks != 0 ? 1u : 0u);
        }
        umma_commit(bar_sfull + 8 * t);
        return true;
      };
      bool ok = true;
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        if (n_of(t) == 0 || !ok) continue;
        ok = mbar_wait(bar_q + 8 * t, 0, abort_flag, status, 43);
        if (ok && f_of(t) == f_min) ok = issue_qk(f_min, t);  // a tile that starts later gets its first product below
      }
      if (ok && f_min < n_max) umma_commit(bar_kempty);                          // the first key block: every product that reads it has been issued
      for (int j = f_min; j < n_max && ok; ++j) {
        const int v = (j - f_min) % kVStages;
        if (!mbar_wait(bar_vfull + 8 * v, ((j - f_min) / kVStages) & 1, abort_flag, status, 44)) break;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          if (j >= n_of(t) || !ok) continue;
          if (j < f_of(t)) {
            if (j + 1 == f_of(t)) ok = issue_qk(j + 1, t);
            continue;
          }
          if (!mbar_wait(bar_pfull + 8 * t, (j - f_of(t)) & 1, abort_flag, status, 45)) { ok = false; break; }
          tc_fence_after();
          const uint32_t tmem_p = tmem_base + t * 128;              // packed bf16 pairs: 8 columns per 16 keys
          const uint32_t tmem_o = tmem_base + 256 + t * 128;
          uint64_t dv = dV + v * (L::kVTileBytes / 16);
          asm volatile("" : "+l"(dv));
#pragma unroll
          for (int ks = 0; ks < kF2Tile / 16; ++ks) {
            // V: 16 key rows of 128 B per step; 64-wide head-dim atoms L::kHalf apart
            umma_bf16_ts(tmem_o, tmem_p + ks * 8, dv + ks * (2048 / 16), idesc_pv, (j > f_of(t) || ks != 0) ? 1u : 0u);
          }
          umma_commit(bar_oready + 8 * t);
          if (j + 1 < n_of(t)) ok = issue_qk(j + 1, t);          // overwrites S_t / P_t: ordered behind PV(j, t)
        }
        if (!ok) break;
        umma_commit(bar_vempty + 8 * v);                        // every MMA that reads this V stage, and the next K stage, is issued
        if (j + 1 < n_max) umma_commit(bar_kempty + 8 * ((j + 1 - f_min) % kStages));
      }
    }
  }
  } else {
    setmaxnreg_inc<224>();
    // ------------------------------------------------------------------ softmax + epilogue, one query row per thread
    const int t = warp >> 2;                                   // query tile of this warp group
    const int wq = warp & 3;                                   // TMEM lane quarter of this warp
    const int row = wq * 32 + lane;
    const int q_idx = q0 + t * kF2Tile + row;
    const uint32_t lane_off = static_cast<uint32_t>(wq * 32) << 16;
    const uint32_t tmem_s = tmem_base + t * 128 + lane_off;
    const uint32_t tmem_o = tmem_base + 256 + t * 128 + lane_off;
    // RULE: scores with a cap or a bias are turned into log2 units when they are read, so the softmax runs with scale 1
    const bool shaped = RULE && (LOG || p.softcap > 0.f || p.slopes != nullptr);
    const float sl2 = shaped ? 1.f : p.scale * kF2Log2e;
    const float rule_c1 = RULE && p.softcap > 0.f ? p.scale / p.softcap : 0.f;
    const float rule_c2 = RULE ? (p.softcap > 0.f ? p.softcap : p.scale) * kF2Log2e : 0.f;
    const float slope2 = RULE && p.slopes ? p.slopes[h] * kF2Log2e : 0.f;
    const float log_amount = LOG ? p.log_amount[h] : 0.f, log_rate = LOG ? p.log_rate[h] : 0.f;
    // first visible key of this row, apart from the kept ones below key_keep
    const int key_lo = !RULE ? 0 : p.chunk > 0 ? (q_idx + shift) / p.chunk * p.chunk : p.window > 0 ? q_idx + shift - p.window + 1 : 0;
    const int key_keep = RULE && p.window > 0 ? p.keep : 0;
    F2Cap cap = {};
    if (RULE) cap.init(rule_c1, rule_c2);
    // a sink is a score 0 met before all keys
    float m_run = RULE && p.sink ? 0.f : -INFINITY, l_run = RULE && p.sink ? 1.f : 0.f;
    const int nt = n_of(t), ft = f_of(t);
    bool ok = true;
    for (int j = ft; j < nt && ok; ++j) {
      if (!mbar_wait(bar_sfull + 8 * t, (j - ft) & 1, abort_flag, status, 46)) { ok = false; break; }
      tc_fence_after();
      const int k0 = block_at(j) * kF2Tile;
      const int key_lim = p.causal ? min(kv_len - 1, q_idx + shift) : kv_len - 1;     // last visible key
      const bool need_mask = (k0 + kF2Tile - 1 > key_lim);
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
      // maximum over 32 scores (masked keys have been set to -inf)
      auto chunk_max = [&](const uint32_t* v) {
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          mx0 = fmaxf(mx0, __uint_as_float(v[i]));
          mx1 = fmaxf(mx1, __uint_as_float(v[i + 1]));
          mx2 = fmaxf(mx2, __uint_as_float(v[i + 2]));
          mx3 = fmaxf(mx3, __uint_as_float(v[i + 3]));
        }
      };
      // the whole row of 128 scores is read from TMEM once and stays in registers (224 per thread after the
      // reallocation above)
      uint32_t r[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32_ptr(tmem_s + c * 32, r + c * 32);
      tmem_ld_wait();
      if (RULE) {
        // cap * tanh(s / cap), then - slope * (query - key)
        const float bias0 = -slope2 * static_cast<float>(q_idx + shift - k0);
        if (p.softcap > 0.f) {
          const uint32_t any = f2_cap_scores(r, cap, slope2, bias0);
          if (__any_sync(0xffffffffu, (any & 0x40000000u) != 0u)) {     // the raw scores are still in TMEM
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_ld_32x32_ptr(tmem_s + c * 32, r + c * 32);
            tmem_ld_wait();
            f2_cap_scores_wide(r, rule_c1, rule_c2, slope2, bias0);
          }
        } else if (LOG ? p.slopes != nullptr : shaped) {
#pragma unroll
          for (int i = 0; i < 128; ++i)
            r[i] = __float_as_uint(fmaf(__uint_as_float(r[i]), rule_c2, fmaf(slope2, static_cast<float>(i), bias0)));
        }
        if (LOG) {
          const float nearest = static_cast<float>(q_idx - lane + shift - k0) - 63.5f;       // of the warp's first row, to the middle key
          f2_log_bias(r, p.softcap > 0.f || p.slopes != nullptr ? 1.f : rule_c2, log_amount, log_rate, static_cast<float>(q_idx + shift - k0),
                      log_rate * 63.5f <= 0.125f * fmaf(log_rate, nearest, 1.f));
        }
        if (k0 < key_lo) {
#pragma unroll
          for (int i = 0; i < 128; ++i)
            if (k0 + i < key_lo && k0 + i >= key_keep) r[i] = 0xff800000u;
        }
      }
      if (need_mask) {                               // only blocks that cross the causal diagonal or the end of the keys
#pragma unroll
        for (int i = 0; i < 128; ++i)
          if (k0 + i > key_lim) r[i] = 0xff800000u;   // -inf: ignored by the maximum, exp2 gives exactly 0
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) chunk_max(r + c * 32);
      const float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3));
      // Keep the old maximum unless the new one is more than 2^threshold larger: exponentials stay <= 2^threshold.
      const bool grow = (mx > m_run) && ((mx - m_run) * sl2 > kF2RescaleThreshold || m_run == -INFINITY);
      float alpha = 1.f;
      if (grow) {
        alpha = (m_run == -INFINITY) ? 0.f : f2_ex2((m_run - mx) * sl2);
        m_run = mx;
        l_run *= alpha;
      }
      if (j > ft && __any_sync(0xffffffffu, grow)) {
        // O_t holds the sum over blocks 0..j-1 once PV(j-1, t) has completed; PV(j, t) cannot start before P below.
        if (!mbar_wait(bar_oready + 8 * t, (j - 1 - ft) & 1, abort_flag, status, 47)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < DV / 32; ++c) {
          uint32_t o[32];
          tmem_ld_32x32_ptr(tmem_o + c * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
          tmem_st_32x32(tmem_o + c * 32, o);
        }
        tmem_st_wait();
      }
      const float msc = (m_run == -INFINITY ? 0.f : m_run) * sl2;
      float rs0 = 0.f, rs1 = 0.f;
      constexpr int kDiv = kPolyEvery > 0 ? kPolyEvery : 1;
      // 32 scores starting at key kb -> probabilities, 16 packed bf16 pairs (chunk index c selects the polynomial share)
      auto chunk_exp = [&](const uint32_t* v, int kb, int c, uint32_t* packed) {
#pragma unroll
        for (int ii = 0; ii < 16; ++ii) {
          const int i = c * 16 + ii;
          const float x0 = fmaf(__uint_as_float(v[2 * ii]), sl2, -msc);
          const float x1 = fmaf(__uint_as_float(v[2 * ii + 1]), sl2, -msc);
          float p0, p1;
          if (kPolyEvery > 0 && (i % kDiv) == kDiv - 1) {
            p0 = f2_ex2_poly(x0);
            p1 = f2_ex2_poly(x1);
          } else {
            p0 = f2_ex2(x0);
            p1 = f2_ex2(x1);
          }
          if (kPolyEvery > 0 && need_mask) {           // the polynomial clamps its argument: zero masked keys explicitly
            if (kb + 2 * ii > key_lim) p0 = 0.f;
            if (kb + 2 * ii + 1 > key_lim) p1 = 0.f;
          }
          rs0 += p0;
          rs1 += p1;
          packed[ii] = pack_bf16x2(p0, p1);
        }
      };
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t packed[16];
        chunk_exp(r + c * 32, k0 + c * 32, c, packed);
        // columns [16c, 16c + 16) of the score buffer: every score is already in registers
        tmem_st_32x16(tmem_s + c * 16, packed);
      }
      l_run += rs0 + rs1;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_pfull + 8 * t);
    }
    uint4 gate_row[RULE ? DV / 8 : 1];                         // the gate of this row, requested while the last product runs
    const bool gated = RULE && p.gate != nullptr && q_idx < p.seq_q;
    if (gated) {
#pragma unroll
      for (int c = 0; c < DV / 8; ++c)
        if (c * 8 < p.dv) gate_row[c % (RULE ? DV / 8 : 1)] = *reinterpret_cast<const uint4*>(p.gate + q_idx * p.ld_gate + h * p.dv + c * 8);
    }
    if (ok && nt > 0) ok = mbar_wait(bar_oready + 8 * t, (nt - 1 - ft) & 1, abort_flag, status, 48);
    if (nt == 0 && q_idx < p.seq_q && q0 + t * kF2Tile < p.seq_q) {
      // no visible key at all (every key of this batch entry is padding): the output row is zero
      __nv_bfloat16* op = p.out + b * p.o_bs + h * p.o_hs + static_cast<long long>(q_idx) * p.o_rs;
#pragma unroll
      for (int c = 0; c < DV / 8; ++c)
        if (!RULE || c * 8 < p.dv) reinterpret_cast<uint4*>(op)[c] = make_uint4(0u, 0u, 0u, 0u);
      if (p.lse != nullptr) p.lse[(static_cast<long long>(b) * p.heads + h) * p.seq_q + q_idx] = 0.f;
    }
    if (ok && nt > 0) {
      tc_fence_after();
      float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      if (RULE) inv *= p.out_scale;
      if (RULE && p.head_gate != nullptr && q_idx < p.seq_q)
        inv *= f2_rcp(1.f + f2_ex2(-p.head_gate[q_idx * p.ld_gate + h] * kF2Log2e));
      __nv_bfloat16* op = p.out + b * p.o_bs + h * p.o_hs + static_cast<long long>(q_idx) * p.o_rs;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32_ptr(tmem_o + c * 32, o);
        tmem_ld_wait();
        if (q_idx < p.seq_q) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            if (RULE && c * 32 + g * 8 >= p.dv) break;
            if (gated) {
              const uint4 gv = gate_row[(c * 4 + g) % (RULE ? DV / 8 : 1)];
              const uint32_t gw[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float2 f = unpack_bf16x2(gw[i]);
                o[g * 8 + 2 * i] = __float_as_uint(__uint_as_float(o[g * 8 + 2 * i]) * f2_rcp(1.f + f2_ex2(-f.x * kF2Log2e)));
                o[g * 8 + 2 * i + 1] = __float_as_uint(__uint_as_float(o[g * 8 + 2 * i + 1]) * f2_rcp(1.f + f2_ex2(-f.y * kF2Log2e)));
              }
            }
            uint4 v;
            v.x = pack_bf16x2(__uint_as_float(o[g * 8 + 0]) * inv, __uint_as_float(o[g * 8 + 1]) * inv);
            v.y = pack_bf16x2(__uint_as_float(o[g * 8 + 2]) * inv, __uint_as_float(o[g * 8 + 3]) * inv);
            v.z = pack_bf16x2(__uint_as_float(o[g * 8 + 4]) * inv, __uint_as_float(o[g * 8 + 5]) * inv);
            v.w = pack_bf16x2(__uint_as_float(o[g * 8 + 6]) * inv, __uint_as_float(o[g * 8 + 7]) * inv);
            reinterpret_cast<uint4*>(op)[c * 4 + g] = v;
          }
        }
      }
      if (p.lse != nullptr && q_idx < p.seq_q)
        p.lse[(static_cast<long long>(b) * p.heads + h) * p.seq_q + q_idx] =
            (m_run == -INFINITY ? 0.f : m_run) * p.scale + logf(fmaxf(l_run, 1e-30f));
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    if (*abort_flag) {
      // a wait gave up: let copies and MMAs in flight land before the accumulators are released
      const unsigned long long t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

}  // namespace rb

namespace {
const CUtensorMap* f2_make_map(const void* base, const long long* strides, int seq, int heads, int batch, int D, int* err) {
  // dims innermost first: (d, head, seq, batch); strides in bytes for head, seq, batch
  const uint64_t dims[4] = {(uint64_t)D, (uint64_t)heads, (uint64_t)seq, (uint64_t)batch};
  const uint64_t str[3] = {(uint64_t)strides[2] * 2, (uint64_t)strides[1] * 2, (uint64_t)strides[0] * 2};
  const uint32_t box[4] = {64, 1, (uint32_t)rb::kF2Tile, 1};
  return rbhost::get_tmap_4d(base, 2, dims, str, box, 1, err);
}

template <int D, int DV, int P, bool RULE, int DR = 0, bool LOG = false>
int f2_launch(const CUtensorMap* tq, const CUtensorMap* tk, const CUtensorMap* tv, const rb::F2Params& p, dim3 grid,
              cudaStream_t stream, const CUtensorMap* tqr = nullptr, const CUtensorMap* tkr = nullptr) {
  auto kern = rb::attn_fwd2_kernel<D, DV, P, RULE, DR, LOG>;
  const int smem = rb::F2Smem<D + DR, DV>::kTotal + 1024;
  static bool cfg_dev[64] = {false};
  bool& cfg = cfg_dev[rbhost::device_slot()];
  if (!cfg) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  kern<<<grid, rb::kF2Threads, smem, stream>>>(*tq, *tk, *tv, tqr ? *tqr : *tq, tkr ? *tkr : *tk, p, rbhost::status_ptr());
  return static_cast<int>(cudaGetLastError());
}
}  // namespace

// Forward pass with two query tiles per CTA.  `poly_every`: 0 = every exponential on the special-function unit,
// 4 = every fourth pair of keys on the FMA-pipe polynomial (measured slower on B200 at both head dims: 218 us against
// 191 us for batch 32 x 12 heads x 1024 x 64; kept for parts whose special-function unit is the limit).  Returns -9 for problems this kernel does not
// take (the caller then uses another forward kernel).
RB_API int rb_attention_fwd_tc2(const RbAttnArgs* a, int poly_every, void* stream_v) {
  if (a->batch <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (a->head_dim != 64 && a->head_dim != 128) return -9;
  if (a->seq_q <= 0 || a->seq_k <= 0 || (a->causal && a->seq_q > a->seq_k)) return -1;
  const void* ptrs[4] = {a->q, a->k, a->v, a->o};
  for (int i = 0; i < 4; ++i)
    if (!ptrs[i] || (reinterpret_cast<uintptr_t>(ptrs[i]) & 15)) return -9;
  const long long* strs[4] = {a->q_strides, a->k_strides, a->v_strides, a->o_strides};
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 3; ++j)
      if (strs[i][j] % 8) return -9;            // TMA strides are multiples of 16 bytes
  auto fix = [](const long long* s, long long* out, int D) {
    out[0] = s[0] > 0 ? s[0] : 8; out[1] = s[1] > 0 ? s[1] : D; out[2] = s[2] > 0 ? s[2] : D;
  };
  long long qs[3], ks[3], vs[3];
  fix(a->q_strides, qs, a->head_dim); fix(a->k_strides, ks, a->head_dim); fix(a->v_strides, vs, a->head_dim);
  int err = 0;
  const CUtensorMap* tq = f2_make_map(a->q, qs, a->seq_q, a->heads, a->batch, a->head_dim, &err);
  const CUtensorMap* tk = f2_make_map(a->k, ks, a->seq_k, a->kv_heads, a->batch, a->head_dim, &err);
  const CUtensorMap* tv = f2_make_map(a->v, vs, a->seq_k, a->kv_heads, a->batch, a->head_dim, &err);
  if (!tq || !tk || !tv) return err ? err : -5;
  rb::F2Params p = {};
  p.out = reinterpret_cast<__nv_bfloat16*>(a->o);
  p.lse = a->lse;
  p.o_bs = a->o_strides[0]; p.o_rs = a->o_strides[1]; p.o_hs = a->o_strides[2];
  p.seq_q = a->seq_q; p.seq_k = a->seq_k; p.heads = a->heads; p.kv_heads = a->kv_heads; p.causal = a->causal;
  p.scale = a->scale;
  p.kv_lens = a->kv_lens;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_v);
  dim3 grid((a->seq_q + 2 * rb::kF2Tile - 1) / (2 * rb::kF2Tile), a->heads, a->batch);
  if (a->head_dim == 64) {
    switch (poly_every) {
      case 0: return f2_launch<64, 64, 0, false>(tq, tk, tv, p, grid, stream);
      case 4: return f2_launch<64, 64, 4, false>(tq, tk, tv, p, grid, stream);
      default: return -1;
    }
  }
  switch (poly_every) {
    case 0: return f2_launch<128, 128, 0, false>(tq, tk, tv, p, grid, stream);
    case 4: return f2_launch<128, 128, 4, false>(tq, tk, tv, p, grid, stream);
    default: return -1;
  }
}

// Causal forward with a score rule (see attention.h).  Returns -9 for operands this kernel does not take.
RB_API int rb_attention_fwd_rule(const RbAttnArgs* a, const RbAttnRule* r, void* stream_v) {
  const int dk = a->head_dim, dv = r->v_dim;
  if (a->batch <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (dk <= 0 || dv <= 0 || dk > 128 || dv > 128 || ((dk | dv) & 7)) return -9;
  if (!a->causal || a->seq_q <= 0 || a->seq_k < a->seq_q || r->chunk < 0 || r->window < 0 || r->keep_first < 0 || (r->window && r->chunk) ||
      !r->log_amount != !r->log_rate || ((r->gate || r->head_gate) && a->batch != 1) || (r->gate && r->head_gate))
    return -1;
  const void* ptrs[5] = {a->q, a->k, a->v, a->o, r->gate};
  for (int i = 0; i < 5; ++i)
    if ((!ptrs[i] && i < 4) || (reinterpret_cast<uintptr_t>(ptrs[i]) & 15)) return -9;
  const long long* strs[4] = {a->q_strides, a->k_strides, a->v_strides, a->o_strides};
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 3; ++j)
      if (strs[i][j] % 8 || strs[i][j] <= 0) return -9;            // TMA strides are multiples of 16 bytes
  if (r->gate && r->ld_gate % 8) return -9;
  const int dr = r->rot_dim;
  if (dr) {
    if (dr < 0 || a->batch != 1 || !r->k_rot || r->softcap > 0.f || r->slopes || r->log_rate || r->window || r->chunk) return -1;
    if (dr > 64 || (dr & 7) || r->ld_k_rot % 8 || r->ld_k_rot < dr || (reinterpret_cast<uintptr_t>(r->k_rot) & 15)) return -9;
  }
  int err = 0;
  const CUtensorMap* tq = f2_make_map(a->q, a->q_strides, a->seq_q, a->heads, a->batch, dk, &err);
  const CUtensorMap* tk = f2_make_map(a->k, a->k_strides, a->seq_k, a->kv_heads, a->batch, dk, &err);
  const CUtensorMap* tv = f2_make_map(a->v, a->v_strides, a->seq_k, a->kv_heads, a->batch, dv, &err);
  if (!tq || !tk || !tv) return err ? err : -5;
  rb::F2Params p = {};
  p.out = reinterpret_cast<__nv_bfloat16*>(a->o);
  p.o_bs = a->o_strides[0]; p.o_rs = a->o_strides[1]; p.o_hs = a->o_strides[2];
  p.seq_q = a->seq_q; p.seq_k = a->seq_k; p.heads = a->heads; p.kv_heads = a->kv_heads; p.causal = 1;
  p.scale = a->scale;
  p.dk = dk; p.dv = dv; p.softcap = r->softcap; p.slopes = r->slopes; p.chunk = r->chunk;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(r->gate); p.ld_gate = r->ld_gate;
  p.dr = dr; p.head_gate = r->head_gate; p.window = r->window; p.keep = r->window > 0 ? r->keep_first : 0; p.sink = r->sink;
  p.log_amount = r->log_amount; p.log_rate = r->log_rate; p.out_scale = r->out_scale;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_v);
  const dim3 grid((a->seq_q + 2 * rb::kF2Tile - 1) / (2 * rb::kF2Tile), a->heads, a->batch);
  if (dr) {
    const long long qr_s[3] = {a->q_strides[0], a->q_strides[1], a->q_strides[2]};
    const long long kr_s[3] = {r->ld_k_rot * a->seq_k, r->ld_k_rot, r->ld_k_rot};
    const CUtensorMap* tqr = f2_make_map(reinterpret_cast<const __nv_bfloat16*>(a->q) + dk, qr_s, a->seq_q, a->heads, 1, dr, &err);
    const CUtensorMap* tkr = f2_make_map(r->k_rot, kr_s, a->seq_k, 1, 1, dr, &err);
    if (!tqr || !tkr) return err ? err : -5;
    if (dk <= 64)
      return dv <= 64 ? f2_launch<64, 64, 0, true, 64>(tq, tk, tv, p, grid, stream, tqr, tkr)
                      : f2_launch<64, 128, 0, true, 64>(tq, tk, tv, p, grid, stream, tqr, tkr);
    return dv <= 64 ? f2_launch<128, 64, 0, true, 64>(tq, tk, tv, p, grid, stream, tqr, tkr)
                    : f2_launch<128, 128, 0, true, 64>(tq, tk, tv, p, grid, stream, tqr, tkr);
  }
  if (r->log_rate) {
    if (dk <= 64)
      return dv <= 64 ? f2_launch<64, 64, 0, true, 0, true>(tq, tk, tv, p, grid, stream)
                      : f2_launch<64, 128, 0, true, 0, true>(tq, tk, tv, p, grid, stream);
    return dv <= 64 ? f2_launch<128, 64, 0, true, 0, true>(tq, tk, tv, p, grid, stream)
                    : f2_launch<128, 128, 0, true, 0, true>(tq, tk, tv, p, grid, stream);
  }
  if (dk <= 64)
    return dv <= 64 ? f2_launch<64, 64, 0, true>(tq, tk, tv, p, grid, stream) : f2_launch<64, 128, 0, true>(tq, tk, tv, p, grid, stream);
  return dv <= 64 ? f2_launch<128, 64, 0, true>(tq, tk, tv, p, grid, stream) : f2_launch<128, 128, 0, true>(tq, tk, tv, p, grid, stream);
}
