// Gated delta rule over prompts, chunked: 64 tokens at a time become matrix products on the tensor cores.
//
// With c_t the running sum of the logarithms of the decays inside a chunk, k and q unit vectors (q scaled) and S0 the state in
// front of it, the corrections u_t = beta_t (v_t - decay_t S_{t-1}^T k_t) of a chunk solve a unit lower triangular system
//   (I + L) U = R,  L_ts = beta_t exp(c_t - c_s) (k_t . k_s) for s < t,  R_t = beta_t (v_t - exp(c_t) S0^T k_t)
// and then
//   o_t = exp(c_t) S0^T q_t + sum_{s <= t} exp(c_t - c_s) (q_t . k_s) u_s,   S = exp(c_end) S0 + sum_s exp(c_end - c_s) k_s u_s^T
// (the WY form of products of Householder-like matrices; Yang et al., "Gated Delta Networks: Improving Mamba2 with Delta Rule").
//
// With T = (I + L)^-1, A the masked products exp(c_t - c_s) (q_t . k_s) and U = T R, nothing but R is needed of a chunk once S0 is
// known: o = exp(c) S0^T q + (A T) R and S = exp(c_end) S0 + W^T R with W = T^T diag(exp(c_end - c)) K.  (A T also has none of the
// cancellation between A and U when keys are much alike.)
//
// Two kernels.  The first works on all chunks of all sequences at once: A T, W and the per-token factors.  The second walks a
// sequence's chunks in order, one CTA (8 warps) per head and value columns, with the state in fp32 accumulator registers.  Queries
// and keys enter the products as the bf16 numbers the convolution left; their norms, the decays and beta are fp32 factors outside.
// R, W, the state and what is added to it are split into two bf16 numbers (about 16 bits).
#include "recurrent.h"

#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace rb {

constexpr int kDcChunk = 64;
constexpr float kDcUnitEps = 1e-6f;
constexpr float kDcLog2e = 1.4426950408889634f;

// scratch of one (chunk, head), rows padded as the second kernel wants them in shared memory (it fetches the block as a whole):
// A T (bf16 [64][72]), W (bf16 [64][DK + 8], high and low half), then fp32 factors
constexpr int kDcMPitch = kDcChunk + 8;
constexpr int kDcMat = kDcChunk * kDcMPitch * 2;
constexpr int kDcFactors = 4;              // [64] each: beta, key read-out, query read-out, and one with exp(c_end) in [0]
__host__ __device__ constexpr int dc_half(int DK) { return kDcChunk * (DK + 8) * 2; }
__host__ __device__ constexpr int dc_scratch(int DK) { return kDcMat + 2 * dc_half(DK) + kDcFactors * kDcChunk * 4; }

// ---- first kernel: one CTA (8 warps) per chunk and head
constexpr int kDpThreads = 256;
template <int DK>
struct DcPrepSmem {
  static constexpr int kPitch = DK + 8, kLPitch = kDcChunk + 4;
  static constexpr int kQ = 0;
  static constexpr int kK = kQ + kDcChunk * kPitch * 2;
  static constexpr int kTPitch = kDcChunk + 8;
  static constexpr int kL = kK + kDcChunk * kPitch * 2;              // fp32 [64][68]: L; later T as bf16 [2][64][72]
  static constexpr int kT = kL + 2 * kDcChunk * kTPitch * 2;         // fp32 [64][68]
  static constexpr int kW = kT + kDcChunk * kLPitch * 4;             // fp32 [48][20] products of blocks
  static constexpr int kF = kW + 48 * 20 * 4;                        // fp32 [4][64]: c, beta, 1 / |k|, scale / |q|
  static constexpr int kTotal = kF + 4 * kDcChunk * 4;
  // W is staged before it leaves: the high half over the queries, the low half over T
  static_assert(kDcChunk * kPitch * 2 <= kW - kT, "staging of the low half");
};

template <int DK>
__global__ void __launch_bounds__(kDpThreads, 3)
delta_rule_prepare_kernel(const RbDeltaRuleArgs a) {
  using L = DcPrepSmem<DK>;
  constexpr int P = L::kPitch, LP = L::kLPitch;
  extern __shared__ __align__(16) uint8_t dp_smem[];
  const uint32_t sQ = smem_u32(dp_smem) + L::kQ, sK = smem_u32(dp_smem) + L::kK;
  float* Lm = reinterpret_cast<float*>(dp_smem + L::kL);
  float* T = reinterpret_cast<float*>(dp_smem + L::kT);
  float* W = reinterpret_cast<float*>(dp_smem + L::kW);
  float* cum = reinterpret_cast<float*>(dp_smem + L::kF);
  float *beta = cum + kDcChunk, *rk = beta + kDcChunk, *rq = rk + kDcChunk;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3;
  const int wr = warp & 3, side = warp >> 2;       // rows wr 16 .. + 16 of the products k . k (side 0) or q . k (side 1)
  const int h = blockIdx.x, tile = blockIdx.y;
  const RcSegment seg = rc_segment(a.segments, a.tiles[2 * tile], a.num_slots);
  const int off = a.tiles[2 * tile + 1];
  if (off >= seg.len) return;
  const int m_rows = min(kDcChunk, seg.len - off);
  const int g = h / (a.heads / a.kv_heads);
  const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(a.qkv) + static_cast<long long>(seg.first + off) * a.ld_qkv;
  const long long offQ = static_cast<long long>(g) * a.dk, offK = static_cast<long long>(a.kv_heads + g) * a.dk;
  for (int i = tid; i < kDcChunk * (DK / 8); i += kDpThreads) {
    const int r = i / (DK / 8), c = (i - r * (DK / 8)) * 8;
    const bool ok = r < m_rows && c < a.dk;
    const __nv_bfloat16* src = rows + (ok ? r * a.ld_qkv + c : 0);
    wm_cp16(sQ + (r * P + c) * 2, ok ? src + offQ : rows, ok);
    wm_cp16(sK + (r * P + c) * 2, ok ? src + offK : rows, ok);
  }
  wm_cp_commit();
  if (warp == 0) {                                 // beta and running log2 decays, two tokens per lane
    const float rate2 = expf(a.a_log[h]) * kDcLog2e, dt_bias = a.dt_bias[h];
    float s[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 2 * lane + i;
      const long long at = static_cast<long long>(seg.first + off + t) * a.ld_ab + h;
      beta[t] = t < m_rows ? rc_sigmoid(a.b_raw[at]) : 0.f;
      s[i] = t < m_rows ? -rate2 * rc_softplus(a.a_raw[at] + dt_bias) : 0.f;
    }
    float run = s[0] + s[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += u;
    }
    cum[2 * lane] = run - s[1];
    cum[2 * lane + 1] = run;
  }
  for (int i = tid; i < kDcChunk * LP; i += kDpThreads) T[i] = 0.f;
  wm_cp_wait<0>();
  __syncthreads();
  {                                                // norms: two threads per row of either
    const int r = (tid & 127) >> 1, half = tid & 1;
    const __nv_bfloat16* row = reinterpret_cast<const __nv_bfloat16*>(dp_smem + (tid < 128 ? L::kQ : L::kK)) + r * P + half * (DK / 2);
    float s = 0.f;
#pragma unroll 4
    for (int c = 0; c < DK / 2; c += 8) {
      float v[8];
      RcVec<__nv_bfloat16, 8>::load(row + c, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) s = fmaf(v[i], v[i], s);
    }
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    const float inv = 1.f / sqrtf(s + kDcUnitEps);
    if (half == 0) {
      if (tid < 128) rq[r] = inv * rsqrtf(static_cast<float>(a.dk));
      else rk[r] = inv;
    }
  }
  __syncthreads();
  uint8_t* scratch = reinterpret_cast<uint8_t*>(a.scratch) + (static_cast<long long>(tile) * a.heads + h) * dc_scratch(DK);
  // ---- L (side 0) and A (side 1); A stays in registers as the A operand of A T, high and low half
  uint32_t ah[4][4], al[4][4];
  {
    float ct[2], ft[2];                            // of the rows gq and gq + 8
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = wr * 16 + gq + 8 * r;
      ct[r] = cum[t];
      ft[r] = side ? rq[t] : beta[t] * rk[t];
    }
    uint32_t xf[DK / 16][4];
#pragma unroll
    for (int k = 0; k < DK / 16; ++k) wm_ldsm_x4(wm_a(side ? sQ : sK, P, wr * 16, k * 16, lane), xf[k]);
#pragma unroll
    for (int sb = 0; sb < 4; ++sb) {
      if (sb > wr) break;                          // what lies above the diagonal is never read
      float acc[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
      for (int k = 0; k < DK / 16; ++k) {
        uint32_t b[4];
        wm_ldsm_x4(wm_b(sK, P, sb * 16, k * 16, lane), b);
        wm_mma(acc[0], xf[k], b[0], b[1]);
        wm_mma(acc[1], xf[k], b[2], b[3]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int s = sb * 16 + i * 8 + 2 * tq;
        const float2 cs = *reinterpret_cast<const float2*>(cum + s), ks = *reinterpret_cast<const float2*>(rk + s);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = wr * 16 + gq + 8 * r;
          const float v0 = s <= t ? wm_ex2(ct[r] - cs.x) * ks.x * ft[r] * acc[i][2 * r] : 0.f;
          const float v1 = s + 1 <= t ? wm_ex2(ct[r] - cs.y) * ks.y * ft[r] * acc[i][2 * r + 1] : 0.f;
          if (side == 0) *reinterpret_cast<float2*>(Lm + t * LP + s) = make_float2(s < t ? v0 : 0.f, s + 1 < t ? v1 : 0.f);
          else wm_split(v0, v1, ah[sb][2 * i + r], al[sb][2 * i + r]);
        }
      }
    }
  }
  __syncthreads();
  // ---- T = (I + L)^-1: the four diagonal blocks of 16 by forward substitution, one thread per column ...
  if (tid < 64) {
    const int b0 = tid & ~15, j = tid & 15;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const float4* row = reinterpret_cast<const float4*>(Lm + (b0 + t) * LP + b0);
      float v0 = t == j ? 1.f : 0.f, v1 = 0.f;
#pragma unroll
      for (int s = 0; s < t; s += 4) {
        const float4 l = row[s / 4];
        v0 = fmaf(-l.x, x[s], v0);
        if (s + 1 < t) v1 = fmaf(-l.y, x[s + 1], v1);
        if (s + 2 < t) v0 = fmaf(-l.z, x[s + 2], v0);
        if (s + 3 < t) v1 = fmaf(-l.w, x[s + 3], v1);
      }
      x[t] = v0 + v1;                              // zero above the diagonal
      T[(b0 + t) * LP + b0 + j] = x[t];
    }
  }
  __syncthreads();
  // ---- ... then the blocks below: T_ij = -T_ii sum_{j <= k < i} L_ik T_kj, one distance i - j after the other
  // 64 threads per block, four neighbouring entries of a row each
  const int gb = tid >> 6, er = (tid >> 2) & 15, ec = (tid & 3) * 4;
  auto dot16 = [&](const float* row, const float* m, int pitch, float4& out) {
#pragma unroll
    for (int k = 0; k < 16; k += 4) {
      const float4 l = *reinterpret_cast<const float4*>(row + k);
      const float lv[4] = {l.x, l.y, l.z, l.w};
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float4 u = *reinterpret_cast<const float4*>(m + (k + q) * pitch);
        out.x = fmaf(lv[q], u.x, out.x); out.y = fmaf(lv[q], u.y, out.y);
        out.z = fmaf(lv[q], u.z, out.z); out.w = fmaf(lv[q], u.w, out.w);
      }
    }
  };
#pragma unroll
  for (int d = 1; d < 4; ++d) {
    const bool mine = gb < 4 - d;                  // block row gb + d, block column gb
    if (mine) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int k = 0; k < d; ++k) dot16(Lm + ((gb + d) * 16 + er) * LP + (gb + k) * 16, T + (gb + k) * 16 * LP + gb * 16 + ec, LP, v);
      *reinterpret_cast<float4*>(W + (gb * 16 + er) * 20 + ec) = v;
    }
    __syncthreads();
    if (mine) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      dot16(T + ((gb + d) * 16 + er) * LP + (gb + d) * 16, W + gb * 16 * 20 + ec, 20, v);
      *reinterpret_cast<float4*>(T + ((gb + d) * 16 + er) * LP + gb * 16 + ec) = make_float4(-v.x, -v.y, -v.z, -v.w);
    }
    __syncthreads();
  }
  const uint32_t sT = smem_u32(dp_smem) + L::kL;
  constexpr int TP = L::kTPitch;
  for (int e = tid; e < kDcChunk * kDcChunk / 8; e += kDpThreads) {
    const int r = e >> 3, c = (e & 7) * 8;
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) wm_split(T[r * LP + c + 2 * k], T[r * LP + c + 2 * k + 1], hi[k], lo[k]);
    *reinterpret_cast<uint4*>(dp_smem + L::kL + (r * TP + c) * 2) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(dp_smem + L::kL + ((kDcChunk + r) * TP + c) * 2) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  // ---- W = T^T diag(1 / |k| exp(c_end - c)) K: rows (columns of T) wr 16 .. + 16; T^T, scaled, is the A operand
  uint32_t th[4][4], tl[4][4];
  {
    const float c_end = cum[kDcChunk - 1];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (k < wr) continue;                        // T is lower triangular
#pragma unroll
      for (int half = 0; half < 2; ++half) {       // columns k 16 + 8 half + 2 tq (+ 1)
        const int t = k * 16 + half * 8 + 2 * tq;
        const float2 ck = *reinterpret_cast<const float2*>(cum + t), kk = *reinterpret_cast<const float2*>(rk + t);
        const float w0 = kk.x * wm_ex2(c_end - ck.x), w1 = kk.y * wm_ex2(c_end - ck.y);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int s = wr * 16 + gq + 8 * r;
          wm_split(w0 * T[t * LP + s], w1 * T[(t + 1) * LP + s], th[k][2 * half + r], tl[k][2 * half + r]);
        }
      }
    }
  }
  __syncthreads();                                 // T is free: staging of W's low half
  // ---- A T: rows wr 16 .. + 16
  if (side == 1) {
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(scratch);
#pragma unroll
    for (int nb = 0; nb < 4; ++nb) {
      float acc[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (k < nb || k > wr) continue;            // both are lower triangular
        uint32_t b[4], bl[4];
        wm_ldsm_x4_t(wm_b_t(sT, TP, nb * 16, k * 16, lane), b);
        wm_ldsm_x4_t(wm_b_t(sT + kDcChunk * TP * 2, TP, nb * 16, k * 16, lane), bl);
        wm_mma(acc[0], ah[k], b[0], b[1]);
        wm_mma(acc[1], ah[k], b[2], b[3]);
        wm_mma(acc[0], al[k], b[0], b[1]);
        wm_mma(acc[1], al[k], b[2], b[3]);
        wm_mma(acc[0], ah[k], bl[0], bl[1]);
        wm_mma(acc[1], ah[k], bl[2], bl[3]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<uint32_t*>(out + (wr * 16 + gq + 8 * r) * kDcMPitch + nb * 16 + i * 8 + 2 * tq) =
              pack_bf16x2(acc[i][2 * r], acc[i][2 * r + 1]);
    }
  }
  {
    // columns: the first five eighths by side 0, the rest by side 1
    constexpr int kCut = DK / 16 * 5 / 8;
    const int nb0 = side ? kCut : 0, nb1 = side ? DK / 16 : kCut;
#pragma unroll 1
    for (int nb = nb0; nb < nb1; ++nb) {
      float acc[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (k < wr) continue;
        uint32_t b[4];
        wm_ldsm_x4_t(wm_b_t(sK, P, nb * 16, k * 16, lane), b);
        wm_mma(acc[0], th[k], b[0], b[1]);
        wm_mma(acc[1], th[k], b[2], b[3]);
        wm_mma(acc[0], tl[k], b[0], b[1]);
        wm_mma(acc[1], tl[k], b[2], b[3]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          wm_split(acc[i][2 * r], acc[i][2 * r + 1], hi, lo);
          const int at = ((wr * 16 + gq + 8 * r) * P + nb * 16 + i * 8 + 2 * tq) * 2;
          *reinterpret_cast<uint32_t*>(dp_smem + L::kQ + at) = hi;
          *reinterpret_cast<uint32_t*>(dp_smem + L::kT + at) = lo;
        }
    }
    __syncwarp();                                  // every warp copies its own rows and columns
    uint8_t* out = scratch + kDcMat;
    // lanes: two rows of 16 at a time, the 16-byte pieces of a row side by side
    const int r0 = wr * 16 + (lane >> 4), c = (nb0 * 2 + (lane & 15)) * 8;
    if (c < nb1 * 16) {
#pragma unroll
      for (int r = r0; r < wr * 16 + 16; r += 2) {
        const int at = (r * P + c) * 2;
        *reinterpret_cast<uint4*>(out + at) = *reinterpret_cast<const uint4*>(dp_smem + L::kQ + at);
        *reinterpret_cast<uint4*>(out + dc_half(DK) + at) = *reinterpret_cast<const uint4*>(dp_smem + L::kT + at);
      }
    }
  }
  if (tid < kDcChunk) {
    float* f = reinterpret_cast<float*>(scratch + kDcMat + 2 * dc_half(DK));
    const float e = wm_ex2(cum[tid]);
    f[tid] = beta[tid];
    f[kDcChunk + tid] = rk[tid] * e;
    f[2 * kDcChunk + tid] = rq[tid] * e;
    f[3 * kDcChunk + tid] = wm_ex2(cum[kDcChunk - 1]);
  }
}

// ---- second kernel
template <int DK, int COLS>
struct DcSmem {
  static constexpr int kPitch = DK + 8, kVPitch = COLS + 8, kMPitch = kDcMPitch;
  static constexpr int kAtom = kDcChunk * 128;                       // 64 rows of 64 bf16, 128-byte swizzle
  // one stage: what a chunk reads; the high half of R replaces V element by element
  static constexpr int kQ = 0;
  static constexpr int kK = kQ + (DK / 64) * kAtom;
  static constexpr int kM = kK + (DK / 64) * kAtom;                  // A T, W (high and low half) and the factors, as in the scratch
  static constexpr int kW = kM + kDcMat;
  static constexpr int kF = kW + 2 * dc_half(DK);
  static constexpr int kV = kF + kDcFactors * kDcChunk * 4;
  static constexpr int kStage = kV + kDcChunk * kVPitch * 2;
  static constexpr int kS = 2 * kStage;                              // state, high and low half
  static constexpr int kR = kS + 2 * DK * kVPitch * 2;               // low half of R
  static constexpr int kBar = kR + kDcChunk * kVPitch * 2;
  static constexpr int kTotal = kBar + 2 * 8 + 16;
  static_assert(kStage % 1024 == 0, "swizzled tiles start at multiples of 1024 bytes");
};

// A fragment, rows [r0, r0 + 16), columns [k0, k0 + 16), of a tile in 128-byte swizzled atoms of 64 columns
__device__ __forceinline__ uint32_t dc_a(uint32_t base, int atom, int r0, int k0, int lane) {
  const int row = r0 + (lane & 15), piece = (k0 >> 3) + (lane >> 4);
  return base + (piece >> 3) * atom + row * 128 + (((piece & 7) ^ (row & 7)) << 4);
}

// untiled copy of a contiguous block, completion counted on an mbarrier
__device__ __forceinline__ void dc_bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

template <int DK, int COLS>
__global__ void __launch_bounds__(256, 1)
delta_rule_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const RbDeltaRuleArgs a,
                        unsigned int* status) {
  using L = DcSmem<DK, COLS>;
  constexpr int P = L::kPitch, VP = L::kVPitch, MP = L::kMPitch;
  constexpr int MT = DK / 64, NJ = COLS / 32;      // state: MT row tiles; columns of a warp: NJ pairs of n-tiles
  extern __shared__ __align__(1024) uint8_t dc_raw[];
  uint8_t* dc_smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(dc_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t base = smem_u32(dc_smem);
  const uint32_t sS = base + L::kS, sRl = base + L::kR, bar = base + L::kBar;      // bar[2]
  volatile int* abort_flag = reinterpret_cast<volatile int*>(dc_smem + L::kBar + 16);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3;
  const int wc = warp >> 2, wr = wc ? 3 - (warp & 3) : (warp & 3);
  const int ctiles = (a.dv + COLS - 1) / COLS;
  const int h = blockIdx.x / ctiles, c0 = (blockIdx.x - h * ctiles) * COLS;
  const RcSegment seg = rc_segment(a.segments, blockIdx.y, a.num_slots);
  if (seg.len <= 0) return;
  int tile0 = 0;                                   // first chunk of this segment in the scratch
  for (int i = 0; i < static_cast<int>(blockIdx.y); ++i) tile0 += (max(0, a.segments[4 * i + 1]) + kDcChunk - 1) / kDcChunk;
  const int g = h / (a.heads / a.kv_heads);
  const __nv_bfloat16* qkv = reinterpret_cast<const __nv_bfloat16*>(a.qkv) + static_cast<long long>(seg.first) * a.ld_qkv;
  const long long offV = 2ll * a.kv_heads * a.dk + static_cast<long long>(h) * a.dv + c0;
  const int chunks = (seg.len + kDcChunk - 1) / kDcChunk;
  if (tid == 0) {
    mbar_init(bar, 1);
    mbar_init(bar + 8, 1);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
  }
  __syncthreads();

  // Everything chunk ci reads, into stage ci & 1.  Rows behind the segment's end are other sequences' queries and keys: beta is
  // zero there and nothing of them is stored.
  auto request = [&](int ci) {
    const uint32_t st = base + (ci & 1) * L::kStage;
    const int t0 = ci * kDcChunk, m_rows = min(kDcChunk, seg.len - t0);
    if (tid == 0) {
      const uint32_t b = bar + 8 * (ci & 1);
      fence_proxy_async_smem();                    // the stage was read (and V written) by ordinary accesses
      mbar_arrive_expect_tx(b, 2 * (DK / 64) * L::kAtom + dc_scratch(DK));
#pragma unroll
      for (int k = 0; k < DK / 64; ++k) {
        tma_load_4d(st + L::kK + k * L::kAtom, &tmK, k * 64, g, seg.first + t0, 0, b);
        tma_load_4d(st + L::kQ + k * L::kAtom, &tmQ, k * 64, g, seg.first + t0, 0, b);
      }
      dc_bulk_load(st + L::kM, reinterpret_cast<const uint8_t*>(a.scratch) + (static_cast<long long>(tile0 + ci) * a.heads + h) * dc_scratch(DK),
                   dc_scratch(DK), b);
    }
    const __nv_bfloat16* rows = qkv + static_cast<long long>(t0) * a.ld_qkv + offV;
    for (int i = tid; i < kDcChunk * (COLS / 8); i += 256) {
      const int r = i / (COLS / 8), c = (i - r * (COLS / 8)) * 8;
      const bool ok = r < m_rows && c0 + c < a.dv;
      wm_cp16(st + L::kV + (r * VP + c) * 2, ok ? rows + r * a.ld_qkv + c : qkv, ok);
    }
    wm_cp_commit();
  };
  request(0);

  // this thread's part of the state: rows n = wr DK/4 + 16 m + gq (+ 8), columns wc COLS/2 + 8 j + 2 tq (+ 1)
  const int n_base = wr * (DK / 4) + gq, v_base = wc * (COLS / 2) + 2 * tq;
  float S[MT][2 * NJ][4];
  float* slot = a.state + (static_cast<long long>(seg.slot) * a.heads + h) * a.dk * a.dv;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int n = n_base + 16 * m + 8 * r, v = c0 + v_base + 8 * j;
        float2 s = make_float2(0.f, 0.f);
        if (seg.start > 0 && n < a.dk && v < a.dv) s = *reinterpret_cast<const float2*>(slot + static_cast<long long>(n) * a.dv + v);
        S[m][j][2 * r] = s.x;
        S[m][j][2 * r + 1] = s.y;
      }
  auto publish = [&]() {                           // the state as two bf16 numbers
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          wm_split(S[m][j][2 * r], S[m][j][2 * r + 1], hi, lo);
          const int at = ((n_base + 16 * m + 8 * r) * VP + v_base + 8 * j) * 2;
          *reinterpret_cast<uint32_t*>(dc_smem + L::kS + at) = hi;
          *reinterpret_cast<uint32_t*>(dc_smem + L::kS + DK * VP * 2 + at) = lo;
        }
  };
  publish();

  bool ok = true;
  for (int ci = 0; ci < chunks; ++ci) {
    wm_cp_wait<0>();
    ok = mbar_wait(bar + 8 * (ci & 1), (ci >> 1) & 1, abort_flag, status, 91) && ok;
    __syncthreads();                               // this chunk's tiles and the state have arrived, for every warp
    if (ci + 1 < chunks) request(ci + 1);
    const uint32_t st = base + (ci & 1) * L::kStage;
    const uint8_t* stp = dc_smem + (ci & 1) * L::kStage;
    const float* f = reinterpret_cast<const float*>(stp + L::kF);
    const int r0 = wr * 16 + gq, r1 = r0 + 8;
    // ---- S0^T k and S0^T q for rows wr 16 .. + 16
    float pm[2 * NJ][4], y[2 * NJ][4];
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) pm[j][i] = y[j][i] = 0.f;
#pragma unroll
    for (int k = 0; k < DK / 16; ++k) {
      uint32_t kf[4], qf[4];
      wm_ldsm_x4(dc_a(st + L::kK, L::kAtom, wr * 16, k * 16, lane), kf);
      wm_ldsm_x4(dc_a(st + L::kQ, L::kAtom, wr * 16, k * 16, lane), qf);
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        uint32_t b[4], bl[4];
        wm_ldsm_x4_t(wm_b_t(sS, VP, wc * (COLS / 2) + j * 16, k * 16, lane), b);
        wm_ldsm_x4_t(wm_b_t(sS + DK * VP * 2, VP, wc * (COLS / 2) + j * 16, k * 16, lane), bl);
        wm_mma(pm[2 * j], kf, b[0], b[1]);
        wm_mma(pm[2 * j + 1], kf, b[2], b[3]);
        wm_mma(y[2 * j], qf, b[0], b[1]);
        wm_mma(y[2 * j + 1], qf, b[2], b[3]);
        wm_mma(pm[2 * j], kf, bl[0], bl[1]);
        wm_mma(pm[2 * j + 1], kf, bl[2], bl[3]);
      }
    }
    // ---- R
    uint8_t* V = dc_smem + (ci & 1) * L::kStage + L::kV;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = r ? r1 : r0;
      const float be = f[t], kd = f[kDcChunk + t];
#pragma unroll
      for (int j = 0; j < 2 * NJ; ++j) {
        const int at = (t * VP + v_base + 8 * j) * 2;
        const float2 v = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(V + at));
        uint32_t hi, lo;
        wm_split(be * (v.x - kd * pm[j][2 * r]), be * (v.y - kd * pm[j][2 * r + 1]), hi, lo);
        *reinterpret_cast<uint32_t*>(V + at) = hi;
        *reinterpret_cast<uint32_t*>(dc_smem + L::kR + at) = lo;
      }
    }
    __syncthreads();
    const uint32_t sRh = st + L::kV;
    // ---- state behind the chunk
    const float e_end = f[3 * kDcChunk];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[m][j][i] *= e_end;
    const float q0 = f[2 * kDcChunk + r0], q1 = f[2 * kDcChunk + r1];
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j) { y[j][0] *= q0; y[j][1] *= q0; y[j][2] *= q1; y[j][3] *= q1; }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t wh[MT][4], wl[MT][4], af[4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        wm_ldsm_x4_t(wm_a_t(st + L::kW, P, wr * (DK / 4) + m * 16, k * 16, lane), wh[m]);
        wm_ldsm_x4_t(wm_a_t(st + L::kW + kDcChunk * P * 2, P, wr * (DK / 4) + m * 16, k * 16, lane), wl[m]);
      }
      if (k <= wr) wm_ldsm_x4(wm_a(st + L::kM, MP, wr * 16, k * 16, lane), af);
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        uint32_t b[4], bl[4];
        wm_ldsm_x4_t(wm_b_t(sRh, VP, wc * (COLS / 2) + j * 16, k * 16, lane), b);
        wm_ldsm_x4_t(wm_b_t(sRl, VP, wc * (COLS / 2) + j * 16, k * 16, lane), bl);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          wm_mma(S[m][2 * j], wh[m], b[0], b[1]);
          wm_mma(S[m][2 * j + 1], wh[m], b[2], b[3]);
          wm_mma(S[m][2 * j], wl[m], b[0], b[1]);
          wm_mma(S[m][2 * j + 1], wl[m], b[2], b[3]);
          wm_mma(S[m][2 * j], wh[m], bl[0], bl[1]);
          wm_mma(S[m][2 * j + 1], wh[m], bl[2], bl[3]);
        }
        if (k <= wr) {                             // o = exp(c) S0^T q + (A T) R
          wm_mma(y[2 * j], af, b[0], b[1]);
          wm_mma(y[2 * j + 1], af, b[2], b[3]);
          wm_mma(y[2 * j], af, bl[0], bl[1]);
          wm_mma(y[2 * j + 1], af, bl[2], bl[3]);
        }
      }
    }
    publish();                                     // every warp has read the old one
    const int t0 = ci * kDcChunk;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.o) + static_cast<long long>(seg.first + t0) * a.ld_o + static_cast<long long>(h) * a.dv + c0;
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j) {
      const int v = v_base + 8 * j;
      if (c0 + v >= a.dv) continue;
      if (t0 + r0 < seg.len) *reinterpret_cast<uint32_t*>(out + r0 * a.ld_o + v) = pack_bf16x2(y[j][0], y[j][1]);
      if (t0 + r1 < seg.len) *reinterpret_cast<uint32_t*>(out + r1 * a.ld_o + v) = pack_bf16x2(y[j][2], y[j][3]);
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int n = n_base + 16 * m + 8 * r, v = c0 + v_base + 8 * j;
        if (ok && n < a.dk && v < a.dv)
          *reinterpret_cast<float2*>(slot + static_cast<long long>(n) * a.dv + v) = make_float2(S[m][j][2 * r], S[m][j][2 * r + 1]);
      }
}

// [rows, heads, dk] part of a packed row-major matrix, 64 columns of 64 rows of one head at a time
const CUtensorMap* dc_map(const void* base, int dk, int heads, long long rows, long long ld, int* err) {
  const uint64_t dims[4] = {(uint64_t)dk, (uint64_t)heads, (uint64_t)rows, 1};
  const uint64_t str[3] = {(uint64_t)dk * 2, (uint64_t)ld * 2, (uint64_t)(rows * ld) * 2};
  const uint32_t box[4] = {64, 1, (uint32_t)kDcChunk, 1};
  return rbhost::get_tmap_4d(base, 2, dims, str, box, 1, err);
}

template <int DK, int COLS>
int dc_main_launch(const RbDeltaRuleArgs& a, const CUtensorMap* tq, const CUtensorMap* tk, cudaStream_t s) {
  const int smem = DcSmem<DK, COLS>::kTotal + 1024;
  static_assert(DcSmem<DK, COLS>::kTotal + 1024 <= 227 * 1024, "shared memory of a CTA");
  auto kern = delta_rule_chunk_kernel<DK, COLS>;
  static bool cfg_dev[64] = {false};
  bool& cfg = cfg_dev[rbhost::device_slot()];
  if (!cfg) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  kern<<<dim3(a.heads * ((a.dv + COLS - 1) / COLS), a.num_segments), 256, smem, s>>>(*tq, *tk, a, rbhost::status_ptr());
  return static_cast<int>(cudaGetLastError());
}

template <int DK>
int dc_launch(const RbDeltaRuleArgs& a, cudaStream_t s) {
  auto prep = delta_rule_prepare_kernel<DK>;
  const int smem = DcPrepSmem<DK>::kTotal;
  static bool cfg_dev[64] = {false};
  bool& cfg = cfg_dev[rbhost::device_slot()];
  if (!cfg) {
    const cudaError_t e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.qkv);
  int err = 0;
  const CUtensorMap* tq = dc_map(q, a.dk, a.kv_heads, a.rows, a.ld_qkv, &err);
  const CUtensorMap* tk = dc_map(q + static_cast<long long>(a.kv_heads) * a.dk, a.dk, a.kv_heads, a.rows, a.ld_qkv, &err);
  if (!tq || !tk) return err ? err : -5;
  prep<<<dim3(a.heads, a.num_tiles), kDpThreads, smem, s>>>(a);
  const int rc = static_cast<int>(cudaGetLastError());
  if (rc) return rc;
  // narrow column tiles (twice the CTAs) while wide ones would leave half of the SMs idle
  const long long wide = static_cast<long long>(a.heads) * ((a.dv + 63) / 64) * a.num_segments;
  return wide * 2 <= rbhost::device_sm_count() || a.dv <= 32 ? dc_main_launch<DK, 32>(a, tq, tk, s)
                                                             : dc_main_launch<DK, 64>(a, tq, tk, s);
}

}  // namespace rb

RB_API long long rb_delta_rule_scratch_bytes(int num_tiles, int heads, int dk) {
  return static_cast<long long>(num_tiles) * heads * rb::dc_scratch(dk <= 64 ? 64 : 128);
}

RB_API int rb_delta_rule_chunked(const RbDeltaRuleArgs* args, void* stream_v) {
  const RbDeltaRuleArgs& a = *args;
  if (a.num_segments <= 0) return 0;
  if (!a.qkv || !a.a_raw || !a.b_raw || !a.dt_bias || !a.a_log || !a.state || !a.o || !a.segments || !a.tiles || !a.scratch || a.f32 ||
      a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dk <= 0 || a.dv <= 0 || a.num_slots <= 0 || a.num_tiles <= 0 || a.rows <= 0 ||
      a.num_segments > 65535 || a.num_tiles > 65535)
    return -1;
  if (a.dk > 128 || ((a.dk | a.dv) & 7) || (a.ld_qkv & 7) || (a.ld_o & 1)) return -9;
  if (((reinterpret_cast<uintptr_t>(a.qkv) | reinterpret_cast<uintptr_t>(a.state) | reinterpret_cast<uintptr_t>(a.scratch)) & 15) ||
      (reinterpret_cast<uintptr_t>(a.o) & 3))
    return -9;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.dk <= 64 ? rb::dc_launch<64>(a, s) : rb::dc_launch<128>(a, s);
}
