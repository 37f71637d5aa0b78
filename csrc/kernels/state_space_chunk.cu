// Mamba-2 state-space recurrence over prompts, chunked: 64 tokens at a time become matrix products on the tensor cores.
//
// With c_t the running sum of the logarithms of the decays inside a chunk and S0 the state in front of it,
//   y_t = exp(c_t) C_t S0 + sum_{s <= t} exp(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//   S   = exp(c_end) S0 + sum_s B_s (exp(c_end - c_s) dt_s x_s)^T
// One CTA (8 warps) owns 64 value columns of one head over a span of chunks.  The state stays in fp32 accumulator registers; its
// bf16 copy in shared memory is the operand of the read-out only.  What enters the state is split into two bf16 numbers (about 16
// bits), decays and step sizes are fp32, so the state itself is good to fp32-like accuracy.
//
// A long segment is cut into spans that run side by side: a first pass computes what every span but the last adds to the state
// (from zero) and its total decay, and each span of the second pass starts from the combination of those before it.
#include "recurrent.h"

#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace rb {

constexpr int kScChunk = 64;
constexpr int kScCols = 64;
constexpr int kScThreads = 256;
constexpr float kScLog2e = 1.4426950408889634f;

template <int N, bool STATE_ONLY>
struct ScSmem {
  static constexpr int kPitch = N + 8, kXPitch = kScCols + 8;
  static constexpr int kB = 0;                                       // two buffers
  static constexpr int kX = kB + 2 * kScChunk * kPitch * 2;          // two buffers
  static constexpr int kXs = kX + 2 * kScChunk * kXPitch * 2;        // scaled x, permuted rows: high half, low half
  static constexpr int kCum = kXs + 2 * kScChunk * kScCols * 2;      // two buffers: fp32 [64] running log2 decays, [64] step sizes
  static constexpr int kC = kCum + 4 * kScChunk * 4;
  static constexpr int kM = kC + (STATE_ONLY ? 0 : kScChunk * kPitch * 2);       // masked products C . B, permuted rows
  static constexpr int kS = kM + (STATE_ONLY ? 0 : kScChunk * kScChunk * 2);     // bf16 copy of the state
  static constexpr int kTotal = kS + (STATE_ONLY ? 0 : N * kXPitch * 2);
};

template <int N, bool STATE_ONLY>
__global__ void __launch_bounds__(kScThreads, STATE_ONLY ? 3 : 2)
state_space_chunk_kernel(const RbStateSpaceArgs a, float* __restrict__ span_state, float* __restrict__ span_decay, int span) {
  using L = ScSmem<N, STATE_ONLY>;
  constexpr int MT = N / 64;                       // 16-row tiles of the state per warp
  constexpr int NP = L::kPitch, XP = L::kXPitch;
  extern __shared__ __align__(16) uint8_t sc_smem[];
  const uint32_t base = smem_u32(sc_smem);
  const uint32_t sC = base + L::kC, sXs = base + L::kXs, sM = base + L::kM, sS = base + L::kS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3;
  const int wc = warp >> 2, wr = wc ? 3 - (warp & 3) : (warp & 3);   // the causal work of a scheduler's two warps adds up evenly
  const int ptiles = (a.p + kScCols - 1) / kScCols;
  const int h = blockIdx.x / ptiles, c0 = (blockIdx.x - h * ptiles) * kScCols;
  const int tile = blockIdx.y;
  const RcSegment seg = rc_segment(a.segments, a.tiles[2 * tile], a.num_slots);
  const int off = a.tiles[2 * tile + 1];
  const int end = min(seg.len, off + span);
  if (off >= seg.len) return;
  if (STATE_ONLY && end == seg.len) return;        // nobody starts from what the last span adds
  const int g = h / (a.heads / a.groups);
  const __nv_bfloat16* xbc = reinterpret_cast<const __nv_bfloat16*>(a.xbc);
  const long long offX = static_cast<long long>(h) * a.p + c0;
  const long long offB = static_cast<long long>(a.heads) * a.p + static_cast<long long>(g) * a.n;
  const long long offC = offB + static_cast<long long>(a.groups) * a.n;
  const float rate2 = expf(a.a_log[h]) * kScLog2e, dt_bias = a.dt_bias[h], dskip = a.D[h];

  // this thread's part of the state: rows n = wr N/4 + 16 m + gq (+ 8), columns wc 32 + 8 j + 2 tq (+ 1)
  const int n_base = wr * (N / 4) + gq, p_base = wc * 32 + 2 * tq;
  float S[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 4; ++j) S[m][j][0] = S[m][j][1] = S[m][j][2] = S[m][j][3] = 0.f;
  auto each = [&](auto f) {                        // f(two neighbouring entries, row, column)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int n = n_base + 16 * m + 8 * r, p = c0 + p_base + 8 * j;
          if (n < a.n && p < a.p) f(S[m][j][2 * r], S[m][j][2 * r + 1], static_cast<long long>(n) * a.p + p);
        }
  };
  const long long state_n = static_cast<long long>(a.n) * a.p;
  float* slot = a.state + (static_cast<long long>(seg.slot) * a.heads + h) * state_n;
  if (!STATE_ONLY) {
    if (seg.start > 0)
      each([&](float& u, float& v, long long i) { const float2 s = *reinterpret_cast<const float2*>(slot + i); u = s.x; v = s.y; });
    for (int t = tile - off / span; t < tile; ++t) {               // spans of this segment in front of this one
      const float d = wm_ex2(span_decay[static_cast<long long>(t) * a.heads + h]);
      const float* add = span_state + (static_cast<long long>(t) * a.heads + h) * state_n;
      each([&](float& u, float& v, long long i) {
        const float2 s = *reinterpret_cast<const float2*>(add + i);
        u = fmaf(u, d, s.x);
        v = fmaf(v, d, s.y);
      });
    }
  }
  float total = 0.f;

  // Tiles of a chunk (rows past the end and columns past the real sizes are zero).  B and x have two buffers; C is free again
  // behind the second barrier of a chunk, so the next chunk's is requested there and arrives under the state's products.
  auto request_bx = [&](int t0) {
    const int m_rows = min(kScChunk, end - t0);
    const __nv_bfloat16* rows = xbc + static_cast<long long>(seg.first + t0) * a.ld_xbc;
    const uint32_t dst = base + L::kB + ((t0 - off) / kScChunk & 1) * kScChunk * NP * 2;
    for (int i = tid; i < kScChunk * (N / 8); i += kScThreads) {
      const int r = i / (N / 8), c = (i - r * (N / 8)) * 8;
      const bool ok = r < m_rows && c < a.n;
      wm_cp16(dst + (r * NP + c) * 2, ok ? rows + r * a.ld_xbc + offB + c : rows, ok);
    }
    const uint32_t dst_x = base + L::kX + ((t0 - off) / kScChunk & 1) * kScChunk * XP * 2;
    for (int i = tid; i < kScChunk * (kScCols / 8); i += kScThreads) {
      const int r = i / (kScCols / 8), c = (i - r * (kScCols / 8)) * 8;
      const bool ok = r < m_rows && c0 + c < a.p;
      wm_cp16(dst_x + (r * XP + c) * 2, ok ? rows + r * a.ld_xbc + offX + c : rows, ok);
    }
  };
  auto request_c = [&](int t0) {
    if (STATE_ONLY) return;
    const int m_rows = min(kScChunk, end - t0);
    const __nv_bfloat16* rows = xbc + static_cast<long long>(seg.first + t0) * a.ld_xbc;
    for (int i = tid; i < kScChunk * (N / 8); i += kScThreads) {
      const int r = i / (N / 8), c = (i - r * (N / 8)) * 8;
      const bool ok = r < m_rows && c < a.n;
      wm_cp16(sC + (r * NP + c) * 2, ok ? rows + r * a.ld_xbc + offC + c : rows, ok);
    }
  };
  // Step sizes and running log2 decays by warp 0, two tokens per lane; the raw values are fetched one chunk earlier still.
  float raw[2] = {0.f, 0.f};
  auto fetch_dt = [&](int t0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = t0 + 2 * lane + i;
      if (t < end) raw[i] = a.dt_raw[static_cast<long long>(seg.first + t) * a.ld_dt + h];
    }
  };
  auto scan_dt = [&](int t0) {
    float* cum = reinterpret_cast<float*>(sc_smem + L::kCum) + ((t0 - off) / kScChunk & 1) * 2 * kScChunk;
    float d[2], s[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      d[i] = t0 + 2 * lane + i < end ? rc_softplus(raw[i] + dt_bias) : 0.f;
      s[i] = -rate2 * d[i];
    }
    float run = s[0] + s[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += u;
    }
    cum[2 * lane] = run - s[1];
    cum[2 * lane + 1] = run;
    cum[kScChunk + 2 * lane] = d[0];
    cum[kScChunk + 2 * lane + 1] = d[1];
  };
  auto publish = [&]() {                           // bf16 copy of the state for the read-out
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<uint32_t*>(sc_smem + L::kS + ((n_base + 16 * m + 8 * r) * XP + p_base + 8 * j) * 2) =
              pack_bf16x2(S[m][j][2 * r], S[m][j][2 * r + 1]);
  };
  request_bx(off);
  request_c(off);
  wm_cp_commit();
  if (warp == 0) {
    fetch_dt(off);
    scan_dt(off);
    fetch_dt(off + kScChunk);
  }
  if (!STATE_ONLY) publish();

  for (int t0 = off; t0 < end; t0 += kScChunk) {
    const int m_rows = min(kScChunk, end - t0);
    const int par = (t0 - off) / kScChunk & 1;
    const uint32_t sB = base + L::kB + par * kScChunk * NP * 2, sX = base + L::kX + par * kScChunk * XP * 2;
    const __nv_bfloat16* xs = reinterpret_cast<const __nv_bfloat16*>(sc_smem + L::kX) + par * kScChunk * XP;
    const float* cum = reinterpret_cast<const float*>(sc_smem + L::kCum) + par * 2 * kScChunk;
    const float* dts = cum + kScChunk;
    const bool more = t0 + kScChunk < end;
    wm_cp_wait<0>();
    __syncthreads();                               // tiles, step sizes and the state in front of the chunk have arrived
    if (more) request_bx(t0 + kScChunk);
    if (warp == 0 && more) {
      scan_dt(t0 + kScChunk);
      fetch_dt(t0 + 2 * kScChunk);
    }
    const float c_end = cum[kScChunk - 1];
    // ---- x scaled by what it adds to the state
    for (int i = tid; i < kScChunk * (kScCols / 8); i += kScThreads) {
      const int r = i / (kScCols / 8), c = (i - r * (kScCols / 8)) * 8;
      const float w = dts[r] * wm_ex2(c_end - cum[r]);
      float v[8];
      RcVec<__nv_bfloat16, 8>::load(xs + r * XP + c, v);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) wm_split(w * v[2 * k], w * v[2 * k + 1], hi[k], lo[k]);
      *reinterpret_cast<uint4*>(sc_smem + L::kXs + wm_swz(r, c >> 3)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(sc_smem + L::kXs + kScChunk * 128 + wm_swz(r, c >> 3)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    float y[4][4];                                 // y of rows wr 16 .. + 16, columns wc 32 .. + 32
    const int r0 = wr * 16 + gq, r1 = r0 + 8;
    if (!STATE_ONLY) {
      // ---- C S0, and one or two of the ten blocks (16 x 16) of C B^T on and below the diagonal: those of the warp's own rows in
      // the same loop, the three that are left by the warps of the first rows, which have the least to do behind the barrier
      const int own = wr > 0 ? wr - wc : (wc == 0 ? 0 : -1);
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
      float gacc[2][4];
      auto clear = [&]() {
#pragma unroll
        for (int i = 0; i < 2; ++i) gacc[i][0] = gacc[i][1] = gacc[i][2] = gacc[i][3] = 0.f;
      };
      auto store_block = [&](int tb, int sb) {     // decays, step sizes and the mask; bf16
        const int ta = tb * 16 + gq, tb8 = ta + 8;
        const float ca = cum[ta], cb = cum[tb8];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int s0 = sb * 16 + i * 8 + 2 * tq;
          const float2 cs = *reinterpret_cast<const float2*>(cum + s0), ds = *reinterpret_cast<const float2*>(dts + s0);
          const float m00 = s0 <= ta ? gacc[i][0] * ds.x * wm_ex2(ca - cs.x) : 0.f;
          const float m01 = s0 + 1 <= ta ? gacc[i][1] * ds.y * wm_ex2(ca - cs.y) : 0.f;
          const float m10 = s0 <= tb8 ? gacc[i][2] * ds.x * wm_ex2(cb - cs.x) : 0.f;
          const float m11 = s0 + 1 <= tb8 ? gacc[i][3] * ds.y * wm_ex2(cb - cs.y) : 0.f;
          *reinterpret_cast<uint32_t*>(sc_smem + L::kM + wm_swz(ta, s0 >> 3) + (s0 & 7) * 2) = pack_bf16x2(m00, m01);
          *reinterpret_cast<uint32_t*>(sc_smem + L::kM + wm_swz(tb8, s0 >> 3) + (s0 & 7) * 2) = pack_bf16x2(m10, m11);
        }
      };
      clear();
#pragma unroll
      for (int k = 0; k < N / 16; ++k) {
        uint32_t cf[4];
        wm_ldsm_x4(wm_a(sC, NP, wr * 16, k * 16, lane), cf);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          uint32_t b[4];
          wm_ldsm_x4_t(wm_b_t(sS, XP, wc * 32 + j * 16, k * 16, lane), b);
          wm_mma(y[2 * j], cf, b[0], b[1]);
          wm_mma(y[2 * j + 1], cf, b[2], b[3]);
        }
        if (own >= 0) {
          uint32_t b[4];
          wm_ldsm_x4(wm_b(sB, NP, own * 16, k * 16, lane), b);
          wm_mma(gacc[0], cf, b[0], b[1]);
          wm_mma(gacc[1], cf, b[2], b[3]);
        }
      }
      if (own >= 0) store_block(wr, own);
      if (wr == 0) {
        for (int e = 0; e <= wc; ++e) {            // (2, 0); (3, 0), (3, 1)
          clear();
#pragma unroll
          for (int k = 0; k < N / 16; ++k) {
            uint32_t cf[4], b[4];
            wm_ldsm_x4(wm_a(sC, NP, (2 + wc) * 16, k * 16, lane), cf);
            wm_ldsm_x4(wm_b(sB, NP, e * 16, k * 16, lane), b);
            wm_mma(gacc[0], cf, b[0], b[1]);
            wm_mma(gacc[1], cf, b[2], b[3]);
          }
          store_block(2 + wc, e);
        }
      }
      const float e0 = wm_ex2(cum[r0]), e1 = wm_ex2(cum[r1]);
#pragma unroll
      for (int j = 0; j < 4; ++j) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
    }
    __syncthreads();                               // the scaled x and the masked products are complete; C and the state's copy are free
    if (more) request_c(t0 + kScChunk);
    wm_cp_commit();
    if (!STATE_ONLY) {
      // ---- + (masked C B^T) x + D x, out
#pragma unroll
      for (int sb = 0; sb < 4; ++sb) {
        if (sb > wr) break;
        uint32_t af[4];
        wm_ldsm_x4(wm_a_swz(sM, wr * 16, sb * 16, lane), af);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          uint32_t b[4];
          wm_ldsm_x4_t(wm_b_t(sX, XP, wc * 32 + j * 16, sb * 16, lane), b);
          wm_mma(y[2 * j], af, b[0], b[1]);
          wm_mma(y[2 * j + 1], af, b[2], b[3]);
        }
      }
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.y) + static_cast<long long>(seg.first + t0) * a.ld_y + offX;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int p = p_base + 8 * j;
        if (c0 + p >= a.p) continue;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = r ? r1 : r0;
          if (t >= m_rows) continue;
          const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(xs + t * XP + p));
          *reinterpret_cast<uint32_t*>(out + static_cast<long long>(t) * a.ld_y + p) =
              pack_bf16x2(fmaf(dskip, x.x, y[j][2 * r]), fmaf(dskip, x.y, y[j][2 * r + 1]));
        }
      }
    }
    // ---- state behind the chunk
    const float e_end = wm_ex2(c_end);
    total += c_end;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[m][j][i] *= e_end;
#pragma unroll
    for (int k = 0; k < kScChunk / 16; ++k) {
      uint32_t af[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) wm_ldsm_x4_t(wm_a_t(sB, NP, wr * (N / 4) + m * 16, k * 16, lane), af[m]);
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          uint32_t b[4];
          wm_ldsm_x4_t(wm_b_t_swz(sXs + half * kScChunk * 128, wc * 32 + j * 16, k * 16, lane), b);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            wm_mma(S[m][2 * j], af[m], b[0], b[1]);
            wm_mma(S[m][2 * j + 1], af[m], b[2], b[3]);
          }
        }
    }
    if (!STATE_ONLY) publish();
  }
  if (STATE_ONLY) {
    float* dst = span_state + (static_cast<long long>(tile) * a.heads + h) * state_n;
    each([&](float& u, float& v, long long i) { *reinterpret_cast<float2*>(dst + i) = make_float2(u, v); });
    if (tid == 0 && c0 == 0) span_decay[static_cast<long long>(tile) * a.heads + h] = total;
  } else if (end == seg.len) {
    each([&](float& u, float& v, long long i) { *reinterpret_cast<float2*>(slot + i) = make_float2(u, v); });
  }
}

template <int N>
int sc_chunk_launch(const RbStateSpaceArgs& a, float* span_state, float* span_decay, int span, cudaStream_t s) {
  const int smem1 = ScSmem<N, true>::kTotal, smem2 = ScSmem<N, false>::kTotal;
  static_assert(2 * (ScSmem<N, false>::kTotal + 1024) <= 228 * 1024, "two CTAs share an SM");
  auto first = state_space_chunk_kernel<N, true>;
  auto second = state_space_chunk_kernel<N, false>;
  static bool cfg_dev[64] = {false};
  bool& cfg = cfg_dev[rbhost::device_slot()];
  if (!cfg) {
    cudaError_t e = cudaFuncSetAttribute(first, cudaFuncAttributeMaxDynamicSharedMemorySize, smem1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(second, cudaFuncAttributeMaxDynamicSharedMemorySize, smem2);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  const dim3 grid(a.heads * ((a.p + kScCols - 1) / kScCols), a.num_tiles);
  if (span_state) first<<<grid, kScThreads, smem1, s>>>(a, span_state, span_decay, span);
  second<<<grid, kScThreads, smem2, s>>>(a, span_state, span_decay, span);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_state_space_chunked(const RbStateSpaceArgs* args, float* span_state, float* span_decay, int span, void* stream_v) {
  const RbStateSpaceArgs& a = *args;
  if (a.num_tiles <= 0) return 0;
  if (!a.xbc || !a.dt_raw || !a.dt_bias || !a.a_log || !a.D || !a.state || !a.y || !a.segments || !a.tiles || a.f32 || a.heads <= 0 ||
      a.groups <= 0 || a.heads % a.groups || a.p <= 0 || a.n <= 0 || a.num_slots <= 0 || a.num_tiles > 65535 || span <= 0 ||
      span % rb::kScChunk || (span_state != nullptr) != (span_decay != nullptr))
    return -1;
  if (a.n > 128 || ((a.n | a.p) & 7) || ((a.ld_xbc | a.ld_y) & 7)) return -9;
  if ((reinterpret_cast<uintptr_t>(a.xbc) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.state) |
       reinterpret_cast<uintptr_t>(span_state)) & 15)
    return -9;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.n <= 64 ? rb::sc_chunk_launch<64>(a, span_state, span_decay, span, s)
                   : rb::sc_chunk_launch<128>(a, span_state, span_decay, span, s);
}
