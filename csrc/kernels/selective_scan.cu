// Mamba's selective scan: one step size per channel and token, one decay per channel and state number.
//
// LP lanes share a channel, each with NI of its state numbers in registers (fp32); the CC = 128 / LP channels of a CTA walk over the tokens
// of a segment.  Prompts: tiles of TT tokens, whose inputs are requested one tile ahead; step sizes (softplus) and dt x are
// formed once per channel and token in shared memory, the skip, the silu gate and the output scale are applied when the tile is stored.
// The lanes' shares of y are summed for four tokens at a time, so that every step of the sum halves what is left.  The time goes to one
// exponential per state number and token on the special-function unit and to the operands from shared memory; the products run on packed
// pairs.  Few segments take more lanes per channel and longer tiles: there a warp's latency counts.  Decoded
// rows take a form without staging, whose traffic is the state, read and written once.
//
// fp32 operands take correctly rounded decays (an error on one side, even of the last bit, adds up over a state's long memory) and plain
// arithmetic.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

constexpr int kSlThreads = 128;
constexpr float kSlLog2e = 1.4426950408889634f;

__device__ __forceinline__ float sl_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two fp32 numbers per instruction
__device__ __forceinline__ uint64_t sl_pack(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void sl_unpack(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t sl_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t sl_mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// NI numbers of a channel's state.  `rate`: A, times log2(e) where the exponential is to base 2.
template <typename T, int NI> struct SlState;
template <int NI> struct SlState<float, NI> {
  float s[NI], rate[NI];
  static constexpr float kRate = 1.f;
  __device__ __forceinline__ void set(int i, float v, float r) { s[i] = v; rate[i] = r; }
  __device__ __forceinline__ float get(int i) const { return s[i]; }
  __device__ __forceinline__ float step(float dt, float u, const float* B, const float* C) {
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      s[i] = fmaf(__double2float_rn(exp(static_cast<double>(dt * rate[i]))), s[i], u * B[i]);
      y = fmaf(s[i], C[i], y);
    }
    return y;
  }
};
template <int NI> struct SlState<__nv_bfloat16, NI> {
  uint64_t s[NI / 2], rate[NI / 2];
  static constexpr float kRate = kSlLog2e;
  __device__ __forceinline__ void set(int i, float v, float r) {
    float a, b, c, d;
    sl_unpack(s[i / 2], a, b);
    sl_unpack(rate[i / 2], c, d);
    s[i / 2] = i & 1 ? sl_pack(a, v) : sl_pack(v, b);
    rate[i / 2] = i & 1 ? sl_pack(c, r) : sl_pack(r, d);
  }
  __device__ __forceinline__ float get(int i) const {
    float a, b;
    sl_unpack(s[i / 2], a, b);
    return i & 1 ? b : a;
  }
  __device__ __forceinline__ float step(float dt, float u, const float* B, const float* C) {
    const uint64_t dt2 = sl_pack(dt, dt), u2 = sl_pack(u, u);
    uint64_t y2 = 0ull;
#pragma unroll
    for (int i = 0; i < NI / 2; ++i) {
      float lo, hi;
      sl_unpack(sl_mul2(dt2, rate[i]), lo, hi);
      s[i] = sl_fma2(sl_pack(sl_ex2(lo), sl_ex2(hi)), s[i], sl_mul2(u2, sl_pack(B[2 * i], B[2 * i + 1])));
      y2 = sl_fma2(s[i], sl_pack(C[2 * i], C[2 * i + 1]), y2);
    }
    float lo, hi;
    sl_unpack(y2, lo, hi);
    return lo + hi;
  }
};

// softplus of a step size: max(x, 0) + ln(1 + e), e = e^-|x|.  With bf16 operands ln(1 + e) = 2 atanh(e / (2 + e)) by the series of atanh,
// whose argument is at most 1/3 (relative error 2e-7).
template <typename T> __device__ __forceinline__ float sl_softplus(float x);
template <> __device__ __forceinline__ float sl_softplus<float>(float x) { return rc_softplus(x); }
template <> __device__ __forceinline__ float sl_softplus<__nv_bfloat16>(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = fmaf(q, 1.f / 15.f, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  return fmaxf(x, 0.f) + 2.f * s * fmaf(p, q, 1.f);
}

// V numbers of a channel at a time: 4, or 2 with NI 2
template <int V> struct SlMany { typedef float4 type; };
template <> struct SlMany<2> { typedef float2 type; };
// VEC: the rows of A hold whole vectors.  Loads are unconditional (numbers past the end come from the row's start and count as zero).
template <typename T, int NI, int VEC>
__device__ __forceinline__ void sl_load_state(SlState<T, NI>& S, const RbSelectiveScanArgs& a, const RcSegment& s, int c, int n0) {
  constexpr int V = NI % 4 ? 2 : 4;
  typedef typename SlMany<V>::type Many;
  const int n4 = (a.n + 3) & ~3;
  const float* st = a.state + (static_cast<long long>(s.slot) * a.inner + c) * n4;
  const float* A = a.A + static_cast<long long>(c) * a.n;
  __align__(16) float w[NI], r[NI];
#pragma unroll
  for (int q = 0; q < NI; q += V) {
    const int n = n0 + q < a.n ? n0 + q : 0;
    *reinterpret_cast<Many*>(w + q) = *reinterpret_cast<const Many*>(st + n);
    if (VEC == 4) {
      *reinterpret_cast<Many*>(r + q) = *reinterpret_cast<const Many*>(A + n);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) r[q + i] = A[n0 + q + i < a.n ? n0 + q + i : 0];
    }
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) S.set(i, s.start > 0 && n0 + i < a.n ? w[i] : 0.f, n0 + i < a.n ? r[i] * SlState<T, NI>::kRate : 0.f);
}
template <typename T, int NI>
__device__ __forceinline__ void sl_store_state(const SlState<T, NI>& S, const RbSelectiveScanArgs& a, const RcSegment& s, int c, int n0) {
  constexpr int V = NI % 4 ? 2 : 4;
  typedef typename SlMany<V>::type Many;
  const int n4 = (a.n + 3) & ~3;
  float* st = a.state + (static_cast<long long>(s.slot) * a.inner + c) * n4;
#pragma unroll
  for (int q = 0; q < NI; q += V) {
    __align__(16) float w[V];
#pragma unroll
    for (int i = 0; i < V; ++i) w[i] = S.get(q + i);
    if (n0 + q < a.n) *reinterpret_cast<Many*>(st + n0 + q) = *reinterpret_cast<const Many*>(w);
  }
}

// VEC consecutive numbers as they lie in memory
template <typename T, int VEC> struct SlRaw;
template <typename T> struct SlRaw<T, 1> {
  T r;
  __device__ __forceinline__ void load(const T* p) { r = *p; }
  __device__ __forceinline__ void get(float (&v)[1]) const { v[0] = static_cast<float>(r); }
};
template <> struct SlRaw<__nv_bfloat16, 4> {
  uint2 r;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { r = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const {
    const float2 a = unpack_bf16x2(r.x), b = unpack_bf16x2(r.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
};
template <> struct SlRaw<float, 4> {
  float4 r;
  __device__ __forceinline__ void load(const float* p) { r = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const { v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w; }
};

template <typename T, int LP, int NI, int TT, int VEC>
__global__ void __launch_bounds__(kSlThreads)
selective_scan_kernel(const RbSelectiveScanArgs a) {
  constexpr int CC = kSlThreads / LP, NP = LP * NI;
  constexpr int kPer = CC / VEC, kUnits = (TT * kPer + kSlThreads - 1) / kSlThreads;        // units of VEC channels per token, per thread
  constexpr int kStride = kSlThreads / kPer;         // tokens between a thread's units
  constexpr int kHalf = TT * NP / VEC, kBC = (2 * kHalf + kSlThreads - 1) / kSlThreads;       // pieces of B (then as many of C), per thread
  __shared__ __align__(16) float sBC[2][TT][NP];
  __shared__ __align__(16) float2 sIn[TT][CC];       // step size, dt x
  __shared__ __align__(16) float sY[TT][CC + 8];      // four tokens of a warp's channels in different banks
  const int tid = threadIdx.x, p = tid % LP, cl = tid / LP, c0 = blockIdx.x * CC, c = c0 + cl, n0 = p * NI;
  const RcSegment s = rc_segment(a.segments, blockIdx.y, a.num_slots);
  if (s.len <= 0) return;
  SlState<T, NI> S;
  sl_load_state<T, NI, VEC>(S, a, s, min(c, a.inner - 1), n0);
  const T *X = reinterpret_cast<const T*>(a.x), *Z = reinterpret_cast<const T*>(a.z), *B = reinterpret_cast<const T*>(a.B),
          *C = reinterpret_cast<const T*>(a.C);
  // a unit: channels c0 + uc .. of token ut + k * kStride of a tile
  const int uc = tid % kPer * VEC, ut = tid / kPer, at = c0 + uc < a.inner ? c0 + uc : 0;
  const bool unit = c0 + uc < a.inner;
  float bias[VEC], skip[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) { bias[i] = a.dt_bias[at + i]; skip[i] = a.D[at + i]; }
  // Loads are unconditional, from places clamped to the segment, and left as they are: nothing waits for them before the next tile.
  SlRaw<T, VEC> x[kUnits], z[kUnits], nx[kUnits], nz[kUnits], bc[kBC];
  SlRaw<float, VEC> dt[kUnits];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < kUnits; ++k) {
      const long long r = s.first + min(t0 + ut + k * kStride, s.len - 1);
      nx[k].load(X + r * a.ld_x + at);
      nz[k].load(Z + r * a.ld_z + at);
      dt[k].load(a.dt_raw + r * a.ld_dt + at);
    }
#pragma unroll
    for (int k = 0; k < kBC; ++k) {
      const int i = tid + k * kSlThreads, h = i % kHalf, n = h * VEC % NP;
      const long long r = s.first + min(t0 + h * VEC / NP, s.len - 1);
      bc[k].load((i < kHalf ? B : C) + r * a.ld_bc + (n < a.n ? n : 0));
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < s.len; t0 += TT) {
#pragma unroll
    for (int k = 0; k < kUnits; ++k) {
      x[k] = nx[k];
      z[k] = nz[k];
      const int t = ut + k * kStride;
      float xv[VEC], dv[VEC];
      x[k].get(xv);
      dt[k].get(dv);
#pragma unroll
      for (int i = 0; i < VEC; ++i) dv[i] = t0 + t < s.len ? sl_softplus<T>(dv[i] + bias[i]) : 0.f;     // a step of 0 leaves the state as it is
      if (t < TT) {
        if constexpr (VEC == 4) {
          float4* dst = reinterpret_cast<float4*>(&sIn[t][uc]);
          dst[0] = make_float4(dv[0], dv[0] * xv[0], dv[1], dv[1] * xv[1]);
          dst[1] = make_float4(dv[2], dv[2] * xv[2], dv[3], dv[3] * xv[3]);
        } else {
          sIn[t][uc] = make_float2(dv[0], dv[0] * xv[0]);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < kBC; ++k) {
      const int i = tid + k * kSlThreads, n = i % kHalf * VEC % NP;
      float v[VEC];
      bc[k].get(v);
#pragma unroll
      for (int q = 0; q < VEC; ++q) v[q] = n + q < a.n ? v[q] : 0.f;
      if (i < 2 * kHalf) RcVec<float, VEC>::store(&sBC[0][0][0] + i * VEC, v);
    }
    __syncthreads();
    if (t0 + TT < s.len) fetch(t0 + TT);
#pragma unroll
    for (int t = 0; t < TT; t += 4) {
      constexpr int V = NI % 4 ? 2 : 4;
      typedef typename SlMany<V>::type Many;
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        __align__(16) float vb[NI], vc[NI];
        const float2 in = sIn[t + k][cl];
#pragma unroll
        for (int q = 0; q < NI; q += V) {
          *reinterpret_cast<Many*>(vb + q) = *reinterpret_cast<const Many*>(&sBC[0][t + k][n0 + q]);
          *reinterpret_cast<Many*>(vc + q) = *reinterpret_cast<const Many*>(&sBC[1][t + k][n0 + q]);
        }
        y[k] = S.step(in.x, in.y, vb, vc);
      }
      if constexpr (LP == 1) {
#pragma unroll
        for (int k = 0; k < 4; ++k) sY[t + k][cl] = y[k];
      } else {
        const bool hi = p & 1;                       // this lane goes on with tokens 2, 3 instead of 0, 1
        const float v0 = (hi ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, hi ? y[0] : y[2], 1);
        const float v1 = (hi ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, hi ? y[1] : y[3], 1);
        if constexpr (LP == 2) {
          sY[t + 2 * hi][cl] = v0;
          sY[t + 2 * hi + 1][cl] = v1;
        } else {
          const bool odd = p & 2;                    // with the second of its two
          float v = (odd ? v1 : v0) + __shfl_xor_sync(0xffffffffu, odd ? v0 : v1, 2);
#pragma unroll
          for (int o = 4; o < LP; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (p < 4) sY[t + 2 * hi + odd][cl] = v;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kUnits; ++k) {
      const int t = ut + k * kStride;
      if (!unit || t >= TT || t0 + t >= s.len) continue;
      float xv[VEC], zv[VEC], o[VEC];
      x[k].get(xv);
      z[k].get(zv);
      RcVec<float, VEC>::load(&sY[t][uc], o);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = a.scale * fmaf(skip[i], xv[i], o[i]) * rc_silu<T>(zv[i]);
      RcVec<T, VEC>::store(reinterpret_cast<T*>(a.y) + (s.first + t0 + t) * a.ld_y + at, o);
    }
  }
  if (c < a.inner) sl_store_state(S, a, s, c, n0);
}

// Segments of one row.  A thread takes NE channels, whose loads are all requested before the first is needed.
template <typename T, int LP, int NI, int NE, int VEC>
__global__ void __launch_bounds__(kSlThreads)
selective_step_kernel(const RbSelectiveScanArgs a) {
  constexpr int CC = kSlThreads / LP;
  const int p = threadIdx.x % LP, cl = blockIdx.x * CC * NE + threadIdx.x / LP, n0 = p * NI;
  const RcSegment s = rc_segment(a.segments, blockIdx.y, a.num_slots);
  if (s.len <= 0) return;
  const long long r = s.first;
  SlState<T, NI> S[NE];
  T x[NE], z[NE];
  float raw[NE], skip[NE], b[NI], cc[NI];
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int c = min(cl + e * CC, a.inner - 1);     // idle lanes stay for the shuffles
    sl_load_state<T, NI, VEC>(S[e], a, s, c, n0);
    x[e] = reinterpret_cast<const T*>(a.x)[r * a.ld_x + c];
    z[e] = reinterpret_cast<const T*>(a.z)[r * a.ld_z + c];
    raw[e] = a.dt_raw[r * a.ld_dt + c] + a.dt_bias[c];
    skip[e] = a.D[c];
  }
  SlRaw<T, VEC> vb[NI / VEC > 0 ? NI / VEC : 1], vc[NI / VEC > 0 ? NI / VEC : 1];
#pragma unroll
  for (int q = 0; q < NI / VEC; ++q) {
    const int n = n0 + q * VEC < a.n ? n0 + q * VEC : 0;
    vb[q].load(reinterpret_cast<const T*>(a.B) + r * a.ld_bc + n);
    vc[q].load(reinterpret_cast<const T*>(a.C) + r * a.ld_bc + n);
  }
#pragma unroll
  for (int q = 0; q < NI / VEC; ++q) {
    float u[VEC], w[VEC];
    vb[q].get(u);
    vc[q].get(w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      b[q * VEC + i] = n0 + q * VEC + i < a.n ? u[i] : 0.f;
      cc[q * VEC + i] = n0 + q * VEC + i < a.n ? w[i] : 0.f;
    }
  }
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int c = cl + e * CC;
    const float dt = sl_softplus<T>(raw[e]), xv = static_cast<float>(x[e]);
    float y = S[e].step(dt, dt * xv, b, cc);
#pragma unroll
    for (int o = 1; o < LP; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (c >= a.inner) continue;
    sl_store_state(S[e], a, s, c, n0);
    if (p == 0) rc_put(reinterpret_cast<T*>(a.y) + r * a.ld_y + c, a.scale * fmaf(skip[e], xv, y) * rc_silu<T>(static_cast<float>(z[e])));
  }
}

template <typename T, int LP, int NI, int TT>
int sl_scan(const RbSelectiveScanArgs& a, bool vec, cudaStream_t s) {
  constexpr int CC = kSlThreads / LP;
  const dim3 grid((a.inner + CC - 1) / CC, a.num_segments);
  if (vec) selective_scan_kernel<T, LP, NI, TT, 4><<<grid, kSlThreads, 0, s>>>(a);
  else selective_scan_kernel<T, LP, NI, TT, 1><<<grid, kSlThreads, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int LP, int NI, int NE>
int sl_step(const RbSelectiveScanArgs& a, bool vec, cudaStream_t s) {
  constexpr int CC = NE * kSlThreads / LP;
  const dim3 grid((a.inner + CC - 1) / CC, a.num_segments);
  if (vec) selective_step_kernel<T, LP, NI, NE, 4><<<grid, kSlThreads, 0, s>>>(a);
  else selective_step_kernel<T, LP, NI, NE, 1><<<grid, kSlThreads, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int sl_pick(const RbSelectiveScanArgs& a, cudaStream_t s) {
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.y) |
                         reinterpret_cast<uintptr_t>(a.B) | reinterpret_cast<uintptr_t>(a.C);
  const bool vec = !(bits & (4 * sizeof(T) - 1)) && !((reinterpret_cast<uintptr_t>(a.dt_raw) | reinterpret_cast<uintptr_t>(a.A)) & 15) &&
                   !((a.ld_x | a.ld_z | a.ld_bc | a.ld_dt | a.ld_y | a.inner | a.n) & 3);
  if (a.single) {
    if (a.n <= 4) return sl_step<T, 1, 4, 1>(a, vec, s);
    if (a.n <= 8) return sl_step<T, 2, 4, 1>(a, vec, s);
    if (a.n <= 16) return sl_step<T, 4, 4, 2>(a, vec, s);
    if (a.n <= 32) return sl_step<T, 8, 4, 2>(a, vec, s);
    if (a.n <= 64) return sl_step<T, 16, 4, 2>(a, vec, s);
    if (a.n <= 128) return sl_step<T, 32, 4, 2>(a, vec, s);
    return sl_step<T, 32, 8, 1>(a, vec, s);
  }
  // channels of all segments in 4 state numbers per lane: less than two warps for every scheduler?
  const bool few = static_cast<long long>(a.inner) * a.num_segments * (a.n <= 16 ? 4 : 8) < 148LL * 4 * 32 * 2;
  if (a.n <= 4) return sl_scan<T, 1, 4, 16>(a, vec, s);
  if (a.n <= 8) return sl_scan<T, 2, 4, 16>(a, vec, s);
  if (a.n <= 16) return few ? sl_scan<T, 8, 2, 64>(a, vec, s) : sl_scan<T, 4, 4, 32>(a, vec, s);
  if (a.n <= 32) return few ? sl_scan<T, 8, 4, 64>(a, vec, s) : sl_scan<T, 4, 8, 32>(a, vec, s);
  if (a.n <= 64) return sl_scan<T, 8, 8, 16>(a, vec, s);
  if (a.n <= 128) return sl_scan<T, 16, 8, 16>(a, vec, s);
  return sl_scan<T, 16, 16, 8>(a, vec, s);
}

}  // namespace rb

RB_API int rb_selective_scan(const RbSelectiveScanArgs* args, void* stream_v) {
  const RbSelectiveScanArgs& a = *args;
  if (a.num_segments <= 0) return 0;
  if (!a.x || !a.z || !a.B || !a.C || !a.dt_raw || !a.dt_bias || !a.A || !a.D || !a.state || !a.y || !a.segments || a.inner <= 0 || a.n <= 0 ||
      a.n > 256 || a.num_slots <= 0 || a.num_segments > 65535)
    return -1;
  if (reinterpret_cast<uintptr_t>(a.state) & 15) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.f32 ? rb::sl_pick<float>(a, s) : rb::sl_pick<__nv_bfloat16>(a, s);
}
