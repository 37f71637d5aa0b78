// Mixture-of-experts routing: router softmax + top-k, a deterministic token -> expert permutation plan whose
// expert segments are padded to whole GEMM tiles, gather / combine with the routing weights, and the backward
// passes of all of them.  The grouped expert GEMM itself is the tcgen05 kernel run over the permuted buffer
// (gemm_tcgen05.cu, grouped mode).
//
// The reference's gating picks experts as `i % E` and dispatches every token to every expert
// (crates/nn/src/moe.rs:122-141,344-348); expert-choice and shared-expert routing run on the host
// (crates/nn/src/expert_choice.rs:205-315, crates/nn/src/shared_expert.rs:279-375).
#include "moe.h"

#include <float.h>

#include "rb_common.cuh"

namespace rb {

constexpr int kMaxK = 8;

__global__ void __launch_bounds__(128)
moe_route_kernel(const float* __restrict__ logits, int T, int E, int k, int renorm, int* __restrict__ idx,
                 float* __restrict__ w, float* __restrict__ probs_out) {
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (t >= T) return;
  const float* x = logits + static_cast<long long>(t) * E;
  float v0 = lane < E ? x[lane] : -INFINITY;
  float v1 = lane + 32 < E ? x[lane + 32] : -INFINITY;
  const float mx = warp_max(fmaxf(v0, v1));
  float p0 = lane < E ? __expf(v0 - mx) : 0.f;
  float p1 = lane + 32 < E ? __expf(v1 - mx) : 0.f;
  const float inv = 1.f / warp_sum(p0 + p1);
  p0 *= inv;
  p1 *= inv;
  if (probs_out) {
    if (lane < E) probs_out[static_cast<long long>(t) * E + lane] = p0;
    if (lane + 32 < E) probs_out[static_cast<long long>(t) * E + lane + 32] = p1;
  }
  float sel_p[kMaxK];
  int sel_i[kMaxK];
  float tot = 0.f;
  float c0 = lane < E ? p0 : -1.f, c1 = lane + 32 < E ? p1 : -1.f;
  for (int j = 0; j < k; ++j) {
    // warp arg-max with ties to the lower expert index
    float bv = c0;
    int bi = lane;
    if (c1 > bv) { bv = c1; bi = lane + 32; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    sel_p[j] = bv;
    sel_i[j] = bi;
    tot += bv;
    if (bi == lane) c0 = -1.f;
    if (bi == lane + 32) c1 = -1.f;
  }
  if (lane == 0) {
    for (int j = 0; j < k; ++j) {
      idx[static_cast<long long>(t) * k + j] = sel_i[j];
      w[static_cast<long long>(t) * k + j] = renorm ? sel_p[j] / tot : sel_p[j];
    }
  }
}

__global__ void __launch_bounds__(128)
moe_route_bwd_kernel(const float* __restrict__ probs, const int* __restrict__ idx, const float* __restrict__ w,
                     const float* __restrict__ dw, const int* __restrict__ counts, int T, int E, int k, int renorm,
                     float aux_grad_scale, float* __restrict__ dlogits) {
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (t >= T) return;
  const float* p = probs + static_cast<long long>(t) * E;
  float dp[2] = {0.f, 0.f};
  // gradient through the (renormalised) selected weights
  float S = 0.f, dot = 0.f;
  for (int j = 0; j < k; ++j) {
    const int e = idx[static_cast<long long>(t) * k + j];
    S += p[e];
    dot += dw[static_cast<long long>(t) * k + j] * w[static_cast<long long>(t) * k + j];
  }
  for (int j = 0; j < k; ++j) {
    const int e = idx[static_cast<long long>(t) * k + j];
    const float g = dw[static_cast<long long>(t) * k + j];
    const float d = renorm ? (g - dot) / S : g;
    if (e == lane) dp[0] += d;
    if (e == lane + 32) dp[1] += d;
  }
  // load-balancing loss: d aux / d p[t, e] = E * f_e / T
  const float denom = static_cast<float>(T) * static_cast<float>(k);
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int e = lane + 32 * h;
    if (e < E) dp[h] += aux_grad_scale * static_cast<float>(E) * (static_cast<float>(counts[e]) / denom) / static_cast<float>(T);
  }
  // softmax backward
  const float pv0 = lane < E ? p[lane] : 0.f, pv1 = lane + 32 < E ? p[lane + 32] : 0.f;
  const float s = warp_sum(dp[0] * pv0 + dp[1] * pv1);
  if (lane < E) dlogits[static_cast<long long>(t) * E + lane] = pv0 * (dp[0] - s);
  if (lane + 32 < E) dlogits[static_cast<long long>(t) * E + lane + 32] = pv1 * (dp[1] - s);
}

// Router with group-limited choice: one warp per token, R experts per lane (expert e = lane + 32 r).  Scores are held as
// order-preserving integer keys (bits of a non-negative float + 1; 0 = not available), so an arg-max is two warp
// reductions.  Shared memory is used for the group maxima only.
template <int R>
__global__ void __launch_bounds__(128)
moe_route_groups_kernel(const float* __restrict__ logits, int T, int E, int k, int groups, int keep, int renorm, float eps,
                        int* __restrict__ idx, float* __restrict__ w) {
  extern __shared__ unsigned int route_sm[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * (blockDim.x >> 5) + warp;
  if (t >= T) return;
  const float* x = logits + static_cast<long long>(t) * E;
  float v[R];
  unsigned int key[R];
  float mx = -INFINITY, sum = 0.f;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    v[r] = lane + 32 * r < E ? x[lane + 32 * r] : -INFINITY;
    mx = fmaxf(mx, v[r]);
  }
  mx = warp_max(mx);
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const float p = lane + 32 * r < E ? __expf(v[r] - mx) : 0.f;
    key[r] = lane + 32 * r < E ? __float_as_uint(p) + 1u : 0u;
    sum += p;
  }
  const float inv = 1.f / warp_sum(sum);
  if (groups > 1 && keep < groups) {
    unsigned int* all = route_sm + warp * (E + groups);
    unsigned int* gkey = all + E;
    const int per = E / groups;
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (lane + 32 * r < E) all[lane + 32 * r] = key[r];
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      unsigned int m = 0u;
      for (int e = g * per; e < (g + 1) * per; ++e) m = max(m, all[e]);
      gkey[g] = m;
    }
    __syncwarp();
    for (int j = 0; j < keep; ++j) {                   // the best groups, ties to the lower one, end up as 0
      unsigned int bv = 0u;
      int bi = groups;
      for (int g = lane; g < groups; g += 32)
        if (gkey[g] > bv) { bv = gkey[g]; bi = g; }
      const unsigned int best = __reduce_max_sync(0xffffffffu, bv);
      const int at = __reduce_min_sync(0xffffffffu, bv == best ? bi : groups);
      if (at < groups && (at & 31) == lane) gkey[at] = 0u;
      __syncwarp();
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (lane + 32 * r < E && gkey[(lane + 32 * r) / per] != 0u) key[r] = 0u;
  }
  float tot = 0.f, mine = 0.f;                         // lane j keeps the j-th weight (written in rounds of 32)
  int mine_e = 0;
  for (int j = 0; j < k; ++j) {
    unsigned int bv = 0u;
    int bi = E;
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (key[r] > bv) { bv = key[r]; bi = lane + 32 * r; }
    const unsigned int best = __reduce_max_sync(0xffffffffu, bv);
    int at = __reduce_min_sync(0xffffffffu, bv == best ? bi : E);
    if (at >= E) at = 0;                               // nothing available (scores that are not numbers)
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (at == lane + 32 * r) key[r] = 0u;
    const float p = best ? __uint_as_float(best - 1u) * inv : 0.f;
    tot += p;
    if ((j & 31) == lane) { mine = p; mine_e = at; }
    if (((j & 31) == 31 || j == k - 1) && (j & ~31) + lane < k) {
      idx[static_cast<long long>(t) * k + (j & ~31) + lane] = mine_e;
      w[static_cast<long long>(t) * k + (j & ~31) + lane] = renorm && k <= 32 ? mine / (tot + eps) : mine;
    }
  }
  if (renorm && k > 32) {
    __syncwarp();
    for (int j = lane; j < k; j += 32) w[static_cast<long long>(t) * k + j] /= tot + eps;
  }
}

// Router with sigmoid scores: one warp per token, R experts per lane.  Choice scores can have either sign, so their keys are the
// float's bits mapped to unsigned order (0 = not available).
__device__ __forceinline__ unsigned int route_key(float v) {
  const unsigned int b = __float_as_uint(v);
  return b & 0x80000000u ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float route_unkey(unsigned int k) { return __uint_as_float(k & 0x80000000u ? k & 0x7fffffffu : ~k); }
template <int R>
__global__ void __launch_bounds__(128)
moe_route_sigmoid_kernel(const float* __restrict__ logits, const float* __restrict__ correction, int T, int E, int k, int groups, int keep,
                         int group_best, int renorm, float eps, int* __restrict__ idx, float* __restrict__ w) {
  extern __shared__ unsigned int route_sm[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * (blockDim.x >> 5) + warp;
  if (t >= T) return;
  const float* x = logits + static_cast<long long>(t) * E;
  float s[R];
  unsigned int key[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int e = lane + 32 * r;
    s[r] = e < E ? 1.f / (1.f + expf(-x[e])) : 0.f;
    key[r] = e < E ? route_key(s[r] + (correction ? correction[e] : 0.f)) : 0u;
  }
  if (groups > 1 && keep < groups) {
    unsigned int* all = route_sm + warp * (E + groups);
    unsigned int* gkey = all + E;
    const int per = E / groups;
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (lane + 32 * r < E) all[lane + 32 * r] = key[r];
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      unsigned int m0 = 0u, m1 = 0u;
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const unsigned int v = all[e];
        m1 = max(m1, min(m0, v));
        m0 = max(m0, v);
      }
      float sum = route_unkey(m0);
      if (group_best > 1 && m1 != 0u) sum += route_unkey(m1);
      gkey[g] = route_key(sum);
    }
    __syncwarp();
    for (int j = 0; j < keep; ++j) {                   // the best groups, ties to the lower one, end up as 0
      unsigned int bv = 0u;
      int bi = groups;
      for (int g = lane; g < groups; g += 32)
        if (gkey[g] > bv) { bv = gkey[g]; bi = g; }
      const unsigned int best = __reduce_max_sync(0xffffffffu, bv);
      const int at = __reduce_min_sync(0xffffffffu, bv == best ? bi : groups);
      if (at < groups && (at & 31) == lane) gkey[at] = 0u;
      __syncwarp();
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (lane + 32 * r < E && gkey[(lane + 32 * r) / per] != 0u) key[r] = 0u;
  }
  float tot = 0.f, mine = 0.f;                         // lane j keeps the j-th weight (written in rounds of 32)
  int mine_e = 0;
  for (int j = 0; j < k; ++j) {
    unsigned int bv = 0u;
    int bi = E;
    float bs = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (key[r] > bv) { bv = key[r]; bi = lane + 32 * r; bs = s[r]; }
    const unsigned int best = __reduce_max_sync(0xffffffffu, bv);
    int at = __reduce_min_sync(0xffffffffu, bv == best ? bi : E);
    if (at >= E) at = 0;                               // nothing available (scores that are not numbers)
    const float p = __shfl_sync(0xffffffffu, bs, at & 31);
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (at == lane + 32 * r) key[r] = 0u;
    tot += p;
    if ((j & 31) == lane) { mine = p; mine_e = at; }
    if (((j & 31) == 31 || j == k - 1) && (j & ~31) + lane < k) {
      idx[static_cast<long long>(t) * k + (j & ~31) + lane] = mine_e;
      w[static_cast<long long>(t) * k + (j & ~31) + lane] = renorm && k <= 32 ? mine / (tot + eps) : mine;
    }
  }
  if (renorm && k > 32) {
    __syncwarp();
    for (int j = lane; j < k; j += 32) w[static_cast<long long>(t) * k + j] /= tot + eps;
  }
}

// act(gate) * up over the rows that hold a token; ACT 0: silu, 1: relu, 2: clamped (both bounded by `limit`, up shifted by one)
template <int ACT>
__device__ __forceinline__ float glu(float g, float u, float limit) {
  if (ACT == 1) return fmaxf(g, 0.f) * u;
  if (ACT == 0) return silu(g) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f);
}
template <int ACT>
__device__ __forceinline__ float glu_exact(float g, float u, float limit) {
  if (ACT == 1) return fmaxf(g, 0.f) * u;
  if (ACT == 0) return g / (1.f + expf(-g)) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}
template <typename T, int N, int ACT>
__global__ void __launch_bounds__(256)
swiglu_slots_kernel(const T* __restrict__ gu, long long ld_gu, T* __restrict__ h, long long ld_h, int n, int F,
                    const int* __restrict__ slot_pos, const float* __restrict__ slot_w, float limit) {
  const int chunks = F / N;
  const long long total = static_cast<long long>(n) * chunks;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
    const long long s = i / chunks;
    const int c = static_cast<int>(i - s * chunks) * N;
    const long long r = slot_pos ? slot_pos[s] : s;
    const float w = slot_w ? slot_w[s] : 1.f;            // of the input of both products
    if (N == 8) {
      const uint4 g = *reinterpret_cast<const uint4*>(gu + r * ld_gu + c), u = *reinterpret_cast<const uint4*>(gu + r * ld_gu + F + c);
      const uint32_t gw[4] = {g.x, g.y, g.z, g.w}, uw[4] = {u.x, u.y, u.z, u.w};
      uint32_t o[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 a = unpack_bf16x2(gw[j]), b = unpack_bf16x2(uw[j]);
        o[j] = pack_bf16x2(glu<ACT>(w * a.x, w * b.x, limit), glu<ACT>(w * a.y, w * b.y, limit));
      }
      *reinterpret_cast<uint4*>(h + r * ld_h + c) = make_uint4(o[0], o[1], o[2], o[3]);
    } else {
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const float g = static_cast<float>(gu[r * ld_gu + c + j]), u = static_cast<float>(gu[r * ld_gu + F + c + j]);
        h[r * ld_h + c + j] = static_cast<T>(glu_exact<ACT>(w * g, w * u, limit));
      }
    }
  }
}

__global__ void __launch_bounds__(256)
moe_scatter_kernel(const uint4* __restrict__ x, const int* __restrict__ slot_pos, uint4* __restrict__ xp, int slots, int k,
                   int chunks) {
  const long long total = static_cast<long long>(slots) * chunks;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
    const long long s = i / chunks;
    const int c = static_cast<int>(i - s * chunks);
    xp[static_cast<long long>(slot_pos[s]) * chunks + c] = x[s / k * chunks + c];
  }
}

// ---- permutation plan ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(1024) moe_count_kernel(const int* __restrict__ idx, int slots, int* __restrict__ counts) {
  __shared__ int sh[32];
  const int e = blockIdx.x;
  int c = 0;
  for (int s = threadIdx.x; s < slots; s += 1024) c += (idx[s] == e);
  for (int o = 16; o > 0; o >>= 1) c += __shfl_xor_sync(0xffffffffu, c, o);
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = c;
  __syncthreads();
  if (threadIdx.x == 0) {
    int t = 0;
    for (int i = 0; i < 32; ++i) t += sh[i];
    counts[e] = t;
  }
}

// One CTA per expert: the expert's segment start from the counts of all experts, then the ranks of its slots in ascending
// order (each warp owns a contiguous range of slots and counts it with ballots, twice: once for the warp's start).  The
// CTAs also share the bookkeeping: -1 in padding rows and in the tail, the tile table, the offsets.
__global__ void __launch_bounds__(1024)
moe_assign_kernel(const int* __restrict__ idx, int slots, int E, const int* __restrict__ counts, int* __restrict__ offsets,
                  int* __restrict__ tile_expert, int* __restrict__ num_tiles, int* __restrict__ slot_pos,
                  int* __restrict__ row_slot, int max_rows) {
  __shared__ int sh_before[32], sh_all[32], warp_cnt[32];
  const int e = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  auto padded = [](int c) { return (c + RB_MOE_ROW_ALIGN - 1) / RB_MOE_ROW_ALIGN * RB_MOE_ROW_ALIGN; };
  int before = 0, all = 0;                             // rows of the experts before this one, rows of all
  for (int i = threadIdx.x; i < E; i += 1024) {
    const int p = padded(counts[i]);
    all += p;
    if (i < e) before += p;
  }
  for (int o = 16; o > 0; o >>= 1) {
    before += __shfl_xor_sync(0xffffffffu, before, o);
    all += __shfl_xor_sync(0xffffffffu, all, o);
  }
  if (lane == 0) { sh_before[warp] = before; sh_all[warp] = all; }
  // this warp's slots, 32 at a time
  const int per = (slots + 1023) / 1024 * 32;
  const int lo = min(slots, warp * per), hi = min(slots, lo + per);
  int cnt = 0;
#pragma unroll 4
  for (int s = lo; s < hi; s += 32) cnt += __popc(__ballot_sync(0xffffffffu, s + lane < hi && idx[s + lane] == e));
  if (lane == 0) warp_cnt[warp] = cnt;
  __syncthreads();
  before = all = 0;
  int rank = 0, count = 0;
  for (int i = 0; i < 32; ++i) {
    before += sh_before[i];
    all += sh_all[i];
    if (i < warp) rank += warp_cnt[i];
    count += warp_cnt[i];
  }
  rank += before;
#pragma unroll 4
  for (int s = lo; s < hi; s += 32) {
    const bool match = s + lane < hi && idx[s + lane] == e;
    const unsigned int m = __ballot_sync(0xffffffffu, match);
    if (match) {
      const int r = rank + __popc(m & ((1u << lane) - 1u));
      slot_pos[s + lane] = r;
      row_slot[r] = s + lane;
    }
    rank += __popc(m);
  }
  const int rows = padded(count);
  for (int r = before + count + threadIdx.x; r < before + rows; r += 1024) row_slot[r] = -1;
  for (int i = threadIdx.x; i < rows / 128; i += 1024) tile_expert[before / 128 + i] = e;
  for (int r = all + e * 1024 + threadIdx.x; r < max_rows; r += E * 1024) row_slot[r] = -1;
  for (int i = all / 128 + e * 1024 + threadIdx.x; i < max_rows / 128; i += E * 1024) tile_expert[i] = -1;
  if (threadIdx.x == 0) {
    offsets[e] = before;
    if (e == E - 1) { offsets[E] = all; num_tiles[0] = all / 128; }
  }
}

__global__ void __launch_bounds__(128)
moe_gather_kernel(const __nv_bfloat16* __restrict__ x, const int* __restrict__ row_slot, const float* __restrict__ slot_scale,
                  __nv_bfloat16* __restrict__ xp, int max_rows, int k, int dim, const int* __restrict__ total_rows) {
  const int chunks = dim / 8;
  const int rows = min(max_rows, total_rows[0]);
  const long long total = static_cast<long long>(rows) * chunks;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
    const int r = static_cast<int>(i / chunks);
    const int c = static_cast<int>(i - static_cast<long long>(r) * chunks) * 8;
    const int s = row_slot[r];
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (s >= 0) {
      v = *reinterpret_cast<const uint4*>(x + static_cast<long long>(s / k) * dim + c);
      if (slot_scale) {
        const float sc = slot_scale[s];
        uint32_t* pv = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = unpack_bf16x2(pv[j]);
          pv[j] = pack_bf16x2(f.x * sc, f.y * sc);
        }
      }
    }
    *reinterpret_cast<uint4*>(xp + static_cast<long long>(r) * dim + c) = v;
  }
}

__global__ void __launch_bounds__(128)
moe_combine_kernel(const __nv_bfloat16* __restrict__ yp, const int* __restrict__ slot_pos, const float* __restrict__ w,
                   const __nv_bfloat16* __restrict__ residual, __nv_bfloat16* __restrict__ y, int T, int k, int dim) {
  const int chunks = dim / 8;
  const long long total = static_cast<long long>(T) * chunks;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
    const int t = static_cast<int>(i / chunks);
    const int c = static_cast<int>(i - static_cast<long long>(t) * chunks) * 8;
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (residual) {
      const uint4 u = *reinterpret_cast<const uint4*>(residual + static_cast<long long>(t) * dim + c);
      const uint32_t* pu = reinterpret_cast<const uint32_t*>(&u);
#pragma unroll
      for (int j = 0; j < 4; ++j) { const float2 f = unpack_bf16x2(pu[j]); acc[2 * j] = f.x; acc[2 * j + 1] = f.y; }
    }
    for (int j = 0; j < k; ++j) {     // fixed order: reproducible
      const int s = t * k + j;
      const float wj = w ? w[s] : 1.f;
      const uint4 u = *reinterpret_cast<const uint4*>(yp + static_cast<long long>(slot_pos[s]) * dim + c);
      const uint32_t* pu = reinterpret_cast<const uint32_t*>(&u);
#pragma unroll
      for (int q = 0; q < 4; ++q) { const float2 f = unpack_bf16x2(pu[q]); acc[2 * q] += wj * f.x; acc[2 * q + 1] += wj * f.y; }
    }
    uint4 o;
    o.x = pack_bf16x2(acc[0], acc[1]); o.y = pack_bf16x2(acc[2], acc[3]);
    o.z = pack_bf16x2(acc[4], acc[5]); o.w = pack_bf16x2(acc[6], acc[7]);
    *reinterpret_cast<uint4*>(y + static_cast<long long>(t) * dim + c) = o;
  }
}

__global__ void __launch_bounds__(128)
moe_weight_grad_kernel(const __nv_bfloat16* __restrict__ dy, const __nv_bfloat16* __restrict__ yp, const int* __restrict__ slot_pos,
                       float* __restrict__ dw, int slots, int k, int dim) {
  const int lane = threadIdx.x & 31;
  const int s = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (s >= slots) return;
  const __nv_bfloat16* a = dy + static_cast<long long>(s / k) * dim;
  const __nv_bfloat16* b = yp + static_cast<long long>(slot_pos[s]) * dim;
  float acc = 0.f;
  for (int c = lane * 8; c < dim; c += 256) {
    const uint4 ua = *reinterpret_cast<const uint4*>(a + c), ub = *reinterpret_cast<const uint4*>(b + c);
    const uint32_t* pa = reinterpret_cast<const uint32_t*>(&ua);
    const uint32_t* pb = reinterpret_cast<const uint32_t*>(&ub);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 fa = unpack_bf16x2(pa[j]), fb = unpack_bf16x2(pb[j]);
      acc += fa.x * fb.x + fa.y * fb.y;
    }
  }
  acc = warp_sum(acc);
  if (lane == 0) dw[s] = acc;
}

inline int grid1d(long long n, int per_block) {
  long long b = (n + per_block - 1) / per_block;
  if (b > 148LL * 32) b = 148LL * 32;
  return static_cast<int>(b < 1 ? 1 : b);
}

}  // namespace rb

#define RB_ST reinterpret_cast<cudaStream_t>(stream_v)

RB_API int rb_moe_route(const float* logits, int T, int E, int k, int renorm, int* idx, float* w, float* probs_out, void* stream_v) {
  if (T <= 0 || E <= 0 || E > 64 || k <= 0 || k > rb::kMaxK || k > E) return -1;
  rb::moe_route_kernel<<<(T + 3) / 4, 128, 0, RB_ST>>>(logits, T, E, k, renorm, idx, w, probs_out);
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_route_groups(const float* logits, int T, int E, int k, int groups, int keep, int renorm, float eps,
                               int* idx, float* w, void* stream_v) {
  if (groups < 1) groups = 1;
  if (keep < 1 || keep > groups) keep = groups;
  if (T <= 0 || E <= 0 || k <= 0 || k > E || E % groups || k > keep * (E / groups)) return -1;
  const size_t smem = groups > 1 && keep < groups ? sizeof(float) * 4 * static_cast<size_t>(E + groups) : 0;
  const int grid = (T + 3) / 4;
  if (E <= 32) rb::moe_route_groups_kernel<1><<<grid, 128, smem, RB_ST>>>(logits, T, E, k, groups, keep, renorm, eps, idx, w);
  else if (E <= 64) rb::moe_route_groups_kernel<2><<<grid, 128, smem, RB_ST>>>(logits, T, E, k, groups, keep, renorm, eps, idx, w);
  else if (E <= 128) rb::moe_route_groups_kernel<4><<<grid, 128, smem, RB_ST>>>(logits, T, E, k, groups, keep, renorm, eps, idx, w);
  else if (E <= 256) rb::moe_route_groups_kernel<8><<<grid, 128, smem, RB_ST>>>(logits, T, E, k, groups, keep, renorm, eps, idx, w);
  else if (E <= 1024) rb::moe_route_groups_kernel<32><<<grid, 128, smem, RB_ST>>>(logits, T, E, k, groups, keep, renorm, eps, idx, w);
  else return -1;
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_route_sigmoid(const float* logits, const float* correction, int T, int E, int k, int groups, int keep,
                                int group_best, int renorm, float eps, int* idx, float* w, void* stream_v) {
  if (groups < 1) groups = 1;
  if (keep < 1 || keep > groups) keep = groups;
  if (T <= 0 || E <= 0 || k <= 0 || k > E || E % groups || k > keep * (E / groups) || group_best < 1 || group_best > 2) return -1;
  const size_t smem = groups > 1 && keep < groups ? sizeof(float) * 4 * static_cast<size_t>(E + groups) : 0;
  auto run = [&](auto kern) {
    kern<<<(T + 3) / 4, 128, smem, RB_ST>>>(logits, correction, T, E, k, groups, keep, group_best, renorm, eps, idx, w);
    return static_cast<int>(cudaGetLastError());
  };
  if (E <= 32) return run(rb::moe_route_sigmoid_kernel<1>);
  if (E <= 64) return run(rb::moe_route_sigmoid_kernel<2>);
  if (E <= 128) return run(rb::moe_route_sigmoid_kernel<4>);
  if (E <= 256) return run(rb::moe_route_sigmoid_kernel<8>);
  if (E <= 1024) return run(rb::moe_route_sigmoid_kernel<32>);
  return -1;
}
namespace {
template <int ACT>
int glu_launch(const void* gu, long long ld_gu, void* h, long long ld_h, int n, int F, int f32, const int* slot_pos, const float* slot_w,
               float limit, cudaStream_t s) {
  const bool vec = !f32 && !((F | ld_gu | ld_h) & 7) && !((reinterpret_cast<uintptr_t>(gu) | reinterpret_cast<uintptr_t>(h)) & 15);
  const int grid = rb::grid1d(static_cast<long long>(n) * (vec ? F / 8 : F), 256);
  if (f32)
    rb::swiglu_slots_kernel<float, 1, ACT><<<grid, 256, 0, s>>>(reinterpret_cast<const float*>(gu), ld_gu,
                                                               reinterpret_cast<float*>(h), ld_h, n, F, slot_pos, slot_w, limit);
  else if (vec)
    rb::swiglu_slots_kernel<__nv_bfloat16, 8, ACT><<<grid, 256, 0, s>>>(reinterpret_cast<const __nv_bfloat16*>(gu), ld_gu,
                                                                       reinterpret_cast<__nv_bfloat16*>(h), ld_h, n, F, slot_pos, slot_w, limit);
  else
    rb::swiglu_slots_kernel<__nv_bfloat16, 1, ACT><<<grid, 256, 0, s>>>(reinterpret_cast<const __nv_bfloat16*>(gu), ld_gu,
                                                                       reinterpret_cast<__nv_bfloat16*>(h), ld_h, n, F, slot_pos, slot_w, limit);
  return static_cast<int>(cudaGetLastError());
}
}  // namespace

RB_API int rb_swiglu_slots(const void* gu, long long ld_gu, void* h, long long ld_h, int n, int F, int f32,
                           const int* slot_pos, const float* slot_w, int act, float limit, void* stream_v) {
  if (n <= 0 || F <= 0 || act < 0 || act > 2) return -1;
  if (act == 2) return glu_launch<2>(gu, ld_gu, h, ld_h, n, F, f32, slot_pos, slot_w, limit, RB_ST);
  return act == 1 ? glu_launch<1>(gu, ld_gu, h, ld_h, n, F, f32, slot_pos, slot_w, limit, RB_ST)
                  : glu_launch<0>(gu, ld_gu, h, ld_h, n, F, f32, slot_pos, slot_w, limit, RB_ST);
}
RB_API int rb_moe_scatter(const void* x, const int* slot_pos, void* xp, int slots, int k, int dim, void* stream_v) {
  if (slots <= 0 || k <= 0 || dim <= 0 || (dim % 8)) return -1;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(xp)) & 15) return -2;
  rb::moe_scatter_kernel<<<rb::grid1d(static_cast<long long>(slots) * (dim / 8), 256), 256, 0, RB_ST>>>(
      reinterpret_cast<const uint4*>(x), slot_pos, reinterpret_cast<uint4*>(xp), slots, k, dim / 8);
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_route_bwd(const float* probs, const int* idx, const float* w, const float* dw, const int* counts, int T,
                            int E, int k, int renorm, float aux_grad_scale, float* dlogits, void* stream_v) {
  if (T <= 0 || E <= 0 || E > 64 || k <= 0 || k > rb::kMaxK) return -1;
  rb::moe_route_bwd_kernel<<<(T + 3) / 4, 128, 0, RB_ST>>>(probs, idx, w, dw, counts, T, E, k, renorm, aux_grad_scale, dlogits);
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_plan(const int* idx, int T, int E, int k, int* counts, int* offsets, int* slot_pos, int* row_slot,
                       int* tile_expert, int* num_tiles, int max_rows, void* stream_v) {
  if (T <= 0 || E <= 0 || k <= 0 || max_rows < T * k + E * RB_MOE_ROW_ALIGN || (max_rows % 128)) return -1;
  rb::moe_count_kernel<<<E, 1024, 0, RB_ST>>>(idx, T * k, counts);
  rb::moe_assign_kernel<<<E, 1024, 0, RB_ST>>>(idx, T * k, E, counts, offsets, tile_expert, num_tiles, slot_pos, row_slot, max_rows);
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_gather(const void* x, const int* row_slot, const float* slot_scale, void* xp, int max_rows, int k, int dim,
                         const int* offsets_last, void* stream_v) {
  if (max_rows <= 0 || dim <= 0 || (dim % 8) || !offsets_last) return -1;
  rb::moe_gather_kernel<<<rb::grid1d(static_cast<long long>(max_rows) * (dim / 8), 128), 128, 0, RB_ST>>>(
      reinterpret_cast<const __nv_bfloat16*>(x), row_slot, slot_scale, reinterpret_cast<__nv_bfloat16*>(xp), max_rows, k, dim,
      offsets_last);
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_combine(const void* yp, const int* slot_pos, const float* w, const void* residual, void* y, int T, int k,
                          int dim, void* stream_v) {
  if (T <= 0 || dim <= 0 || (dim % 8)) return -1;
  rb::moe_combine_kernel<<<rb::grid1d(static_cast<long long>(T) * (dim / 8), 128), 128, 0, RB_ST>>>(
      reinterpret_cast<const __nv_bfloat16*>(yp), slot_pos, w, reinterpret_cast<const __nv_bfloat16*>(residual),
      reinterpret_cast<__nv_bfloat16*>(y), T, k, dim);
  return static_cast<int>(cudaGetLastError());
}
RB_API int rb_moe_weight_grad(const void* dy, const void* yp, const int* slot_pos, float* dw, int T, int k, int dim, void* stream_v) {
  if (T <= 0 || dim <= 0 || (dim % 8)) return -1;
  rb::moe_weight_grad_kernel<<<(T * k + 3) / 4, 128, 0, RB_ST>>>(reinterpret_cast<const __nv_bfloat16*>(dy),
                                                                  reinterpret_cast<const __nv_bfloat16*>(yp), slot_pos, dw,
                                                                  T * k, k, dim);
  return static_cast<int>(cudaGetLastError());
}
