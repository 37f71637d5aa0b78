// Per-head work between the packed attention projection and the attention kernels, in one pass: RMS norm of every query
// and key head, rotary positions on them (neighbours paired, cosines and sines from a table that all layers share), mixing of the
// values with an earlier layer's values of the same token, and the append of keys and values to their cache slots.  All of it is fp32.  A group of 8 or 16 lanes owns one head of one token with 16-byte accesses;
// head sizes that are not whole vectors take the scalar form (one warp per head).
//
// Where halves of a head turn together, a lane holds the vectors of both.  Where a norm spans the whole projection, a CTA owns a token.
#include "head_prep.h"

#include "rb_common.cuh"

namespace rb {

constexpr int kHpMaxVec = 4;                       // vectors per lane: head sizes up to 512 (bf16) / 256 (fp32)

template <typename T> struct HpVec;
template <> struct HpVec<__nv_bfloat16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = unpack_bf16x2(w[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                              pack_bf16x2(v[6], v[7]));
  }
};
template <> struct HpVec<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
__device__ __forceinline__ float hp_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float hp_get(const float* p) { return *p; }
__device__ __forceinline__ void hp_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void hp_put(float* p, float v) { *p = v; }

struct HpItem {
  int kind, head;                                  // 0 query, 1 key, 2 value
};
// query heads without a norm and positions need no work at all
__host__ __device__ __forceinline__ int hp_queries(const RbHeadPrepArgs& a) { return a.q_gamma || a.rot ? a.heads : 0; }
// (u, v) at columns c, c + 1 of token t
__device__ __forceinline__ void hp_rotate(const RbHeadPrepArgs& a, long long t, int c, float& u, float& v) {
  const float2 cs = __ldg(reinterpret_cast<const float2*>(a.rot + t * a.rot_dims + c));
  const float x = u;
  u = x * cs.x - v * cs.y;
  v = v * cs.x + x * cs.y;
}
__device__ __forceinline__ HpItem hp_item(int i, const RbHeadPrepArgs& a) {
  if (i < hp_queries(a)) return {0, i};
  i -= hp_queries(a);
  if (i < a.kv_heads) return {1, i};
  return {2, i - a.kv_heads};
}

template <typename T, int LANES>
__global__ void __launch_bounds__(128)
head_prep_kernel(const RbHeadPrepArgs a RB_BOUNDS_PARAM) {
  using V = HpVec<T>;
  const int sub = threadIdx.x & (LANES - 1);
  const int items = hp_queries(a) + 2 * a.kv_heads;
  const long long total = a.tokens * items;
  const long long per_grid = static_cast<long long>(gridDim.x) * (blockDim.x / LANES);
  const long long rounds = (total + per_grid - 1) / per_grid;
  long long g = static_cast<long long>(blockIdx.x) * (blockDim.x / LANES) + threadIdx.x / LANES;
  for (long long r = 0; r < rounds; ++r, g += per_grid) {
    const bool live = g < total;                   // idle groups stay in the loop: the shuffles below are warp-wide
    const long long t = live ? g / items : 0;
    const HpItem it = hp_item(static_cast<int>(live ? g - t * items : 0), a);
    const int dim = it.kind == 2 ? a.dv : a.dk;
    const long long off = it.kind == 0 ? a.off_q : it.kind == 1 ? a.off_k : a.off_v;
    T* row = reinterpret_cast<T*>(a.p) + t * a.ld + off + static_cast<long long>(it.head) * dim;
    const T* gamma = reinterpret_cast<const T*>(it.kind == 0 ? a.q_gamma : it.kind == 1 ? a.k_gamma : nullptr);
    const int rotated = it.kind != 2 && a.rot ? a.rot_dims : 0;
    const int used = it.kind == 0 && !gamma ? rotated : dim;   // the rest of a query without a norm stays as it is
    float v[kHpMaxVec][V::N];
    float sq = 0.f;
#pragma unroll
    for (int c = 0; c < kHpMaxVec; ++c) {
      const int col = (c * LANES + sub) * V::N;
      if (live && col < used) {
        V::load(row + col, v[c]);
#pragma unroll
        for (int i = 0; i < V::N; ++i) sq += v[c][i] * v[c][i];
      }
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (!live) continue;
    const bool mixed = it.kind == 2 && a.v_first != nullptr;
    const float rstd = gamma ? rsqrtf(sq / static_cast<float>(dim) + a.eps) : 1.f;
    const float lam = mixed ? a.mix[0] : 0.f;
    const T* first = mixed ? reinterpret_cast<const T*>(a.v_first) + t * a.ld_vf + static_cast<long long>(it.head) * dim : nullptr;
    T* cache = nullptr;
    if (it.kind != 0 && a.k_cache) {
      const long long slot = a.slots[t];
      if (slot >= a.num_slots && sub == 0) RB_BOUNDS_HIT(103);       // a negative slot means "skip this token"
      if (slot >= 0 && slot < a.num_slots)
        cache = reinterpret_cast<T*>(it.kind == 1 ? a.k_cache : a.v_cache) + (slot * a.kv_heads + it.head) * dim;
    }
#pragma unroll
    for (int c = 0; c < kHpMaxVec; ++c) {
      const int col = (c * LANES + sub) * V::N;
      if (col >= used) continue;
      if (gamma) {
        float w[V::N];
        V::load(gamma + col, w);
#pragma unroll
        for (int i = 0; i < V::N; ++i) v[c][i] = v[c][i] * rstd * w[i];
      }
      if (mixed) {
        float w[V::N];
        V::load(first + col, w);
#pragma unroll
        for (int i = 0; i < V::N; ++i) v[c][i] = (1.f - lam) * v[c][i] + lam * w[i];
      }
      if (col < rotated) {
#pragma unroll
        for (int i = 0; i < V::N; i += 2)
          if (col + i < rotated) hp_rotate(a, t, col + i, v[c][i], v[c][i + 1]);
      }
      if (gamma || mixed || col < rotated) V::store(row + col, v[c]);
      if (cache) V::store(cache + col, v[c]);
    }
  }
}

// any head size and alignment: one warp per head, pair by pair
template <typename T>
__global__ void __launch_bounds__(128)
head_prep_scalar_kernel(const RbHeadPrepArgs a RB_BOUNDS_PARAM) {
  const int lane = threadIdx.x & 31;
  const int items = hp_queries(a) + 2 * a.kv_heads;
  const long long total = a.tokens * items;
  const long long stride = static_cast<long long>(gridDim.x) * (blockDim.x >> 5);
  for (long long g = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5); g < total; g += stride) {
    const long long t = g / items;
    const HpItem it = hp_item(static_cast<int>(g - t * items), a);
    const int dim = it.kind == 2 ? a.dv : a.dk;
    const long long off = it.kind == 0 ? a.off_q : it.kind == 1 ? a.off_k : a.off_v;
    T* row = reinterpret_cast<T*>(a.p) + t * a.ld + off + static_cast<long long>(it.head) * dim;
    const T* gamma = reinterpret_cast<const T*>(it.kind == 0 ? a.q_gamma : it.kind == 1 ? a.k_gamma : nullptr);
    float rstd = 1.f;
    if (gamma) {
      float sq = 0.f;
      for (int c = lane; c < dim; c += 32) { const float x = hp_get(row + c); sq += x * x; }
      rstd = rsqrtf(warp_sum(sq) / static_cast<float>(dim) + a.eps);
    }
    const bool mixed = it.kind == 2 && a.v_first != nullptr;
    const float lam = mixed ? a.mix[0] : 0.f;
    T* cache = nullptr;
    if (it.kind != 0 && a.k_cache) {
      const long long slot = a.slots[t];
      if (slot >= a.num_slots && lane == 0) RB_BOUNDS_HIT(103);
      if (slot >= 0 && slot < a.num_slots)
        cache = reinterpret_cast<T*>(it.kind == 1 ? a.k_cache : a.v_cache) + (slot * a.kv_heads + it.head) * dim;
    }
    const int rotated = it.kind != 2 && a.rot ? a.rot_dims : 0;
    for (int c = 2 * lane; c < dim; c += 64) {
      float x[2] = {0.f, 0.f};
      const int n = min(2, dim - c);
      for (int i = 0; i < n; ++i) {
        x[i] = hp_get(row + c + i);
        if (gamma) x[i] = x[i] * rstd * hp_get(gamma + c + i);
        if (mixed) x[i] = (1.f - lam) * x[i] + lam * hp_get(reinterpret_cast<const T*>(a.v_first) + t * a.ld_vf +
                                                            static_cast<long long>(it.head) * dim + c + i);
      }
      if (c < rotated) hp_rotate(a, t, c, x[0], x[1]);
      for (int i = 0; i < n; ++i) {
        hp_put(row + c + i, x[i]);
        if (cache) hp_put(cache + c + i, x[i]);
      }
    }
  }
}

// Without norms and mixing: positions and append only.  One CTA per token, a thread per vector: the rotated vectors of the queries, then
// those of the keys and the values.
template <typename T>
__global__ void __launch_bounds__(256)
head_rotate_append_kernel(const RbHeadPrepArgs a RB_BOUNDS_PARAM) {
  using V = HpVec<T>;
  const long long t = blockIdx.x;
  T* row = reinterpret_cast<T*>(a.p) + t * a.ld;
  const int rotated = a.rot ? a.rot_dims : 0;
  const int uq = (rotated + V::N - 1) / V::N, uk = a.dk / V::N, uv = a.dv / V::N;
  const int nq = a.heads * uq, nk = a.kv_heads * uk, total = nq + nk + a.kv_heads * uv;
  bool stored = false;
  long long slot = 0;
  if (a.k_cache) {
    slot = a.slots[t];
    if (slot >= a.num_slots && threadIdx.x == 0) RB_BOUNDS_HIT(103);       // a negative slot means "skip this token"
    stored = slot >= 0 && slot < a.num_slots;
  }
  for (int u = threadIdx.x; u < total; u += blockDim.x) {
    int head, col;
    T* src;
    T* dst = nullptr;
    if (u < nq) {
      head = u / uq;
      col = (u - head * uq) * V::N;
      src = row + a.off_q + head * a.dk + col;
    } else if (u < nq + nk) {
      head = (u - nq) / uk;
      col = (u - nq - head * uk) * V::N;
      src = row + a.off_k + head * a.dk + col;
      if (stored) dst = reinterpret_cast<T*>(a.k_cache) + (slot * a.kv_heads + head) * a.dk + col;
    } else {
      col = (u - nq - nk) * V::N;                                          // the value heads are contiguous on both sides
      src = row + a.off_v + col;
      if (stored) dst = reinterpret_cast<T*>(a.v_cache) + slot * a.kv_heads * a.dv + col;
    }
    const bool turn = u < nq + nk && col < rotated;
    if (!turn && !dst) continue;
    float v[V::N];
    V::load(src, v);
    if (turn) {
#pragma unroll
      for (int i = 0; i < V::N; i += 2)
        if (col + i < rotated) hp_rotate(a, t, col + i, v[i], v[i + 1]);
      V::store(src, v);
    }
    if (dst) V::store(dst, v);
  }
}

// ---- halves: numbers i and i + rot_dims / 2 of a head turn together ------------------------------------------------------------------
__host__ __device__ __forceinline__ int hp_half_items(const RbHeadPrepArgs& a) {
  return hp_queries(a) + a.kv_heads + (a.k_cache && !a.values_are_keys ? a.kv_heads : 0);
}

// A group of LANES lanes owns a head.  Its units: a vector of the first half with its partner of the second, then single vectors.
template <typename T, int LANES, int CH>
__global__ void __launch_bounds__(128)
head_half_kernel(const RbHeadPrepArgs a RB_BOUNDS_PARAM) {
  using V = HpVec<T>;
  const int sub = threadIdx.x & (LANES - 1);
  const int items = hp_half_items(a), half = a.rot ? a.rot_dims / 2 : 0, pairs = half / V::N;
  const long long total = a.tokens * items;
  const long long per_grid = static_cast<long long>(gridDim.x) * (blockDim.x / LANES);
  const long long rounds = (total + per_grid - 1) / per_grid;
  long long g = static_cast<long long>(blockIdx.x) * (blockDim.x / LANES) + threadIdx.x / LANES;
  for (long long r = 0; r < rounds; ++r, g += per_grid) {
    const bool live = g < total;                   // idle groups stay in the loop: the shuffles below are warp-wide
    const long long t = live ? g / items : 0;
    const HpItem it = hp_item(static_cast<int>(live ? g - t * items : 0), a);
    const int dim = it.kind == 2 ? a.dv : a.dk, turned = it.kind == 2 ? 0 : pairs;
    const int units = turned + (dim - 2 * turned * V::N) / V::N;
    const long long off = it.kind == 0 ? a.off_q : it.kind == 1 ? a.off_k : a.off_v;
    T* base = reinterpret_cast<T*>(a.p) + t * a.ld;
    T* row = base + off + static_cast<long long>(it.head) * dim;
    const T* gamma = reinterpret_cast<const T*>(it.kind == 0 ? a.q_gamma : it.kind == 1 ? a.k_gamma : nullptr);
    float v[CH][2][V::N];
    float sq = 0.f;
    auto column = [&](int u) { return u < turned ? u * V::N : (u + turned) * V::N; };
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int u = c * LANES + sub;
      if (!live || u >= units) continue;
      V::load(row + column(u), v[c][0]);
      if (u < turned) V::load(row + column(u) + half, v[c][1]);
#pragma unroll
      for (int i = 0; i < V::N; ++i) {
        sq += v[c][0][i] * v[c][0][i];
        if (u < turned) sq += v[c][1][i] * v[c][1][i];
      }
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (!live) continue;
    const float rstd = gamma ? rsqrtf(sq / static_cast<float>(dim) + a.eps) : 1.f;
    T *cache = nullptr, *raw = nullptr, *raw_cache = nullptr;
    if (it.kind != 0 && a.k_cache) {
      const long long slot = a.slots[t];
      if (slot >= a.num_slots && sub == 0) RB_BOUNDS_HIT(103);       // a negative slot means "skip this token"
      if (slot >= 0 && slot < a.num_slots) {
        const long long at = (slot * a.kv_heads + it.head) * dim;
        cache = reinterpret_cast<T*>(it.kind == 1 ? a.k_cache : a.v_cache) + at;
        if (a.values_are_keys) raw_cache = reinterpret_cast<T*>(a.v_cache) + at;
      }
    }
    if (it.kind == 1 && a.values_are_keys) raw = base + a.off_v + static_cast<long long>(it.head) * dim;
    const float scale = it.kind == 1 ? a.k_scale : 1.f;
    const bool changed = gamma || scale != 1.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int u = c * LANES + sub;
      if (u >= units) continue;
      const bool turn = u < turned;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (e && !turn) continue;
        const int col = column(u) + e * half;
        if (raw) V::store(raw + col, v[c][e]);
        if (raw_cache) V::store(raw_cache + col, v[c][e]);
        if (gamma) {
          float w[V::N];
          V::load(gamma + col, w);
#pragma unroll
          for (int i = 0; i < V::N; ++i) v[c][e][i] = v[c][e][i] * rstd * w[i];
        }
      }
      if (turn) {
        const float4* cs = reinterpret_cast<const float4*>(a.rot + t * a.rot_dims + 2 * column(u));
#pragma unroll
        for (int i = 0; i < V::N; i += 2) {
          const float4 f = __ldg(cs + i / 2);
          const float x0 = v[c][0][i], x1 = v[c][0][i + 1];
          v[c][0][i] = x0 * f.x - v[c][1][i] * f.y;
          v[c][1][i] = v[c][1][i] * f.x + x0 * f.y;
          v[c][0][i + 1] = x1 * f.z - v[c][1][i + 1] * f.w;
          v[c][1][i + 1] = v[c][1][i + 1] * f.z + x1 * f.w;
        }
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (e && !turn) continue;
        const int col = column(u) + e * half;
#pragma unroll
        for (int i = 0; i < V::N; ++i) v[c][e][i] *= scale;
        if (changed || turn) V::store(row + col, v[c][e]);
        if (cache) V::store(cache + col, v[c][e]);
      }
    }
  }
}

// any head size and alignment: one warp per head
template <typename T>
__global__ void __launch_bounds__(128)
head_half_scalar_kernel(const RbHeadPrepArgs a RB_BOUNDS_PARAM) {
  const int lane = threadIdx.x & 31;
  const int items = hp_half_items(a), half = a.rot ? a.rot_dims / 2 : 0;
  const long long total = a.tokens * items;
  const long long stride = static_cast<long long>(gridDim.x) * (blockDim.x >> 5);
  for (long long g = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5); g < total; g += stride) {
    const long long t = g / items;
    const HpItem it = hp_item(static_cast<int>(g - t * items), a);
    const int dim = it.kind == 2 ? a.dv : a.dk, turned = it.kind == 2 ? 0 : half;
    const long long off = it.kind == 0 ? a.off_q : it.kind == 1 ? a.off_k : a.off_v;
    T* base = reinterpret_cast<T*>(a.p) + t * a.ld;
    T* row = base + off + static_cast<long long>(it.head) * dim;
    const T* gamma = reinterpret_cast<const T*>(it.kind == 0 ? a.q_gamma : it.kind == 1 ? a.k_gamma : nullptr);
    float rstd = 1.f;
    if (gamma) {
      float sq = 0.f;
      for (int c = lane; c < dim; c += 32) { const float x = hp_get(row + c); sq += x * x; }
      rstd = rsqrtf(warp_sum(sq) / static_cast<float>(dim) + a.eps);
    }
    T *cache = nullptr, *raw = nullptr, *raw_cache = nullptr;
    if (it.kind != 0 && a.k_cache) {
      const long long slot = a.slots[t];
      if (slot >= a.num_slots && lane == 0) RB_BOUNDS_HIT(103);
      if (slot >= 0 && slot < a.num_slots) {
        const long long at = (slot * a.kv_heads + it.head) * dim;
        cache = reinterpret_cast<T*>(it.kind == 1 ? a.k_cache : a.v_cache) + at;
        if (a.values_are_keys) raw_cache = reinterpret_cast<T*>(a.v_cache) + at;
      }
    }
    if (it.kind == 1 && a.values_are_keys) raw = base + a.off_v + static_cast<long long>(it.head) * dim;
    const float scale = it.kind == 1 ? a.k_scale : 1.f;
    for (int u = lane; u < dim - turned; u += 32) {        // a number of the first half with its partner, or one behind both halves
      const bool turn = u < turned;
      const int col[2] = {turn ? u : u + turned, u + turned};
      float x[2] = {0.f, 0.f};
      for (int e = 0; e < (turn ? 2 : 1); ++e) {
        x[e] = hp_get(row + col[e]);
        if (raw) hp_put(raw + col[e], x[e]);
        if (raw_cache) hp_put(raw_cache + col[e], x[e]);
        if (gamma) x[e] = x[e] * rstd * hp_get(gamma + col[e]);
      }
      if (turn) {
        const float2 f = __ldg(reinterpret_cast<const float2*>(a.rot + t * a.rot_dims) + u);
        const float first = x[0];
        x[0] = first * f.x - x[1] * f.y;
        x[1] = x[1] * f.x + first * f.y;
      }
      for (int e = 0; e < (turn ? 2 : 1); ++e) {
        hp_put(row + col[e], x[e] * scale);
        if (cache) hp_put(cache + col[e], x[e] * scale);
      }
    }
  }
}

template <typename T>
int hp_half_launch(const RbHeadPrepArgs& a, cudaStream_t s) {
  constexpr int N = HpVec<T>::N;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.q_gamma) | reinterpret_cast<uintptr_t>(a.k_gamma) |
                         reinterpret_cast<uintptr_t>(a.k_cache) | reinterpret_cast<uintptr_t>(a.v_cache) | reinterpret_cast<uintptr_t>(a.rot);
  const int half = a.rot ? a.rot_dims / 2 : 0;
  const bool values = a.k_cache && !a.values_are_keys;
  const bool vec = !(bits & 15) && !((a.ld | a.off_q | a.off_k | a.off_v | a.dk | a.dv | half) % N);
  const int units = max((a.dk - half) / N, values ? a.dv / N : 0);
  const long long total = a.tokens * hp_half_items(a);
  auto blocks = [&](int per) { const long long b = (total + per - 1) / per; return static_cast<int>(b > 148LL * 16 ? 148LL * 16 : b); };
  if (vec && units <= 8) head_half_kernel<T, 8, 1><<<blocks(16), 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (vec && units <= 16) head_half_kernel<T, 16, 1><<<blocks(8), 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (vec && units <= 64) head_half_kernel<T, 16, 4><<<blocks(8), 128, 0, s>>>(a RB_BOUNDS_ARG);
  else head_half_scalar_kernel<T><<<blocks(4), 128, 0, s>>>(a RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

// ---- norms over whole rows -------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ float rp_temperature(const RbRowPrepArgs& a, long long t) {
  return a.temp_every > 0 ? fmaf(a.temp_coef, logf(static_cast<float>((a.pos[t] + 1) / a.temp_every + 1)), 1.f) : 1.f;
}
// two sums over the CTA; `red` holds one pair per warp
__device__ __forceinline__ float2 rp_sums(float v, float w, float2* red) {
  v = warp_sum(v);
  w = warp_sum(w);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(v, w);
  __syncthreads();
  float2 s = make_float2(0.f, 0.f);
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) { s.x += red[i].x; s.y += red[i].y; }
  return s;
}

// One CTA per token, VEC numbers per thread and step (1: any size and alignment); q and k stay in registers when CH steps hold them.
template <typename T, int VEC, int CH>
__global__ void __launch_bounds__(256)
row_prep_kernel(const RbRowPrepArgs a RB_BOUNDS_PARAM) {
  using V = HpVec<T>;
  __shared__ float2 red[8];
  const long long t = blockIdx.x;
  T* row = reinterpret_cast<T*>(a.p) + t * a.ld;
  const int nqk = a.nq + a.nk;
  auto load = [&](const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 1) v[0] = hp_get(p);
    else V::load(p, v);
  };
  auto store = [&](T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 1) hp_put(p, v[0]);
    else V::store(p, v);
  };
  long long slot = -1;
  if (a.k_cache) {
    slot = a.slots[t];
    if (slot >= a.num_slots) {
      if (threadIdx.x == 0) RB_BOUNDS_HIT(103);                      // a negative slot means "skip this token"
      slot = -1;
    }
  }
  if (slot >= 0)
    for (int col = threadIdx.x * VEC; col < a.nv; col += blockDim.x * VEC) {
      float u[VEC];
      load(row + nqk + col, u);
      store(reinterpret_cast<T*>(a.v_cache) + slot * a.nv + col, u);
    }
  float v[CH > 0 ? CH : 1][VEC];
  float sq = 0.f, sk = 0.f;
  auto square = [&](int col, const float (&u)[VEC]) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) s = fmaf(u[i], u[i], s);
    if (col < a.nq) sq += s;
    else sk += s;
  };
  if constexpr (CH > 0) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int col = (c * blockDim.x + threadIdx.x) * VEC;
      if (col >= nqk) continue;
      load(row + col, v[c]);
      square(col, v[c]);
    }
  } else {
    for (int col = threadIdx.x * VEC; col < nqk; col += blockDim.x * VEC) {
      load(row + col, v[0]);
      square(col, v[0]);
    }
  }
  const float2 sums = rp_sums(sq, sk, red);
  const float fq = rp_temperature(a, t) / sqrtf(sums.x / static_cast<float>(a.nq) + a.eps);
  const float fk = a.nk > 0 ? 1.f / sqrtf(sums.y / static_cast<float>(a.nk) + a.eps) : 0.f;
  auto finish = [&](int col, float (&u)[VEC]) {
    const bool query = col < a.nq;
    const float* gamma = query ? a.q_gamma + col : a.k_gamma + (col - a.nq);
    const float f = query ? fq : fk;
#pragma unroll
    for (int i = 0; i < VEC; ++i) u[i] = u[i] * f * gamma[i];
    store(row + col, u);
    if (!query && slot >= 0) store(reinterpret_cast<T*>(a.k_cache) + slot * a.nk + (col - a.nq), u);
  };
  if constexpr (CH > 0) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int col = (c * blockDim.x + threadIdx.x) * VEC;
      if (col < nqk) finish(col, v[c]);
    }
  } else {
    for (int col = threadIdx.x * VEC; col < nqk; col += blockDim.x * VEC) {
      load(row + col, v[0]);
      finish(col, v[0]);
    }
  }
}

template <typename T>
int rp_launch(const RbRowPrepArgs& a, cudaStream_t s) {
  constexpr int N = HpVec<T>::N;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.k_cache) | reinterpret_cast<uintptr_t>(a.v_cache);
  const int grid = static_cast<int>(a.tokens);
  if ((bits & 15) || ((a.ld | a.nq | a.nk | a.nv) % N)) {
    row_prep_kernel<T, 1, 0><<<grid, 256, 0, s>>>(a RB_BOUNDS_ARG);
    return static_cast<int>(cudaGetLastError());
  }
  const int units = (a.nq + a.nk) / N, threads = units <= 64 ? 64 : units <= 128 ? 128 : 256, ch = (units + threads - 1) / threads;
  if (ch <= 1) row_prep_kernel<T, N, 1><<<grid, threads, 0, s>>>(a RB_BOUNDS_ARG);
  else if (ch <= 2) row_prep_kernel<T, N, 2><<<grid, threads, 0, s>>>(a RB_BOUNDS_ARG);
  else if (ch <= 4) row_prep_kernel<T, N, 4><<<grid, threads, 0, s>>>(a RB_BOUNDS_ARG);
  else if (ch <= 8) row_prep_kernel<T, N, 8><<<grid, threads, 0, s>>>(a RB_BOUNDS_ARG);
  else row_prep_kernel<T, N, 0><<<grid, threads, 0, s>>>(a RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int hp_launch(const RbHeadPrepArgs& a, cudaStream_t s) {
  constexpr int N = HpVec<T>::N;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.q_gamma) |
                         reinterpret_cast<uintptr_t>(a.k_gamma) | reinterpret_cast<uintptr_t>(a.v_first) |
                         reinterpret_cast<uintptr_t>(a.k_cache) | reinterpret_cast<uintptr_t>(a.v_cache);
  const bool vec = !(bits & 15) && !((a.ld | a.off_q | a.off_k | a.off_v | a.dk | a.dv | (a.v_first ? a.ld_vf : 0)) % N) &&
                   a.dk <= 16 * N * kHpMaxVec && a.dv <= 16 * N * kHpMaxVec;
  const long long total = a.tokens * (hp_queries(a) + 2 * a.kv_heads);
  const bool narrow = a.dk <= 8 * N && a.dv <= 8 * N;        // one vector per lane of a group of 8
  const int per_block = vec ? (narrow ? 16 : 8) : 4;
  long long blocks = (total + per_block - 1) / per_block;
  if (blocks > 148LL * 16) blocks = 148LL * 16;
  const int units = (a.rot ? a.heads * ((a.rot_dims + N - 1) / N) : 0) + a.kv_heads * (a.dk + a.dv) / N;
  if (vec && !a.q_gamma && !a.k_gamma && !a.v_first && a.tokens <= 0x7fffffffLL)
    head_rotate_append_kernel<T><<<static_cast<int>(a.tokens), units <= 64 ? 64 : units <= 128 ? 128 : 256, 0, s>>>(a RB_BOUNDS_ARG);
  else if (vec && narrow)
    head_prep_kernel<T, 8><<<static_cast<int>(blocks), 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (vec)
    head_prep_kernel<T, 16><<<static_cast<int>(blocks), 128, 0, s>>>(a RB_BOUNDS_ARG);
  else
    head_prep_scalar_kernel<T><<<static_cast<int>(blocks), 128, 0, s>>>(a RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_head_prep(const RbHeadPrepArgs* args, void* stream_v) {
  const RbHeadPrepArgs& a = *args;
  if (a.tokens <= 0) return 0;
  if (!a.p || a.heads <= 0 || a.kv_heads <= 0 || a.dk <= 0 || a.dv <= 0) return -1;
  if (a.rot && (a.rot_dims <= 0 || (a.rot_dims & 1) || a.rot_dims > a.dk || (reinterpret_cast<uintptr_t>(a.rot) & 7))) return -1;
  if ((a.k_cache == nullptr) != (a.v_cache == nullptr) || (a.k_cache && !a.slots) || (a.v_first && !a.mix)) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  if (a.half) {
    if (a.v_first || (a.values_are_keys && a.dk != a.dv)) return -1;
    return a.f32 ? rb::hp_half_launch<float>(a, s) : rb::hp_half_launch<__nv_bfloat16>(a, s);
  }
  return a.f32 ? rb::hp_launch<float>(a, s) : rb::hp_launch<__nv_bfloat16>(a, s);
}

RB_API int rb_row_prep(const RbRowPrepArgs* args, void* stream_v) {
  const RbRowPrepArgs& a = *args;
  if (a.tokens <= 0) return 0;
  if (!a.p || a.nq <= 0 || a.nk < 0 || a.nv < 0 || !a.q_gamma || (a.nk > 0 && !a.k_gamma) || (a.temp_every > 0 && !a.pos) ||
      (a.k_cache == nullptr) != (a.v_cache == nullptr) || (a.k_cache && !a.slots) || a.tokens > 0x7fffffffLL)
    return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.f32 ? rb::rp_launch<float>(a, s) : rb::rp_launch<__nv_bfloat16>(a, s);
}
