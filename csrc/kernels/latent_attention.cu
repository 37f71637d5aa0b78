// Latent attention: what stands between its matrix products, and decoding on the cached vectors.
//
// Decoding never forms the heads' keys and values.  A head's query is multiplied by its key product once (rb_head_product), scores are
// taken against the cached vectors themselves, the weighted sum of the vectors goes through the head's value product.  All heads share
// one "key" of rank + rot numbers per token whose first `rank` are the "value" too, so every cached byte is read once for both.  Prompts
// form keys and values (attention_fwd2.cu takes the shared rotated part as it is).
#include "latent_attention.h"

#include "latent_common.cuh"
#include "rb_common.cuh"
#include "warp_mma.cuh"

namespace rb {

__device__ __forceinline__ float la_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float la_get(const float* p) { return *p; }
__device__ __forceinline__ void la_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void la_put(float* p, float v) { *p = v; }

template <typename T, int VEC> struct LaVec {
  static __device__ __forceinline__ void load(const T* p, float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = la_get(p + i);
  }
  static __device__ __forceinline__ void store(T* p, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) la_put(p + i, v[i]);
  }
};
template <> struct LaVec<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = unpack_bf16x2(w[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  }
};

// ---- norms, positions, append: one CTA per token, values stay in registers between the sum and the store ---------------------------
template <typename T, int VEC, int CH>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const RbLatentPrepArgs a RB_BOUNDS_PARAM) {
  using V = LaVec<T, VEC>;
  __shared__ float2 red[4];
  const long long t = blockIdx.x;
  T* row = reinterpret_cast<T*>(a.p) + t * a.ld;
  const int units_q = (a.q_rank + VEC - 1) / VEC, units_c = (a.rank + VEC - 1) / VEC;
  float v[CH][VEC];
  float sq = 0.f, sc = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {                      // units: the query latent's, then the cached vector's
    const int u = c * 128 + threadIdx.x;
    if (u < units_q) {
      V::load(row + a.off_q + u * VEC, v[c]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) sq = fmaf(v[c][i], v[c][i], sq);
    } else if (u < units_q + units_c) {
      V::load(row + a.off_kv + (u - units_q) * VEC, v[c]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) sc = fmaf(v[c][i], v[c][i], sc);
    }
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(sq, sc);
  __syncthreads();
  sq = red[0].x + red[1].x + red[2].x + red[3].x;
  sc = red[0].y + red[1].y + red[2].y + red[3].y;
  const float rq = 1.f / sqrtf(sq / static_cast<float>(a.q_rank) + a.eps), rc = 1.f / sqrtf(sc / static_cast<float>(a.rank) + a.eps);
  T* cache = nullptr;
  if (a.cache) {
    const long long slot = a.slots[t];
    if (slot >= a.num_slots && threadIdx.x == 0) RB_BOUNDS_HIT(103);      // a negative slot means "skip this token"
    if (slot >= 0 && slot < a.num_slots) cache = reinterpret_cast<T*>(a.cache) + slot * (a.rank + a.rot);
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int u = c * 128 + threadIdx.x;
    if (u >= units_q + units_c) continue;
    const bool is_q = u < units_q;
    const int col = (is_q ? u : u - units_q) * VEC;
    const float* g = (is_q ? a.q_gamma : a.kv_gamma) + col;
    const float r = is_q ? rq : rc;
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[c][i] *= r * __ldg(g + i);
    V::store(row + (is_q ? a.off_q : a.off_kv) + col, v[c]);
    if (!is_q && cache) V::store(cache + col, v[c]);
  }
  // the rotated part: pairs, then what is left of it
  T* kr = row + a.off_kv + a.rank;
  for (int c = 2 * threadIdx.x; c < a.rot; c += 256) {
    float x[2] = {la_get(kr + c), c + 1 < a.rot ? la_get(kr + c + 1) : 0.f};
    if (c < 2 * a.pairs) {
      const float2 cs = __ldg(reinterpret_cast<const float2*>(a.table) + t * a.pairs + c / 2);
      const float u = x[0];
      x[0] = u * cs.x - x[1] * cs.y;
      x[1] = x[1] * cs.x + u * cs.y;
    }
    for (int i = 0; i < 2 && c + i < a.rot; ++i) {
      la_put(kr + c + i, x[i]);
      if (cache) la_put(cache + a.rank + c + i, x[i]);
    }
  }
}

template <typename T, int VEC>
int lp_launch(const RbLatentPrepArgs& a, cudaStream_t s) {
  const int units = (a.q_rank + VEC - 1) / VEC + (a.rank + VEC - 1) / VEC;
  const int grid = static_cast<int>(a.tokens);
  if (units <= 128) latent_prep_kernel<T, VEC, 1><<<grid, 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (units <= 256) latent_prep_kernel<T, VEC, 2><<<grid, 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (units <= 512) latent_prep_kernel<T, VEC, 4><<<grid, 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (units <= 1024) latent_prep_kernel<T, VEC, 8><<<grid, 128, 0, s>>>(a RB_BOUNDS_ARG);
  else if (units <= 4096) latent_prep_kernel<T, VEC, 32><<<grid, 128, 0, s>>>(a RB_BOUNDS_ARG);
  else return -6;
  return static_cast<int>(cudaGetLastError());
}

// ---- one small product per head ------------------------------------------------------------------------------------------------
// 64 tokens x BN columns of one head per CTA, 64-deep slices through a ring of shared-memory stages, a warp owns 16 tokens.  Batches of
// decoded tokens are far smaller than a tcgen05 tile's 128 rows per head; the kernel is bound by reading the weights.
constexpr int kHpRows = 64, kHpK = 64, kHpPitch = 72;

template <int BN, bool TR>
struct HpSmem {
  static constexpr int kStages = BN == 32 ? 8 : 4;       // narrow tiles serve few heads: depth instead of CTAs
  static constexpr int kWRows = TR ? kHpK : BN, kWPitch = TR ? BN + 8 : kHpPitch;
  static constexpr int kX = kHpRows * kHpPitch, kStage = kX + kWRows * kWPitch;
  static constexpr int kBytes = kStages * kStage * 2;
};

template <int BN, bool TR>
__global__ void __launch_bounds__(128)
head_product_kernel(const RbHeadProductArgs a) {
  using S = HpSmem<BN, TR>;
  extern __shared__ __align__(16) __nv_bfloat16 hp_sm[];
  const int h = blockIdx.y, n0 = blockIdx.x * BN, r0 = blockIdx.z * kHpRows;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* X = reinterpret_cast<const __nv_bfloat16*>(a.x) + h * a.x_head;
  const __nv_bfloat16* W = reinterpret_cast<const __nv_bfloat16*>(a.w) + h * a.w_head;
  const int steps = (a.k + kHpK - 1) / kHpK;
  auto request = [&](int st) {
    if (st < steps) {
      __nv_bfloat16* xs = hp_sm + (st % S::kStages) * S::kStage;
      const uint32_t xb = smem_u32(xs), wb = smem_u32(xs + S::kX);
      const int k0 = st * kHpK;
#pragma unroll
      for (int i = 0; i < kHpRows * 8 / 128; ++i) {
        const int idx = i * 128 + threadIdx.x, r = idx >> 3, c = (idx & 7) * 8;
        const bool ok = r0 + r < a.rows && k0 + c < a.k;
        wm_cp16(xb + (r * kHpPitch + c) * 2, ok ? X + static_cast<long long>(r0 + r) * a.ld_x + k0 + c : X, ok);
      }
      constexpr int PER = S::kWPitch / 8 - 1;            // 16-byte pieces per row of the weight slice
#pragma unroll
      for (int i = 0; i < S::kWRows * PER / 128; ++i) {
        const int idx = i * 128 + threadIdx.x, r = idx / PER, c = (idx - r * PER) * 8;
        const int n = TR ? n0 + c : n0 + r, k = TR ? k0 + r : k0 + c;
        const bool ok = n < a.n && k < a.k;
        wm_cp16(wb + (r * S::kWPitch + c) * 2, ok ? W + (TR ? k * a.ld_w + n : n * a.ld_w + k) : W, ok);
      }
    }
    wm_cp_commit();
  };
  float acc[BN / 8][4];
#pragma unroll
  for (int i = 0; i < BN / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < S::kStages - 1; ++i) request(i);
  const bool active = r0 + warp * 16 < a.rows;
  const int g = lane >> 2, tq = lane & 3;
  const __nv_bfloat16* G = a.gate ? reinterpret_cast<const __nv_bfloat16*>(a.gate) + static_cast<long long>(h) * a.n : nullptr;
  uint32_t gates[BN / 8][2];                             // requested under the first slices
#pragma unroll
  for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int n = n0 + nt * 8 + 2 * tq, r = r0 + warp * 16 + g + 8 * half;
      gates[nt][half] = G && n < a.n && r < a.rows ? *reinterpret_cast<const uint32_t*>(G + r * a.ld_g + n) : 0u;
    }
  for (int st = 0; st < steps; ++st) {
    wm_cp_wait<S::kStages - 2>();
    __syncthreads();                                     // slice st has landed for everyone, slice st - 1 is no longer read
    request(st + S::kStages - 1);
    if (!active) continue;
    const uint32_t xb = smem_u32(hp_sm + (st % S::kStages) * S::kStage), wb = xb + S::kX * 2;
#pragma unroll
    for (int k0 = 0; k0 < kHpK; k0 += 16) {
      uint32_t af[4];
      wm_ldsm_x4(wm_a(xb, kHpPitch, warp * 16, k0, lane), af);
#pragma unroll
      for (int nb = 0; nb < BN / 16; ++nb) {
        uint32_t bf[4];
        if (TR) wm_ldsm_x4_t(wm_b_t(wb, S::kWPitch, nb * 16, k0, lane), bf);
        else wm_ldsm_x4(wm_b(wb, S::kWPitch, nb * 16, k0, lane), bf);
        wm_mma(acc[2 * nb], af, bf[0], bf[1]);
        wm_mma(acc[2 * nb + 1], af, bf[2], bf[3]);
      }
    }
  }
  __nv_bfloat16* Y = reinterpret_cast<__nv_bfloat16*>(a.y) + h * a.y_head;
#pragma unroll
  for (int nt = 0; nt < BN / 8; ++nt) {
    const int n = n0 + nt * 8 + 2 * tq;
    if (n >= a.n) continue;                              // n is a multiple of 8
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = r0 + warp * 16 + g + 8 * half;
      if (r >= a.rows) continue;
      float u = acc[nt][2 * half], v = acc[nt][2 * half + 1];
      if (G) {
        const float2 z = unpack_bf16x2(gates[nt][half]);
        u = __fdividef(u, 1.f + __expf(-z.x));
        v = __fdividef(v, 1.f + __expf(-z.y));
      }
      *reinterpret_cast<uint32_t*>(Y + r * a.ld_y + n) = pack_bf16x2(u, v);
    }
  }
  if (a.tail) {                                          // 8 columns of one row per thread, spread over the head's CTAs
    const int units = a.tail / 8, total = min(kHpRows, a.rows - r0) * units;
    for (int i = blockIdx.x * 128 + threadIdx.x; i < total; i += gridDim.x * 128) {
      const int r = r0 + i / units, c = i % units * 8;
      uint4 u = *reinterpret_cast<const uint4*>(X + r * a.ld_x + a.tail_off + c);
      uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (c / 2 + q >= a.pairs) break;
        const float2 cs = __ldg(reinterpret_cast<const float2*>(a.table) + static_cast<long long>(r) * a.pairs + c / 2 + q);
        const float2 z = unpack_bf16x2(w[q]);
        w[q] = pack_bf16x2(z.x * cs.x - z.y * cs.y, z.y * cs.x + z.x * cs.y);
      }
      *reinterpret_cast<uint4*>(Y + r * a.ld_y + a.n + c) = u;
    }
  }
}

template <int BN, bool TR>
int hp_run(const RbHeadProductArgs& a, cudaStream_t s) {
  auto kern = head_product_kernel<BN, TR>;
  constexpr int smem = HpSmem<BN, TR>::kBytes;
  static bool cfg[64] = {};
  bool& done = cfg[rbhost::device_slot()];
  if (!done) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    done = true;
  }
  kern<<<dim3((a.n + BN - 1) / BN, a.heads, (a.rows + kHpRows - 1) / kHpRows), 128, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// any sizes, bf16 or fp32: one thread per output
template <typename T>
__global__ void __launch_bounds__(128)
head_product_plain_kernel(const RbHeadProductArgs a) {
  const int width = a.n + a.tail;
  const long long total = static_cast<long long>(a.rows) * a.heads * width;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
    const int n = static_cast<int>(i % width), h = static_cast<int>(i / width % a.heads);
    const long long t = i / width / a.heads;
    const T* x = reinterpret_cast<const T*>(a.x) + t * a.ld_x + h * a.x_head;
    float v = 0.f;
    if (n < a.n) {
      const T* w = reinterpret_cast<const T*>(a.w) + h * a.w_head;
      for (int k = 0; k < a.k; ++k) v = fmaf(la_get(x + k), la_get(w + (a.transposed ? k * a.ld_w + n : n * a.ld_w + k)), v);
      if (a.gate) v /= 1.f + expf(-la_get(reinterpret_cast<const T*>(a.gate) + t * a.ld_g + static_cast<long long>(h) * a.n + n));
    } else {
      const int c = n - a.n;
      v = la_get(x + a.tail_off + c);
      if (c < 2 * a.pairs) {
        const float2 cs = __ldg(reinterpret_cast<const float2*>(a.table) + t * a.pairs + c / 2);
        const float o = la_get(x + a.tail_off + (c ^ 1));
        v = c & 1 ? v * cs.x + o * cs.y : v * cs.x - o * cs.y;
      }
    }
    la_put(reinterpret_cast<T*>(a.y) + t * a.ld_y + h * a.y_head + n, v);
  }
}

// ---- decode: page sizes and rotated parts that latent_decode_tc.cu does not take --------------------------------------------------------
// One CTA = (slice of the context, sequence, 16 MT heads).  64 tokens at a time are copied into one of two shared-memory tiles (the next
// tile flies while this one is used) and serve all heads, for the scores and for the weighted sum.
//   scores: the warps form 4 groups over the columns times 2 over the tokens; a warp's share of the queries stays in registers, the
//           column groups' partial sums meet in shared memory
//   softmax: 16 (MT 1) or 8 (MT 2) threads per head, running maximum and sum in registers
//   sum:    a warp owns VW columns of the vectors for all heads and tokens
// A second kernel merges the slices.
constexpr int kLdTile = 64, kLdWarps = 8;

template <int MT>
struct LdSmem {
  static constexpr int kRows = 16 * MT;
  static constexpr int kScorePitch = kLdTile + 4, kProbPitch = kLdTile + 8;
  static constexpr int kScores = 4 * kRows * kScorePitch * 4;      // bytes
  static constexpr int kProbs = kRows * kProbPitch * 2;
  static int bytes(int width16) { return 2 * kLdTile * (width16 + 8) * 2 + kScores + kProbs + kRows * 4; }
};

template <int MT, int VW, int KMAX>
__global__ void __launch_bounds__(kLdWarps * 32, 1)
latent_decode_kernel(const RbLatentDecodeArgs a, int nsplit RB_BOUNDS_PARAM) {
  using S = LdSmem<MT>;
  extern __shared__ __align__(16) uint8_t ld_sm[];
  const int width = a.rank + a.rot, width16 = (width + 15) / 16 * 16, pitch = width16 + 8;
  const int tile_bytes = kLdTile * pitch * 2;
  float* scores = reinterpret_cast<float*>(ld_sm + 2 * tile_bytes);
  __nv_bfloat16* probs = reinterpret_cast<__nv_bfloat16*>(ld_sm + 2 * tile_bytes + S::kScores);
  float* alpha_sh = reinterpret_cast<float*>(ld_sm + 2 * tile_bytes + S::kScores + S::kProbs);
  const uint32_t tiles = smem_u32(ld_sm), probs_u32 = smem_u32(probs);
  const int sp = blockIdx.y, b = blockIdx.z, h0 = blockIdx.x * S::kRows;   // a slice's head groups are neighbours: they meet in L2
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gq = lane >> 2, tq = lane & 3;
  const int ctx = a.context_lens[b];
  const int slice = latent_chunk(ctx, nsplit);
  const int t_begin = sp * slice;
  if (t_begin >= ctx) return;
  const int t_end = min(ctx, t_begin + slice);
  const int nheads = min(S::kRows, a.heads - h0);
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache);
  const int* table = a.block_tables + static_cast<long long>(b) * a.max_blocks;

  // a warp copies 8 tokens of a tile, 16 bytes per lane at a time
  const int pieces = width16 / 8;
  auto request = [&](int first, int buf) {
    const int tok = first + warp * 8 + (lane & 7);
    int slot = -1;
    if (tok < t_end) {
      const int bi = tok / a.block_size;
      int blk = bi < a.max_blocks ? table[bi] : -1;
      if (blk < 0 || blk >= a.num_blocks) {                          // corrupt tables read block 0 instead of faulting
        RB_BOUNDS_HIT(104);
        blk = 0;
      }
      slot = blk * a.block_size + (tok - bi * a.block_size);
    }
    const uint32_t dst = tiles + buf * tile_bytes + warp * 8 * pitch * 2;
    int r = 0, c = lane;
    const int rounds = (8 * pieces + 31) / 32;
    for (int i = 0; i < rounds; ++i, c += 32) {
      while (c >= pieces) { c -= pieces; ++r; }
      const int s = __shfl_sync(0xffffffffu, slot, r & 7);
      if (r < 8) {
        const bool ok = s >= 0 && c * 8 < width;
        wm_cp16(dst + (r * pitch + c * 8) * 2, ok ? cache + static_cast<long long>(s) * width + c * 8 : cache, ok);
      }
    }
  };
  request(t_begin, 0);
  wm_cp_commit();

  // this warp's share of the queries as A fragments: columns [16 kb, 16 (kb + kn))
  const int kg = warp & 3, tg = warp >> 2;
  const int ksteps = width16 / 16, per = (ksteps + 3) / 4;
  const int kb = min(kg * per, ksteps), kn = min(per, ksteps - kb);
  uint32_t qf[MT][KMAX][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int ks = 0; ks < KMAX; ++ks)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int head = m * 16 + gq + (j & 1) * 8, col = (kb + ks) * 16 + 2 * tq + (j >> 1) * 8;
        qf[m][ks][j] = ks < kn && head < nheads && col < width
                           ? __ldg(reinterpret_cast<const uint32_t*>(reinterpret_cast<const __nv_bfloat16*>(a.q) + b * a.ld_q +
                                                                     static_cast<long long>(h0 + head) * width + col))
                           : 0u;
      }

  constexpr int TPH = kLdWarps * 32 / S::kRows;        // threads per head in the softmax
  constexpr int CPT = kLdTile / TPH;                   // scores per thread
  const int sm_row = threadIdx.x / TPH, sm_c = (threadIdx.x % TPH) * CPT;
  float m_run = -INFINITY, l_run = 0.f;
  const float sl2 = a.scale * 1.4426950408889634f;
  constexpr int NT = VW / 8;
  const bool summing = warp * VW < a.rank;
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;

  int buf = 0;
  for (int base = t_begin; base < t_end; base += kLdTile, buf ^= 1) {
    wm_cp_wait<0>();
    __syncthreads();                                   // this tile has landed; nobody reads the other one any more
    if (base + kLdTile < t_end) request(base + kLdTile, buf ^ 1);
    wm_cp_commit();
    const uint32_t tile = tiles + buf * tile_bytes;
    // ---- partial scores of 32 tokens over this warp's columns
    float s[MT][4][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n) s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KMAX; ++ks) {
      if (ks < kn) {
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t bf[4];
          wm_ldsm_x4(wm_b(tile, pitch, tg * 32 + np * 16, (kb + ks) * 16, lane), bf);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            wm_mma(s[m][2 * np], qf[m][ks], bf[0], bf[1]);
            wm_mma(s[m][2 * np + 1], qf[m][ks], bf[2], bf[3]);
          }
        }
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        float* p = scores + (kg * S::kRows + m * 16 + gq) * S::kScorePitch + tg * 32 + n * 8 + 2 * tq;
        *reinterpret_cast<float2*>(p) = make_float2(s[m][n][0], s[m][n][1]);
        *reinterpret_cast<float2*>(p + 8 * S::kScorePitch) = make_float2(s[m][n][2], s[m][n][3]);
      }
    __syncthreads();
    // ---- softmax over the tile
    {
      float x[CPT];
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < CPT; i += 4) {
        const float* p = scores + sm_row * S::kScorePitch + sm_c + i;
        float4 v = *reinterpret_cast<const float4*>(p);
#pragma unroll
        for (int g = 1; g < 4; ++g) {
          const float4 w = *reinterpret_cast<const float4*>(p + g * S::kRows * S::kScorePitch);
          v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
        }
        x[i] = v.x; x[i + 1] = v.y; x[i + 2] = v.z; x[i + 3] = v.w;
      }
#pragma unroll
      for (int i = 0; i < CPT; ++i) {
        x[i] = base + sm_c + i < t_end ? x[i] * sl2 : -INFINITY;
        mx = fmaxf(mx, x[i]);
      }
#pragma unroll
      for (int o = TPH / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float mn = fmaxf(m_run, mx);               // finite: the tile's first token is always visible
      const float al = wm_ex2(m_run - mn);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < CPT; ++i) { x[i] = wm_ex2(x[i] - mn); sum += x[i]; }
#pragma unroll
      for (int o = TPH / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      l_run = fmaf(l_run, al, sum);
      m_run = mn;
#pragma unroll
      for (int i = 0; i < CPT; i += 2)
        *reinterpret_cast<uint32_t*>(probs + sm_row * S::kProbPitch + sm_c + i) = pack_bf16x2(x[i], x[i + 1]);
      if (threadIdx.x % TPH == 0) alpha_sh[sm_row] = al;
    }
    __syncthreads();
    // ---- weighted sum over this warp's columns
    if (summing) {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = alpha_sh[m * 16 + gq], a1 = alpha_sh[m * 16 + gq + 8];
#pragma unroll
        for (int n = 0; n < NT; ++n) { acc[m][n][0] *= a0; acc[m][n][1] *= a0; acc[m][n][2] *= a1; acc[m][n][3] *= a1; }
      }
#pragma unroll
      for (int ks = 0; ks < kLdTile / 16; ++ks) {
        uint32_t pf[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) wm_ldsm_x4(wm_a(probs_u32, S::kProbPitch, m * 16, ks * 16, lane), pf[m]);
#pragma unroll
        for (int n2 = 0; n2 < NT / 2; ++n2) {
          uint32_t bf[4];
          wm_ldsm_x4_t(wm_b_t(tile, pitch, warp * VW + n2 * 16, ks * 16, lane), bf);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            wm_mma(acc[m][2 * n2], pf[m], bf[0], bf[1]);
            wm_mma(acc[m][2 * n2 + 1], pf[m], bf[2], bf[3]);
          }
        }
      }
    }
  }
  // ---- this slice's (maximum, sum, weighted sum) per head, or the result when there is one slice only
  __syncthreads();
  float* lsum = alpha_sh;
  if (threadIdx.x % TPH == 0) {
    lsum[sm_row] = l_run;
    if (nsplit > 1 && sm_row < nheads) {
      float* pp = a.scratch + ((static_cast<long long>(b) * a.heads + h0 + sm_row) * nsplit + sp) * (a.rank + 2);
      pp[0] = m_run;
      pp[1] = l_run;
    }
  }
  __syncthreads();
  if (!summing) return;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int head = m * 16 + gq + 8 * half;
      if (head >= nheads) continue;
      const float inv = nsplit > 1 ? 1.f : 1.f / lsum[head];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int col = warp * VW + n * 8 + 2 * tq;
        if (col >= a.rank) continue;                   // rank is a multiple of 8
        const float u = acc[m][n][2 * half] * inv, v = acc[m][n][2 * half + 1] * inv;
        if (nsplit > 1) {
          float* pp = a.scratch + ((static_cast<long long>(b) * a.heads + h0 + head) * nsplit + sp) * (a.rank + 2);
          *reinterpret_cast<float2*>(pp + 2 + col) = make_float2(u, v);
        } else {
          *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(a.out) + b * a.ld_o + static_cast<long long>(h0 + head) * a.rank + col) =
              pack_bf16x2(u, v);
        }
      }
    }
}

// out[b, h, :] = merge over the slices that hold tokens of sequence b (at most 64); a thread owns two columns
__global__ void __launch_bounds__(256)
latent_merge_kernel(const float* __restrict__ partial, const int* __restrict__ context_lens, int heads, int rank, int nsplit,
                    __nv_bfloat16* __restrict__ out, long long ld_o) {
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31;
  const int ctx = context_lens[b], slice = latent_chunk(ctx, nsplit);
  const int n = min(nsplit, (ctx + slice - 1) / slice);
  const long long pitch = rank + 2;
  const float* base = partial + (static_cast<long long>(b) * heads + h) * nsplit * pitch;
  // every warp by itself: lane s has the factors of slices s and s + 32
  const float m0 = lane < n ? base[lane * pitch] : -INFINITY, m1 = lane + 32 < n ? base[(lane + 32) * pitch] : -INFINITY;
  const float l0 = lane < n ? base[lane * pitch + 1] : 0.f, l1 = lane + 32 < n ? base[(lane + 32) * pitch + 1] : 0.f;
  const float mx = warp_max(fmaxf(m0, m1));
  float s0 = wm_ex2(m0 - mx), s1 = wm_ex2(m1 - mx);
  const float den = warp_sum(fmaf(l0, s0, l1 * s1));
  const float inv = den > 0.f ? 1.f / den : 0.f;
  s0 *= inv;
  s1 *= inv;
  for (int c0 = 0; c0 < rank; c0 += 2 * blockDim.x) {
    const int c = c0 + 2 * threadIdx.x;
    float u = 0.f, v = 0.f;
#pragma unroll 4
    for (int s = 0; s < n; ++s) {
      const float sc = __shfl_sync(0xffffffffu, s < 32 ? s0 : s1, s & 31);
      if (c < rank) {
        const float2 z = *reinterpret_cast<const float2*>(base + s * pitch + 2 + c);
        u = fmaf(z.x, sc, u);
        v = fmaf(z.y, sc, v);
      }
    }
    if (c < rank) *reinterpret_cast<uint32_t*>(out + b * ld_o + static_cast<long long>(h) * rank + c) = pack_bf16x2(u, v);
  }
}

template <int MT, int VW, int KMAX>
int ld_launch(const RbLatentDecodeArgs& a, int nsplit, cudaStream_t s) {
  auto kern = latent_decode_kernel<MT, VW, KMAX>;
  const int smem = LdSmem<MT>::bytes((a.rank + a.rot + 15) / 16 * 16);
  static bool cfg[64] = {};
  bool& done = cfg[rbhost::device_slot()];
  if (!done) {
    // the widest tile this form takes
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LdSmem<MT>::bytes(KMAX * 64));
    if (e != cudaSuccess) return static_cast<int>(e);
    done = true;
  }
  kern<<<dim3((a.heads + 16 * MT - 1) / (16 * MT), nsplit, a.batch), kLdWarps * 32, smem, s>>>(a, nsplit RB_BOUNDS_ARG);
  return static_cast<int>(cudaGetLastError());
}

// Slices per sequence: as many as make a launch of one CTA per SM shortest, for contexts of 4096 tokens (or what the tables can hold).
// It depends on the batch and the tables' width only, which a captured graph keeps.
inline int ld_splits(int batch, int heads, long long capacity) {
  const long long ctas = static_cast<long long>(batch) * ((heads + 31) / 32);
  const long long ctx = capacity < 4096 ? capacity : 4096;
  int best = 1;
  long long best_cost = 0;
  for (int s = 1; s <= 64 && (s == 1 || (s - 1) * 128 < capacity); ++s) {
    const long long cost = (ctas * s + 147) / 148 * ((ctx + s - 1) / s + 256);
    if (s == 1 || cost < best_cost) { best = s; best_cost = cost; }
  }
  return best;
}

}  // namespace rb

RB_API int rb_latent_prep(const RbLatentPrepArgs* args, void* stream_v) {
  const RbLatentPrepArgs& a = *args;
  if (a.tokens <= 0) return 0;
  if (!a.p || !a.q_gamma || !a.kv_gamma || a.q_rank <= 0 || a.rank <= 0 || a.rot < 0 || a.pairs < 0 || 2 * a.pairs > a.rot ||
      (a.pairs && !a.table) || (a.cache && !a.slots) || a.tokens > 0x7fffffffLL)
    return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  const bool vec = !((reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.cache)) & 15) &&
                   !((a.ld | a.off_q | a.off_kv | a.q_rank | a.rank | (a.rank + a.rot)) & 7);
  if (a.f32) return rb::lp_launch<float, 1>(a, s);
  return vec ? rb::lp_launch<__nv_bfloat16, 8>(a, s) : rb::lp_launch<__nv_bfloat16, 1>(a, s);
}

RB_API int rb_head_product(const RbHeadProductArgs* args, void* stream_v) {
  const RbHeadProductArgs& a = *args;
  if (a.rows <= 0) return 0;
  if (!a.x || !a.w || !a.y || a.heads <= 0 || a.n <= 0 || a.k <= 0 || a.tail < 0 || a.pairs < 0 || 2 * a.pairs > a.tail || (a.pairs && !a.table))
    return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  const bool fast = !a.f32 && !((a.n | a.k | a.tail | a.tail_off) & 7) && !((a.ld_x | a.x_head | a.ld_w | a.w_head | a.ld_y | a.y_head) & 7) &&
                    !((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.y)) & 15) &&
                    (!a.gate || (!(a.ld_g & 1) && !(reinterpret_cast<uintptr_t>(a.gate) & 3))) && a.heads <= 65535 && a.rows <= 65535 * 64;
  if (fast) {
    const long long wide = static_cast<long long>((a.n + 63) / 64) * a.heads * ((a.rows + 63) / 64);
    if (wide < 148) return a.transposed ? rb::hp_run<32, true>(a, s) : rb::hp_run<32, false>(a, s);
    return a.transposed ? rb::hp_run<64, true>(a, s) : rb::hp_run<64, false>(a, s);
  }
  long long blocks = (static_cast<long long>(a.rows) * a.heads * (a.n + a.tail) + 127) / 128;
  if (blocks > 148LL * 64) blocks = 148LL * 64;
  if (a.f32) rb::head_product_plain_kernel<float><<<static_cast<int>(blocks), 128, 0, s>>>(a);
  else rb::head_product_plain_kernel<__nv_bfloat16><<<static_cast<int>(blocks), 128, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

RB_API long long rb_latent_decode_scratch_floats(int batch, int heads, int rank, int max_blocks, int block_size) {
  const int nsplit = rb::ld_splits(batch, heads, static_cast<long long>(max_blocks) * block_size);
  return nsplit > 1 ? static_cast<long long>(batch) * heads * nsplit * (rank + 2) : 1;
}

RB_API int rb_latent_decode(const RbLatentDecodeArgs* args, void* stream_v) {
  const RbLatentDecodeArgs& a = *args;
  if (a.batch <= 0) return 0;
  if (!a.q || !a.out || !a.cache || !a.block_tables || !a.context_lens || !a.scratch || a.heads <= 0 || a.rank <= 0 || a.rot < 0 ||
      a.rank > 512 || a.rank + a.rot > 640 || ((a.rank | a.rot) & 7) || a.block_size <= 0 || a.max_blocks <= 0 || a.batch > 65535 ||
      a.num_blocks * a.block_size >= (1ll << 31) || ((a.ld_q | a.ld_o) & 1))
    return -1;
  if ((reinterpret_cast<uintptr_t>(a.cache) & 15) || ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.out)) & 3) ||
      (reinterpret_cast<uintptr_t>(a.scratch) & 7))
    return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  const int n = rb::ld_splits(a.batch, a.heads, static_cast<long long>(a.max_blocks) * a.block_size), width = a.rank + a.rot;
  int rc = rb::latent_decode_tc(a, n, s);
  if (rc == -9) {
    const bool two = a.heads > 16;
    if (a.rank <= 128 && width <= 256) rc = two ? rb::ld_launch<2, 16, 4>(a, n, s) : rb::ld_launch<1, 16, 4>(a, n, s);
    else if (a.rank <= 256 && width <= 384) rc = two ? rb::ld_launch<2, 32, 6>(a, n, s) : rb::ld_launch<1, 32, 6>(a, n, s);
    else rc = two ? rb::ld_launch<2, 64, 10>(a, n, s) : rb::ld_launch<1, 64, 10>(a, n, s);
  }
  if (rc || n == 1) return rc;
  rb::latent_merge_kernel<<<dim3(a.heads, a.batch), a.rank <= 128 ? 64 : 256, 0, s>>>(a.scratch, a.context_lens, a.heads, a.rank, n,
                                                                                    reinterpret_cast<__nv_bfloat16*>(a.out), a.ld_o);
  return static_cast<int>(cudaGetLastError());
}
