// C interface of the preparation of a packed attention projection, per head or over whole rows (head_prep.cu).
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
typedef struct RbHeadPrepArgs {
  void* p;                    // packed projection [tokens, ld]: query heads at off_q, key heads at off_k, value heads at off_v
  const void* q_gamma;        // [dk] RMS-norm weight of every query head, or NULL (no norm); type of p
  const void* k_gamma;        // same for the key heads
  const void* v_first;        // [tokens, kv_heads * dv] values to mix in (pitch ld_vf), type of p, or NULL
  const float* mix;           // [1] share of v_first
  void* k_cache;              // [num_slots, kv_heads, dk] / [num_slots, kv_heads, dv], type of p, or both NULL
  void* v_cache;
  const long long* slots;     // cache slot of every token (negative: not stored)
  const float* rot;           // [tokens, rot_dims / 2] pairs (cos, sin) (rb_rotary_table), or NULL: queries and keys are not rotated
  long long ld, off_q, off_k, off_v, ld_vf, tokens, num_slots;
  int f32, heads, kv_heads, dk, dv, rot_dims;
  float eps;
  int half;                   // numbers i and i + rot_dims / 2 turn together instead of neighbours (no v_first then)
  int values_are_keys;        // with half, dk == dv: the value columns and v_cache receive the keys as they were
  float k_scale;              // with half: of the keys, behind the rotation
} RbHeadPrepArgs;
// In place: q <- rms(q) * q_gamma, k <- rms(k) * k_gamma, then neighbouring pairs of their first rot_dims numbers are rotated;
// v <- (1 - mix) v + mix v_first; k and v also go to their slots.
int rb_head_prep(const RbHeadPrepArgs* args, void* stream);
// Rows q [nq] | k [nk] | v [nv] (nk = nv = 0: queries only), in place: q <- rms(q) * q_gamma * (1 + temp_coef ln(floor((pos + 1) /
// temp_every) + 1)), k <- rms(k) * k_gamma, each norm over the whole part; k and v also go to their slots.
typedef struct RbRowPrepArgs {
  void* p;                    // [tokens, ld], bf16 or fp32 (f32)
  const float* q_gamma;       // [nq]
  const float* k_gamma;       // [nk]
  void* k_cache;              // [num_slots, nk] / [num_slots, nv], type of p, or both NULL
  void* v_cache;
  const long long* slots;     // cache slot of every token (negative: not stored)
  const long long* pos;       // position of every token (read with temp_every > 0)
  long long ld, tokens, num_slots;
  int f32, nq, nk, nv, temp_every;   // temp_every 0: no factor
  float temp_coef, eps;
} RbRowPrepArgs;
int rb_row_prep(const RbRowPrepArgs* args, void* stream);
#ifdef __cplusplus
}
#endif
