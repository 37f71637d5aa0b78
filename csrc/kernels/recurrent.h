// C interface of the layers that carry state from token to token (short_conv.cu, state_space.cu, selective_scan.cu, delta_rule.cu) and of the
// gated norm behind them (gated_norm.cu).  All pointers are device pointers.
//
// A batch is a list of segments, each the next tokens of one sequence: table row {first row of the batch, number of rows, state
// slot, position of the first row in its sequence}.  At position 0 the state counts as zero, whatever the slot holds; after the
// call the slot holds the state behind the segment's last row.
#pragma once
#ifdef __cplusplus
extern "C" {
#endif

// out[t, c] = act(bias[c] + sum_i w[c, i] x[t - (taps - 1) + i, c]): causal convolution per channel over a sequence.
typedef struct RbShortConvArgs {
  const void* x;             // [rows, channels], pitch ld_x, bf16 or fp32 (f32)
  void* out;                 // same type, pitch ld_o
  void* state;               // [slots, taps - 1, channels] of the same type: the last inputs, oldest first
  const float* w;            // [channels, taps]
  const float* bias;         // [channels] or NULL
  const int* segments;       // [n, 4]
  const int* tiles;          // [num_tiles, 2]: segment, first row inside it (multiples of RB_CONV_TILE, every one listed)
  long long ld_x, ld_o;
  int num_tiles, channels, taps, f32, silu, num_slots;
} RbShortConvArgs;
#define RB_CONV_TILE 16
int rb_short_conv(const RbShortConvArgs* args, void* stream);

// Mamba-2 recurrence.  Per head h of group g = h / (heads / groups), with dt = softplus(dt_raw + dt_bias[h]):
//   S <- exp(-exp(a_log[h]) dt) S + dt B_g x^T   (S [n, p]),   y = S^T C_g + D[h] x
// xbc [rows, heads p + 2 groups n] = x | B | C, bf16 or fp32; dt_raw fp32; y in the type of xbc; the state is fp32
// [slots, heads, n, p4], p4 = p rounded up to a multiple of 4.  `decay` (fp32 [heads], in (0, 1]) instead of dt_raw, dt_bias and a_log
// (NULL): S <- decay[h] S + B_g x^T.  D may be NULL (0).
typedef struct RbStateSpaceArgs {
  const void* xbc;
  const float* dt_raw;
  const float* dt_bias;
  const float* a_log;
  const float* D;
  float* state;
  void* y;
  const int* segments;
  const int* tiles;          // chunked form: [num_tiles, 2]: segment, first row inside it
  long long ld_xbc, ld_dt, ld_y;
  long long rows;            // chunked form: rows of xbc
  int num_segments, num_tiles, heads, groups, p, n, f32, num_slots;
  const float* decay;
} RbStateSpaceArgs;
int rb_state_space_scan(const RbStateSpaceArgs* args, void* stream);
// The same for prompts on the tensor cores: bf16, n <= 128, n and p multiples of 8 (-9 otherwise).  `tiles` lists spans of `span`
// rows (a multiple of 128, in order, every one listed), which run side by side.  span_state fp32 [num_tiles, heads, n, p] and
// span_decay fp32 [num_tiles, heads] are scratch; both may be NULL when no segment has more than one span.
int rb_state_space_chunked(const RbStateSpaceArgs* args, float* span_state, float* span_decay, int span, void* stream);

// Mamba's selective scan.  Per channel c, with dt = softplus(dt_raw[c] + dt_bias[c]):
//   S[c, :] <- exp(dt A[c, :]) S[c, :] + dt x_c B,   y_c = S[c, :] . C + D[c] x_c,   out_c = scale y_c silu(z_c)
// x, z, out [rows, inner] and B, C [rows, n] (same pitch) are bf16 or fp32 (f32); dt_raw fp32 [rows, inner]; A fp32 [inner, n], negative;
// the state is fp32 [slots, inner, n4], n4 = n rounded up to a multiple of 4.  n at most 256.
typedef struct RbSelectiveScanArgs {
  const void* x;
  const void* z;
  const void* B;
  const void* C;
  const float* dt_raw;
  const float* dt_bias;
  const float* A;
  const float* D;
  float* state;
  void* y;
  const int* segments;
  long long ld_x, ld_z, ld_bc, ld_dt, ld_y;
  int num_segments, num_slots, inner, n, f32;
  int single;                // every segment is one row
  float scale;
} RbSelectiveScanArgs;
int rb_selective_scan(const RbSelectiveScanArgs* args, void* stream);

// Gated delta rule.  Per value head h of query / key head g = h / (heads / kv_heads), with beta = sigmoid(b_raw),
// decay = exp(-exp(a_log[h]) softplus(a_raw + dt_bias[h])), k' = k / sqrt(|k|^2 + 1e-6), q' = dk^(-1/2) q / sqrt(|q|^2 + 1e-6):
//   S <- decay S;  u = beta (v - S^T k');  S <- S + k' u^T;  o = S^T q'   (S [dk, dv])
// qkv [rows, 2 kv_heads dk + heads dv] = q | k | v, bf16 or fp32; a_raw, b_raw fp32 (same pitch); o in the type of qkv; the state
// is fp32 [slots, heads, dk, dv4], dv4 = dv rounded up to a multiple of 4.
typedef struct RbDeltaRuleArgs {
  const void* qkv;
  const float* a_raw;
  const float* b_raw;
  const float* dt_bias;
  const float* a_log;
  float* state;
  void* o;
  const int* segments;
  const int* tiles;
  void* scratch;             // chunked form
  long long ld_qkv, ld_ab, ld_o;
  long long rows;            // chunked form: rows of qkv
  int num_segments, num_tiles, heads, kv_heads, dk, dv, f32, num_slots;
} RbDeltaRuleArgs;
int rb_delta_rule_scan(const RbDeltaRuleArgs* args, void* stream);
// The same for prompts on the tensor cores: bf16, dk <= 128, dk and dv multiples of 8 (-9 otherwise).  `tiles` lists pieces of 64
// rows, in order, every one listed; scratch: rb_delta_rule_scratch_bytes(num_tiles, heads, dk) bytes.
long long rb_delta_rule_scratch_bytes(int num_tiles, int heads, int dk);
int rb_delta_rule_chunked(const RbDeltaRuleArgs* args, void* stream);

// Every row of y consists of `parts` equal parts.  gate_first: u = y silu(z), out = u / rms(u) * weight; else:
// out = y / rms(y) * weight * silu(z); rms over a part, with eps inside the root.  weight fp32 [weight_n]: the whole row or one
// part's (shared by all parts), or NULL (no weight; weight_n is part_n then).
typedef struct RbGatedNormArgs {
  const void* y;
  const void* z;
  void* out;                 // all bf16 or fp32 (f32)
  const float* weight;
  long long ld_y, ld_z, ld_o;
  int rows, parts, part_n, weight_n, f32, gate_first;
  float eps;
} RbGatedNormArgs;
int rb_gated_norm(const RbGatedNormArgs* args, void* stream);
#ifdef __cplusplus
}
#endif
