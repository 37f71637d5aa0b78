// C interface of the flash-attention kernels (attention.cu).  bf16 tensors addressed by element
// strides {batch, row, head}; the head dimension is contiguous.  lse / delta are fp32 [batch, heads, seq_q].
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
typedef struct RbAttnArgs {
  const void* q; const void* k; const void* v;
  void* o;                 // forward: output; backward: the forward output (read)
  const void* d_o;         // backward: gradient of o (same strides as o)
  void* dq; void* dk; void* dv;
  float* lse;              // forward: written (may be NULL); backward: read
  float* delta;            // backward scratch, fp32 [batch, heads, seq_q]
  long long q_strides[3], k_strides[3], v_strides[3], o_strides[3];
  long long dq_strides[3], dk_strides[3], dv_strides[3];
  int batch, heads, kv_heads, seq_q, seq_k, head_dim;
  int causal;              // with seq_q < seq_k the queries are aligned to the end of the keys
  float scale;             // softmax scale, usually 1/sqrt(head_dim)
  const int* kv_lens;      // optional [batch]: keys at positions >= kv_lens[b] are padding and invisible (NULL: all seq_k
                           // keys are real).  Taken by the "tc2" kernels; the others return -9 when it is set.
} RbAttnArgs;
// Score rule of an inference forward pass (causal, queries aligned to the end of the keys, key 0 is the start of a chunk):
//   s = q . k * scale; softcap > 0: s <- softcap * tanh(s / softcap); slopes (fp32 [heads]): s <- s - slopes[h] * (i - j);
//   chunk > 0: i sees j only when i / chunk == j / chunk; window > 0 (without chunk): i sees j only when i - j < window or
//   j < keep_first; sink: a further score 0 without a value takes part in the softmax; gate (bf16 [seq_q, heads * v_dim], pitch
//   ld_gate, batch 1) or head_gate (fp32 [seq_q, heads], pitch ld_gate, batch 1): the output is multiplied by sigmoid(gate)
//   With window and keep_first the keys may leave out positions between the kept ones and the first query's window.
typedef struct RbAttnRule {
  int v_dim;               // value head size (RbAttnArgs.head_dim is the query / key size)
  float softcap;
  const float* slopes;
  int chunk;
  const void* gate;
  const float* head_gate;
  long long ld_gate;
  int window, keep_first, sink;
  // rot_dim > 0: queries and keys have a second part of rot_dim numbers.  A head's follows the head_dim numbers of its query (heads of q
  // are head_dim + rot_dim or more apart); the keys share k_rot [seq_k, rot_dim], pitch ld_k_rot (batch 1).  The score is the sum of both.
  int rot_dim;
  const void* k_rot;
  long long ld_k_rot;
  // fp32 [heads] each, or both NULL: s <- s - log_amount[h] * ln(1 + log_rate[h] * (i - j)), log_rate not negative (without rot_dim)
  const float* log_amount;
  const float* log_rate;
  float out_scale;         // of the output
} RbAttnRule;
int rb_attention_fwd_rule(const RbAttnArgs* args, const RbAttnRule* rule, void* stream);
int rb_attention_fwd(const RbAttnArgs* args, void* stream);
int rb_attention_bwd(const RbAttnArgs* args, void* stream);
// tcgen05 paths (attention_tc.cu, attention_fwd2.cu, attention_bwd_tc.cu, attention_bwd2.cu); -9: shape not taken
int rb_attention_fwd_tc(const RbAttnArgs* args, void* stream);
int rb_attention_fwd_tc2(const RbAttnArgs* args, int poly_every, void* stream);
int rb_attention_bwd_tc(const RbAttnArgs* args, void* stream);
int rb_attention_delta_tc(const RbAttnArgs* args, void* stream);
int rb_attention_bwd_tc2(const RbAttnArgs* args, void* stream);
#ifdef __cplusplus
}
#endif
