// C interface of the paged KV-cache kernels (paged_attention.cu).
// Cache layout per layer: [num_blocks, block_size, kv_heads, head_dim] bf16 for K and for V.
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
// Copies new keys / values into their cache slots.  k_new / v_new: [tokens, kv_heads, head_dim] with row pitch
// ld_k / ld_v (so they may be column ranges of a packed QKV projection).  slot_mapping[t] = block * block_size + offset,
// negative slots are skipped.
int rb_kv_append(const void* k_new, long long ld_k, const void* v_new, long long ld_v, void* k_cache, void* v_cache,
                 const long long* slot_mapping, long long tokens, int kv_heads, int head_dim, long long num_slots,
                 void* stream);
// Decode attention: one query token per sequence.
//   q [batch, heads, head_dim] (row pitch ld_q), out [batch, heads, head_dim] (row pitch ld_o), both bf16
//   block_tables [batch, max_blocks] int32, context_lens [batch] int32 (tokens already in the cache, incl. the new one)
//   scratch: fp32 [rb_paged_attention_scratch_floats(...)] for the per-slice partial results of the split-KV kernel
long long rb_paged_attention_scratch_floats(int batch, int heads, int head_dim, int max_blocks, int block_size);
int rb_paged_attention_decode(const void* q, long long ld_q, void* out, long long ld_o, const void* k_cache,
                              const void* v_cache, const int* block_tables, int max_blocks, const int* context_lens,
                              int batch, int heads, int kv_heads, int head_dim, int block_size, long long num_blocks,
                              float scale, float* scratch, void* stream);
// The same decode attention with separate key / value head sizes (multiples of 8, at most 128), a score rule and an output
// gate; softcap, slopes, log bias, chunk, window, sink, gates and out_scale as in RbPagedRowsArgs below.  bf16 operands.  scratch: fp32
// [rb_paged_attention_scratch_floats(batch, heads, dv, max_blocks, block_size)].
typedef struct RbPagedDecodeArgs {
  const void* q;             // [batch, heads * dk], pitch ld_q
  void* out;                 // [batch, heads * dv], pitch ld_o
  const void* k_cache;
  const void* v_cache;
  const int* block_tables;
  const int* context_lens;
  const float* slopes;
  const void* gate;          // [batch, heads * dv], pitch ld_g
  const float* head_gate;    // [batch, heads], pitch ld_g
  float* scratch;
  long long ld_q, ld_o, ld_g, num_blocks;
  int batch, max_blocks, heads, kv_heads, dk, dv, block_size, chunk, window, keep_first, sink;
  float scale, softcap;
  const float* log_amount;
  const float* log_rate;
  float out_scale;
} RbPagedDecodeArgs;
int rb_paged_attention_decode_rule(const RbPagedDecodeArgs* args, void* stream);
// Attention over the pages for any rows of a batch (prompt portions and decoded tokens alike), any head sizes, bf16 or
// fp32 operands, fp32 arithmetic: the 32-bit mode and the fallback for head sizes the tensor-core kernels do not take.
//   row r is the token at position row_pos[r] of the sequence whose pages are block_tables[row_seq[r]]; it sees the keys
//   j <= pos, and with chunk > 0 only those with j / chunk == pos / chunk, with window > 0 only those with pos - j < window or
//   j < keep_first
//   sink: a further score 0 without a value takes part in the softmax
//   score = q . k * scale; softcap > 0: score <- softcap * tanh(score / softcap); slopes (fp32 [heads], or NULL):
//   score <- score - slopes[h] * (pos - j); log_amount, log_rate (fp32 [heads] each, or both NULL):
//   score <- score - log_amount[h] * ln(1 + log_rate[h] * (pos - j)), log_rate not negative; out_scale multiplies the output
//   gate (type of q, pitch ld_g, [rows, heads * dv], or NULL) or head_gate (fp32 [rows, heads], pitch ld_g, or NULL): the output
//   is multiplied by sigmoid(gate)
typedef struct RbPagedRowsArgs {
  const void* q;
  void* out;
  const void* k_cache;       // [num_blocks, block_size, kv_heads, dk], consecutive slots ld_kc apart (0: kv_heads * dk)
  const void* v_cache;       // [num_blocks, block_size, kv_heads, dv], ld_vc apart; both may be columns of one array
  const int* block_tables;   // [sequences, max_blocks]
  const int* row_seq;
  const long long* row_pos;
  const float* slopes;
  const void* gate;
  const float* head_gate;
  long long ld_q, ld_o, ld_g, num_blocks, ld_kc, ld_vc;
  int f32, rows, max_blocks, heads, kv_heads, dk, dv, block_size, chunk, window, keep_first, sink;
  float scale, softcap;
  const float* log_amount;
  const float* log_rate;
  float out_scale;
} RbPagedRowsArgs;
int rb_paged_attention_rows(const RbPagedRowsArgs* args, void* stream);
#ifdef __cplusplus
}
#endif
