// C interface of the latent attention kernels (latent_attention.cu): keys and values of all heads are products of one cached vector per
// token, beside a rotated key part that the heads share.  A slot of the cache holds [vector (rank) | rotated part (rot)].
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
// Norms, positions and cache append behind the packed projection, in place on p (bf16 or fp32, pitch ld):
//   p[t, off_q .. + q_rank) <- rms * q_gamma;  p[t, off_kv .. + rank) <- rms * kv_gamma;  the next `rot` columns: the neighbouring pairs of
//   the first 2 * pairs are rotated by `table` (rb_rotary_table);  p[t, off_kv .. + rank + rot) goes to cache slot slots[t]
typedef struct RbLatentPrepArgs {
  void* p;
  const float* q_gamma;      // [q_rank]
  const float* kv_gamma;     // [rank]
  const float* table;        // [tokens, pairs, 2]
  void* cache;               // [num_slots, rank + rot], type of p
  const long long* slots;    // negative: not stored
  long long ld, off_q, off_kv, tokens, num_slots;
  int f32, q_rank, rank, rot, pairs;
  float eps;
} RbLatentPrepArgs;
int rb_latent_prep(const RbLatentPrepArgs* args, void* stream);

// One small product per head: y[t, h, n] = sum_k x[t, h, k] * w[h](n, k), where w[h] is stored [n, k] or, transposed, [k, n] (pitch ld_w,
// heads w_head apart).  x and y have row pitches ld_x / ld_y and heads x_head / y_head apart.  Optional: y is multiplied by sigmoid(gate)
// (gate [t, h * n], pitch ld_g); `tail` further columns behind x's first tail_off ones are copied behind y's n columns, the neighbouring
// pairs of their first 2 * pairs rotated by `table`.  bf16 (fp32 sums) or fp32.
typedef struct RbHeadProductArgs {
  const void* x;
  const void* w;
  void* y;
  const void* gate;
  const float* table;        // [rows, pairs, 2]
  long long ld_x, x_head, ld_w, w_head, ld_y, y_head, ld_g;
  int f32, rows, heads, n, k, transposed, tail, tail_off, pairs;
} RbHeadProductArgs;
int rb_head_product(const RbHeadProductArgs* args, void* stream);

// Decode attention on the cached vectors: q [batch, heads, rank + rot] (the heads' queries as seen by the cached vector, then the rotated
// part), score = q . slot * scale, out [batch, heads, rank] = softmax-weighted sum of the vectors.  bf16; rank <= 512, rank + rot <= 640,
// both multiples of 8.  scratch: fp32 [rb_latent_decode_scratch_floats(...)].
typedef struct RbLatentDecodeArgs {
  const void* q;             // pitch ld_q, heads rank + rot apart
  void* out;                 // pitch ld_o, heads rank apart
  const void* cache;         // [num_blocks, block_size, rank + rot]
  const int* block_tables;   // [batch, max_blocks]
  const int* context_lens;   // [batch], the new token included
  float* scratch;
  long long ld_q, ld_o, num_blocks;
  int batch, max_blocks, heads, rank, rot, block_size;
  float scale;
} RbLatentDecodeArgs;
long long rb_latent_decode_scratch_floats(int batch, int heads, int rank, int max_blocks, int block_size);
int rb_latent_decode(const RbLatentDecodeArgs* args, void* stream);
#ifdef __cplusplus
}
#endif
