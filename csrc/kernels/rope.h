// C interface of the rotary-embedding and SwiGLU kernels (rope.cu).
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
// In-place rotary position embedding on bf16 x viewed as [tokens, heads, head_dim] with row pitch ld
// (head h starts at column h*head_dim).  Pairs are (i, i + head_dim/2) ("rotate half").  The position of
// token t is positions[t] when positions != NULL, else pos_offset + (t % seq_len).  inverse = 1 applies the
// transposed rotation, which is the backward pass.
int rb_rope(void* x, long long ld, const long long* positions, long long tokens, int heads, int head_dim, int seq_len,
            long long pos_offset, float theta, int inverse, void* stream);
// out[t, i] = magnitude * (cos, sin)(positions[t] * freqs[i]): fp32 [rows, pairs, 2], the table of the pairwise rotations below and in
// head_prep.h, latent_attention.h
int rb_rotary_table(const long long* positions, const double* freqs, float magnitude, float* out, long long rows, int pairs,
                    void* stream);
// In place on x[t, h * pitch + 2i], x[t, h * pitch + 2i + 1], i < pairs (bf16 or fp32; x points at the first rotated column of head 0)
int rb_rotate_pairs(void* x, long long ld, const float* table, long long rows, int heads, long long pitch, int pairs, int f32,
                    void* stream);
// h[t, f] = silu(gu[t, f]) * gu[t, F + f]   with gu [tokens, 2F] (gate | up), bf16
int rb_swiglu_fwd(const void* gu, long long ld_gu, void* h, long long ld_h, long long tokens, int F, void* stream);
// dgu[t, f] = dh * up * silu'(gate);  dgu[t, F + f] = dh * silu(gate)
int rb_swiglu_bwd(const void* dh, long long ld_dh, const void* gu, long long ld_gu, void* dgu, long long ld_dgu,
                  long long tokens, int F, void* stream);
#ifdef __cplusplus
}
#endif
