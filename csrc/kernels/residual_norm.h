// C interface of the sublayer-output norm with a 32-bit residual stream (residual_norm.cu).
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
typedef struct RbResidualNormArgs {
  // source row t: y[t] (slot_pos NULL), or the routed sum  sum_j slot_w[t k + j] * y[slot_pos[t k + j]]; plus add[t] if given
  const void* y;
  const int* slot_pos;
  const float* slot_w;      // NULL: all are 1
  const void* add;
  const void* gamma;        // bf16 or fp32 [n] (param_f32); NULL: x += source
  const void* beta;         // same type, or NULL
  const void* next_gamma;   // with x: h receives rms(new x) * next_gamma, the next sublayer's input; or NULL
  float* x;                 // fp32 residual [rows, n], updated in place: x += norm(source); NULL: no residual
  void* h;                  // copy of the new residual (without x: the normalised row), bf16 or fp32, or NULL
  long long ldy, ld_add, ldx, ldh;
  int y_f32, param_f32, h_f32;   // y and add share y_f32
  int k, rows, n, rms;
  float eps;
} RbResidualNormArgs;
int rb_residual_norm(const RbResidualNormArgs* args, void* stream);
// Update of a residual stream behind a block whose sublayers were computed side by side, and the dynamic tanh in front of the
// next block:  x += mult * (normed * rms(a) * wa + normed * rms(b) * wb + c),   h = tanh(alpha x) * gamma + beta
// a, b, c share their type (y_f32); any may be NULL; rms over the row with eps inside the root; a and b come with a weight.
typedef struct RbStreamUpdateArgs {
  const void* a;
  const void* b;
  const void* c;
  const float* wa;          // [n]
  const float* wb;          // [n]
  float* x;                 // fp32 [rows, n], in place (only read when a, b and c are NULL)
  const float* alpha;       // [1]
  const float* gamma;       // [n]
  const float* beta;        // [n]
  void* h;                  // bf16 or fp32 [rows, n], or NULL (then alpha, gamma and beta are not read)
  long long lda, ldb, ldc, ldx, ldh;
  int y_f32, h_f32, rows, n;
  float mult, normed, eps;
} RbStreamUpdateArgs;
int rb_stream_update(const RbStreamUpdateArgs* args, void* stream);
#ifdef __cplusplus
}
#endif
