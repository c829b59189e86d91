/* nativebit_b200 — C ABI of the kernels of layered decoders (models that list their layers one by one: latent
 * attention, gated linear attention, dense feed-forward, norms before and after every sublayer).
 *
 * Same rules as nativebit_b200.h: plain device pointers, sizes and a CUDA stream handle; asynchronous; no
 * allocation, no synchronisation; every call returns an nb_status; no CPU path.  Weights are bf16, row-major
 * (out, in) with a row stride that is a multiple of 8 elements; activations are bf16 or fp32 (NB_BF16 / NB_F32:
 * with NB_F32 every product is a true 32-bit one); norms, positions, attention scores and weights, decays and the
 * recurrent state are fp32 in both cases. */
#ifndef NATIVEBIT_B200_LAYERED_H_
#define NATIVEBIT_B200_LAYERED_H_

#include "nativebit_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef enum { NB_NORM_RMS = 0, NB_NORM_LAYER = 1 } nb_norm;   /* LAYER: mean taken off, weight, no bias */
typedef enum { NB_ACT_NONE = 0, NB_ACT_SWIGLU_PAIRS = 1 } nb_act;
/* NB_ACT_SWIGLU_PAIRS: rows 2i and 2i + 1 of the weight are gate and up of channel i; y has N / 2 columns,
 * silu(gate + bias) * (up + bias). */

/* ---- x (rows, C) fp32 = table[token] * scale for a bf16 (V, C) table; token ids are clamped to [0, V). */
int nb_embed_scaled(const void* table_bf16, const int64_t* token, int rows, int V, int C, float scale, float* x, void* stream);

/* ---- one step of the residual chain, per row: x += norm(y) * wy (if y), then h = norm(x) * w (if h).
 * x, y (rows, C) fp32; h (rows, ldh) of h_dtype. */
int nb_residual_norm(float* x, const float* y, const float* wy, const float* w, int norm, float eps, void* h, int h_dtype, int ldh,
                     int rows, int C, void* stream);

/* ---- y (M, N) = x (M, K) . w (N, K)^T (+ bias) for many rows.
 * nb_linear_bf16: bf16 x on the tcgen05 tensor cores, fp32 accumulation, y NB_BF16 or NB_F32; x and w 16-byte
 * aligned, ldx and ldw multiples of 8; `status`: device int, NB_ERR_TIMEOUT if a bounded wait ran out, or NULL.
 * nb_linear_f32: fp32 x and y, fp32 multiply-adds. */
int nb_linear_bf16(const void* x, int ldx, const void* w, int ldw, const float* bias, int act, int M, int N, int K, void* y, int y_dtype,
                   int ldy, int* status, void* stream);
int nb_linear_f32(const float* x, int ldx, const void* w, int ldw, const float* bias, int act, int M, int N, int K, float* y, int ldy,
                  void* stream);

/* ---- y (N) = w (N, K) . act for ONE row (decode), fp32 activations, with the element-wise step in front folded in:
 *   norm_w NULL:            act = x
 *   norm_w, delta NULL:     act = norm(x) * norm_w
 *   norm_w, delta:          r = x + norm(delta) * delta_w; x_out = r; act = norm(r) * norm_w   (x_out != x)
 * The weights are requested before the launch waits for earlier work of the stream. */
typedef struct {
  const void* w;        /* bf16 (N, ldw), 16-byte aligned, columns K .. ldw zero */
  const float* bias;    /* N or NULL */
  float* y;
  const float* x;       /* K */
  const float* delta;   /* K or NULL */
  const float* delta_w; /* K or NULL */
  float* x_out;         /* K or NULL */
  const float* norm_w;  /* K or NULL */
  float eps;
  int N, K, ldw, act, norm;
} nb_matvec_args;
int nb_matvec_bf16(const nb_matvec_args* a, void* stream);

/* ---- latent attention -------------------------------------------------------------------------------------
 * Cache of a layer: (B, ctx, ldc) rows [latent (rank) | rotated key part (rot)] of the activation dtype, ldc a
 * multiple of 8, columns past them zero.  cos2 / sin2: (ctx, rot) fp32, every pair's entry twice (interleaved pairs).
 *
 * nb_latent_prepare, per row b * T + t: cq = RMSNorm(a[q_off ..]) * q_norm (q_rank values); if kv_off >= 0:
 * cache[b][pos0 + t] = [RMSNorm(a[kv_off ..]) * kv_norm | rotate(a[kv_off + rank ..])]. */
typedef struct {
  const void* a;
  void* cq;
  void* cache;
  const float *q_norm, *kv_norm, *cos2, *sin2;
  float eps;
  int dtype, B, T, lda, q_off, q_rank, ldcq, kv_off, rank, rot, ctx, ldc, pos0;
} nb_latent_prepare_args;
int nb_latent_prepare(const nb_latent_prepare_args* a, void* stream);

/* Attention of T new positions pos0 .. pos0 + T - 1 over keys within `window` (0: all earlier ones): query i sees
 * keys j with 0 <= i - j < window.  q: (B * T, ldq), head h at h * (dim + rot), [unrotated | to be rotated].
 * kv: (B, kv_rows, ldkv), row r = position kv_pos0 + r, up-projected keys of head h at h * dim and values at
 * v_off + h * vdim; the shared rotated key part is read from `cache`.  out (B * T, ldo): head h at h * vdim, multiplied
 * by sigmoid(gate[row * ldg + h]) if gate.  NB_BF16 runs on the tensor cores (scores, softmax in fp32; the softmax
 * weights enter the second product as two bf16 terms), NB_F32 in fp32 multiply-adds.  vdim <= 256. */
typedef struct {
  const void* q;
  const void* kv;
  const void* cache;
  const void* gate;
  void* out;
  const float *cos2, *sin2;
  float scale;
  int dtype, B, T, H, dim, rot, vdim, rank, ctx, ldc, ldq, ldkv, v_off, kv_rows, kv_pos0, ldg, ldo, pos0, window;
} nb_latent_attention_args;
int nb_latent_attention(const nb_latent_attention_args* a, void* stream);

/* One new position per sequence, in latent space: per head, q' = W_uk^T q_unrotated, scores against the cached rows,
 * the weighted latent through W_uv, the output gate; a cluster of CTAs per head splits the keys.  kv_off >= 0: the
 * launch also norms and rotates a[kv_off ..] and writes it into the cache at *pos (otherwise another layer already
 * did).  q (B, ldq) and a (B, lda) fp32; gate logits at a[g_off + h]; uk (H * dim, ldu), uv (H * vdim, ldu) bf16 with
 * ldu >= rank; out (B, ldo) fp32.  Does nothing when *pos is outside [0, ctx). */
typedef struct {
  const float* q;
  const float* a;
  void* cache;
  const void *uk, *uv;
  const float *kv_norm, *cos2, *sin2;
  const int64_t* pos;
  float* out;
  float scale, eps;
  int cache_dtype, B, H, dim, rot, vdim, rank, ctx, ldc, ldq, lda, kv_off, g_off, ldu, ldo, window;
} nb_latent_decode_args;
int nb_latent_decode(const nb_latent_decode_args* a, void* stream);

/* ---- gated linear attention -------------------------------------------------------------------------------
 * p: (B * T, ldp) projections, q at q_off (H * dim), k at k_off, v at v_off (H * vdim), g at g_off, a at a_off
 * (a_rank); decay alpha = sigmoid(a2 . a + a2_b)^(1 / tau) per key channel; per head S <- diag(alpha) S + k v^T,
 * o = S^T (q * dim^-1/2); out (B * T, ldo) = RMSNorm(o) * norm_w * silu(g).  state: (B, H, dim, lds) fp32, lds a
 * multiple of 4, columns vdim .. lds zero; read and updated.
 * nb_gla_prefill works in chunks of 64 tokens; workspace of nb_gla_workspace_bytes().
 * nb_gla_decode: one token per sequence, fp32 p and out. */
typedef struct {
  const void* p;
  void* out;
  float* state;
  const void* a2;      /* bf16 (H * dim, lda2) */
  const float *a2_b, *norm_w;
  float tau, eps;
  int dtype, B, T, H, dim, vdim, ldp, q_off, k_off, v_off, g_off, a_off, a_rank, lda2, lds, ldo;
} nb_gla_args;
size_t nb_gla_workspace_bytes(int B, int T, int H, int dim, int vdim);
int nb_gla_prefill(const nb_gla_args* a, void* workspace, size_t workspace_bytes, void* stream);
int nb_gla_decode(const nb_gla_args* a, void* stream);

/* ---- greedy choice: token[b] = index of the largest of logits (B, V) fp32 (lowest index among equals); *pos += 1
 * if pos != NULL. */
int nb_argmax(const float* logits, int B, int V, int64_t* token, int64_t* pos, void* stream);

#ifdef __cplusplus
}
#endif
#endif
