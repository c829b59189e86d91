/* nativebit_b200 — C ABI of the kernels of layered decoders (models that list their layers one by one: latent
 * attention, grouped attention with scores mixed across heads, gated linear attention, dense feed-forward, norms before and
 * after every sublayer or hyper-connections).
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
typedef enum { NB_ACT_NONE = 0, NB_ACT_SWIGLU_PAIRS = 1, NB_ACT_CLAMPED_GLU_PAIRS = 2 } nb_act;
/* .._PAIRS: rows 2i and 2i + 1 of the weight are gate and up of channel i (g = gate + bias, u = up + bias); y has N / 2
 * columns.  SWIGLU: silu(g) * u.  CLAMPED_GLU: g = min(g, limit), u clamped to +-limit, g * sigmoid(alpha * g) * (u + 1)
 * (alpha and limit are not read by the other activations). */

/* ---- x (rows, streams, C) fp32 = table[token] * scale, once per stream, for a bf16 (V, C) table; token ids are clamped
 * to [0, V). */
int nb_embed_scaled(const void* table_bf16, const int64_t* token, int rows, int V, int C, float scale, int streams, float* x, void* stream);

/* ---- one step of the residual chain, per row: x += norm(y) * wy (if y), then h = norm(x) * w (if h).
 * x, y (rows, C) fp32; h (rows, ldh) of h_dtype. */
int nb_residual_norm(float* x, const float* y, const float* wy, const float* w, int norm, float eps, void* h, int h_dtype, int ldh,
                     int rows, int C, void* stream);

/* ---- hyper-connections: a residual of `streams` vectors per row, mixed at every sublayer.  With the result y of the
 * sublayer before (the sum of one or two branches, each through an optional norm of its own and times its weight; none if
 * y0 is NULL), per row:
 *   x_out_t = sum_s mix[s][t] x_s + share_t * y        the streams behind it (not written if x_out is NULL)
 *   u       = sum_s read_s x_s + direct * y            what the next sublayer reads: its weights applied to those streams
 *   h       = norm(u) * norm_w
 * coef: fp32 [read (streams) | direct | share (streams) | mix (streams, streams)].  x, x_out (rows, streams, C), y (rows, C).
 * nb_stream_norm: many rows, h (rows, ldh) of h_dtype; x_out may be x. */
enum { NB_MAX_STREAMS = 8 };
typedef struct {
  const float* x;
  float* x_out;
  const float *y0, *w0, *y1, *w1, *coef, *norm_w;
  float eps;
  int streams, C, y_norm, norm;   /* y_norm: nb_norm, or -1 for none */
} nb_stream_args;
int nb_stream_norm(const nb_stream_args* a, void* h, int h_dtype, int ldh, int rows, void* stream);

/* ---- y (M, N) = x (M, K) . w (N, K)^T (+ bias) for many rows.
 * nb_linear_bf16: bf16 x on the tcgen05 tensor cores, fp32 accumulation, y NB_BF16 or NB_F32; x and w 16-byte
 * aligned, ldx and ldw multiples of 8; `status`: device int, NB_ERR_TIMEOUT if a bounded wait ran out, or NULL.
 * nb_linear_f32: fp32 x and y, fp32 multiply-adds. */
int nb_linear_bf16(const void* x, int ldx, const void* w, int ldw, const float* bias, int act, float alpha, float limit, int M, int N, int K,
                   void* y, int y_dtype, int ldy, int* status, void* stream);
int nb_linear_f32(const float* x, int ldx, const void* w, int ldw, const float* bias, int act, float alpha, float limit, int M, int N, int K,
                  float* y, int ldy, void* stream);

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
  float eps, alpha, limit;
  int N, K, ldw, act, norm;
} nb_matvec_args;
int nb_matvec_bf16(const nb_matvec_args* a, void* stream);
/* The same behind hyper-connections: act = the h of nb_stream_norm for one row (s->x_out != s->x); of `a` the launch reads
 * w, bias, y, N, K, ldw and the activation. */
int nb_matvec_streams(const nb_matvec_args* a, const nb_stream_args* s, void* stream);
/* Two products of plain rows (no norm, no delta) in one launch. */
int nb_matvec_pair(const nb_matvec_args* a, const nb_matvec_args* b, void* stream);

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

/* ---- grouped attention with scores mixed across heads ---------------------------------------------------------
 * Cache of a layer: (B, ctx, ldc) rows [keys of the G heads (G * dim) | .. | values from v_off (G * vdim)] of the activation
 * dtype, ldc and v_off multiples of 8.  Query head h reads key/value head h / (H / G).  Per query i and key j of the window
 * (0 <= i - j < window): s_h = softcap * tanh(q_h . k * scale / softcap) - penalty[h][i - j], then s'_h = sum_g talk[h][g] s_g,
 * softmax of s'_h over the keys, out_h = sum of values * sigmoid(gate), the gate per element.  softcap <= 0: no cap;
 * penalty NULL: none; gate NULL (g_off < 0): none.  penalty: (H, n_pen) fp32 with n_pen >= min(window, ctx); talk (H, H).
 *
 * nb_cache_append: cache[b][pos0 + t][0 .. cols) = src row b * T + t, columns off .. (16 bytes at a time: off and both row
 * strides are multiples of 8, the row's last eight columns are copied whole).
 * nb_talk_attention: T new positions pos0 .. whose keys and values are in the cache.  NB_BF16 runs on the tensor cores
 * (scores, mixing and softmax in fp32; the softmax weights enter the second product as two bf16 terms), NB_F32 in fp32
 * multiply-adds.  The mixed scores of a block of queries pass through the workspace (any size from
 * nb_talk_attention_workspace_bytes(.., 1) on; with more, more queries at a time).
 * nb_talk_decode: one new position per sequence from fp32 projections p: appends its keys and values (p at k_off, in the
 * cache row's layout) and attends, a cluster of CTAs per sequence.  Does nothing when *pos is outside [0, ctx). */
typedef struct {
  const void *q, *cache, *gate;
  void* out;
  const float *penalty, *talk;
  float scale, softcap;
  int dtype, B, T, H, G, dim, vdim, ctx, ldc, v_off, ldq, ldg, ldo, pos0, window, n_pen;
} nb_talk_attention_args;
int nb_cache_append(const void* src, int ld, int off, int cols, void* cache, int ldc, int dtype, int B, int T, int ctx, int pos0, void* stream);
size_t nb_talk_attention_workspace_bytes(int B, int T, int H, int pos0, int window, int query_tiles);
int nb_talk_attention(const nb_talk_attention_args* a, void* workspace, size_t workspace_bytes, void* stream);

typedef struct {
  const float* p;
  void* cache;
  const float *penalty, *talk;
  const int64_t* pos;
  float* out;
  float scale, softcap;
  int cache_dtype, B, H, G, dim, vdim, ctx, ldc, v_off, ldp, q_off, k_off, g_off, ldo, window, n_pen;
} nb_talk_decode_args;
int nb_talk_decode(const nb_talk_decode_args* a, void* stream);

/* ---- gated linear attention -------------------------------------------------------------------------------
 * p: (B * T, ldp) projections, q at q_off (H * dim), k at k_off, v at v_off (H * vdim), g at g_off, a at a_off
 * (a_rank); decay alpha = sigmoid(a2 . a + a2_b)^(1 / tau) per key channel; per head S <- diag(alpha) S + k v^T,
 * o = S^T (q * dim^-1/2); out (B * T, ldo) = RMSNorm(o) * norm_w * silu(g).  state: (B, H, dim, lds) fp32, lds a
 * multiple of 4, columns vdim .. lds zero; read and updated.
 * kind NB_GLA_FORGET: the decay decides what is written as well.  z = p at k_off (H * dim) + a2_b, alpha = lower +
 * (1 - lower) sigmoid(z), k = 1 - alpha, o = S^T silu(q) without a scale; no low-rank projection (a2, a_off and a_rank are
 * not read, nor is tau) and, with g_off < 0, no output gate. */
typedef enum { NB_GLA_LOW_RANK = 0, NB_GLA_FORGET = 1 } nb_gla_kind;
/*
 * nb_gla_prefill works in chunks of 64 tokens; workspace of nb_gla_workspace_bytes().
 * nb_gla_decode: one token per sequence, fp32 p and out. */
typedef struct {
  const void* p;
  void* out;
  float* state;
  const void* a2;      /* bf16 (H * dim, lda2) */
  const float *a2_b, *norm_w, *lower;
  float tau, eps;
  int kind, dtype, B, T, H, dim, vdim, ldp, q_off, k_off, v_off, g_off, a_off, a_rank, lda2, lds, ldo;
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
