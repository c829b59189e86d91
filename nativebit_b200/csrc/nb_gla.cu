// Gated linear attention: per head a (dim x vdim) state S, S <- diag(alpha) S + k v^T, o = S^T q, with a decay alpha per
// key channel: from a low-rank projection beside a projected key (NB_GLA_LOW_RANK), or a forget gate above a lower bound
// with the key 1 - alpha (NB_GLA_FORGET, the HGRN2 recurrence).
//
// Prompts run in chunks of 64 tokens (the chunkwise form of "Gated Linear Attention Transformers with Hardware-Efficient
// Training", Yang, Wang, Shen, Panda and Kim): every chunk's contribution to the state in parallel, a scan over the chunks,
// then every chunk's outputs in parallel from the state at its start and the scores inside it.  Decays are carried as
// logarithms, summed inside sub-blocks of 16 tokens, and every exponential taken is of a number <= 0: a strongly decaying
// channel underflows to zero instead of overflowing, and neighbouring tokens never subtract two large sums.
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <cooperative_groups.h>

#include <algorithm>

#include "nb_layered.cuh"
#include "nb_mma.cuh"

namespace nb {

namespace cg = cooperative_groups;

constexpr int kGC = 64, kGS = 16, kGSubs = kGC / kGS;   // chunk, sub-block, sub-blocks per chunk

struct GlaWs {
  float* bl;    // (B * T, H * dim) log decays, summed from the start of the token's sub-block to the token itself
  float* u;     // (B, chunks, H, dim, lds) contributions of the chunks; the scan turns them into the states at their starts
  float* dec;   // (B, chunks, H, dim) log decay over the chunk
  float* o;     // (B * T, H * vdim) outputs before the norm
};

__host__ __device__ inline int gla_chunks(int T) { return (T + kGC - 1) / kGC; }

// ---- the forget gate: alpha = 1 - om * sigmoid(-z) with om = 1 - lower; the key is om * sigmoid(-z), without the
// cancellation of 1 - alpha.
__device__ __forceinline__ float forget_key(float z, float om) { return om * sigmoid_f(-z); }
__device__ __forceinline__ float forget_key_fast(float z, float om) { return __fdividef(om, 1.f + __expf(z)); }
// log alpha; a gate that closes completely counts as the smallest normal number
__device__ __forceinline__ float forget_log(float z, float lower) {
  const float om = 1.f - lower, k = forget_key(z, om);
  return k < 0.5f ? log1pf(-k) : logf(fmaxf(lower + om * sigmoid_f(z), 1.17549435e-38f));
}
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// q and k as the recurrence takes them, from what the projection left (fp32 functions): `ch` counts all heads' channels.
template <int kKind> __device__ __forceinline__ float gla_q(float q, float scale) { return kKind == NB_GLA_FORGET ? silu_f(q) : q * scale; }
template <int kKind> __device__ __forceinline__ float gla_k(const nb_gla_args& p, float k, int ch) {
  return kKind == NB_GLA_FORGET ? forget_key(k + p.a2_b[ch], 1.f - p.lower[ch]) : k;
}

// ---- decays.  grid (sub-blocks, channel tiles, B); a thread owns one channel of 16 tokens.
constexpr int kDecThreads = 128;
template <typename T> __global__ void __launch_bounds__(kDecThreads) gla_forget_kernel(const nb_gla_args p, GlaWs w) {
  const int t0 = blockIdx.x * kGS, b = blockIdx.z, ch = blockIdx.y * kDecThreads + threadIdx.x, HD = p.H * p.dim;
  if (ch >= HD) return;
  const int cnt = min(kGS, p.T - t0);
  const T* z = reinterpret_cast<const T*>(p.p) + (size_t)(b * p.T + t0) * p.ldp + p.k_off + ch;
  float* out = w.bl + (size_t)(b * p.T + t0) * HD + ch;
  const float bias = p.a2_b[ch], lower = p.lower[ch];
  float v[kGS], sum = 0.f;
#pragma unroll
  for (int t = 0; t < kGS; ++t) v[t] = t < cnt ? to_f(z[(size_t)t * p.ldp]) : 0.f;
#pragma unroll
  for (int t = 0; t < kGS; ++t) {
    sum += forget_log(v[t] + bias, lower);
    if (t < cnt) out[(size_t)t * HD] = sum;
  }
}

template <typename T> __global__ void __launch_bounds__(kDecThreads) gla_decay_kernel(const nb_gla_args p, GlaWs w) {
  extern __shared__ __align__(16) float as[];           // [kGS][a_rank]
  const int t0 = blockIdx.x * kGS, b = blockIdx.z, ch = blockIdx.y * kDecThreads + threadIdx.x, HD = p.H * p.dim;
  const int cnt = min(kGS, p.T - t0);
  const T* base = reinterpret_cast<const T*>(p.p) + (size_t)(b * p.T + t0) * p.ldp + p.a_off;
  for (int i = threadIdx.x; i < kGS * p.a_rank; i += kDecThreads) {
    const int t = i / p.a_rank, r = i - t * p.a_rank;
    as[i] = t < cnt ? to_f(base[(size_t)t * p.ldp + r]) : 0.f;
  }
  __syncthreads();
  if (ch >= HD) return;
  float z[kGS];
  const float bias = p.a2_b[ch];
#pragma unroll
  for (int t = 0; t < kGS; ++t) z[t] = bias;
  const bf16* w2 = reinterpret_cast<const bf16*>(p.a2) + (size_t)ch * p.lda2;
  for (int r = 0; r < p.a_rank; ++r) {
    const float x = to_f(w2[r]);
#pragma unroll
    for (int t = 0; t < kGS; ++t) z[t] = fmaf(x, as[t * p.a_rank + r], z[t]);
  }
  float sum = 0.f;
  const float inv_tau = 1.0f / p.tau;
  float* out = w.bl + (size_t)(b * p.T + t0) * HD + ch;
#pragma unroll
  for (int t = 0; t < kGS; ++t) {
    // with bf16 projections log(1 + e^-|z|) goes through the hardware functions: absolute errors of 1e-7
    sum += (sizeof(T) == 2 ? fminf(z[t], 0.f) - __logf(1.f + __expf(-fabsf(z[t]))) : log_sigmoid_f(z[t])) * inv_tau;
    if (t < cnt) out[(size_t)t * HD] = sum;
  }
}

// ---- what a chunk adds to the state: U[d][v] = sum_t k_t[d] exp(decay from t to the chunk's end) v_t[v].
// grid (chunks, H * d tiles * v tiles, B), 64 x 64 outputs per CTA.
template <typename T, int kKind> __global__ void __launch_bounds__(256) gla_state_kernel(const nb_gla_args p, GlaWs w, int dtiles, int vtiles) {
  __shared__ __align__(16) float ks[kGC][64 + 4], vs[kGC][64 + 4];
  __shared__ float tot[kGSubs][64];                     // log decay of a whole sub-block
  const int n = blockIdx.x, b = blockIdx.z, tid = threadIdx.x;
  const int h = blockIdx.y / (dtiles * vtiles), rest = blockIdx.y - h * dtiles * vtiles;
  const int d0 = (rest / vtiles) * 64, v0 = (rest % vtiles) * 64;
  const int t0 = n * kGC, cnt = min(kGC, p.T - t0), HD = p.H * p.dim;
  const T* base = reinterpret_cast<const T*>(p.p) + (size_t)(b * p.T + t0) * p.ldp;
  const float* bl = w.bl + (size_t)(b * p.T + t0) * HD + h * p.dim;
  for (int i = tid; i < kGSubs * 64; i += 256) {
    const int s = i >> 6, d = d0 + (i & 63), t = min(cnt, (s + 1) * kGS) - 1;
    tot[s][i & 63] = (s * kGS < cnt && d < p.dim) ? bl[(size_t)t * HD + d] : 0.f;
  }
  __syncthreads();
  for (int i = tid; i < kGC * 64; i += 256) {
    const int t = i >> 6, c = i & 63, d = d0 + c, v = v0 + c, s = t / kGS;
    float kv = 0.f;
    if (t < cnt && d < p.dim) {
      float e = tot[s][c] - bl[(size_t)t * HD + d];
      for (int m = s + 1; m < kGSubs; ++m) e += tot[m][c];
      kv = gla_k<kKind>(p, to_f(base[(size_t)t * p.ldp + p.k_off + h * p.dim + d]), h * p.dim + d) * expf(e);
    }
    ks[t][c] = kv;
    vs[t][c] = (t < cnt && v < p.vdim) ? to_f(base[(size_t)t * p.ldp + p.v_off + h * p.vdim + v]) : 0.f;
  }
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
#pragma unroll 8
  for (int t = 0; t < kGC; ++t) {
    const float4 a = *reinterpret_cast<const float4*>(&ks[t][ty * 4]), c = *reinterpret_cast<const float4*>(&vs[t][tx * 4]);
    const float av[4] = {a.x, a.y, a.z, a.w}, cv[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], cv[j], acc[i][j]);
  }
  const size_t head = ((size_t)b * gridDim.x + n) * p.H + h;
  float* u = w.u + head * p.dim * p.lds;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int d = d0 + ty * 4 + i, v = v0 + tx * 4;
    if (d < p.dim && v < p.lds) *reinterpret_cast<float4*>(u + (size_t)d * p.lds + v) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
  }
  if (v0 == 0 && tid < 64 && d0 + tid < p.dim) w.dec[head * p.dim + d0 + tid] = tot[0][tid] + tot[1][tid] + tot[2][tid] + tot[3][tid];
}

// ---- scan over the chunks, element by element: u[n] becomes the state at the start of chunk n, state the final one.
__global__ void __launch_bounds__(256) gla_scan_kernel(const nb_gla_args p, GlaWs w, int chunks) {
  const int per = p.dim * (p.lds / 4), i = blockIdx.x * 256 + threadIdx.x, bh = blockIdx.y;
  if (i >= per) return;
  const int b = bh / p.H, h = bh - b * p.H, d = i / (p.lds / 4);
  float4* st = reinterpret_cast<float4*>(p.state) + (size_t)bh * per + i;
  float4 s = *st;
  constexpr int kAhead = 8;            // chunks requested at a time: the loads do not depend on one another
  for (int n0 = 0; n0 < chunks; n0 += kAhead) {
    float4 u[kAhead];
    float a[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const size_t head = ((size_t)b * chunks + min(n0 + j, chunks - 1)) * p.H + h;
      u[j] = reinterpret_cast<const float4*>(w.u)[head * per + i];
      a[j] = w.dec[head * p.dim + d];
    }
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (n0 + j < chunks) {
        const size_t head = ((size_t)b * chunks + n0 + j) * p.H + h;
        reinterpret_cast<float4*>(w.u)[head * per + i] = s;
        const float e = expf(a[j]);
        s.x = fmaf(s.x, e, u[j].x); s.y = fmaf(s.y, e, u[j].y); s.z = fmaf(s.z, e, u[j].z); s.w = fmaf(s.w, e, u[j].w);
      }
    }
  }
  *st = s;
}

// ---- outputs of a chunk: o_t = S^T (q_t decayed from the chunk's start) + sum_{s <= t} A[t][s] v_s, with
// A[t][s] = sum_d q_t[d] k_s[d] exp(decay from s to t).  grid (chunks, H, B).  A is built 4 x 4 per thread; for tokens of
// different sub-blocks the decay is split at the start of t's sub-block, inside a sub-block at the start of t's group of
// four, and inside a group of four it is taken pair by pair.
template <typename T, int kKind> __global__ void __launch_bounds__(256) gla_output_kernel(const nb_gla_args p, GlaWs w) {
  extern __shared__ __align__(16) float gsm[];
  constexpr int ld = 64 + 4;
  float* as = gsm;                      // [64][ld]  A, transposed: as[s][t]
  float* qt = as + kGC * ld;            // [64][ld]  q of a tile of 64 channels, transposed: qt[d][t]
  float* kt = qt + kGC * ld;            // [64][ld]  k, later v: [s][v]
  float* bt = kt + kGC * ld;            // [64][ld]  summed log decays, transposed, later a tile of S
  float* tot = bt + kGC * ld;           // [kGSubs][64]
  const int n = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int t0 = n * kGC, cnt = min(kGC, p.T - t0), HD = p.H * p.dim;
  const T* base = reinterpret_cast<const T*>(p.p) + (size_t)(b * p.T + t0) * p.ldp;
  const float* bl = w.bl + (size_t)(b * p.T + t0) * HD + h * p.dim;
  const float qscale = 1.0f / sqrtf((float)p.dim);
  const int tb = ty * 4, sb = tx * 4, si = tb / kGS, sj = sb / kGS;   // this thread's tokens t (rows) and s (columns)

  auto load_tile = [&](int d0) {
    for (int i = tid; i < kGC * 64; i += 256) {
      const int t = i >> 6, c = i & 63, d = d0 + c;
      const bool in = t < cnt && d < p.dim;
      qt[c * ld + t] = in ? gla_q<kKind>(to_f(base[(size_t)t * p.ldp + p.q_off + h * p.dim + d]), qscale) : 0.f;
      bt[c * ld + t] = in ? bl[(size_t)t * HD + d] : 0.f;
    }
    for (int i = tid; i < kGSubs * 64; i += 256) {
      const int s = i >> 6, d = d0 + (i & 63), t = min(cnt, (s + 1) * kGS) - 1;
      tot[i] = (s * kGS < cnt && d < p.dim) ? bl[(size_t)t * HD + d] : 0.f;
    }
  };

  float a[4][4] = {};
  for (int d0 = 0; d0 < p.dim; d0 += 64) {
    __syncthreads();
    load_tile(d0);
    for (int i = tid; i < kGC * 64; i += 256) {
      const int t = i >> 6, c = i & 63, d = d0 + c;
      kt[c * ld + t] = (t < cnt && d < p.dim) ? gla_k<kKind>(p, to_f(base[(size_t)t * p.ldp + p.k_off + h * p.dim + d]), h * p.dim + d) : 0.f;
    }
    __syncthreads();
    const int dn = min(64, p.dim - d0);
    if (sb <= tb) {
      for (int d = 0; d < dn; ++d) {
        const float4 q4 = *reinterpret_cast<const float4*>(qt + d * ld + tb), bq4 = *reinterpret_cast<const float4*>(bt + d * ld + tb);
        const float4 k4 = *reinterpret_cast<const float4*>(kt + d * ld + sb), bk4 = *reinterpret_cast<const float4*>(bt + d * ld + sb);
        float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w};
        const float bq[4] = {bq4.x, bq4.y, bq4.z, bq4.w}, bk[4] = {bk4.x, bk4.y, bk4.z, bk4.w};
        if (sb == tb) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            a[i][i] = fmaf(q[i], k[i], a[i][i]);
#pragma unroll
            for (int j = 0; j < i; ++j) a[i][j] = fmaf(q[i] * expf(bq[i] - bk[j]), k[j], a[i][j]);
          }
        } else {
          float ref_q, ref_k;             // the decay is split there: both parts are <= 0
          if (si == sj) {
            ref_q = ref_k = bt[d * ld + tb - 1];   // tb is not the first group of its sub-block here
          } else {
            ref_q = 0.f;
            ref_k = tot[sj * 64 + d];
            for (int m = sj + 1; m < si; ++m) ref_k += tot[m * 64 + d];
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) { q[i] *= expf(bq[i] - ref_q); k[i] *= expf(ref_k - bk[i]); }
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) a[i][j] = fmaf(q[i], k[j], a[i][j]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) as[(sb + j) * ld + tb + i] = (tb + i < cnt && sb + j <= tb + i) ? a[i][j] : 0.f;

  const float* S = w.u + (((size_t)b * gridDim.x + n) * p.H + h) * p.dim * p.lds;
  for (int v0 = 0; v0 < p.vdim; v0 += 64) {
    float o[4][4] = {};
    for (int d0 = 0; d0 < p.dim; d0 += 64) {
      __syncthreads();
      load_tile(d0);
      __syncthreads();
      for (int i = tid; i < kGC * 64; i += 256) {       // q decayed from the chunk's start; then a tile of S over the decays
        const int c = i & 63, t = i >> 6;
        float e = bt[c * ld + t];
        for (int m = 0; m < t / kGS; ++m) e += tot[m * 64 + c];
        qt[c * ld + t] *= expf(e);
      }
      __syncthreads();
      for (int i = tid; i < 64 * 64; i += 256) {
        const int d = i >> 6, v = i & 63;
        bt[d * ld + v] = (d0 + d < p.dim && v0 + v < p.vdim) ? S[(size_t)(d0 + d) * p.lds + v0 + v] : 0.f;
      }
      __syncthreads();
      const int dn = min(64, p.dim - d0);
      for (int d = 0; d < dn; ++d) {
        const float4 q4 = *reinterpret_cast<const float4*>(qt + d * ld + tb), s4 = *reinterpret_cast<const float4*>(bt + d * ld + tx * 4);
        const float q[4] = {q4.x, q4.y, q4.z, q4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) o[i][j] = fmaf(q[i], s[j], o[i][j]);
      }
    }
    __syncthreads();
    for (int i = tid; i < kGC * 64; i += 256) {
      const int t = i >> 6, c = i & 63;
      kt[t * ld + c] = (t < cnt && v0 + c < p.vdim) ? to_f(base[(size_t)t * p.ldp + p.v_off + h * p.vdim + v0 + c]) : 0.f;
    }
    __syncthreads();
    for (int s = 0; s < tb + 4; ++s) {
      const float4 a4 = *reinterpret_cast<const float4*>(as + s * ld + tb), v4 = *reinterpret_cast<const float4*>(kt + s * ld + tx * 4);
      const float av[4] = {a4.x, a4.y, a4.z, a4.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = fmaf(av[i], vv[j], o[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (tb + i < cnt && v0 + tx * 4 + j < p.vdim)
          w.o[(size_t)(b * p.T + t0 + tb + i) * p.H * p.vdim + h * p.vdim + v0 + tx * 4 + j] = o[i][j];
  }
}

// ---- out = RMSNorm(o) * norm_w * silu(g) (no gate with g_off < 0), one warp per (row, head)
template <typename T> __global__ void __launch_bounds__(256) gla_finish_kernel(const nb_gla_args p, GlaWs w) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const size_t rh = (size_t)blockIdx.x * 8 + warp;
  if (rh >= (size_t)p.B * p.T * p.H) return;
  const size_t row = rh / p.H;
  const int h = (int)(rh - row * p.H);
  const float* o = w.o + rh * p.vdim;
  float ss = 0.f;
  for (int i = lane; i < p.vdim; i += 32) ss += o[i] * o[i];
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  const T* g = reinterpret_cast<const T*>(p.p) + row * p.ldp + p.g_off + h * p.vdim;
  T* out = reinterpret_cast<T*>(p.out) + row * p.ldo + h * p.vdim;
  for (int i = lane; i < p.vdim; i += 32) out[i] = from_f<T>(o[i] * inv * p.norm_w[i] * (p.g_off < 0 ? 1.f : silu_f(to_f(g[i]))));
}

// ---- the same two kernels for bf16 projections on the tensor cores.  q, k and v are bf16 as they are; everything the
// recurrence adds — decayed q and k, the state, the scores — stays fp32 and enters a product as two bf16 terms (the
// product of two such pairs as three).  Four warps per CTA; vdim <= VD.
constexpr int kGmThreads = 128;
constexpr int kGmLd = 64 + 8;          // row stride of a staged tile of 64 channels, in elements
constexpr int kGbLd = 64 + 4;          // row stride of staged log decays
constexpr float kSplitLimit = -60.f;   // a sub-block that decays further is taken pair by pair

template <int VD> struct GlaStateSmem {
  bf16 k[kGC * kGmLd], khi[kGC * kGmLd], klo[kGC * kGmLd], v[kGC * (VD + 8)];
  float bl[kGC * kGbLd], tot[kGSubs * 64];
};

// Copies rows of `cols` bf16 (zero past `valid` columns and `cnt` rows) into shared memory; vec: 16-byte aligned, cols % 8 == 0,
// asynchronous: complete after stage_wait() and a barrier.
__device__ __forceinline__ void stage_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

__device__ __forceinline__ void stage_rows(bf16* dst, int ldd, const bf16* src, int lds, int cols, int valid, int cnt, bool vec) {
  if (vec) {
    const int c8 = (threadIdx.x & 7) * 8;
#pragma unroll
    for (int tr = 0; tr < kGC; tr += kGmThreads / 8) {
      const int t = tr + (threadIdx.x >> 3);
      for (int c = c8; c < cols; c += 64) {
        if (t < cnt && c < valid) cp16(dst + t * ldd + c, src + (size_t)t * lds + c);
        else *reinterpret_cast<uint4*>(dst + t * ldd + c) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
  } else {
    for (int i = threadIdx.x; i < kGC * cols; i += kGmThreads) {
      const int t = i / cols, c = i - t * cols;
      dst[t * ldd + c] = (t < cnt && c < valid) ? src[(size_t)t * lds + c] : from_f<bf16>(0.f);
    }
  }
}

// Summed log decays of a chunk, 64 channels from `src` (zero past cnt rows and dn channels), into shared memory.
__device__ __forceinline__ void stage_decays(float* dst, const float* src, int HD, int dn, int cnt, bool vec) {
  if (vec) {
    const int c = (threadIdx.x & 15) * 4;
#pragma unroll
    for (int tr = 0; tr < kGC; tr += kGmThreads / 16) {
      const int t = tr + (threadIdx.x >> 4);
      if (t < cnt && c < dn) cp16(dst + t * kGbLd + c, src + (size_t)t * HD + c);
      else *reinterpret_cast<float4*>(dst + t * kGbLd + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int i = threadIdx.x; i < kGC * 64; i += kGmThreads) {
      const int t = i >> 6, d = i & 63;
      dst[t * kGbLd + d] = (t < cnt && d < dn) ? src[(size_t)t * HD + d] : 0.f;
    }
  }
}

// Log decay of the chunk's sub-blocks (their last token's sum).
__device__ __forceinline__ bool sub_block_totals(float* tot, const float* bl, int cnt) {
  bool deep = false;
  for (int i = threadIdx.x; i < kGSubs * 64; i += kGmThreads) {
    const int s = i >> 6, t = min(cnt, (s + 1) * kGS) - 1;
    const float x = s * kGS < cnt ? bl[t * kGbLd + (i & 63)] : 0.f;
    tot[i] = x;
    deep |= x < kSplitLimit;
  }
  return deep;
}

// Bias and 1 - lower bound of two neighbouring channels, and the keys of the pair.
struct ForgetPair {
  float2 bias, om;
  __device__ ForgetPair(const nb_gla_args& p, int kind, int ch, int d, int dn) {
    bias = om = make_float2(0.f, 0.f);
    if (kind != NB_GLA_FORGET) return;
    if (d < dn) { bias.x = p.a2_b[ch]; om.x = 1.f - p.lower[ch]; }
    if (d + 1 < dn) { bias.y = p.a2_b[ch + 1]; om.y = 1.f - p.lower[ch + 1]; }
  }
  template <int kKind> __device__ __forceinline__ float2 key(uint32_t kk) const {
    if (kKind != NB_GLA_FORGET) return make_float2(bf_lo(kk), bf_hi(kk));
    return make_float2(forget_key_fast(bf_lo(kk) + bias.x, om.x), forget_key_fast(bf_hi(kk) + bias.y, om.y));
  }
};

// grid (chunks, H * d tiles, B): 64 channels x vdim of a chunk's contribution.
template <int VD, int kKind> __global__ void __launch_bounds__(kGmThreads) gla_state_mma_kernel(const nb_gla_args p, GlaWs w, int dtiles, int vec) {
  extern __shared__ __align__(16) uint8_t gsm_raw[];
  GlaStateSmem<VD>& sm = *reinterpret_cast<GlaStateSmem<VD>*>(gsm_raw);
  const int n = blockIdx.x, h = blockIdx.y / dtiles, d0 = (blockIdx.y - h * dtiles) * 64, b = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = n * kGC, cnt = min(kGC, p.T - t0), HD = p.H * p.dim;
  const bf16* base = reinterpret_cast<const bf16*>(p.p) + (size_t)(b * p.T + t0) * p.ldp;
  const float* bl = w.bl + (size_t)(b * p.T + t0) * HD + h * p.dim + d0;
  const int dn = min(64, p.dim - d0);
  stage_decays(sm.bl, bl, HD, dn, cnt, vec);
  stage_rows(sm.k, kGmLd, base + p.k_off + h * p.dim + d0, p.ldp, 64, dn, cnt, vec);
  stage_rows(sm.v, VD + 8, base + p.v_off + h * p.vdim, p.ldp, VD, p.vdim, cnt, vec);
  const ForgetPair fp(p, kKind, h * p.dim + d0 + 2 * lane, 2 * lane, dn);   // of this thread's pair of channels below
  stage_wait();
  __syncthreads();
  sub_block_totals(sm.tot, sm.bl, cnt);
  __syncthreads();
#pragma unroll 4
  for (int i = tid; i < kGC * 32; i += kGmThreads) {      // pairs of channels
    const int t = i >> 5, d = (i & 31) * 2, s = t / kGS;
    const float2 bb = *reinterpret_cast<const float2*>(sm.bl + t * kGbLd + d);
    const uint32_t kk = *reinterpret_cast<const uint32_t*>(sm.k + t * kGmLd + d);
    float ex = sm.tot[s * 64 + d] - bb.x, ey = sm.tot[s * 64 + d + 1] - bb.y;
#pragma unroll
    for (int m = 1; m < kGSubs; ++m)
      if (m > s) { ex += sm.tot[m * 64 + d]; ey += sm.tot[m * 64 + d + 1]; }
    uint32_t hi, lo;
    const float2 key = fp.key<kKind>(kk);
    split_bf16(key.x * __expf(ex), key.y * __expf(ey), hi, lo);
    if (t >= cnt) hi = lo = 0u;
    *reinterpret_cast<uint32_t*>(sm.khi + t * kGmLd + d) = hi;
    *reinterpret_cast<uint32_t*>(sm.klo + t * kGmLd + d) = lo;
  }
  __syncthreads();
  float acc[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  // rows of the product are channels: the A fragment is k transposed
  const int at = ((lane >> 4) << 3) + (lane & 7), ac = warp * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
  for (int kk = 0; kk < kGC; kk += 16) {
    uint32_t hi[4], lo[4];
    ldsm_x4_t(hi, sm.khi + (kk + at) * kGmLd + ac);
    ldsm_x4_t(lo, sm.klo + (kk + at) * kGmLd + ac);
#pragma unroll
    for (int v = 0; v < VD / 16; ++v) {
      uint32_t bb[4];
      ldsm_x4_t(bb, sm.v + (kk + (lane & 15)) * (VD + 8) + v * 16 + (lane >> 4) * 8);
      mma_bf16(acc[2 * v], hi, bb[0], bb[1]);
      mma_bf16(acc[2 * v + 1], hi, bb[2], bb[3]);
      mma_bf16(acc[2 * v], lo, bb[0], bb[1]);
      mma_bf16(acc[2 * v + 1], lo, bb[2], bb[3]);
    }
  }
  const size_t head = ((size_t)b * gridDim.x + n) * p.H + h;
  float* u = w.u + (head * p.dim + d0) * p.lds;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int d = warp * 16 + (lane >> 2) + 8 * half;
    if (d < dn) {
#pragma unroll
      for (int i = 0; i < VD / 8; ++i) {
        const int v = i * 8 + (lane & 3) * 2;              // lds is a multiple of 4: a pair never straddles the end
        if (v < p.lds) *reinterpret_cast<float2*>(u + (size_t)d * p.lds + v) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
      }
    }
  }
  if (tid < dn) w.dec[head * p.dim + d0 + tid] = sm.tot[tid] + sm.tot[64 + tid] + sm.tot[128 + tid] + sm.tot[192 + tid];
}

template <int VD> struct GlaOutSmem {
  bf16 q[kGC * kGmLd], k[kGC * kGmLd];           // as they are
  bf16 khi[kGC * kGmLd], klo[kGC * kGmLd];       // k decayed to the end of its sub-block
  float bl[kGC * kGbLd];                         // summed log decays
  float tot[kGSubs * 64];                        // log decay of a whole sub-block
  float fac[10 * 64];                            // factors of the block pairs and of the chunk's start, see below
  bf16 shi[64 * (VD + 8)], slo[64 * (VD + 8)];   // a tile of the state; at the end v
};

// grid (chunks, H, B).  Warp i owns sub-block i: its 16 queries against the keys of sub-blocks 0 .. i and against the state
// at the chunk's start; then the scores against the values, the norm over the head's outputs and the gate.
//   q . k over sub-blocks i > j: (q exp(bl)) . (k exp(tot_j - bl)) * exp(tot_{j+1} + .. + tot_{i-1}), the last on q's side;
//   i == j: the same with exp(-tot_i), as long as no channel of the tile decays past kSplitLimit inside the sub-block.
template <int VD, int kKind> __global__ void __launch_bounds__(kGmThreads) gla_output_mma_kernel(const nb_gla_args p, GlaWs w, int vec) {
  extern __shared__ __align__(16) uint8_t gsm_raw[];
  GlaOutSmem<VD>& sm = *reinterpret_cast<GlaOutSmem<VD>*>(gsm_raw);
  const int n = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = n * kGC, cnt = min(kGC, p.T - t0), HD = p.H * p.dim;
  const bf16* base = reinterpret_cast<const bf16*>(p.p) + (size_t)(b * p.T + t0) * p.ldp;
  const float* blg = w.bl + (size_t)(b * p.T + t0) * HD + h * p.dim;
  const float* S = w.u + (((size_t)b * gridDim.x + n) * p.H + h) * p.dim * p.lds;
  const float qscale = 1.0f / sqrtf((float)p.dim);
  const int ra = warp * 16 + (lane >> 2), rb = ra + 8, c2 = (lane & 3) * 2;   // this lane's two query rows, its column pair

  float sc[kGSubs][2][4];              // scores: key sub-block, half of it, fragment
  float o[VD / 8][4];
#pragma unroll
  for (int j = 0; j < kGSubs; ++j)
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[j][x][e] = 0.f;
#pragma unroll
  for (int i = 0; i < VD / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;

  for (int d0 = 0; d0 < p.dim; d0 += 64) {
    const int dn = min(64, p.dim - d0);
    __syncthreads();                   // the tile before is no longer read
    stage_rows(sm.q, kGmLd, base + p.q_off + h * p.dim + d0, p.ldp, 64, dn, cnt, vec);
    stage_rows(sm.k, kGmLd, base + p.k_off + h * p.dim + d0, p.ldp, 64, dn, cnt, vec);
    stage_decays(sm.bl, blg + d0, HD, dn, cnt, vec);
#pragma unroll 8
    for (int i = tid; i < 64 * (VD / 4); i += kGmThreads) {     // state, four columns at a time (a row is padded to fours)
      const int d = i / (VD / 4), v = (i - d * (VD / 4)) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d < dn && v < p.lds) x = *reinterpret_cast<const float4*>(S + (size_t)(d0 + d) * p.lds + v);
      uint32_t h0, l0, h1, l1;
      split_bf16(x.x, x.y, h0, l0);
      split_bf16(x.z, x.w, h1, l1);
      *reinterpret_cast<uint2*>(sm.shi + d * (VD + 8) + v) = make_uint2(h0, h1);
      *reinterpret_cast<uint2*>(sm.slo + d * (VD + 8) + v) = make_uint2(l0, l1);
    }
    stage_wait();
    __syncthreads();
    const bool deep = __syncthreads_or(sub_block_totals(sm.tot, sm.bl, cnt));   // some channel decays past the limit in a sub-block
    if (tid < 64) {
      const float a0 = sm.tot[tid], a1 = sm.tot[64 + tid], a2 = sm.tot[128 + tid], a3 = sm.tot[192 + tid];
      float* f = sm.fac + tid;
      f[0 * 64] = __expf(a1);            // between sub-blocks 2 and 0
      f[1 * 64] = __expf(a2);            // 3 and 1
      f[2 * 64] = __expf(a1 + a2);       // 3 and 0
      f[3 * 64] = __expf(a0);            // from the chunk's start to sub-block 1, 2, 3
      f[4 * 64] = __expf(a0 + a1);
      f[5 * 64] = __expf(a0 + a1 + a2);
      f[6 * 64] = deep ? 0.f : __expf(-a0);      // inside sub-block 0 .. 3
      f[7 * 64] = deep ? 0.f : __expf(-a1);
      f[8 * 64] = deep ? 0.f : __expf(-a2);
      f[9 * 64] = deep ? 0.f : __expf(-a3);
    }
    const ForgetPair fp(p, kKind, h * p.dim + d0 + 2 * lane, 2 * lane, dn);
    for (int i = tid; i < kGC * 32; i += kGmThreads) {
      const int t = i >> 5, d = (i & 31) * 2;
      const uint32_t kk = *reinterpret_cast<const uint32_t*>(sm.k + t * kGmLd + d);
      const float* tt = sm.tot + (t / kGS) * 64 + d;
      uint32_t hi, lo;
      const float2 key = fp.key<kKind>(kk);
      split_bf16(key.x * __expf(tt[0] - sm.bl[t * kGbLd + d]), key.y * __expf(tt[1] - sm.bl[t * kGbLd + d + 1]), hi, lo);
      if (t >= cnt) hi = lo = 0u;
      *reinterpret_cast<uint32_t*>(sm.khi + t * kGmLd + d) = hi;
      *reinterpret_cast<uint32_t*>(sm.klo + t * kGmLd + d) = lo;
    }
    __syncthreads();
#pragma unroll 1
    for (int kk = 0; kk < 64; kk += 16) {
      if (kk >= dn) break;
      // decayed queries of this step, fp32, in the A fragment's places: (row a, row b) x (columns c2, c2 + 8)
      float qd[4][2];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = (j & 1) ? rb : ra, c = kk + c2 + (j >> 1) * 8;
        const uint32_t qq = *reinterpret_cast<const uint32_t*>(sm.q + r * kGmLd + c);
        qd[j][0] = (kKind == NB_GLA_FORGET ? silu_fast(bf_lo(qq)) : bf_lo(qq) * qscale) * __expf(sm.bl[r * kGbLd + c]);
        qd[j][1] = (kKind == NB_GLA_FORGET ? silu_fast(bf_hi(qq)) : bf_hi(qq) * qscale) * __expf(sm.bl[r * kGbLd + c + 1]);
      }
      auto fragment = [&](const float* f, uint32_t (&hi)[4], uint32_t (&lo)[4]) {   // f: per-channel factor or null
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int c = kk + c2 + (j >> 1) * 8;
          const float fx = f ? f[c] : 1.f, fy = f ? f[c + 1] : 1.f;
          split_bf16(qd[j][0] * fx, qd[j][1] * fy, hi[j], lo[j]);
        }
      };
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < kGSubs; ++j) {
        if (j > warp) break;
        const float* f = j == warp ? sm.fac + (6 + warp) * 64
                         : j + 1 == warp ? nullptr
                         : sm.fac + (warp == 2 ? 0 : j == 1 ? 1 : 2) * 64;
        if (j == warp && deep) continue;
        fragment(f, hi, lo);
        uint32_t kh[4], kl[4];         // sixteen keys: row = token, column = channel
        const int off = (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * kGmLd + kk + ((lane >> 3) & 1) * 8;
        ldsm_x4(kh, sm.khi + off);
        ldsm_x4(kl, sm.klo + off);
        mma_bf16(sc[j][0], hi, kh[0], kh[1]);
        mma_bf16(sc[j][1], hi, kh[2], kh[3]);
        mma_bf16(sc[j][0], hi, kl[0], kl[1]);
        mma_bf16(sc[j][1], hi, kl[2], kl[3]);
        mma_bf16(sc[j][0], lo, kh[0], kh[1]);
        mma_bf16(sc[j][1], lo, kh[2], kh[3]);
      }
      fragment(warp == 0 ? nullptr : sm.fac + (2 + warp) * 64, hi, lo);
#pragma unroll
      for (int v = 0; v < VD / 16; v += 2) {         // eight independent products before an accumulator comes again
        uint32_t sh[2][4], sl[2][4];
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int off = (kk + (lane & 15)) * (VD + 8) + (v + y) * 16 + (lane >> 4) * 8;
          ldsm_x4_t(sh[y], sm.shi + off);
          ldsm_x4_t(sl[y], sm.slo + off);
        }
#pragma unroll
        for (int term = 0; term < 3; ++term)
#pragma unroll
          for (int y = 0; y < 2; ++y)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
              const uint32_t(&bb)[4] = term == 1 ? sl[y] : sh[y];
              mma_bf16(o[2 * (v + y) + x], term == 2 ? lo : hi, bb[2 * x], bb[2 * x + 1]);
            }
      }
    }
    if (deep) {                        // the pairs of this warp's own sub-block, one exponential each
#pragma unroll
      for (int j = 0; j < kGSubs; ++j) {
        if (j != warp) continue;
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int t = e < 2 ? ra : rb, s = j * 16 + x * 8 + c2 + (e & 1);
            if (s > t || t >= cnt) continue;
            float sum = 0.f;
            for (int d = 0; d < dn; ++d)
              sum += gla_q<kKind>(to_f(sm.q[t * kGmLd + d]), qscale) * __expf(sm.bl[t * kGbLd + d] - sm.bl[s * kGbLd + d]) *
                     gla_k<kKind>(p, to_f(sm.k[s * kGmLd + d]), h * p.dim + d0 + d);
            sc[j][x][e] += sum;
          }
      }
    }
  }
  __syncthreads();
  // the values, the gate and the norm's weights take the place of the state and the factors
  stage_rows(sm.shi, VD + 8, base + p.v_off + h * p.vdim, p.ldp, VD, p.vdim, cnt, vec);
  const bool gated = p.g_off >= 0;
  if (gated) stage_rows(sm.slo, VD + 8, base + p.g_off + h * p.vdim, p.ldp, VD, p.vdim, cnt, vec);
  for (int i = tid; i < VD; i += kGmThreads) sm.fac[i] = i < p.vdim ? p.norm_w[i] : 0.f;
  stage_wait();
  __syncthreads();
#pragma unroll
  for (int j = 0; j < kGSubs; ++j) {
    if (j > warp) break;
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int f = 0; f < 4; ++f) {
      const int half = f & 1, x = f >> 1, t = half ? rb : ra, s = j * 16 + x * 8 + c2;
      const float u = s <= t ? sc[j][x][2 * half] : 0.f, v = s + 1 <= t ? sc[j][x][2 * half + 1] : 0.f;
      split_bf16(u, v, hi[f], lo[f]);
    }
#pragma unroll
    for (int v = 0; v < VD / 16; ++v) {
      uint32_t bb[4];
      ldsm_x4_t(bb, sm.shi + (j * 16 + (lane & 15)) * (VD + 8) + v * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        mma_bf16(o[2 * v + x], hi, bb[2 * x], bb[2 * x + 1]);
        mma_bf16(o[2 * v + x], lo, bb[2 * x], bb[2 * x + 1]);
      }
    }
  }
  float sa = 0.f, sb = 0.f;            // columns past vdim are zero
#pragma unroll
  for (int i = 0; i < VD / 8; ++i) {
    sa += o[i][0] * o[i][0] + o[i][1] * o[i][1];
    sb += o[i][2] * o[i][2] + o[i][3] * o[i][3];
  }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    sa += __shfl_xor_sync(0xffffffffu, sa, x);
    sb += __shfl_xor_sync(0xffffffffu, sb, x);
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = half ? rb : ra;
    if (t >= cnt) continue;
    const float inv = 1.0f / sqrtf((half ? sb : sa) / (float)p.vdim + p.eps);
    const bf16* g = sm.slo + t * (VD + 8);
    bf16* out = reinterpret_cast<bf16*>(p.out) + (size_t)(b * p.T + t0 + t) * p.ldo + h * p.vdim;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) {
      const int v = i * 8 + c2;
      const uint32_t gg = *reinterpret_cast<const uint32_t*>(g + v);
      const float2 nw = *reinterpret_cast<const float2*>(sm.fac + v);
      const float gx = bf_lo(gg), gy = bf_hi(gg);
      const float x = o[i][2 * half] * inv * nw.x * (gated ? __fdividef(gx, 1.f + __expf(-gx)) : 1.f);
      const float y = o[i][2 * half + 1] * inv * nw.y * (gated ? __fdividef(gy, 1.f + __expf(-gy)) : 1.f);
      if (vec) {
        if (v < p.vdim) *reinterpret_cast<uint32_t*>(out + v) = pack_bf16(x, y);
      } else {
        if (v < p.vdim) out[v] = from_f<bf16>(x);
        if (v + 1 < p.vdim) out[v + 1] = from_f<bf16>(y);
      }
    }
  }
}

// ---- one token per sequence.  grid (H, B, S) in clusters of S CTAs along z: a CTA owns a range of value columns of the
// head's state, reads it once and writes it once; the squares of the outputs are summed over the cluster for the norm.
// The state was written in the step before (or by the prompt), so it is requested ahead of the dependency wait, and so are
// the decay's weights, as far as they fit the registers.
constexpr int kGdThreads = 256, kGdWarps = kGdThreads / 32;
constexpr int kGdPre = 8;              // rows of the state (four columns each) a thread may hold ahead of the wait

template <int kKind> __global__ void __launch_bounds__(kGdThreads) gla_decode_kernel(const nb_gla_args p) {
  extern __shared__ __align__(16) float gdm[];
  __shared__ float red[kGdWarps], ssq;
  cg::cluster_group cluster = cg::this_cluster();
  const int S = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int quads = p.lds / 4, qper = (quads + S - 1) / S, c0 = rank * qper, cn = max(0, min(quads, c0 + qper) - c0);   // columns in fours
  float* al = gdm;                     // [dim] decays
  float* ks = al + p.dim;              // [dim]
  float* qs = ks + p.dim;              // [dim]
  float* os = qs + p.dim;              // [4 * qper] outputs
  float4* part = reinterpret_cast<float4*>(gdm + ((3 * p.dim + 4 * qper + 3) & ~3));   // [kGdThreads]
  float4* st = reinterpret_cast<float4*>(p.state) + ((size_t)b * p.H + h) * p.dim * quads;
  const int cols0 = min(cn, kGdThreads), groups0 = cols0 ? kGdThreads / cols0 : 1, g0 = cols0 ? tid / cols0 : 0, cc0 = cols0 ? tid - g0 * cols0 : 0;
  const bool pre = cn > 0 && cn <= kGdThreads && (p.dim + groups0 - 1) / groups0 <= kGdPre;
  float4 sreg[kGdPre];
#pragma unroll
  for (int i = 0; i < kGdPre; ++i) {
    const int d = g0 + i * groups0;
    sreg[i] = (pre && g0 < groups0 && d < p.dim) ? st[(size_t)d * quads + c0 + cc0] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const bool short_rank = kKind == NB_GLA_LOW_RANK && p.lda2 <= 16 && p.dim <= kGdThreads;   // a row of W_a2 is one or two 16-byte loads
  const bf16* w2 = reinterpret_cast<const bf16*>(p.a2) + (size_t)(h * p.dim) * p.lda2;
  uint4 wa = make_uint4(0u, 0u, 0u, 0u), wb = wa;
  float bias = 0.f;
  if (short_rank && tid < p.dim) {
    wa = *reinterpret_cast<const uint4*>(w2 + (size_t)tid * p.lda2);
    if (p.lda2 > 8) wb = *reinterpret_cast<const uint4*>(w2 + (size_t)tid * p.lda2 + 8);
    bias = p.a2_b[h * p.dim + tid];
  }
  float lower = 0.f;
  if (kKind == NB_GLA_FORGET && tid < p.dim) { bias = p.a2_b[h * p.dim + tid]; lower = p.lower[h * p.dim + tid]; }
  pdl_enter();
  const float* row = reinterpret_cast<const float*>(p.p) + (size_t)b * p.ldp;
  const float* vrow = row + p.v_off + h * p.vdim;
  const float qscale = 1.0f / sqrtf((float)p.dim);
  const int vp = 4 * (c0 + cc0);
  float4 vpre = make_float4(0.f, 0.f, 0.f, 0.f);
  if (pre && g0 < groups0)
    vpre = make_float4(vp < p.vdim ? vrow[vp] : 0.f, vp + 1 < p.vdim ? vrow[vp + 1] : 0.f, vp + 2 < p.vdim ? vrow[vp + 2] : 0.f,
                       vp + 3 < p.vdim ? vrow[vp + 3] : 0.f);
  for (int d = tid; d < p.dim; d += kGdThreads) {
    const int ch = h * p.dim + d;
    const float k = row[p.k_off + ch], q = row[p.q_off + ch];
    if constexpr (kKind == NB_GLA_FORGET) {
      const float lo = d == tid ? lower : p.lower[ch], zf = k + (d == tid ? bias : p.a2_b[ch]), om = 1.f - lo;
      al[d] = lo + om * sigmoid_f(zf);
      ks[d] = forget_key(zf, om);
      qs[d] = silu_f(q);
      continue;
    }
    float z;
    if (short_rank) {
      z = bias;
      const uint32_t u[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        if (2 * r < p.a_rank) z = fmaf(bf_lo(u[r]), row[p.a_off + 2 * r], z);
        if (2 * r + 1 < p.a_rank) z = fmaf(bf_hi(u[r]), row[p.a_off + 2 * r + 1], z);
      }
    } else {
      z = p.a2_b[ch];
      for (int r = 0; r < p.a_rank; ++r) z = fmaf(to_f(w2[(size_t)d * p.lda2 + r]), row[p.a_off + r], z);
    }
    al[d] = expf(log_sigmoid_f(z) / p.tau);
    ks[d] = k;
    qs[d] = q * qscale;
  }
  __syncthreads();
  for (int base = 0; base < cn; base += kGdThreads) {
    const int cols = min(cn - base, kGdThreads), groups = kGdThreads / cols, gi = tid / cols, c = tid - gi * cols;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto advance = [&](float4 s, const float4& vv, int d) {
      const float a = al[d], k = ks[d], q = qs[d];
      s.x = fmaf(s.x, a, k * vv.x); s.y = fmaf(s.y, a, k * vv.y); s.z = fmaf(s.z, a, k * vv.z); s.w = fmaf(s.w, a, k * vv.w);
      st[(size_t)d * quads + c0 + base + c] = s;
      o.x = fmaf(s.x, q, o.x); o.y = fmaf(s.y, q, o.y); o.z = fmaf(s.z, q, o.z); o.w = fmaf(s.w, q, o.w);
    };
    if (pre) {
#pragma unroll
      for (int i = 0; i < kGdPre; ++i) {
        const int d = g0 + i * groups0;
        if (g0 < groups0 && d < p.dim) advance(sreg[i], vpre, d);
      }
    } else if (gi < groups) {
      const int v = 4 * (c0 + base + c);
      const float4 vv = make_float4(v < p.vdim ? vrow[v] : 0.f, v + 1 < p.vdim ? vrow[v + 1] : 0.f, v + 2 < p.vdim ? vrow[v + 2] : 0.f,
                                    v + 3 < p.vdim ? vrow[v + 3] : 0.f);
#pragma unroll 4
      for (int d = gi; d < p.dim; d += groups) advance(st[(size_t)d * quads + c0 + base + c], vv, d);
    }
    part[tid] = o;
    __syncthreads();
    if (tid < cols) {
      float4 v = part[tid];
      for (int g = 1; g < groups; ++g) {
        const float4 x = part[g * cols + tid];
        v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w;
      }
      float* od = os + 4 * (base + tid);
      od[0] = v.x; od[1] = v.y; od[2] = v.z; od[3] = v.w;
    }
    __syncthreads();
  }
  float ss = 0.f;
  for (int i = tid; i < 4 * cn; i += kGdThreads) ss += os[i] * os[i];    // columns past vdim are zero
  ss = block_sum<kGdWarps>(ss, red);
  if (tid == 0) ssq = ss;
  cluster.sync();
  float tot = 0.f;
  for (int r = 0; r < S; ++r) tot += *cluster.map_shared_rank(&ssq, r);
  cluster.sync();                      // nobody reads another CTA's shared memory after this
  const float inv = 1.0f / sqrtf(tot / (float)p.vdim + p.eps);
  for (int i = tid; i < 4 * cn; i += kGdThreads) {
    const int v = 4 * c0 + i;
    if (v < p.vdim)
      reinterpret_cast<float*>(p.out)[(size_t)b * p.ldo + h * p.vdim + v] = os[i] * inv * p.norm_w[v] * (p.g_off < 0 ? 1.f : silu_f(row[p.g_off + h * p.vdim + v]));
  }
}

template <typename T, int kKind> static int launch_decays(const nb_gla_args& a, const GlaWs& w, cudaStream_t st) {
  const dim3 grid((a.T + kGS - 1) / kGS, (a.H * a.dim + kDecThreads - 1) / kDecThreads, a.B);
  if (kKind == NB_GLA_FORGET) gla_forget_kernel<T><<<grid, kDecThreads, 0, st>>>(a, w);
  else gla_decay_kernel<T><<<grid, kDecThreads, (size_t)kGS * a.a_rank * 4, st>>>(a, w);
  return check_launch();
}

template <typename T, int kKind> static int gla_prefill(const nb_gla_args& a, const GlaWs& w, cudaStream_t st) {
  const int chunks = gla_chunks(a.T), dt = (a.dim + 63) / 64, vt = (a.vdim + 63) / 64;
  if (int rc = launch_decays<T, kKind>(a, w, st)) return rc;
  gla_state_kernel<T, kKind><<<dim3(chunks, a.H * dt * vt, a.B), 256, 0, st>>>(a, w, dt, vt);
  if (int rc = check_launch()) return rc;
  gla_scan_kernel<<<dim3((a.dim * (a.lds / 4) + 255) / 256, a.B * a.H), 256, 0, st>>>(a, w, chunks);
  if (int rc = check_launch()) return rc;
  constexpr size_t smem = ((size_t)4 * kGC * (64 + 4) + kGSubs * 64) * 4;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(gla_output_kernel<T, kKind>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) return record_cuda_error(e);
    done[dev & 63] = true;
  }
  gla_output_kernel<T, kKind><<<dim3(chunks, a.H, a.B), 256, smem, st>>>(a, w);
  if (int rc = check_launch()) return rc;
  const size_t rh = (size_t)a.B * a.T * a.H;
  gla_finish_kernel<T><<<(unsigned)((rh + 7) / 8), 256, 0, st>>>(a, w);
  return check_launch();
}

// bf16 projections with vdim <= VD: decay, state, scan and output kernels, the last with the norm and the gate.
template <int VD, int kKind> static int gla_prefill_mma(const nb_gla_args& a, const GlaWs& w, cudaStream_t st) {
  const int chunks = gla_chunks(a.T), dt = (a.dim + 63) / 64;
  const int vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ldp % 8 == 0 && a.q_off % 8 == 0 && a.k_off % 8 == 0 && a.v_off % 8 == 0 &&
                  (a.g_off < 0 || a.g_off % 8 == 0) && a.ldo % 2 == 0 && (uintptr_t)a.p % 16 == 0 && (uintptr_t)a.out % 4 == 0;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(gla_state_mma_kernel<VD, kKind>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(GlaStateSmem<VD>)))
      return record_cuda_error(e);
    if (cudaError_t e = cudaFuncSetAttribute(gla_output_mma_kernel<VD, kKind>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(GlaOutSmem<VD>)))
      return record_cuda_error(e);
    done[dev & 63] = true;
  }
  if (int rc = launch_decays<bf16, kKind>(a, w, st)) return rc;
  gla_state_mma_kernel<VD, kKind><<<dim3(chunks, a.H * dt, a.B), kGmThreads, sizeof(GlaStateSmem<VD>), st>>>(a, w, dt, vec);
  if (int rc = check_launch()) return rc;
  gla_scan_kernel<<<dim3((a.dim * (a.lds / 4) + 255) / 256, a.B * a.H), 256, 0, st>>>(a, w, chunks);
  if (int rc = check_launch()) return rc;
  gla_output_mma_kernel<VD, kKind><<<dim3(chunks, a.H, a.B), kGmThreads, sizeof(GlaOutSmem<VD>), st>>>(a, w, vec);
  return check_launch();
}

template <int kKind> static int gla_prefill_kind(const nb_gla_args& a, const GlaWs& w, cudaStream_t st) {
  if (a.dtype == NB_F32) return gla_prefill<float, kKind>(a, w, st);
  return a.vdim <= 64    ? gla_prefill_mma<64, kKind>(a, w, st)
         : a.vdim <= 128 ? gla_prefill_mma<128, kKind>(a, w, st)
         : a.vdim <= 256 ? gla_prefill_mma<256, kKind>(a, w, st)
                         : gla_prefill<bf16, kKind>(a, w, st);
}

static int gla_check(const nb_gla_args* a) {
  if (!a || !a->p || !a->out || !a->state || !a->a2_b || !a->norm_w || a->B < 1 || a->T < 1 || a->H < 1 || a->dim < 1 || a->vdim < 1)
    return NB_ERR_ARG;
  const bool low_rank = a->kind == NB_GLA_LOW_RANK;
  if (low_rank ? !a->a2 || a->a_rank < 1 || !(a->tau > 0.f) : a->kind != NB_GLA_FORGET || !a->lower) return NB_ERR_ARG;
  if (a->dtype != NB_BF16 && a->dtype != NB_F32) return NB_ERR_ARG;
  const int hd = a->H * a->dim, hv = a->H * a->vdim;
  if (a->q_off < 0 || a->k_off < 0 || a->v_off < 0 || (low_rank && (a->g_off < 0 || a->a_off < 0)) || a->q_off + hd > a->ldp ||
      a->k_off + hd > a->ldp || a->v_off + hv > a->ldp || (a->g_off >= 0 && a->g_off + hv > a->ldp) ||
      (low_rank && (a->a_off + a->a_rank > a->ldp || a->lda2 < a->a_rank)) || a->ldo < hv ||
      a->lds < a->vdim || a->lds % 4 || a->H > 65535 || a->B > 65535 || (long long)a->B * a->H > 65535)
    return NB_ERR_SHAPE;
  if ((uintptr_t)a->state % 16 || (low_rank && ((uintptr_t)a->a2 % 16 || a->lda2 % 8))) return NB_ERR_ALIGN;
  return NB_OK;
}

static size_t round256(size_t n) { return (n + 255) & ~(size_t)255; }

}  // namespace nb

using namespace nb;

extern "C" size_t nb_gla_workspace_bytes(int B, int T, int H, int dim, int vdim) {
  if (B < 1 || T < 1 || H < 1 || dim < 1 || vdim < 1) return 0;
  const size_t rows = (size_t)B * T, ch = (size_t)B * gla_chunks(T) * H, lds = (vdim + 3) & ~3;
  return round256(rows * H * dim * 4) + round256(ch * dim * lds * 4) + round256(ch * dim * 4) + round256(rows * H * vdim * 4);
}

extern "C" int nb_gla_prefill(const nb_gla_args* a, void* workspace, size_t workspace_bytes, void* stream) {
  if (int rc = gla_check(a)) return rc;
  if (a->lds != ((a->vdim + 3) & ~3)) return NB_ERR_SHAPE;
  if (!workspace || workspace_bytes < nb_gla_workspace_bytes(a->B, a->T, a->H, a->dim, a->vdim)) return NB_ERR_WORKSPACE;
  if ((uintptr_t)workspace % 256) return NB_ERR_ALIGN;
  const int dt = (a->dim + 63) / 64, vt = (a->vdim + 63) / 64;
  if ((long long)a->H * dt * vt > 65535 || (a->kind == NB_GLA_LOW_RANK && (size_t)kGS * a->a_rank * 4 > 48 * 1024) || (a->H * a->dim + kDecThreads - 1) / kDecThreads > 65535)
    return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  const size_t rows = (size_t)a->B * a->T, ch = (size_t)a->B * gla_chunks(a->T) * a->H;
  char* base = reinterpret_cast<char*>(workspace);
  GlaWs w;
  w.bl = reinterpret_cast<float*>(base);
  base += round256(rows * a->H * a->dim * 4);
  w.u = reinterpret_cast<float*>(base);
  base += round256(ch * a->dim * a->lds * 4);
  w.dec = reinterpret_cast<float*>(base);
  base += round256(ch * a->dim * 4);
  w.o = reinterpret_cast<float*>(base);
  cudaStream_t st = (cudaStream_t)stream;
  return a->kind == NB_GLA_FORGET ? gla_prefill_kind<NB_GLA_FORGET>(*a, w, st) : gla_prefill_kind<NB_GLA_LOW_RANK>(*a, w, st);
}

extern "C" int nb_gla_decode(const nb_gla_args* a, void* stream) {
  if (int rc = gla_check(a)) return rc;
  if (a->dtype != NB_F32) return NB_ERR_ARG;
  const int want = 592 / std::max(1, a->B * a->H), quads = a->lds / 4;
  const int S = std::min(want >= 8 ? 8 : want >= 4 ? 4 : want >= 2 ? 2 : 1, quads >= 8 ? 8 : quads >= 4 ? 4 : quads >= 2 ? 2 : 1);
  const size_t smem = (size_t)((3 * a->dim + 4 * ((quads + S - 1) / S) + 3) & ~3) * 4 + kGdThreads * 16;
  if (smem > 48 * 1024) return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a->H, a->B, S);
  cfg.blockDim = dim3(kGdThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = (cudaStream_t)stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = 1;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = S;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  return record_cuda_error(cudaLaunchKernelEx(&cfg, a->kind == NB_GLA_FORGET ? gla_decode_kernel<NB_GLA_FORGET> : gla_decode_kernel<NB_GLA_LOW_RANK>, *a));
}
