// Gated linear attention: per head a (dim x vdim) state S, S <- diag(alpha) S + k v^T, o = S^T q, with a decay alpha per
// key channel from a low-rank projection.
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

// ---- decays.  grid (sub-blocks, channel tiles, B); a thread owns one channel of 16 tokens.
constexpr int kDecThreads = 128;
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
  float* out = w.bl + (size_t)(b * p.T + t0) * HD + ch;
#pragma unroll
  for (int t = 0; t < kGS; ++t) {
    sum += log_sigmoid_f(z[t]) / p.tau;
    if (t < cnt) out[(size_t)t * HD] = sum;
  }
}

// ---- what a chunk adds to the state: U[d][v] = sum_t k_t[d] exp(decay from t to the chunk's end) v_t[v].
// grid (chunks, H * d tiles * v tiles, B), 64 x 64 outputs per CTA.
template <typename T> __global__ void __launch_bounds__(256) gla_state_kernel(const nb_gla_args p, GlaWs w, int dtiles, int vtiles) {
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
      kv = to_f(base[(size_t)t * p.ldp + p.k_off + h * p.dim + d]) * expf(e);
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
  for (int n = 0; n < chunks; ++n) {
    const size_t head = ((size_t)b * chunks + n) * p.H + h;
    float4* up = reinterpret_cast<float4*>(w.u) + head * per + i;
    const float a = expf(w.dec[head * p.dim + d]);
    const float4 u = *up;
    *up = s;
    s.x = fmaf(s.x, a, u.x); s.y = fmaf(s.y, a, u.y); s.z = fmaf(s.z, a, u.z); s.w = fmaf(s.w, a, u.w);
  }
  *st = s;
}

// ---- outputs of a chunk: o_t = S^T (q_t decayed from the chunk's start) + sum_{s <= t} A[t][s] v_s, with
// A[t][s] = sum_d q_t[d] k_s[d] exp(decay from s to t).  grid (chunks, H, B).  A is built 4 x 4 per thread; for tokens of
// different sub-blocks the decay is split at the start of t's sub-block, inside a sub-block at the start of t's group of
// four, and inside a group of four it is taken pair by pair.
template <typename T> __global__ void __launch_bounds__(256) gla_output_kernel(const nb_gla_args p, GlaWs w) {
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
      qt[c * ld + t] = in ? to_f(base[(size_t)t * p.ldp + p.q_off + h * p.dim + d]) * qscale : 0.f;
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
      kt[c * ld + t] = (t < cnt && d < p.dim) ? to_f(base[(size_t)t * p.ldp + p.k_off + h * p.dim + d]) : 0.f;
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

// ---- out = RMSNorm(o) * norm_w * silu(g), one warp per (row, head)
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
  for (int i = lane; i < p.vdim; i += 32) out[i] = from_f<T>(o[i] * inv * p.norm_w[i] * silu_f(to_f(g[i])));
}

// ---- one token per sequence.  grid (H, B, S) in clusters of S CTAs along z: a CTA owns a range of value columns of the
// head's state, reads it once and writes it once; the squares of the outputs are summed over the cluster for the norm.
constexpr int kGdThreads = 256, kGdWarps = kGdThreads / 32;

__global__ void __launch_bounds__(kGdThreads) gla_decode_kernel(const nb_gla_args p) {
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
  pdl_enter();
  const float* row = reinterpret_cast<const float*>(p.p) + (size_t)b * p.ldp;
  const float qscale = 1.0f / sqrtf((float)p.dim);
  for (int d = tid; d < p.dim; d += kGdThreads) {
    const int ch = h * p.dim + d;
    const bf16* w2 = reinterpret_cast<const bf16*>(p.a2) + (size_t)ch * p.lda2;
    float z = p.a2_b[ch];
    for (int r = 0; r < p.a_rank; ++r) z = fmaf(to_f(w2[r]), row[p.a_off + r], z);
    al[d] = expf(log_sigmoid_f(z) / p.tau);
    ks[d] = row[p.k_off + ch];
    qs[d] = row[p.q_off + ch] * qscale;
  }
  __syncthreads();
  float4* st = reinterpret_cast<float4*>(p.state) + ((size_t)b * p.H + h) * p.dim * quads;
  const float* vrow = row + p.v_off + h * p.vdim;
  for (int base = 0; base < cn; base += kGdThreads) {
    const int cols = min(cn - base, kGdThreads), groups = kGdThreads / cols, gi = tid / cols, c = tid - gi * cols;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (gi < groups) {
      const int v = 4 * (c0 + base + c);
      const float4 vv = make_float4(v < p.vdim ? vrow[v] : 0.f, v + 1 < p.vdim ? vrow[v + 1] : 0.f, v + 2 < p.vdim ? vrow[v + 2] : 0.f,
                                    v + 3 < p.vdim ? vrow[v + 3] : 0.f);
#pragma unroll 8
      for (int d = gi; d < p.dim; d += groups) {
        float4* sp = st + (size_t)d * quads + c0 + base + c;
        float4 s = *sp;
        const float a = al[d], k = ks[d], q = qs[d];
        s.x = fmaf(s.x, a, k * vv.x); s.y = fmaf(s.y, a, k * vv.y); s.z = fmaf(s.z, a, k * vv.z); s.w = fmaf(s.w, a, k * vv.w);
        *sp = s;
        o.x = fmaf(s.x, q, o.x); o.y = fmaf(s.y, q, o.y); o.z = fmaf(s.z, q, o.z); o.w = fmaf(s.w, q, o.w);
      }
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
      reinterpret_cast<float*>(p.out)[(size_t)b * p.ldo + h * p.vdim + v] = os[i] * inv * p.norm_w[v] * silu_f(row[p.g_off + h * p.vdim + v]);
  }
}

template <typename T> static int gla_prefill(const nb_gla_args& a, const GlaWs& w, cudaStream_t st) {
  const int chunks = gla_chunks(a.T), subs = (a.T + kGS - 1) / kGS, dt = (a.dim + 63) / 64, vt = (a.vdim + 63) / 64;
  const int HD = a.H * a.dim;
  gla_decay_kernel<T><<<dim3(subs, (HD + kDecThreads - 1) / kDecThreads, a.B), kDecThreads, (size_t)kGS * a.a_rank * 4, st>>>(a, w);
  if (int rc = check_launch()) return rc;
  gla_state_kernel<T><<<dim3(chunks, a.H * dt * vt, a.B), 256, 0, st>>>(a, w, dt, vt);
  if (int rc = check_launch()) return rc;
  gla_scan_kernel<<<dim3((a.dim * (a.lds / 4) + 255) / 256, a.B * a.H), 256, 0, st>>>(a, w, chunks);
  if (int rc = check_launch()) return rc;
  constexpr size_t smem = ((size_t)4 * kGC * (64 + 4) + kGSubs * 64) * 4;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(gla_output_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) return record_cuda_error(e);
    done[dev & 63] = true;
  }
  gla_output_kernel<T><<<dim3(chunks, a.H, a.B), 256, smem, st>>>(a, w);
  if (int rc = check_launch()) return rc;
  const size_t rh = (size_t)a.B * a.T * a.H;
  gla_finish_kernel<T><<<(unsigned)((rh + 7) / 8), 256, 0, st>>>(a, w);
  return check_launch();
}

static int gla_check(const nb_gla_args* a) {
  if (!a || !a->p || !a->out || !a->state || !a->a2 || !a->a2_b || !a->norm_w || a->B < 1 || a->T < 1 || a->H < 1 || a->dim < 1 || a->vdim < 1 ||
      a->a_rank < 1 || !(a->tau > 0.f))
    return NB_ERR_ARG;
  if (a->dtype != NB_BF16 && a->dtype != NB_F32) return NB_ERR_ARG;
  const int hd = a->H * a->dim, hv = a->H * a->vdim;
  if (a->q_off < 0 || a->k_off < 0 || a->v_off < 0 || a->g_off < 0 || a->a_off < 0 || a->q_off + hd > a->ldp || a->k_off + hd > a->ldp ||
      a->v_off + hv > a->ldp || a->g_off + hv > a->ldp || a->a_off + a->a_rank > a->ldp || a->lda2 < a->a_rank || a->ldo < hv ||
      a->lds < a->vdim || a->lds % 4 || a->H > 65535 || a->B > 65535 || (long long)a->B * a->H > 65535)
    return NB_ERR_SHAPE;
  if ((uintptr_t)a->state % 16) return NB_ERR_ALIGN;
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
  if ((long long)a->H * dt * vt > 65535 || (size_t)kGS * a->a_rank * 4 > 48 * 1024 || (a->H * a->dim + kDecThreads - 1) / kDecThreads > 65535)
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
  return a->dtype == NB_BF16 ? gla_prefill<bf16>(*a, w, (cudaStream_t)stream) : gla_prefill<float>(*a, w, (cudaStream_t)stream);
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
  return record_cuda_error(cudaLaunchKernelEx(&cfg, gla_decode_kernel, *a));
}
